"""A mixture of experts as a decoder's layer uses it: the grouped products, the routing buffers, and the launches between router logits
and the experts' outputs (csrc/moe.cu and the grouped linears)."""
import torch

from . import ops


class Experts:
    """`experts` units of one shape, of which every token uses `top`: gated ones, or (gates None) the square of a relu.

    gates, ups: [ff, width] per expert; downs: [width, ff].  glu, limit: the gated unit.  score: how router logits become weights.
    weigh_input: a token's weight multiplies an expert's input (its output is then summed as it is) instead of its output.
    With score MOE_SOFTMAX_ALL: correction, groups, keep (see pt_moe_route), and `identity` more router outputs whose experts give their
    input back."""

    def __init__(self, dtype, top, gates, ups, downs, glu=ops.GLU_CLAMPED, limit=0.0, score=ops.MOE_SOFTMAX, weigh_input=False, correction=None, groups=0, keep=0, identity=0):
        if identity and weigh_input:
            raise ops.PtError("experts without matrices have no input that a weight could multiply")
        self.dtype, self.experts, self.top, self.score, self.weigh_input, self.identity = dtype, len(ups), top, score, weigh_input, identity
        self.choice = dict(score=score, correction=correction, groups=groups, keep=keep, identity=identity)
        self.logits = self.experts + identity
        ff, self.width = ups[0].shape
        self.ff = ops.pad_to(ff, ops.DenseLinear.K_PAD if dtype == torch.bfloat16 else 16)      # features: the padded input of the next product

        def down(w):
            full = torch.zeros((self.width, self.ff), dtype=dtype, device=w.device)
            full[:, :ff] = w
            return full

        if gates is None:
            self.up, self.epilogue = ops.GroupedLinear(ups, dtype, pad_rows=self.ff), ops.EPI_RELU2
        else:
            self.up, self.epilogue = ops.GroupedLinear([ops.glu_rows(g, u, self.ff) for g, u in zip(gates, ups)], dtype, limit=limit, glu=glu), ops.EPI_GLU
        self.back = ops.GroupedLinear([down(w) for w in downs], dtype)

    def step_bytes(self, rows):
        """Weight bytes that a step of `rows` tokens reads at most."""
        return min(self.experts, rows * self.top) * (self.up.nbytes + self.back.nbytes)

    def tile(self, n):
        """Rows of a tile of the grouped products for n tokens: 1 for the skinny-matmul kernel, else about an expert's share."""
        if self.dtype == torch.float32:
            return 64
        if n <= ops.DenseLinear.SKINNY_ROWS:
            return 1
        share, tile = n * self.top / self.logits, 16
        while tile < 128 and tile < share:
            tile *= 2
        return tile

    @staticmethod
    def buffers(r, rows, groups, h_ld, device, ws=None):
        """Adds to `r` what `groups` (of one decoder) need for up to `rows` tokens whose activations have row stride h_ld; `ws` (default: r)
        is the object whose lin_ws the skinny products use."""
        dt, ws = groups[0].dtype, ws or r
        f32, i32 = dict(dtype=torch.float32, device=device), dict(dtype=torch.int32, device=device)
        top, experts = max(g.top for g in groups), max(g.logits for g in groups)
        padded = [g.tile(rows) * ops.moe_max_tiles(rows, g.experts, g.top, g.tile(rows)) for g in groups]
        r.logits = torch.empty(rows * experts, **f32)
        r.expert, r.pair_row, r.weight = torch.empty(rows * top, **i32), torch.empty(rows * top, **i32), torch.empty(rows * top, **f32)
        r.tile_expert, r.tile_rows, r.row_token = (torch.empty(max(padded), **i32) for _ in range(3))
        r.row_weight = torch.empty(max(padded), **f32)
        r.counts = torch.empty(experts, **i32)
        r.gathered = torch.empty(max(padded) * h_ld, dtype=dt, device=device)
        r.act = torch.empty(max(p * g.ff for p, g in zip(padded, groups)), dtype=dt, device=device)
        r.pair_y = torch.empty((max(padded), groups[0].width), dtype=dt, device=device)
        if dt == torch.bfloat16:
            pairs = min(rows, ops.DenseLinear.SKINNY_ROWS) * top
            n = max(ops._lib.lib().pt_linear_workspace_bytes(pairs, x.n_out, 4) for g in groups for x in (g.up, g.back))
            if ws.lin_ws is None or n > ws.lin_ws.numel():
                ws.lin_ws = torch.zeros(n, dtype=torch.uint8, device=device)

    def __call__(self, r, n, h_ld, error_flag, ws=None, h=None):
        """From r.logits [n, router outputs] and the tokens' activations h (default: r.h) to the experts' outputs; returns what `post_norm` or
        `shift_norm` adds up."""
        ws, tile, W, h = ws or r, self.tile(n), self.width, r.h if h is None else h
        logits = r.logits[:n * self.logits].view(n, self.logits)
        kw = dict(linear_ws=ws.lin_ws, gemm_ws=ws.gemm_ws, error_flag=error_flag, pdl=1)
        pair_row = r.pair_row if tile > 1 or self.identity else None
        if tile == 1:
            ops.moe_route(logits, n, self.experts, self.top, r.expert, r.weight, pair_row=pair_row, **self.choice)
            self.up(h, r.act, n * self.top, self.ff, 1, r.expert, x_div=self.top, epilogue=self.epilogue, row_scale=r.weight if self.weigh_input else None, **kw)
            self.back(r.act, r.pair_y, n * self.top, W, 1, r.expert, **kw)
        else:
            rows = tile * ops.moe_max_tiles(n, self.experts, self.top, tile)
            ops.moe_route(logits, n, self.experts, self.top, r.expert, r.weight, tile, pair_row, r.tile_expert, r.tile_rows, r.row_token, r.counts, h, h_ld, r.gathered,
                          row_weight=r.row_weight if self.weigh_input else None, **self.choice)
            self.up(r.gathered, r.act, rows, self.ff, tile, r.tile_expert, r.tile_rows, epilogue=self.epilogue, row_scale=r.row_weight if self.weigh_input else None, **kw)
            self.back(r.act, r.pair_y, rows, W, tile, r.tile_expert, r.tile_rows, **kw)
        return dict(pair_y=r.pair_y, pair_ld=W, top=self.top, pair_w=None if self.weigh_input else r.weight, pair_row=pair_row)
