"""A mixture of experts as a decoder's layer uses it: the grouped products, the routing buffers, and the launches between router logits
and the experts' outputs (csrc/moe.cu and the grouped linears)."""
import torch

from . import ops


class Experts:
    """`experts` gated units of one shape, of which every token uses `top`.

    gates, ups: [ff, width] per expert; downs: [width, ff].  glu, limit: the gated unit.  score: how router logits become weights.
    weigh_input: a token's weight multiplies an expert's input (its output is then summed as it is) instead of its output."""

    def __init__(self, dtype, top, gates, ups, downs, glu=ops.GLU_CLAMPED, limit=0.0, score=ops.MOE_SOFTMAX, weigh_input=False):
        self.dtype, self.experts, self.top, self.score, self.weigh_input = dtype, len(gates), top, score, weigh_input
        ff, self.width = gates[0].shape
        self.ff = ops.pad_to(ff, ops.DenseLinear.K_PAD if dtype == torch.bfloat16 else 16)      # features: the padded input of the next product

        def down(w):
            full = torch.zeros((self.width, self.ff), dtype=dtype, device=w.device)
            full[:, :ff] = w
            return full

        self.up = ops.GroupedLinear([ops.glu_rows(g, u, self.ff) for g, u in zip(gates, ups)], dtype, limit=limit, glu=glu)
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
        share, tile = n * self.top / self.experts, 16
        while tile < 128 and tile < share:
            tile *= 2
        return tile

    @staticmethod
    def buffers(r, rows, groups, h_ld, device, ws=None):
        """Adds to `r` what `groups` (of one decoder) need for up to `rows` tokens whose activations have row stride h_ld; `ws` (default: r)
        is the object whose lin_ws the skinny products use."""
        dt, ws = groups[0].dtype, ws or r
        f32, i32 = dict(dtype=torch.float32, device=device), dict(dtype=torch.int32, device=device)
        top, experts = max(g.top for g in groups), max(g.experts for g in groups)
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

    def __call__(self, r, n, h_ld, error_flag, ws=None):
        """From r.logits [n, experts] and the tokens' activations r.h to the experts' outputs; returns what `post_norm` adds up."""
        ws, tile, W = ws or r, self.tile(n), self.width
        logits = r.logits[:n * self.experts].view(n, self.experts)
        kw = dict(linear_ws=ws.lin_ws, gemm_ws=ws.gemm_ws, error_flag=error_flag, pdl=1)
        if tile == 1:
            ops.moe_route(logits, n, self.experts, self.top, r.expert, r.weight, score=self.score)
            self.up(r.h, r.act, n * self.top, self.ff, 1, r.expert, x_div=self.top, epilogue=ops.EPI_GLU, row_scale=r.weight if self.weigh_input else None, **kw)
            self.back(r.act, r.pair_y, n * self.top, W, 1, r.expert, **kw)
        else:
            rows = tile * ops.moe_max_tiles(n, self.experts, self.top, tile)
            ops.moe_route(logits, n, self.experts, self.top, r.expert, r.weight, tile, r.pair_row, r.tile_expert, r.tile_rows, r.row_token, r.counts, r.h, h_ld, r.gathered,
                          score=self.score, row_weight=r.row_weight if self.weigh_input else None)
            self.up(r.gathered, r.act, rows, self.ff, tile, r.tile_expert, r.tile_rows, epilogue=ops.EPI_GLU, row_scale=r.row_weight if self.weigh_input else None, **kw)
            self.back(r.act, r.pair_y, rows, W, tile, r.tile_expert, r.tile_rows, **kw)
        return dict(pair_y=r.pair_y, pair_ld=W, top=self.top, pair_w=None if self.weigh_input else r.weight, pair_row=None if tile == 1 else r.pair_row)
