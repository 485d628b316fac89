"""Host-side mirror of the reference's custom-op surface (poptransformer/ops/customized.py)
on CUDA tensors.  Same op names and argument meanings; every function enqueues kernels of
libpt_b200.so on torch's current stream.  PyTorch is used for device memory and streams only.

Reference op            -> function here
  KVCache               -> kv_cache            (dense reference layout, bit-exact)
  KVCachePipeline       -> kv_cache_pipeline
  Int4ToHalf            -> int4_to_half
  SoftmaxV3             -> softmax_ce
  NormCE                -> layer_norm_ce
  CastToUint8...        -> half_to_uint8
  FP8MatMul...          -> fp8_matmul
  BeamSearch            -> beam_search
  Remap                 -> remap_tensor        (layout hint on IPU; identity here)
plus the fused decode stages that replace chains of reference ops: PackedLinear / linear,
rms_norm, kv_append_attn, topk, embedding, step_containers, wkv.
"""
import ctypes

import torch

from . import _lib
from ._lib import (AttnArgs, BatchView, ContextRows, DenseExt, GemmArgs, HyperArgs, LatentAttnArgs, LatentContextArgs, LatentPrepArgs, LinearArgs, MlstmArgs,
                   MoeRouteArgs, PostNormArgs, PtError, ShiftNormArgs, SsmArgs, WindowAttnArgs, check)

W_INT4, W_FP16, W_FP8, W_BF16 = 0, 1, 2, 3
DT_F16, DT_F32, DT_BF16 = 0, 1, 2
PRO_NONE, PRO_RMSNORM, PRO_CAST_FP8, PRO_RMSNORM_CAST_FP8, PRO_NORMCE = 0, 1, 2, 3, 4
EPI_STORE, EPI_RESIDUAL, EPI_SWIGLU, EPI_BIAS, EPI_BIAS_GELU, EPI_BIAS_RESIDUAL, EPI_RELU2, EPI_GLU, EPI_GELU_MUL, EPI_SOFTCAP, EPI_XIELU = range(11)
GLU_CLAMPED, GLU_SILU, GLU_GELU = 0, 1, 2
MOE_SOFTMAX, MOE_SIGMOID, MOE_SOFTMAX_ALL = 0, 1, 2
ROPE_NONE, ROPE_LLAMA, ROPE_CHATGLM2 = 0, 1, 2
SOFTMAX_F32, SOFTMAX_F16 = 0, 1


def _stream():
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def _ptr(t):
    if t is None:
        return None
    if not t.is_cuda:
        raise PtError("libpt_b200 ops need CUDA tensors (there is no CPU path)")
    if not t.is_contiguous():
        raise PtError("libpt_b200 ops need contiguous tensors")
    return ctypes.c_void_p(t.data_ptr())


def dtype_code(dt):
    code = {torch.float16: DT_F16, torch.float32: DT_F32, torch.bfloat16: DT_BF16}.get(dt)
    if code is None:
        raise PtError(f"unsupported element type {dt}")
    return code


def launch_count():
    return int(_lib.lib().pt_launch_count())


# ------------------------------------------------------------------------------------------ Int4ToHalf
def int4_to_half(x, scale, ref=None, axis=1, remap=1, group=0):
    """ops.int4_to_half (customized.py:115-124).  x int8 [n, m]; scale fp16 [n] (axis 1) / [m]
    (axis 0) or [n, 2m/group].  `ref` and `remap` only steer the IPU layout and are ignored."""
    n, m = x.shape
    out = torch.empty((2 * m, n) if axis == 1 else (2 * n, m), dtype=torch.float16, device=x.device)
    check(_lib.lib().pt_int4_to_half(_ptr(x), _ptr(scale), n, m, axis, group, _ptr(out), _stream()), "Int4ToHalf")
    return out


# ------------------------------------------------------------------------------------------ linear
class PackedLinear:
    """A weight matrix in the streaming kernel's tile order (built once at load time).

    w: [n_out, k] with k contiguous — INT4: int8 [n_out, k/2] in the reference checkpoint format
    (precision_strategy.py:24-42) with fp16 scales [n_out] or [n_out, k/group]; FP16: fp16 [n_out, k]
    (the HF [out, in] layout, i.e. before the reference's load-time transpose, layers/linear.py:32);
    FP8: uint8 E4M3 [n_out, k] with a per-tensor scale; BF16: bfloat16 [n_out, k]."""

    def __init__(self, wfmt, w, scale=None, group=0, interleave_gate_up=False, w_scale=1.0):
        L = _lib.lib()
        self.wfmt = wfmt
        self.n_out = w.shape[0]
        self.k_in = w.shape[1] * 2 if wfmt == W_INT4 else w.shape[1]
        self.w_scale = float(w_scale)
        self.interleaved = bool(interleave_gate_up)
        if wfmt == W_INT4:
            self.group = int(group) if group else self.k_in
            scale = scale.reshape(self.n_out, self.k_in // self.group).contiguous()
        else:
            self.group = 0
        nbytes = L.pt_linear_packed_bytes(wfmt, self.n_out, self.k_in)
        self.packed_w = torch.empty(nbytes, dtype=torch.uint8, device=w.device)
        check(L.pt_linear_repack(wfmt, _ptr(w.contiguous()), _ptr(scale) if scale is not None else None, self.n_out, self.k_in,
                                 self.group, 1 if interleave_gate_up else 0, _ptr(self.packed_w), _stream()), "pt_linear_repack")

    @property
    def nbytes(self):
        """Algorithmic bytes one launch streams from HBM: weights plus one fp16 scale per row and group.  (The
        packed tiles repeat a scale for every 128-k chunk of its group, so the buffer itself can be larger.)"""
        sb = self.n_out * (self.k_in // self.group) * 2 if self.wfmt == W_INT4 else 0
        wb = self.n_out * self.k_in // 2 if self.wfmt == W_INT4 else self.n_out * self.k_in * (1 if self.wfmt == W_FP8 else 2)
        return wb + sb


def linear_workspace(batch, n_out_max, max_ksplit=16, device="cuda"):
    """Zero-initialised split-k workspace shared by all linears of a stream (counters must start at 0;
    every launch leaves them at 0)."""
    n = _lib.lib().pt_linear_workspace_bytes(batch, n_out_max, max_ksplit)
    return torch.zeros(n, dtype=torch.uint8, device=device)


def linear_args(x, pl, out, prologue=PRO_NONE, epilogue=EPI_STORE, gamma=None, eps=0.0, act_scale=0.0, bias=None,
                residual=None, workspace=None, ksplit=0, out_ld=0, pdl=0, error_flag=None, beta=None, alpha=1.0, ext=None):
    a = LinearArgs()
    a.wfmt, a.batch, a.n_out, a.k_in, a.group = pl.wfmt, x.shape[0], pl.n_out, pl.k_in, pl.group
    a.prologue, a.epilogue, a.ksplit = prologue, epilogue, ksplit
    a.x, a.packed_w = _ptr(x), _ptr(pl.packed_w)
    a.norm_gamma, a.norm_eps, a.act_scale, a.w_scale = _ptr(gamma), eps, act_scale, pl.w_scale
    a.bias, a.residual, a.out, a.out_ld, a.pdl = _ptr(bias), _ptr(residual), _ptr(out), out_ld, pdl
    a.error_flag, a.norm_beta = _ptr(error_flag), _ptr(beta)
    a.out_dtype, a.alpha = dtype_code(out.dtype), float(alpha)
    if ext is not None:
        a.ext = ctypes.pointer(ext)
    a.workspace = _ptr(workspace)
    a.workspace_bytes = workspace.numel() if workspace is not None else 0
    return a


def linear(x, pl, out=None, **kw):
    """y = epilogue(prologue(x) @ W^T).  x fp16 [batch <= 32, k]."""
    if x.shape[1] != pl.k_in:
        raise PtError(f"linear: x has k={x.shape[1]}, weight has k={pl.k_in}")
    n = pl.n_out // 2 if kw.get("epilogue", EPI_STORE) == EPI_SWIGLU else pl.n_out
    if out is None:
        out = torch.empty((x.shape[0], n), dtype=torch.float16, device=x.device)
    a = linear_args(x, pl, out, **kw)
    check(_lib.lib().pt_linear(ctypes.byref(a), _stream()), "pt_linear")
    return out


# ------------------------------------------------------------------------------------------ tensor-core GEMMs (16+ rows)
class GemmWeight:
    """A weight matrix tiled once for pt_gemm (pt_gemm_repack): FP8 bytes [n_out, k], or INT4 rows in the reference's int8
    [n_out, k/2] format plus fp16 scales [n_out, k/group], or bfloat16 [n_out, k]."""

    def __init__(self, wfmt, w, scale=None, group=0, w_scale=1.0):
        L = _lib.lib()
        self.wfmt, self.n_out, self.w_scale = wfmt, w.shape[0], float(w_scale)
        if wfmt == W_INT4:
            self.k_in = w.shape[1] * 2
            self.group = int(group) if group else self.k_in
            self.scales = scale.reshape(self.n_out, self.k_in // self.group).to(torch.float16).contiguous()
        elif wfmt in (W_FP8, W_BF16):
            self.k_in, self.group, self.scales = w.shape[1], 0, None
        else:
            raise PtError("GemmWeight: INT4, FP8 or BF16")
        self.w = torch.empty(L.pt_gemm_packed_bytes(wfmt, self.n_out, self.k_in), dtype=torch.uint8, device=w.device)
        check(L.pt_gemm_repack(wfmt, _ptr(w.contiguous()), self.n_out, self.k_in, _ptr(self.w), _stream()), "pt_gemm_repack")

    @property
    def nbytes(self):
        """Algorithmic bytes one launch streams from HBM."""
        wb = self.n_out * self.k_in // 2 if self.wfmt == W_INT4 else self.n_out * self.k_in * (2 if self.wfmt == W_BF16 else 1)
        return wb + (self.scales.numel() * 2 if self.scales is not None else 0)


def gemm_workspace(m, n_out_max, max_ksplit=8, device="cuda"):
    return torch.zeros(_lib.lib().pt_gemm_workspace_bytes(m, n_out_max, max_ksplit), dtype=torch.uint8, device=device)


def gemm(x, gw, out=None, x_scale=1.0, epilogue=EPI_STORE, residual=None, workspace=None, ksplit=0, error_flag=None, bias=None,
         out_ld=0, alpha=1.0, ext=None, pdl=0):
    """y = x @ W^T on the tcgen05 GEMM.  INT4: x fp16 [m, k]; FP8: x E4M3 bytes [m, k] quantised with `x_scale`; BF16: x bfloat16,
    `out` bfloat16 or float32."""
    m = x.shape[0]
    if x.shape[1] != gw.k_in:
        raise PtError(f"gemm: x has k={x.shape[1]}, weight has k={gw.k_in}")
    if out is None:
        out = torch.empty((m, gw.n_out), dtype=torch.float16, device=x.device)
    a = GemmArgs()
    a.wfmt, a.m, a.n_out, a.k_in, a.group, a.epilogue, a.ksplit = gw.wfmt, m, gw.n_out, gw.k_in, gw.group, epilogue, ksplit
    a.w_tiled = 1
    a.x, a.w, a.scales = _ptr(x), _ptr(gw.w), _ptr(gw.scales)
    a.x_scale, a.w_scale = float(x_scale), gw.w_scale
    a.residual, a.out, a.out_ld = _ptr(residual), _ptr(out), out_ld
    a.out_dtype, a.alpha = dtype_code(out.dtype), float(alpha)
    a.workspace, a.workspace_bytes = _ptr(workspace), (workspace.numel() if workspace is not None else 0)
    a.error_flag, a.bias = _ptr(error_flag), _ptr(bias)
    if ext is not None:
        a.ext = ctypes.pointer(ext)
    a.pdl = pdl
    check(_lib.lib().pt_gemm(ctypes.byref(a), _stream()), "pt_gemm")
    return out


# ------------------------------------------------------------------------------------------ linears of bf16 / fp32 models
def pad_to(n, m):
    return (n + m - 1) // m * m


def glu_rows(gate, up, features):
    """Weight rows of a gated product (EPI_GLU): blocks of eight gate features and the same eight up features, with zero rows up to
    `features` (a multiple of eight)."""
    n, k = gate.shape
    out = torch.zeros((features // 8, 2, 8, k), dtype=gate.dtype, device=gate.device)
    for j, w in enumerate((gate, up)):
        full = torch.zeros((features, k), dtype=w.dtype, device=w.device)
        full[:n] = w
        out[:, j] = full.view(-1, 8, k)
    return out.reshape(-1, k)


class DenseLinear:
    """W [n_out, k] of a model whose activations are bfloat16 or float32.  bfloat16: the skinny-matmul kernel up to `skinny_rows` rows
    and the tcgen05 GEMM beyond (one tiling of the weights each), k padded to `K_PAD` with zero columns, so inputs have `ld` columns.
    float32: true 32-bit products, no padding.  Outputs may have more columns than n_out (`out_ld`)."""
    K_PAD = 64
    # Measured on B200 over 2048 x 4096 .. 32000 x 4096: at 8 rows the GEMM is level (2048-wide) to 20 % faster, at 32 rows 10 % to 3x.
    # Up to a million weights (128 x 2048, 2048 x 128, 1024 x 1024) the skinny kernel takes 0.6 - 0.75 of the GEMM's time at 8 and 16 rows.
    SKINNY_ROWS, SMALL_ROWS, SMALL_SIZE = 7, 16, 1 << 20

    def __init__(self, w, dtype, pad_rows=0, keep=False, bias=None, split=None, limit=0.0, glu=GLU_CLAMPED, xielu=None):
        """pad_rows: zero rows are appended up to this many outputs (an output that is the padded input of the next linear).
        keep: keep the padded matrix itself as `w` (a table that also serves look-ups).  bias: fp32 [n_out].  split: outputs from this
        row on (a multiple of 32) go to a second, fp32 output and skip the epilogue.  limit, glu: of a gated epilogue (rows as glu_rows);
        limit also of the softcap.  xielu: (pos, neg) of that epilogue."""
        self.dtype, self.n_out, self.k_in = dtype, w.shape[0], w.shape[1]
        self.split, self.limit, self.glu, self.xielu = split, float(limit), glu, xielu
        self.ld = pad_to(self.k_in, self.K_PAD) if dtype == torch.bfloat16 else self.k_in
        if self.ld != self.k_in or pad_rows > self.n_out:
            full = torch.zeros((max(pad_rows, self.n_out), self.ld), dtype=w.dtype, device=w.device)
            full[:self.n_out, :self.k_in] = w
            w, self.n_out = full, full.shape[0]
        self.bias = None
        if bias is not None:
            self.bias = torch.zeros(self.n_out, dtype=torch.float32, device=w.device)
            self.bias[:len(bias)] = bias
        w = w.to(dtype).contiguous()
        self.skinny_rows = self.SMALL_ROWS if self.n_out * self.ld <= self.SMALL_SIZE else self.SKINNY_ROWS
        if dtype == torch.bfloat16:
            self.skinny, self.gemm = PackedLinear(W_BF16, w), GemmWeight(W_BF16, w)
            self.w = w if keep else None
        elif dtype == torch.float32:
            self.w = w
        else:
            raise PtError(f"DenseLinear: bfloat16 or float32, got {dtype}")

    @property
    def nbytes(self):
        """Algorithmic bytes of one launch: the weights once."""
        return self.n_out * self.k_in * (2 if self.dtype == torch.bfloat16 else 4)

    def _ext(self, out2, out2_ld, mul, mul_ids, bias):
        """mul: (a table of the output's type, its row stride, its first column)."""
        bias = self.bias if bias is None else bias
        if bias is None and self.split is None and mul is None and not self.limit and self.glu == GLU_CLAMPED and self.xielu is None:
            return None
        e = DenseExt()
        e.bias, e.limit, e.glu = _ptr(bias), self.limit, self.glu
        if self.xielu is not None:
            e.pos, e.neg = self.xielu
        if self.split is not None:
            e.out2, e.out2_ld, e.split_n = _ptr(out2), out2_ld, self.split
        if mul is not None:
            table, ld, col = mul
            e.mul, e.mul_ld, e.mul_ids = table.data_ptr() + col * table.element_size(), ld, _ptr(mul_ids)
        return e

    def __call__(self, x, out, rows, out_ld, epilogue=EPI_STORE, alpha=1.0, linear_ws=None, gemm_ws=None, error_flag=None, out2=None, out2_ld=0, mul=None,
                 mul_ids=None, pdl=0, bias=None):
        """out[:rows, :n_out] = epilogue(alpha * x[:rows] @ W^T + bias); x and out are flat or 2-D buffers of row strides `ld` and
        `out_ld`.  bias: fp32 [n_out] in place of the linear's own.  pdl: programmatic dependent launch behind the kernel before it in the stream (bfloat16)."""
        x = x.reshape(-1)[:rows * self.ld].view(rows, self.ld)
        L = _lib.lib()
        ext = self._ext(out2, out2_ld, mul, mul_ids, bias)
        if self.dtype == torch.float32:
            check(L.pt_gemm_f32(_ptr(x), self.ld, _ptr(self.w), self.ld, rows, self.n_out, self.k_in, float(alpha), epilogue, _ptr(out), out_ld,
                                ctypes.byref(ext) if ext else None, _stream()), "pt_gemm_f32")
        elif rows <= self.skinny_rows:
            a = linear_args(x, self.skinny, out, epilogue=epilogue, workspace=linear_ws, out_ld=out_ld, error_flag=error_flag, alpha=alpha, ext=ext, pdl=pdl)
            check(L.pt_linear(ctypes.byref(a), _stream()), "pt_linear")
        else:
            gemm(x, self.gemm, out=out, epilogue=epilogue, workspace=gemm_ws, error_flag=error_flag, out_ld=out_ld, alpha=alpha, ext=ext, pdl=pdl)


class GroupedLinear:
    """Matrices [n_out, k] of one shape (experts), one after the other in a buffer: every tile of activation rows is multiplied with
    the matrix that `group_of` names for it.  bfloat16: tiles of one row on the skinny-matmul kernel, tiles of 16 .. 256 rows on the
    tcgen05 GEMM; float32: tiles of 64 rows."""
    skinny_rows = DenseLinear.SKINNY_ROWS

    def __init__(self, ws, dtype, pad_rows=0, limit=0.0, glu=GLU_CLAMPED):
        self.dtype, self.groups, self.k_in, self.limit, self.glu = dtype, len(ws), ws[0].shape[1], float(limit), glu
        self.n_out = max(pad_rows, ws[0].shape[0])
        self.ld = pad_to(self.k_in, DenseLinear.K_PAD) if dtype == torch.bfloat16 else self.k_in
        L = _lib.lib()
        dev = ws[0].device
        if dtype == torch.bfloat16:
            skinny, tiled = L.pt_linear_packed_bytes(W_BF16, self.n_out, self.ld), L.pt_gemm_packed_bytes(W_BF16, self.n_out, self.ld)
            self.skinny = torch.empty((self.groups, skinny), dtype=torch.uint8, device=dev)
            self.tiled = torch.empty((self.groups, tiled), dtype=torch.uint8, device=dev)
        elif dtype == torch.float32:
            self.w = torch.zeros((self.groups, self.n_out, self.k_in), dtype=dtype, device=dev)
        else:
            raise PtError(f"GroupedLinear: bfloat16 or float32, got {dtype}")
        for g, w in enumerate(ws):
            if dtype == torch.float32:
                self.w[g, :w.shape[0]] = w
                continue
            full = torch.zeros((self.n_out, self.ld), dtype=dtype, device=dev)
            full[:w.shape[0], :self.k_in] = w
            check(L.pt_linear_repack(W_BF16, _ptr(full), None, self.n_out, self.ld, 0, 0, _ptr(self.skinny[g]), _stream()), "pt_linear_repack")
            check(L.pt_gemm_repack(W_BF16, _ptr(full), self.n_out, self.ld, _ptr(self.tiled[g]), _stream()), "pt_gemm_repack")

    @property
    def nbytes(self):
        """Bytes of one matrix."""
        return self.n_out * self.k_in * (2 if self.dtype == torch.bfloat16 else 4)

    def __call__(self, x, out, rows, out_ld, tile, group_of, used=None, x_div=1, epilogue=EPI_STORE, linear_ws=None, gemm_ws=None, error_flag=None, pdl=0,
                 row_scale=None):
        """out[:rows] = epilogue(x rows @ matrix^T).  tile: rows per entry of group_of; with tile 1 row r reads x row r // x_div.
        used: rows of every tile that matter (the GEMM leaves the others out).  row_scale: fp32, a factor on every row's sums."""
        L = _lib.lib()
        e = DenseExt()
        e.limit, e.n_groups, e.group_rows, e.group_x_div, e.group_of, e.group_used = self.limit, self.groups, tile, x_div, _ptr(group_of), _ptr(used)
        e.glu, e.row_scale = self.glu, _ptr(row_scale)
        if self.dtype == torch.float32:
            check(L.pt_gemm_f32(_ptr(x), self.ld, _ptr(self.w), self.ld, rows, self.n_out, self.k_in, 1.0, epilogue, _ptr(out), out_ld, ctypes.byref(e), _stream()),
                  "pt_gemm_f32")
        elif tile == 1:
            a = LinearArgs()
            a.wfmt, a.batch, a.n_out, a.k_in, a.epilogue, a.x, a.packed_w = W_BF16, rows, self.n_out, self.ld, epilogue, _ptr(x), _ptr(self.skinny)
            a.out, a.out_ld, a.out_dtype, a.alpha, a.error_flag = _ptr(out), out_ld, dtype_code(out.dtype), 1.0, _ptr(error_flag)
            a.workspace, a.workspace_bytes = _ptr(linear_ws), linear_ws.numel() if linear_ws is not None else 0
            a.ext, a.pdl = ctypes.pointer(e), pdl
            check(L.pt_linear(ctypes.byref(a), _stream()), "pt_linear")
        else:
            a = GemmArgs()
            a.wfmt, a.m, a.n_out, a.k_in, a.epilogue, a.w_tiled, a.x, a.w = W_BF16, rows, self.n_out, self.ld, epilogue, 1, _ptr(x), _ptr(self.tiled)
            a.out, a.out_ld, a.out_dtype, a.alpha, a.error_flag = _ptr(out), out_ld, dtype_code(out.dtype), 1.0, _ptr(error_flag)
            a.workspace, a.workspace_bytes = _ptr(gemm_ws), gemm_ws.numel() if gemm_ws is not None else 0
            a.ext, a.pdl = ctypes.pointer(e), pdl
            check(L.pt_gemm(ctypes.byref(a), _stream()), "pt_gemm")


# ------------------------------------------------------------------------------------------ layers with per-sequence positions
def batch_view(n_seq, n_tok, cu, start, slot, tok_seq):
    """The packed tokens of one launch (pt_batch_view): device int32 tensors."""
    v = BatchView()
    v.n_seq, v.n_tok = n_seq, n_tok
    v.cu, v.start, v.slot, v.tok_seq = _ptr(cu), _ptr(start), _ptr(slot), _ptr(tok_seq)
    v.keep = (cu, start, slot, tok_seq)
    return v


def hyper(xs, rows, eps, norm_w=None, h=None, h_ld=0, w_in=None, y=None, y_ld=0, mix=None, w_out=None, mult=1.0, table=None, ids=None, ids_ld=1,
          step=None, pos_out=None, row_index=None, sum_out=None, vocab=0):
    """Hyper-connection step on the fp32 streams xs [rows, streams, width] (see pt_hyper): write the finished sublayer's y, read and
    normalise the next one's input into h.  `table` starts tokens from an embedding table instead."""
    a = HyperArgs()
    a.rows, a.width, a.streams = rows, xs.shape[2], xs.shape[1]
    a.dtype = dtype_code(h.dtype if h is not None else (table.dtype if table is not None else torch.float32))
    a.eps, a.mult, a.xs = float(eps), float(mult), _ptr(xs)
    if table is not None:
        a.table, a.table_ld, a.vocab = _ptr(table), table.shape[1], vocab or table.shape[0]
        a.ids, a.ids_ld, a.step_dev, a.pos_out = _ptr(ids), ids_ld, _ptr(step), _ptr(pos_out)
    a.row_index, a.y, a.y_ld, a.mix, a.w_out, a.w_in = _ptr(row_index), _ptr(y), y_ld, _ptr(mix), _ptr(w_out), _ptr(w_in)
    a.norm_w, a.h, a.h_ld, a.sum_out = _ptr(norm_w), _ptr(h), h_ld, _ptr(sum_out)
    check(_lib.lib().pt_hyper(ctypes.byref(a), _stream()), "pt_hyper")


def window_attn_workspace(n_seq, n_head, vdim, page_size, max_len, window, keep_first, device="cuda"):
    n = _lib.lib().pt_window_attn_workspace_bytes(n_seq, n_head, vdim, page_size, max_len, window, keep_first)
    return torch.zeros(n, dtype=torch.uint8, device=device)


def window_attn(view, qkv, qkv_ld, cache, out, out_ld, n_head, scale, window=0, keep_first=0, sink=None, append=True, max_tokens_per_seq=0,
                workspace=None, error_flag=None, plain=False, values_are_keys=False, q_norm=None, k_norm=None, eps=0.0, rope=None, rope_dims=0, out_scale=1.0,
                out_cols=0, softcap=0.0, gate=None, gate_ld=0, gate_per_head=False, context=None):
    """Masked attention of the packed tokens of `view` over a paged cache (see pt_window_attn).  qkv rows hold [q | k | v]
    (append=True: k and v go to the cache first), [q | k] (values_are_keys: the keys as they are in the row are the values) or only q
    (a layer that reads another layer's cache).  q_norm, k_norm, rope: per-head norm and rotation of q and k; q is then rewritten.  gate: rows
    whose sigmoid multiplies the output (a view that starts at its first column).  context: an object with k, v, shared, ld, shared_dim
    and cu that names rows of the whole context as keys and values of a prompt, in place of the cache's pages (see pt_context_rows)."""
    a = WindowAttnArgs()
    a.batch, a.dtype = view, dtype_code(qkv.dtype)
    a.n_head, a.n_kv, a.dim, a.vdim = n_head, cache.n_kv, cache.head_dim, cache.v_dim
    a.page_size, a.max_pages, a.max_len = cache.page_size, cache.page_table.shape[1], cache.max_len
    a.window, a.keep_first, a.scale, a.sink = window, keep_first, float(scale), _ptr(sink)
    a.q, a.q_ld, a.kv_ld = _ptr(qkv), qkv_ld, qkv_ld
    if append:
        k = qkv.data_ptr() + n_head * cache.head_dim * qkv.element_size()
        a.k, a.v = k, k if values_are_keys else k + cache.n_kv * cache.head_dim * qkv.element_size()
    a.q_norm, a.k_norm, a.norm_eps, a.rope, a.rope_dims = _ptr(q_norm), _ptr(k_norm), float(eps), _ptr(rope), rope_dims
    a.out_scale, a.out_cols = float(out_scale), out_cols
    a.softcap, a.gate, a.gate_ld, a.gate_per_head = float(softcap), gate.data_ptr() if gate is not None else None, gate_ld, 1 if gate_per_head else 0
    if context is not None:
        c = ContextRows()
        c.k, c.v, c.shared, c.ld, c.shared_ld, c.shared_dim, c.cu = context.k.data_ptr(), context.v.data_ptr(), context.shared.data_ptr(), context.ld, context.shared_dim, context.shared_dim, _ptr(context.cu)
        a.n_kv, a.dim, a.vdim, a.context = n_head, context.dim, context.vdim, ctypes.pointer(c)
    a.pool, a.page_table, a.out, a.out_ld = _ptr(cache.pool), _ptr(cache.page_table), _ptr(out), out_ld
    a.max_tokens_per_seq, a.plain = max_tokens_per_seq, 1 if plain else 0
    a.workspace, a.workspace_bytes = _ptr(workspace), workspace.numel() if workspace is not None else 0
    a.error_flag = _ptr(error_flag)
    check(_lib.lib().pt_window_attn(ctypes.byref(a), _stream()), "pt_window_attn")


def latent_cache(rows, w, max_len, page_size=64, device="cuda", page_table=None, dtype=torch.bfloat16, n_pages=None):
    """Page pool of a latent attention layer: per position one row [rotated key part | latent] and padding."""
    return PagedKVCache(rows, 1, _lib.lib().pt_latent_row(w.rot_dim, w.rank), max_len, page_size, device, page_table, v_dim=0, dtype=dtype, n_pages=n_pages)


def latent_prep(view, rows, ld, q_col, kv_col, w, cq, cq_ld, cache, eps, rope, error_flag=None):
    """Norms of both latents, rotation of the shared key part, append (see pt_latent_prep).  q_col, kv_col: first columns of the query latent
    and of [latent | key part] in `rows` (kv_col None: the layer reads what another one caches); w: an object with q_rank, rank, rot_dim and the fp32 tensors q_norm, kv_norm."""
    a = LatentPrepArgs()
    es = rows.element_size()
    a.batch, a.dtype, a.q_rank, a.rank, a.rot_dim, a.eps = view, dtype_code(rows.dtype), w.q_rank, w.rank, w.rot_dim, float(eps)
    a.q, a.kv, a.ld = rows.data_ptr() + q_col * es, None if kv_col is None else rows.data_ptr() + kv_col * es, ld
    a.q_norm, a.kv_norm, a.rope, a.cq, a.cq_ld = _ptr(w.q_norm), None if kv_col is None else _ptr(w.kv_norm), _ptr(rope), _ptr(cq), cq_ld
    a.pool, a.page_table, a.page_size, a.max_pages, a.max_len = _ptr(cache.pool), _ptr(cache.page_table), cache.page_size, cache.page_table.shape[1], cache.max_len
    a.error_flag = _ptr(error_flag)
    check(_lib.lib().pt_latent_prep(ctypes.byref(a), _stream()), "pt_latent_prep")


def latent_context(view, ctx_cu, n_ctx, w, cache, shared, latent, latent_ld):
    """The cached rows of every sequence's context, one after the other (see pt_latent_context)."""
    a = LatentContextArgs()
    a.batch, a.ctx_cu, a.n_ctx, a.rot_dim, a.rank = view, _ptr(ctx_cu), n_ctx, w.rot_dim, w.rank
    a.page_size, a.max_pages, a.pool, a.page_table = cache.page_size, cache.page_table.shape[1], _ptr(cache.pool), _ptr(cache.page_table)
    a.shared, a.latent, a.latent_ld = _ptr(shared), _ptr(latent), latent_ld
    check(_lib.lib().pt_latent_context(ctypes.byref(a), _stream()), "pt_latent_context")


def latent_workspace_bytes(n_tok, w, dtype):
    return _lib.lib().pt_latent_attn_workspace_bytes(n_tok, w.heads, w.rot_dim, w.rank, dtype_code(dtype))


def latent_attn(view, q, q_ld, w, cache, out, out_ld, scale, rope, workspace, gate=None, gate_ld=0, out_cols=0, error_flag=None, plain=False, gate_per_value=False):
    """Attention over the cached latents (see pt_latent_attn).  w: an object with heads, dim, rot_dim, vdim, rank and the tensors w_k [heads,
    rank, dim] and w_v [heads, vdim, rank].  gate: a view that starts at the heads' gates (gate_per_value: one per output)."""
    a = LatentAttnArgs()
    a.batch, a.dtype, a.n_head, a.dim, a.rot_dim, a.vdim, a.rank, a.scale = view, dtype_code(q.dtype), w.heads, w.dim, w.rot_dim, w.vdim, w.rank, float(scale)
    a.q, a.q_ld, a.rope, a.w_k, a.w_v = _ptr(q), q_ld, _ptr(rope), _ptr(w.w_k), _ptr(w.w_v)
    a.gate, a.gate_ld, a.gate_per_value = gate.data_ptr() if gate is not None else None, gate_ld, 1 if gate_per_value else 0
    a.pool, a.page_table, a.page_size, a.max_pages, a.max_len = _ptr(cache.pool), _ptr(cache.page_table), cache.page_size, cache.page_table.shape[1], cache.max_len
    a.out, a.out_ld, a.out_cols, a.plain, a.error_flag = _ptr(out), out_ld, out_cols, 1 if plain else 0, _ptr(error_flag)
    a.workspace, a.workspace_bytes = _ptr(workspace), workspace.numel()
    check(_lib.lib().pt_latent_attn(ctypes.byref(a), _stream()), "pt_latent_attn")


def ssm(view, zx, zx_ld, out, out_ld, w, ring, state, y, xbc=None, dt=None, workspace=None, plain=False):
    """State-space mixer between its projections (see pt_ssm).  w: an object with heads, vdim, state, groups, taps, norm_groups, eps
    and the fp32 tensors conv_w, conv_b, dt_bias, A_log, D, norm_w."""
    a = SsmArgs()
    a.batch, a.dtype = view, dtype_code(zx.dtype)
    a.heads, a.vdim, a.state_dim, a.groups, a.taps, a.norm_groups, a.eps = w.heads, w.vdim, w.state, w.groups, w.taps, w.norm_groups, float(w.eps)
    a.zx, a.zx_ld, a.out, a.out_ld = _ptr(zx), zx_ld, _ptr(out), out_ld
    a.conv_w, a.conv_b, a.dt_bias, a.A_log, a.D, a.norm_w = (_ptr(t) for t in (w.conv_w, w.conv_b, w.dt_bias, w.A_log, w.D, w.norm_w))
    a.ring, a.state, a.xbc, a.dt, a.y = _ptr(ring), _ptr(state), _ptr(xbc), _ptr(dt), _ptr(y)
    a.plain = 1 if plain else 0
    a.workspace, a.workspace_bytes = _ptr(workspace), workspace.numel() if workspace is not None else 0
    check(_lib.lib().pt_ssm(ctypes.byref(a), _stream()), "pt_ssm")


def mlstm(view, rows, ld, cols, gates, gate_ld, out, out_ld, w, state, nm, y, workspace, out_scale=1.0, out_cols=0, plain=False):
    """Matrix memory between its projections (see pt_mlstm).  cols: first columns of q, k, v and the output gate in `rows`; gates: fp32
    rows [log input | log forget]; w: an object with heads, dim, vdim, cap, eps and the fp32 tensor norm_w.  out: a view that starts
    at the output's first column."""
    a = MlstmArgs()
    es = rows.element_size()
    a.batch, a.dtype, a.heads, a.dim, a.vdim = view, dtype_code(rows.dtype), w.heads, w.dim, w.vdim
    a.gate_cap, a.q_scale, a.eps, a.out_scale = float(w.cap), float(w.dim) ** -0.5, float(w.eps), float(out_scale)
    a.q, a.k, a.v, a.gate = (rows.data_ptr() + c * es for c in cols)
    a.ld, a.log_i, a.log_f, a.gate_ld = ld, gates.data_ptr(), gates.data_ptr() + w.heads * 4, gate_ld
    a.norm_w, a.state, a.nm, a.y = _ptr(w.norm_w), _ptr(state), _ptr(nm), _ptr(y)
    a.out, a.out_ld, a.out_cols, a.plain = out.data_ptr(), out_ld, out_cols, 1 if plain else 0
    a.workspace, a.workspace_bytes = _ptr(workspace), workspace.numel() if workspace is not None else 0
    check(_lib.lib().pt_mlstm(ctypes.byref(a), _stream()), "pt_mlstm")


def post_norm(rows, width, eps, dtype, x_in=None, x_out=None, y=None, y_ld=0, pair_y=None, pair_ld=0, top=0, pair_w=None, pair_row=None, norm_w=None,
              final_w=None, h=None, h_ld=0, row_index=None, table=None, vocab=0, ids=None, ids_ld=1, step=None, pos_out=None, id_out=None, h_cols=0,
              copy=None, copy_ld=0, copy_cols=0):
    """Residual step with a norm on the sublayer's output, on the next one's input or both (see pt_post_norm), or the start of a token
    from an embedding table.  copy: a view that starts at the first column of the second copy."""
    a = PostNormArgs()
    a.rows, a.width, a.dtype, a.eps, a.x_in, a.x_out = rows, width, dtype_code(dtype), float(eps), _ptr(x_in), _ptr(x_out)
    if table is not None:
        a.table, a.table_ld, a.vocab, a.ids, a.ids_ld = _ptr(table), table.shape[1], vocab or table.shape[0], _ptr(ids), ids_ld
        a.step_dev, a.pos_out, a.id_out = _ptr(step), _ptr(pos_out), _ptr(id_out)
    a.row_index, a.y, a.y_ld = _ptr(row_index), _ptr(y), y_ld
    if pair_y is not None:
        a.pair_dtype = dtype_code(pair_y.dtype)
    a.pair_y, a.pair_ld, a.top, a.pair_w, a.pair_row = _ptr(pair_y), pair_ld, top, _ptr(pair_w), _ptr(pair_row)
    a.norm_w, a.final_w, a.h, a.h_ld, a.h_cols = _ptr(norm_w), _ptr(final_w), _ptr(h), h_ld, h_cols
    a.copy, a.copy_ld, a.copy_cols = copy.data_ptr() if copy is not None else None, copy_ld, copy_cols
    check(_lib.lib().pt_post_norm(ctypes.byref(a), _stream()), "pt_post_norm")


def shift_norm(view, rows, width, groups, eps, dtype, x_in=None, x_out=None, y=None, y_ld=0, pair_y=None, pair_ld=0, top=0, pair_w=None, pair_row=None, self_rows=None,
               self_ld=0, w1=None, shift=None, h1=None, h1_ld=0, state_in=None, state_out=None, state_by_seq=False, w2=None, h2=None, h2_ld=0, row_index=None, table=None, vocab=0,
               ids=None, ids_ld=1, step=None, pos_out=None, embed_w=None):
    """Residual step with two grouped norms of the stream, the first mixed with the token before, or the start of a token from an embedding
    table (see pt_shift_norm).  view: needed with h1.  self_rows: what the experts without matrices give back."""
    a = ShiftNormArgs()
    if view is not None:
        a.batch = view
    a.rows, a.width, a.groups, a.dtype, a.eps, a.x_in, a.x_out = rows, width, groups, dtype_code(dtype), float(eps), _ptr(x_in), _ptr(x_out)
    if table is not None:
        a.table, a.table_ld, a.vocab, a.ids, a.ids_ld = _ptr(table), table.shape[1], vocab or table.shape[0], _ptr(ids), ids_ld
        a.step_dev, a.pos_out, a.embed_w = _ptr(step), _ptr(pos_out), _ptr(embed_w)
    a.row_index, a.y, a.y_ld = _ptr(row_index), _ptr(y), y_ld
    if pair_y is not None:
        a.pair_dtype = dtype_code(pair_y.dtype)
    a.pair_y, a.pair_ld, a.top, a.pair_w, a.pair_row, a.self, a.self_ld = _ptr(pair_y), pair_ld, top, _ptr(pair_w), _ptr(pair_row), _ptr(self_rows), self_ld
    a.w1, a.shift, a.h1, a.h1_ld, a.state_in, a.state_out, a.state_by_seq = _ptr(w1), _ptr(shift), _ptr(h1), h1_ld, _ptr(state_in), _ptr(state_out), 1 if state_by_seq else 0
    a.w2, a.h2, a.h2_ld = _ptr(w2), _ptr(h2), h2_ld
    check(_lib.lib().pt_shift_norm(ctypes.byref(a), _stream()), "pt_shift_norm")


def moe_max_tiles(n_tok, experts, top, tile):
    return int(_lib.lib().pt_moe_max_tiles(n_tok, experts, top, tile))


def moe_route(logits, n_tok, experts, top, expert, weight, tile=0, pair_row=None, tile_expert=None, tile_rows=None, row_token=None, counts=None, h=None, h_ld=0, gathered=None,
              score=MOE_SOFTMAX, row_weight=None, correction=None, groups=0, keep=0, identity=0):
    """Experts and weights of every token, and with `tile` the rows of the grouped products (see pt_moe_route)."""
    a = MoeRouteArgs()
    a.n_tok, a.experts, a.top, a.logits, a.logits_ld = n_tok, experts, top, _ptr(logits), logits.shape[-1]     # experts: those with matrices
    a.expert, a.weight, a.tile, a.score, a.row_weight = _ptr(expert), _ptr(weight), tile, score, _ptr(row_weight)
    a.correction, a.groups, a.keep, a.identity, a.pair_row = _ptr(correction), groups, keep, identity, _ptr(pair_row)
    if tile:
        a.max_tiles = moe_max_tiles(n_tok, experts, top, tile)
        a.tile_expert, a.tile_rows, a.row_token = _ptr(tile_expert), _ptr(tile_rows), _ptr(row_token)
        a.counts = _ptr(counts)
        if h is not None:
            a.h, a.h_bytes, a.gathered = _ptr(h), h_ld * h.element_size(), _ptr(gathered)
    check(_lib.lib().pt_moe_route(ctypes.byref(a), _stream()), "pt_moe_route")


# ------------------------------------------------------------------------------------------ norms / softmax
def layer_norm_ce(x, gamma, beta, eps, batch_size=None, sequence_length=None, input_size=None):
    """ops.layer_norm_ce (customized.py:69-102): LayerNorm over the last dim with the NormCE arithmetic."""
    dim = x.shape[-1]
    rows = x.numel() // dim
    out = torch.empty_like(x)
    check(_lib.lib().pt_norm_ce(_ptr(x), _ptr(gamma), _ptr(beta), rows, dim, float(eps), _ptr(out), _stream()), "NormCE")
    return out


def rms_norm(x, gamma, eps, residual=None):
    """RMSLayerNorm (layers/rms_layer_norm.py:26-36); with `residual` returns (norm(x + residual), x + residual)."""
    dim = x.shape[-1]
    rows = x.numel() // dim
    out = torch.empty_like(x)
    s = torch.empty_like(x) if residual is not None else None
    check(_lib.lib().pt_rms_norm(_ptr(x), _ptr(residual), _ptr(gamma), rows, dim, float(eps), _ptr(out), _ptr(s), _stream()), "pt_rms_norm")
    return (out, s) if residual is not None else out


def softmax_ce(x, dim=-1, stable_mode=True):
    """ops.softmax_ce (customized.py:57-65) over the last axis; fp16 or fp32 input."""
    if dim not in (-1, x.dim() - 1):
        raise PtError("SoftmaxV3: only the last axis is supported (the reference flattens to [rows, last])")
    n = x.shape[-1]
    out = torch.empty_like(x)
    dt = {torch.float16: 0, torch.float32: 1}.get(x.dtype)
    if dt is None:
        raise PtError("SoftmaxV3: dtype must be fp16 or fp32")
    check(_lib.lib().pt_softmax(_ptr(x), x.numel() // n, n, 1 if stable_mode else 0, dt, _ptr(out), _stream()), "SoftmaxV3")
    return out


# ------------------------------------------------------------------------------------------ KV cache (reference layout)
class KVCacheOp:
    """One `KVCache` call site: owns the persistent cache like the reference op instance
    (custom_ops/kv_cache.cpp:108-116), re-zeroed when step == 0."""

    def __init__(self, max_len, sequence_axis, step_len=1, fp8=False, fp8_scale=1.0):
        """fp8=True is the op's `fp8` attribute (customized.py:32; kv_cache.cpp:100-104, :183-185): the cache is kept as 8-bit floats
        (E4M3 bytes of updater / fp8_scale) and returned cast back to fp16."""
        self.max_len, self.axis, self.step_len = max_len, sequence_axis, step_len
        self.fp8, self.fp8_scale = bool(fp8), float(fp8_scale)
        self.cache = self.scratch = None

    def __call__(self, step, updater):
        shape = list(updater.shape)
        if shape[self.axis] != self.step_len:
            raise PtError(f"KVCache: updater has {shape[self.axis]} positions on axis {self.axis}, step_len is {self.step_len}")
        outer = 1
        for d in shape[: self.axis]:
            outer *= d
        inner = 1
        for d in shape[self.axis + 1:]:
            inner *= d
        shape[self.axis] = self.max_len
        if self.fp8:
            if self.cache is None:
                self.cache = torch.zeros(shape, dtype=torch.uint8, device=updater.device)
            out = torch.empty(shape, dtype=torch.float16, device=updater.device)
            check(_lib.lib().pt_kv_cache_fp8(_ptr(step), _ptr(updater), _ptr(self.cache), _ptr(out), self.fp8_scale, outer, self.max_len,
                                             self.step_len, inner, _stream()), "KVCache")
            return out
        if self.cache is None:
            self.cache = torch.zeros(shape, dtype=updater.dtype, device=updater.device)
            self.scratch = torch.empty_like(self.cache)
        check(_lib.lib().pt_kv_cache(_ptr(step), _ptr(updater), _ptr(self.cache), _ptr(self.scratch), outer, self.max_len,
                                     self.step_len, inner, _stream()), "KVCache")
        return self.cache


def kv_cache(state, step, updater):
    """ops.kv_cache (customized.py:21-35) with the op instance's state made explicit."""
    return state(step, updater)


class KVCachePipelineOp:
    """One `KVCachePipeline` call site (custom_ops/kv_cache_pipeline.cpp:374-451): `max_bps` caches, cache step % max_bps receives the
    shifted insert and is returned.  transpose=1 is the op's second storage layout (kv_cache_pipeline.hpp:107-113, vertex
    GetBpsKvCacheLastDim, kv_cache_codelet.cpp:170-212): the caches are kept as [..., H, max_len] and shifted along their LAST
    dimension; the op returns the tensor transposed back (kv_cache_pipeline.cpp:441-446), so callers see the same values."""

    def __init__(self, max_len, max_bps, sequence_axis, step_len=1, transpose=0, fp8=False, fp8_scale=1.0):
        """fp8=True: the caches hold E4M3 bytes of updater / fp8_scale and the op returns fp16 (kv_cache_pipeline.cpp:386-388, :437-439)."""
        self.max_len, self.max_bps, self.axis, self.step_len, self.transpose = max_len, max_bps, sequence_axis, step_len, int(transpose)
        self.fp8, self.fp8_scale = bool(fp8), float(fp8_scale)
        self.caches = None

    def __call__(self, step, updater):
        shape = list(updater.shape)
        if self.axis != len(shape) - 2:
            raise PtError("KVCachePipeline: sequence_axis must be rank - 2 (kv_cache_pipeline.hpp:83-88)")
        if shape[self.axis] != self.step_len:
            raise PtError(f"KVCachePipeline: updater has {shape[self.axis]} positions on axis {self.axis}, step_len is {self.step_len}")
        if self.transpose:
            upd = updater.transpose(-1, -2).contiguous()           # [..., H, step_len]: the sequence is the last dimension
            outer, inner = upd.numel() // self.step_len, 1
            store = list(upd.shape[:-1]) + [self.max_len]
        else:
            upd = updater
            outer = 1
            for d in shape[: self.axis]:
                outer *= d
            inner = shape[-1]
            store = shape[: self.axis] + [self.max_len, shape[-1]]
        if self.caches is None:
            self.caches = torch.zeros([self.max_bps] + store, dtype=torch.uint8 if self.fp8 else updater.dtype, device=updater.device)
        out = torch.empty(store, dtype=updater.dtype, device=updater.device)
        if self.fp8:
            check(_lib.lib().pt_kv_cache_pipeline_fp8(_ptr(step), _ptr(upd), _ptr(self.caches), _ptr(out), self.fp8_scale, self.max_bps, outer,
                                                      self.max_len, self.step_len, inner, _stream()), "KVCachePipeline")
        else:
            check(_lib.lib().pt_kv_cache_pipeline(_ptr(step), _ptr(upd), _ptr(self.caches), _ptr(out), self.max_bps, outer, self.max_len,
                                                  self.step_len, inner, _stream()), "KVCachePipeline")
        return out.transpose(-1, -2).contiguous() if self.transpose else out


def kv_cache_pipeline(state, step, updater):
    return state(step, updater)


# ------------------------------------------------------------------------------------------ paged cache + attention
class PagedKVCache:
    """Page pool of one layer plus the (shared) page table.  pool[page][2][n_kv][page_size][head_dim]; with a value width of its own
    (v_dim) a page is K [n_kv][page_size][head_dim] followed by V [n_kv][page_size][v_dim].  n_pages: size of the pool where pages
    are handed out on demand (cache.SequenceSlots) instead of max_len tokens per row."""

    def __init__(self, rows, n_kv, head_dim, max_len, page_size=64, device="cuda", page_table=None, extra_pages=0, v_dim=None, dtype=torch.float16,
                 n_pages=None):
        self.rows, self.n_kv, self.head_dim, self.page_size = rows, n_kv, head_dim, page_size
        self.v_dim = head_dim if v_dim is None else v_dim
        self.max_len = max_len
        self.max_pages = (max_len + page_size - 1) // page_size
        n_pages = (rows * self.max_pages if n_pages is None else n_pages) + extra_pages
        shape = (n_pages, 2, n_kv, page_size, head_dim) if self.v_dim == head_dim else (n_pages, n_kv * page_size * (head_dim + self.v_dim))
        self.pool = torch.zeros(shape, dtype=dtype, device=device)
        if page_table is None:
            page_table = torch.arange(rows * self.max_pages, dtype=torch.int32, device=device).reshape(rows, self.max_pages)
        self.page_table = page_table

    def export(self, step, max_len):
        """Reference-layout view [2, rows, n_kv, max_len, head_dim], newest first, zeros beyond step."""
        out = torch.empty((2, self.rows, self.n_kv, max_len, self.head_dim), dtype=torch.float16, device=self.pool.device)
        check(_lib.lib().pt_kv_export(_ptr(self.pool), _ptr(self.page_table), _ptr(step), self.rows, self.n_kv, self.head_dim,
                                      self.page_size, self.max_pages, max_len, _ptr(out), _stream()), "pt_kv_export")
        return out


def attn_workspace(batch, n_head, head_dim, max_pages, device="cuda"):
    n = _lib.lib().pt_attn_workspace_bytes(batch, n_head, head_dim, max_pages)
    return torch.zeros(n, dtype=torch.uint8, device=device)


def attn_args(qkv, step, cache, out, n_head, rope_mode, softmax_mode, score_scale, rope_sin, rope_cos, workspace, error_flag, pdl=0,
              out_fp8=None, out_fp8_scale=0.0):
    a = AttnArgs()
    a.batch, a.n_head, a.n_kv, a.head_dim = qkv.shape[0], n_head, cache.n_kv, cache.head_dim
    a.page_size, a.max_pages, a.rope_mode, a.softmax_mode = cache.page_size, cache.max_pages, rope_mode, softmax_mode
    a.score_scale = score_scale
    a.step_dev, a.qkv, a.rope_sin, a.rope_cos = _ptr(step), _ptr(qkv), _ptr(rope_sin), _ptr(rope_cos)
    a.pool, a.page_table, a.out, a.out_ld = _ptr(cache.pool), _ptr(cache.page_table), _ptr(out), 0
    a.workspace, a.workspace_bytes = _ptr(workspace), workspace.numel()
    a.error_flag = _ptr(error_flag)
    a.pdl = pdl
    a.max_len = cache.max_len
    a.out_fp8, a.out_fp8_scale = _ptr(out_fp8), float(out_fp8_scale)
    return a


def kv_append_attn(qkv, step, cache, n_head, rope_mode=ROPE_NONE, softmax_mode=SOFTMAX_F32, score_scale=1.0, rope_sin=None,
                   rope_cos=None, workspace=None, error_flag=None, out=None):
    """RoPE + KV append + decode attention for one new token per row.  qkv fp16 [rows, (n_head + 2 n_kv) * H]."""
    if out is None:
        out = torch.empty((qkv.shape[0], n_head * cache.head_dim), dtype=torch.float16, device=qkv.device)
    if workspace is None:
        workspace = attn_workspace(qkv.shape[0], n_head, cache.head_dim, cache.max_pages, qkv.device)
    a = attn_args(qkv, step, cache, out, n_head, rope_mode, softmax_mode, score_scale, rope_sin, rope_cos, workspace, error_flag)
    check(_lib.lib().pt_kv_append_attn(ctypes.byref(a), _stream()), "pt_kv_append_attn")
    return out


def prefill_attn(qkv, cache, batch, n_tokens, start, n_head, score_scale, rope_sin, rope_cos, out=None):
    """Causal attention over a whole prompt chunk (the reference's sequence_length != 1 attention, llama2/attention.py:64-114):
    qkv fp16 [batch * n_tokens, 3 * n_head * H], row b * n_tokens + t = position start + t of sequence b.  Rotates q in place,
    appends rotated k and v to the paged cache and returns softmax(q K^T * scale + causal mask) V, [batch * n_tokens, n_head * H]."""
    if qkv.shape != (batch * n_tokens, 3 * n_head * cache.head_dim) or cache.n_kv != n_head:
        raise PtError(f"prefill_attn: qkv {tuple(qkv.shape)} does not match batch={batch} n_tokens={n_tokens} n_head={n_head} (no grouped KV heads)")
    if out is None:
        out = torch.empty((batch * n_tokens, n_head * cache.head_dim), dtype=torch.float16, device=qkv.device)
    a = _lib.PrefillAttnArgs()
    a.batch, a.n_tokens, a.start, a.n_head, a.head_dim = batch, n_tokens, start, n_head, cache.head_dim
    a.page_size, a.max_pages, a.max_len, a.score_scale = cache.page_size, cache.max_pages, cache.max_len, score_scale
    a.qkv, a.rope_sin, a.rope_cos, a.pool, a.page_table, a.out = _ptr(qkv), _ptr(rope_sin), _ptr(rope_cos), _ptr(cache.pool), _ptr(cache.page_table), _ptr(out)
    check(_lib.lib().pt_prefill_attn(ctypes.byref(a), _stream()), "pt_prefill_attn")
    return out


# ------------------------------------------------------------------------------------------ top-k / beam search
def topk(x, k, axis=-1):
    """ops.topk (popart.py:135-137) on the last axis: (values, int32 indices), ties -> lowest index."""
    if axis not in (-1, x.dim() - 1):
        raise PtError("topk: only the last axis is supported")
    dim = x.shape[-1]
    rows = x.numel() // dim
    dt = {torch.float16: 0, torch.float32: 1}[x.dtype]
    vals = torch.empty(x.shape[:-1] + (k,), dtype=x.dtype, device=x.device)
    ids = torch.empty(x.shape[:-1] + (k,), dtype=torch.int32, device=x.device)
    check(_lib.lib().pt_topk(_ptr(x), rows, dim, k, dt, _ptr(vals), _ptr(ids), _stream()), "topk")
    return vals, ids


def beam_search(logits, hyp_container, prob_container, step, beam_size, parent=None, workspace=None):
    """`BeamSearch` custom op (beam_search_custom_op.cpp:333-478).  logits [B, beam, V]; hyp int32
    [B, max_len, beam] and prob [B, beam] are updated in place.  Returns (next_id, global_best_id, hyp, prob)."""
    b, beam, vocab = logits.shape
    if beam != beam_size:
        raise PtError("BeamSearch: logits.shape[1] must equal beam_size")
    max_len = hyp_container.shape[1]
    dt = {torch.float16: 0, torch.float32: 1}[logits.dtype]
    L = _lib.lib()
    if workspace is None:
        workspace = torch.empty(L.pt_beam_search_workspace_bytes(b, beam, max_len), dtype=torch.uint8, device=logits.device)
    next_id = torch.empty((b, beam), dtype=torch.int32, device=logits.device)
    gbest = torch.empty((b, beam), dtype=torch.int32, device=logits.device)
    check(L.pt_beam_search(_ptr(logits), _ptr(hyp_container), _ptr(prob_container), _ptr(step), b, beam, vocab, max_len, dt,
                           _ptr(next_id), _ptr(gbest), _ptr(parent), _ptr(workspace), workspace.numel(), _stream()), "BeamSearch")
    return next_id, gbest, hyp_container, prob_container


# ------------------------------------------------------------------------------------------ FP8
def _require_e4m3(op, fp8_format):
    """The reference's formats are Graphcore's F143 / F152 (exponent bias and range differ from OCP E4M3, the arithmetic is
    closed): bytes in those formats would decode to other values here, so they are refused instead of silently misread."""
    if fp8_format in ("F143", "F152"):
        raise PtError(f"{op}: Graphcore {fp8_format} bytes are not OCP E4M3 and are not supported; re-quantise the fp16/fp32 tensor "
                      "with poptransformer_b200.quant.quantize_fp8 (E4M3, per-tensor scale amax/448)")
    if fp8_format != "E4M3":
        raise PtError(f"{op}: unsupported format {fp8_format}")


def half_to_uint8(x, fp8_scale, fp8_format="E4M3"):
    """ops.half_to_uint8 (customized.py:127-135) with OCP E4M3 and a float per-tensor scale."""
    _require_e4m3("CastToUint8", fp8_format)
    out = torch.empty(x.shape, dtype=torch.uint8, device=x.device)
    check(_lib.lib().pt_cast_fp8(_ptr(x), float(fp8_scale), x.numel(), _ptr(out), _stream()), "CastToUint8")
    return out


def fp8_matmul(input_l, input_r, fp8_scale_lhs, fp8_scale_rhs, fp8_format_lhs="E4M3", fp8_format_rhs="E4M3"):
    """ops.fp8_matmul (customized.py:137-148): input_l e4m3 [m, k], input_r e4m3 [n, k] (k contiguous) -> fp16 [m, n]."""
    _require_e4m3("FP8MatMul", fp8_format_lhs)
    _require_e4m3("FP8MatMul", fp8_format_rhs)
    m, k = input_l.shape
    n = input_r.shape[0]
    out = torch.empty((m, n), dtype=torch.float16, device=input_l.device)
    check(_lib.lib().pt_fp8_matmul(_ptr(input_l), _ptr(input_r), float(fp8_scale_lhs), float(fp8_scale_rhs), m, n, k, _ptr(out), _stream()),
          "FP8MatMul")
    return out


# ------------------------------------------------------------------------------------------ misc
def wkv(k, v, time_first, time_decay, num, den, max_state):
    out = torch.empty_like(k)
    b, c = k.shape
    check(_lib.lib().pt_wkv(_ptr(k), _ptr(v), _ptr(time_first), _ptr(time_decay), _ptr(num), _ptr(den), _ptr(max_state), b, c, _ptr(out),
                            _stream()), "pt_wkv")
    return out


def embedding(table, ids, step=None, out=None):
    """ids int32 [batch, stride]; gathers table[ids[b, *step]] (step None -> column 0)."""
    batch, stride = ids.shape
    vocab, dim = table.shape
    if out is None:
        out = torch.empty((batch, dim), dtype=table.dtype, device=table.device)
    check(_lib.lib().pt_embedding(_ptr(table), _ptr(ids), stride, _ptr(step), batch, dim, vocab, _ptr(out), _stream()), "pt_embedding")
    return out


def step_containers(ids, step, next_ids, pad_id, eos_id=-1, stop_mask=None, done_flag=None):
    """step_containers + step_loop_cond (models/base_model.py:313-355).  With `done_flag` (device int32, zeroed per generation)
    the reference's early stop applies: the flag is set by the iteration that found every sequence already stopped, and the
    calls after it change nothing."""
    batch, max_len = ids.shape
    if done_flag is None:
        check(_lib.lib().pt_step_containers(_ptr(ids), batch, max_len, _ptr(step), _ptr(next_ids), int(pad_id), int(eos_id), _ptr(stop_mask),
                                            _stream()), "pt_step_containers")
    else:
        check(_lib.lib().pt_step_containers_early_stop(_ptr(ids), batch, max_len, _ptr(step), _ptr(next_ids), int(pad_id), int(eos_id),
                                                       _ptr(stop_mask), _ptr(done_flag), _stream()), "pt_step_containers_early_stop")


def lm_head_tp_merge(dec):
    """TPLMHead.__call__ after the matmul (layers/lm_head.py:86-115) for a decoder holding its vocab shard's logits: exact-zero
    logits -> -10000, local top-1, + rank * vocab_per_rank, all-gather of (value, id) over the TP group, arg-max over ranks.
    Uses the decoder's logits, next_val, next_ids, gather_val, gather_ids, vocab_loc, rank, tp and group."""
    L = _lib.lib()
    check(L.pt_lm_head_local_topk(_ptr(dec.logits), dec.batch, dec.vocab_loc, dec.rank * dec.vocab_loc, _ptr(dec.next_val),
                                  _ptr(dec.next_ids), _stream()), "pt_lm_head_local_topk")
    torch.distributed.all_gather_into_tensor(dec.gather_val, dec.next_val.view(1, -1), group=dec.group)
    torch.distributed.all_gather_into_tensor(dec.gather_ids, dec.next_ids.view(1, -1), group=dec.group)
    check(L.pt_lm_head_tp_pick(_ptr(dec.gather_val), _ptr(dec.gather_ids), dec.tp, dec.batch, _ptr(dec.next_ids), _stream()),
          "pt_lm_head_tp_pick")


def random_sample(logits, k, generator=None):
    """ops.random_sample (popart.py:25-29): top-k of the logits on their last axis, then one of the k candidates picked by the arg-max
    of k standard-normal draws (one draw vector shared by all rows, shape [1, k] as in the reference).  The draws come from torch's
    generator (the reference's come from PopART's RNG: the choice is not reproducible across the two, the candidate set is)."""
    vals, ids = topk(logits, k)
    noise = torch.randn((1, k), generator=generator, device=logits.device, dtype=torch.float32)
    pick = torch.argmax(noise, dim=1)                               # [1]
    return ids[..., pick.item()].unsqueeze(-1).contiguous()


def add(a, b):
    out = torch.empty_like(a)
    check(_lib.lib().pt_add_f16(_ptr(a), _ptr(b), a.numel(), _ptr(out), _stream()), "pt_add_f16")
    return out


def remap_tensor(x, fwd_after_matmul=0, name="remap"):
    """ops.remap_tensor (customized.py:38-54): an IPU tile-layout hint with no numeric effect."""
    return x
