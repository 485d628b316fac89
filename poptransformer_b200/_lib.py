"""ctypes binding of libpt_b200.so (the C-ABI declared in include/pt_b200.h).

There is no CPU fallback: if the library cannot be loaded every op raises.
"""
import ctypes
import os

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.environ.get("PT_B200_LIB", os.path.join(HERE, "libpt_b200.so"))

c_void_p, c_int, c_float, c_size_t, c_int64 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_size_t, ctypes.c_int64


class PtError(RuntimeError):
    """Raised when a libpt_b200 entry point reports an error (the reference raises
    popart::error / poplar_error at graph-build time for the same violations)."""


class DenseExt(ctypes.Structure):
    _fields_ = [("bias", c_void_p), ("out2", c_void_p), ("out2_ld", c_int), ("split_n", c_int), ("limit", c_float), ("mul", c_void_p), ("mul_ld", c_int),
                ("mul_ids", c_void_p), ("n_groups", c_int), ("group_rows", c_int), ("group_x_div", c_int), ("group_of", c_void_p),
                ("group_used", c_void_p), ("glu", c_int), ("row_scale", c_void_p), ("pos", c_float), ("neg", c_float)]


class LinearArgs(ctypes.Structure):
    _fields_ = [
        ("wfmt", c_int), ("batch", c_int), ("n_out", c_int), ("k_in", c_int), ("group", c_int),
        ("prologue", c_int), ("epilogue", c_int), ("ksplit", c_int),
        ("x", c_void_p), ("packed_w", c_void_p), ("norm_gamma", c_void_p),
        ("norm_eps", c_float), ("act_scale", c_float), ("w_scale", c_float),
        ("bias", c_void_p), ("residual", c_void_p), ("out", c_void_p), ("out_ld", c_int), ("pdl", c_int),
        ("workspace", c_void_p), ("workspace_bytes", c_size_t), ("error_flag", c_void_p), ("norm_beta", c_void_p),
        ("out_dtype", c_int), ("alpha", c_float), ("ext", ctypes.POINTER(DenseExt)),
    ]


class AttnArgs(ctypes.Structure):
    _fields_ = [
        ("batch", c_int), ("n_head", c_int), ("n_kv", c_int), ("head_dim", c_int),
        ("page_size", c_int), ("max_pages", c_int), ("rope_mode", c_int), ("softmax_mode", c_int),
        ("score_scale", c_float),
        ("step_dev", c_void_p), ("qkv", c_void_p), ("rope_sin", c_void_p), ("rope_cos", c_void_p),
        ("pool", c_void_p), ("page_table", c_void_p), ("out", c_void_p), ("out_ld", c_int),
        ("workspace", c_void_p), ("workspace_bytes", c_size_t), ("error_flag", c_void_p), ("pdl", c_int), ("max_len", c_int),
        ("out_fp8", c_void_p), ("out_fp8_scale", c_float),
    ]


class GemmArgs(ctypes.Structure):
    _fields_ = [
        ("wfmt", c_int), ("m", c_int), ("n_out", c_int), ("k_in", c_int), ("group", c_int), ("epilogue", c_int), ("ksplit", c_int),
        ("w_tiled", c_int), ("x", c_void_p), ("w", c_void_p), ("scales", c_void_p), ("x_scale", c_float), ("w_scale", c_float),
        ("residual", c_void_p), ("out", c_void_p), ("out_ld", c_int), ("workspace", c_void_p), ("workspace_bytes", c_size_t),
        ("error_flag", c_void_p), ("bias", c_void_p), ("out_dtype", c_int), ("alpha", c_float), ("ext", ctypes.POINTER(DenseExt)),
        ("pdl", c_int),
    ]


class PrefillAttnArgs(ctypes.Structure):
    _fields_ = [(n, c_int) for n in ("batch", "n_tokens", "start", "n_head", "head_dim", "page_size", "max_pages", "max_len")] + \
               [("score_scale", c_float), ("qkv", c_void_p), ("rope_sin", c_void_p), ("rope_cos", c_void_p), ("pool", c_void_p),
                ("page_table", c_void_p), ("out", c_void_p)]


class BatchView(ctypes.Structure):
    _fields_ = [("n_seq", c_int), ("n_tok", c_int)] + [(n, c_void_p) for n in ("cu", "start", "slot", "tok_seq")]


class HyperArgs(ctypes.Structure):
    _fields_ = [("rows", c_int), ("width", c_int), ("streams", c_int), ("dtype", c_int), ("eps", c_float), ("mult", c_float), ("xs", c_void_p),
                ("table", c_void_p), ("table_ld", c_int), ("vocab", c_int), ("ids", c_void_p), ("ids_ld", c_int), ("step_dev", c_void_p),
                ("pos_out", c_void_p), ("row_index", c_void_p), ("y", c_void_p), ("y_ld", c_int)] + \
               [(n, c_void_p) for n in ("mix", "w_out", "w_in", "norm_w", "h")] + [("h_ld", c_int), ("sum_out", c_void_p)]


class ContextRows(ctypes.Structure):
    _fields_ = [("k", c_void_p), ("v", c_void_p), ("shared", c_void_p), ("ld", c_int), ("shared_ld", c_int), ("shared_dim", c_int), ("cu", c_void_p)]


class WindowAttnArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("dtype", "n_head", "n_kv", "dim", "vdim", "page_size", "max_pages", "window", "keep_first")] + \
               [("scale", c_float), ("sink", c_void_p), ("q", c_void_p), ("q_ld", c_int), ("k", c_void_p), ("v", c_void_p), ("kv_ld", c_int),
                ("pool", c_void_p), ("page_table", c_void_p), ("out", c_void_p), ("out_ld", c_int), ("max_tokens_per_seq", c_int), ("max_len", c_int),
                ("plain", c_int), ("workspace", c_void_p), ("workspace_bytes", c_size_t), ("error_flag", c_void_p), ("q_norm", c_void_p), ("k_norm", c_void_p),
                ("norm_eps", c_float), ("rope_dims", c_int), ("rope", c_void_p), ("out_scale", c_float), ("out_cols", c_int),
                ("softcap", c_float), ("gate", c_void_p), ("gate_ld", c_int), ("gate_per_head", c_int), ("values_in_keys", c_int), ("value_col", c_int), ("row_ld", c_int),
                ("context", ctypes.POINTER(ContextRows))]


class LatentPrepArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("dtype", "q_rank", "rank", "rot_dim")] + [("eps", c_float), ("q", c_void_p), ("kv", c_void_p), ("ld", c_int)] + \
               [(n, c_void_p) for n in ("q_norm", "kv_norm", "rope", "cq")] + [("cq_ld", c_int), ("pool", c_void_p), ("page_table", c_void_p)] + \
               [(n, c_int) for n in ("page_size", "max_pages", "max_len")] + [("error_flag", c_void_p)]


class LatentContextArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView), ("ctx_cu", c_void_p)] + [(n, c_int) for n in ("n_ctx", "rot_dim", "rank", "page_size", "max_pages")] + \
               [(n, c_void_p) for n in ("pool", "page_table", "shared", "latent")] + [("latent_ld", c_int)]


class LatentAttnArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("dtype", "n_head", "dim", "rot_dim", "vdim", "rank")] + \
               [("scale", c_float), ("q", c_void_p), ("q_ld", c_int)] + [(n, c_void_p) for n in ("rope", "w_k", "w_v", "gate")] + \
               [("gate_ld", c_int), ("pool", c_void_p), ("page_table", c_void_p)] + [(n, c_int) for n in ("page_size", "max_pages", "max_len")] + \
               [("out", c_void_p), ("out_ld", c_int), ("out_cols", c_int), ("plain", c_int), ("workspace", c_void_p), ("workspace_bytes", c_size_t),
                ("error_flag", c_void_p), ("gate_per_value", c_int)]


class SsmArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("dtype", "heads", "vdim", "state_dim", "groups", "taps", "norm_groups")] + \
               [("eps", c_float), ("zx", c_void_p), ("zx_ld", c_int)] + \
               [(n, c_void_p) for n in ("conv_w", "conv_b", "dt_bias", "A_log", "D", "norm_w", "ring", "state", "xbc", "dt", "y", "out")] + \
               [("out_ld", c_int), ("plain", c_int), ("workspace", c_void_p), ("workspace_bytes", c_size_t)]


class MlstmArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("dtype", "heads", "dim", "vdim")] + [(n, c_float) for n in ("gate_cap", "q_scale", "eps", "out_scale")] + \
               [(n, c_void_p) for n in ("q", "k", "v", "gate")] + [("ld", c_int), ("log_i", c_void_p), ("log_f", c_void_p), ("gate_ld", c_int)] + \
               [(n, c_void_p) for n in ("norm_w", "state", "nm", "y", "out")] + [("out_ld", c_int), ("out_cols", c_int), ("plain", c_int), ("workspace", c_void_p),
                                                                                 ("workspace_bytes", c_size_t)]


class PostNormArgs(ctypes.Structure):
    _fields_ = [("rows", c_int), ("width", c_int), ("dtype", c_int), ("eps", c_float), ("x_in", c_void_p), ("x_out", c_void_p), ("table", c_void_p),
                ("table_ld", c_int), ("vocab", c_int), ("ids", c_void_p), ("ids_ld", c_int)] + \
               [(n, c_void_p) for n in ("step_dev", "pos_out", "id_out", "row_index", "y")] + [("y_ld", c_int), ("pair_y", c_void_p), ("pair_dtype", c_int), ("pair_ld", c_int), ("top", c_int)] + \
               [(n, c_void_p) for n in ("pair_w", "pair_row", "norm_w", "final_w", "h")] + [("h_ld", c_int), ("h_cols", c_int), ("copy", c_void_p), ("copy_ld", c_int), ("copy_cols", c_int)]


class ShiftNormArgs(ctypes.Structure):
    _fields_ = [("batch", BatchView)] + [(n, c_int) for n in ("rows", "width", "groups", "dtype")] + \
               [("eps", c_float), ("x_in", c_void_p), ("x_out", c_void_p), ("table", c_void_p), ("table_ld", c_int), ("vocab", c_int), ("ids", c_void_p), ("ids_ld", c_int)] + \
               [(n, c_void_p) for n in ("step_dev", "pos_out", "embed_w", "row_index", "y")] + [("y_ld", c_int), ("pair_y", c_void_p), ("pair_dtype", c_int), ("pair_ld", c_int), ("top", c_int)] + \
               [(n, c_void_p) for n in ("pair_w", "pair_row", "self")] + [("self_ld", c_int), ("w1", c_void_p), ("shift", c_void_p), ("h1", c_void_p), ("h1_ld", c_int)] + \
               [("state_in", c_void_p), ("state_out", c_void_p), ("state_by_seq", c_int), ("w2", c_void_p), ("h2", c_void_p), ("h2_ld", c_int)]


class MoeRouteArgs(ctypes.Structure):
    _fields_ = [("n_tok", c_int), ("experts", c_int), ("top", c_int), ("logits", c_void_p), ("logits_ld", c_int), ("expert", c_void_p), ("weight", c_void_p),
                ("tile", c_int), ("max_tiles", c_int), ("pair_row", c_void_p), ("tile_expert", c_void_p), ("tile_rows", c_void_p), ("row_token", c_void_p), ("counts", c_void_p), ("h", c_void_p), ("h_bytes", c_int),
                ("gathered", c_void_p), ("score", c_int), ("row_weight", c_void_p), ("correction", c_void_p), ("groups", c_int), ("keep", c_int), ("identity", c_int)]


class LlamaLayer(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("qkv", "o", "gu", "down", "ln1", "ln2", "pool")]


class LlamaStepArgs(ctypes.Structure):
    _fields_ = [(n, c_int) for n in ("batch", "d_model", "n_head", "head_dim", "ffn", "vocab", "n_layer", "max_len", "page_size",
                                     "max_pages", "pad_id", "eos_id")] + [("norm_eps", c_float), ("score_scale", c_float)] + \
               [(n, c_void_p) for n in ("layers", "norm", "head", "emb", "rope_sin", "rope_cos", "ids", "step_dev", "stop_mask", "next_ids",
                                        "page_table", "x", "qkv", "attn", "act", "logits", "workspace")] + \
               [("workspace_bytes", c_size_t), ("error_flag", c_void_p), ("trace", c_void_p), ("debug", c_int)] + \
               [(n, c_int) for n in ("tp_size", "tp_rank", "ffn_offset", "ffn_valid", "vocab_offset", "emb_rows")] + [("tp_buffers", c_void_p * 8)] + \
               [("done_flag", c_void_p), ("wait_limit", c_int)]


# name -> (restype, argtypes); mirrors include/pt_b200.h one to one
SIGNATURES = {
    "pt_last_error": (ctypes.c_char_p, []),
    "pt_version": (c_int, []),
    "pt_launch_count": (ctypes.c_uint64, []),
    "pt_int4_to_half": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_linear_packed_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_linear_repack": (c_int, [c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_linear_workspace_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_linear": (c_int, [ctypes.POINTER(LinearArgs), c_void_p]),
    "pt_linear_static_scratch": (c_int, [ctypes.POINTER(LinearArgs), c_void_p]),
    "pt_gemm_workspace_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_gemm": (c_int, [ctypes.POINTER(GemmArgs), c_void_p]),
    "pt_gemm_packed_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_gemm_repack": (c_int, [c_int, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "pt_gemm_f32": (c_int, [c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_float, c_int, c_void_p, c_int, ctypes.POINTER(DenseExt), c_void_p]),
    "pt_post_norm": (c_int, [ctypes.POINTER(PostNormArgs), c_void_p]),
    "pt_shift_norm": (c_int, [ctypes.POINTER(ShiftNormArgs), c_void_p]),
    "pt_moe_max_tiles": (c_int, [c_int] * 4),
    "pt_moe_route": (c_int, [ctypes.POINTER(MoeRouteArgs), c_void_p]),
    "pt_mlstm_workspace_bytes": (c_size_t, [c_int] * 5),
    "pt_mlstm_state_floats": (c_size_t, [c_int] * 4),
    "pt_mlstm": (c_int, [ctypes.POINTER(MlstmArgs), c_void_p]),
    "pt_hyper": (c_int, [ctypes.POINTER(HyperArgs), c_void_p]),
    "pt_window_attn_workspace_bytes": (c_size_t, [c_int] * 7),
    "pt_window_attn": (c_int, [ctypes.POINTER(WindowAttnArgs), c_void_p]),
    "pt_latent_row": (c_int, [c_int] * 2),
    "pt_latent_prep": (c_int, [ctypes.POINTER(LatentPrepArgs), c_void_p]),
    "pt_latent_context": (c_int, [ctypes.POINTER(LatentContextArgs), c_void_p]),
    "pt_latent_attn_workspace_bytes": (c_size_t, [c_int] * 5),
    "pt_latent_attn": (c_int, [ctypes.POINTER(LatentAttnArgs), c_void_p]),
    "pt_ssm_workspace_bytes": (c_size_t, [c_int] * 5),
    "pt_ssm": (c_int, [ctypes.POINTER(SsmArgs), c_void_p]),
    "pt_norm_ce": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p, c_void_p]),
    "pt_rms_norm": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p, c_void_p, c_void_p]),
    "pt_softmax": (c_int, [c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_kv_cache": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_int, c_int, c_int64, c_void_p]),
    "pt_kv_cache_pipeline": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int64, c_int, c_int, c_int64, c_void_p]),
    "pt_kv_cache_fp8": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_int64, c_int, c_int, c_int64, c_void_p]),
    "pt_kv_cache_pipeline_fp8": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_int, c_int64, c_int, c_int, c_int64, c_void_p]),
    "pt_attn_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int]),
    "pt_kv_append_attn": (c_int, [ctypes.POINTER(AttnArgs), c_void_p]),
    "pt_prefill_attn": (c_int, [ctypes.POINTER(PrefillAttnArgs), c_void_p]),
    "pt_prefill_embed": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "pt_kv_export": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_kv_reorder_pages": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p]),
    "pt_kv_reorder_table": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "pt_llama_stream_permute": (c_int, [c_int, c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "pt_llama_step_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int]),
    "pt_llama_tp_buffer_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_llama_decode_step": (c_int, [ctypes.POINTER(LlamaStepArgs), c_void_p]),
    "pt_topk": (c_int, [c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "pt_lm_head_local_topk": (c_int, [c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "pt_lm_head_tp_pick": (c_int, [c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "pt_beam_search_workspace_bytes": (c_size_t, [c_int, c_int, c_int]),
    "pt_beam_search": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p,
                               c_void_p, c_size_t, c_void_p]),
    "pt_cast_fp8": (c_int, [c_void_p, c_float, c_int64, c_void_p, c_void_p]),
    "pt_fp8_matmul": (c_int, [c_void_p, c_void_p, c_float, c_float, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_rwkv_mix": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "pt_rwkv_act": (c_int, [c_int, c_void_p, c_void_p, c_void_p, ctypes.c_int64, c_void_p]),
    "pt_wkv": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "pt_embedding": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p]),
    "pt_step_containers": (c_int, [c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "pt_step_containers_early_stop": (c_int, [c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "pt_swiglu": (c_int, [c_void_p, c_int, c_int, c_void_p, c_int, c_void_p]),
    "pt_rms_norm_fp8": (c_int, [c_void_p, c_void_p, c_int, c_int, c_float, c_float, c_void_p, c_void_p]),
    "pt_swiglu_fp8": (c_int, [c_void_p, c_int, c_int, c_float, c_void_p, c_int, c_void_p]),
    "pt_add_f16": (c_int, [c_void_p, c_void_p, c_int64, c_void_p, c_void_p]),
}

_lib = None
_partial = False


def use_library(path):
    """Loads `path` instead of the full library (before the first call of lib()): it may lack the kernels of other models."""
    global LIB_PATH, _partial
    if _lib is not None and path != LIB_PATH:
        raise PtError(f"{LIB_PATH} is already loaded")
    _partial = path != LIB_PATH
    LIB_PATH = path


def lib():
    """Loads libpt_b200.so (building it with nvcc if it is missing and nvcc is present)."""
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(LIB_PATH):
        from . import build as _build
        _build.build()
    try:
        handle = ctypes.CDLL(LIB_PATH)
    except OSError as e:  # no fallback on purpose
        raise PtError(f"libpt_b200.so could not be loaded from {LIB_PATH}: {e}") from e
    for name, (res, args) in SIGNATURES.items():
        if _partial and not hasattr(handle, name):
            continue                     # calling it raises AttributeError
        fn = getattr(handle, name)
        fn.restype, fn.argtypes = res, args
    _lib = handle
    return _lib


def check(code, what=""):
    if code != 0:
        msg = lib().pt_last_error().decode(errors="replace")
        raise PtError(f"{what or 'libpt_b200'} failed ({code}): {msg}")
