// What the linears of bf16 and fp32 models (pt_linear and pt_gemm with PT_W_BF16, pt_gemm_f32) do with a finished sum.
//
//     y = alpha * sum + bias[n]                                   then, by epilogue:
//   STORE      out[m, n] = y
//   RELU2      out[m, n] = max(y, 0)^2
//   GELU_MUL   out[m, n] = gelu_tanh(y) * mul[mul_ids[m], n]
//   SOFTCAP    out[m, n] = limit * tanh(y / limit)
//   XIELU      out[m, n] = y / 2 + (y > 0 ? pos y^2 : neg (exp(y) - 1 - y))
//   GLU        weight rows alternate in blocks of eight, eight gate features and then the same eight up features; by `glu`:
//     CLAMPED    out[m, f] = g sigmoid(1.702 g) (u + 1),  g = min(gate, limit), u = clamp(up, -limit, limit)
//     SILU       out[m, f] = gate sigmoid(gate) up
//     GELU       out[m, f] = gelu_tanh(gate) up
// row_scale (optional, one factor per activation row) multiplies the sum before the bias: the product of a scaled row.
// Outputs from split_n on skip the epilogue and go to a second, fp32 matrix: out2[m, n - split_n] = y.
#pragma once
#include <limits.h>

#include "elem.cuh"

namespace pt {

struct DenseOut {
  void *out;
  float *out2;
  const float *bias;
  const void *mul;
  const int *mul_ids;
  int out_ld, out2_ld, split_n, mul_ld, epilogue, out_dt;
  float alpha, limit;
  int glu;
  const float *row_scale;
  float pos, neg;
};

static inline DenseOut make_dense_out(void *out, int out_ld, int out_dt, int epilogue, float alpha, const pt_dense_ext *e) {
  DenseOut o{};
  o.out = out; o.out_ld = out_ld; o.out_dt = out_dt; o.epilogue = epilogue;
  o.alpha = alpha != 0.f ? alpha : 1.0f;
  o.split_n = INT_MAX;
  if (e) {
    o.bias = e->bias; o.mul = e->mul; o.mul_ids = e->mul_ids; o.mul_ld = e->mul_ld; o.limit = e->limit;
    o.glu = e->glu; o.row_scale = e->row_scale; o.pos = e->pos; o.neg = e->neg;
    if (e->out2) { o.out2 = e->out2; o.out2_ld = e->out2_ld; o.split_n = e->split_n; }
  }
  return o;
}
static inline bool dense_needs_ext(int epilogue, const pt_dense_ext *e) { return e && (e->row_scale || epilogue == PT_EPI_SOFTCAP || epilogue == PT_EPI_XIELU || (epilogue == PT_EPI_GLU && e->glu != PT_GLU_CLAMPED)); }
static inline bool dense_epilogue_known(int e) { return e == PT_EPI_STORE || e == PT_EPI_RELU2 || e == PT_EPI_GLU || e == PT_EPI_GELU_MUL || e == PT_EPI_SOFTCAP || e == PT_EPI_XIELU; }
// nullptr, or what is wrong with the combination.
static inline const char *dense_ext_error(int epilogue, int n_out, const pt_dense_ext *e) {
  if ((epilogue == PT_EPI_GLU || epilogue == PT_EPI_GELU_MUL || epilogue == PT_EPI_SOFTCAP || epilogue == PT_EPI_XIELU) && !e) return "the epilogue needs its extra arguments";
  if (!e) return nullptr;
  if (epilogue == PT_EPI_GELU_MUL && !(e->mul && e->mul_ids)) return "a gelu-times-row epilogue needs mul and mul_ids";
  if (e->out2 && (e->split_n < 0 || e->split_n % 32 || e->split_n > n_out || e->out2_ld < n_out - e->split_n))
    return "split_n must be a multiple of 32 within n_out, and out2_ld hold the rest";
  if (epilogue == PT_EPI_GLU && (e->out2 ? e->split_n : n_out) % 16) return "gated features come in blocks of eight";
  if (epilogue == PT_EPI_GLU && (e->glu < PT_GLU_CLAMPED || e->glu > PT_GLU_GELU)) return "unknown kind of gated unit";
  if (((epilogue == PT_EPI_GLU && e->glu == PT_GLU_CLAMPED) || epilogue == PT_EPI_SOFTCAP) && !(e->limit > 0.f)) return "the epilogue needs a positive limit";
  if (e->n_groups < 0 || (e->n_groups > 0 && (!e->group_of || e->group_rows < 1))) return "groups need group_of and group_rows";
  return nullptr;
}

#ifdef __CUDACC__
__device__ __forceinline__ float gelu_tanh_f(float x) {
  return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * x * x, x, x)));
}
// tanh(z) = 2 sigmoid(2 z) - 1, with the fast exponential and quotient (a few units in the last place): what the bf16 kernels use, also
// because their epilogues stay short
__device__ __forceinline__ float gelu_tanh_fast(float x) {
  return __fdividef(x, 1.0f + __expf(-1.5957691216057308f * fmaf(0.044715f * x * x, x, x)));
}
template <bool FAST, int GLU> __device__ __forceinline__ float glu_unit(float gate, float up, float limit) {
  if (GLU == PT_GLU_SILU) return (FAST ? __fdividef(gate, 1.0f + __expf(-gate)) : gate / (1.0f + expf(-gate))) * up;
  if (GLU == PT_GLU_GELU) return (FAST ? gelu_tanh_fast(gate) : gelu_tanh_f(gate)) * up;
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  if (FAST) return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (u + 1.0f);   // (rounded to bf16 by the caller; for g very negative the quotient is 0)
  return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}
// EXT: the kernel serves what dense_needs_ext names (an instantiation of its own, so that the others' epilogues stay short)
template <bool FAST, bool EXT> __device__ __forceinline__ float glu_f(const DenseOut &o, float gate, float up) {
  if (!EXT) return glu_unit<FAST, PT_GLU_CLAMPED>(gate, up, o.limit);
  if (o.glu == PT_GLU_SILU) return glu_unit<FAST, PT_GLU_SILU>(gate, up, 0.f);
  if (o.glu == PT_GLU_GELU) return glu_unit<FAST, PT_GLU_GELU>(gate, up, 0.f);
  return glu_unit<FAST, PT_GLU_CLAMPED>(gate, up, o.limit);
}
__device__ __forceinline__ void dense_put(const DenseOut &o, int m, int n, float y) {
  const size_t i = (size_t)m * o.out_ld + n;
  if (o.out_dt == PT_DT_F32) reinterpret_cast<float *>(o.out)[i] = y;
  else reinterpret_cast<__nv_bfloat16 *>(o.out)[i] = __float2bfloat16_rn(y);
}
template <bool EXT> __device__ __forceinline__ float dense_factor(const DenseOut &o, int m) { return EXT && o.row_scale ? o.alpha * __ldcg(o.row_scale + m) : o.alpha; }
template <bool EXT> __device__ __forceinline__ float dense_value(const DenseOut &o, int m, int n, float acc) { return fmaf(acc, dense_factor<EXT>(o, m), o.bias ? __ldg(o.bias + n) : 0.f); }
__device__ __forceinline__ float softcap_fast(float x, float limit) { return limit * (1.0f - __fdividef(2.0f, 1.0f + __expf(__fdividef(2.0f * x, limit)))); }
template <bool EXACT> __device__ __forceinline__ float xielu_f(float y, float pos, float neg) {
  const float e = EXACT ? expm1f(y) - y : __expf(y) - 1.0f - y;       // (not used for y > 0, where it may overflow)
  return fmaf(0.5f, y, y > 0.f ? pos * y * y : neg * e);
}
// One finished sum (any epilogue but GLU, whose sums come in pairs).  EXACT: for models that run in 32-bit.
template <bool EXT, bool EXACT = false> __device__ __forceinline__ void dense_store(const DenseOut &o, int m, int n, float acc) {
  float y = dense_value<EXT>(o, m, n, acc);
  if (n >= o.split_n) {
    o.out2[(size_t)m * o.out2_ld + n - o.split_n] = y;
    return;
  }
  if (o.epilogue == PT_EPI_RELU2) {
    y = fmaxf(y, 0.f);
    y *= y;
  } else if (EXT && o.epilogue == PT_EPI_SOFTCAP) {
    y = EXACT ? o.limit * tanhf(y / o.limit) : softcap_fast(y, o.limit);
  } else if (EXT && o.epilogue == PT_EPI_XIELU) {
    y = xielu_f<EXACT>(y, o.pos, o.neg);
  } else if (o.epilogue == PT_EPI_GELU_MUL) {
    const size_t i = (size_t)o.mul_ids[m] * o.mul_ld + n;
    y = (EXACT ? gelu_tanh_f(y) : gelu_tanh_fast(y)) * (o.out_dt == PT_DT_F32 ? reinterpret_cast<const float *>(o.mul)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16 *>(o.mul)[i]));
  }
  dense_put(o, m, n, y);
}
// Sums of the gate row n (n % 16 < 8) and the up row n + 8.
template <bool EXT, bool EXACT = false> __device__ __forceinline__ void dense_store_glu(const DenseOut &o, int m, int n, float gate, float up) {
  const int f = n / 16 * 8 + n % 8;
  const float g = dense_value<EXT>(o, m, n, gate), u = dense_value<EXT>(o, m, n + 8, up);
  dense_put(o, m, f, glu_f<!EXACT, EXT>(o, g, u));
}
// Four consecutive outputs n .. n + 3 (n a multiple of four).  The plain epilogues leave as one store where the rows allow it.
__device__ __forceinline__ void dense_put4(void *out, size_t i, bool f32, const float (&y)[4]) {
  if (f32) {
    float *o = reinterpret_cast<float *>(out) + i;
    if (((uintptr_t)o & 15) == 0) *reinterpret_cast<float4 *>(o) = make_float4(y[0], y[1], y[2], y[3]);
    else {
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = y[j];
    }
  } else {
    __nv_bfloat16 *o = reinterpret_cast<__nv_bfloat16 *>(out) + i;
    if (((uintptr_t)o & 7) == 0) *reinterpret_cast<uint2 *>(o) = make_uint2(pack_bf2(y[0], y[1]), pack_bf2(y[2], y[3]));
    else {
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = __float2bfloat16_rn(y[j]);
    }
  }
}
template <bool EXT> __device__ __forceinline__ void dense_store4(const DenseOut &o, int m, int n, const float4 &acc) {
  const float a[4] = {acc.x, acc.y, acc.z, acc.w};
  const bool second = n >= o.split_n;
  if (!second && o.epilogue != PT_EPI_STORE && o.epilogue != PT_EPI_RELU2 && !(EXT && o.epilogue == PT_EPI_XIELU)) {
#pragma unroll 1
    for (int j = 0; j < 4; ++j) dense_store<EXT>(o, m, n + j, j == 0 ? acc.x : j == 1 ? acc.y : j == 2 ? acc.z : acc.w);
    return;
  }
  const float f = dense_factor<EXT>(o, m);
  float y[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    y[j] = fmaf(a[j], f, o.bias ? __ldg(o.bias + n + j) : 0.f);
    if (!second && o.epilogue == PT_EPI_RELU2) {
      y[j] = fmaxf(y[j], 0.f);
      y[j] *= y[j];
    }
    if (EXT && !second && o.epilogue == PT_EPI_XIELU) y[j] = xielu_f<false>(y[j], o.pos, o.neg);
  }
  if (second) dense_put4(o.out2, (size_t)m * o.out2_ld + n - o.split_n, true, y);
  else dense_put4(o.out, (size_t)m * o.out_ld + n, o.out_dt == PT_DT_F32, y);
}
// Four gate rows n .. n + 3 and the up rows n + 8 ..
template <bool EXT> __device__ __forceinline__ void dense_store_glu4(const DenseOut &o, int m, int n, const float4 &gate, const float4 &up) {
  const float f = dense_factor<EXT>(o, m), g[4] = {gate.x, gate.y, gate.z, gate.w}, u[4] = {up.x, up.y, up.z, up.w};
  float y[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) y[j] = glu_f<true, EXT>(o, fmaf(g[j], f, o.bias ? __ldg(o.bias + n + j) : 0.f), fmaf(u[j], f, o.bias ? __ldg(o.bias + n + 8 + j) : 0.f));
  dense_put4(o.out, (size_t)m * o.out_ld + n / 16 * 8 + n % 8, o.out_dt == PT_DT_F32, y);
}
#endif

}  // namespace pt
