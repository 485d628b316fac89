// Residual step between two sublayers' matrix products, with a norm on what is added, on what is read next, or on both:
//     x <- x + rms(y) * norm_w  or  x + y        and h = x  or  rms(x) * final_w in the activation type, the input of the next product.
// y may be a sum: a dense output plus a (weighted) sum over the experts a token went to (their rows lie where the router put them).
// The same kernel starts a token (y is its embedding row, there is no x yet) and ends the model (h = rms(x) * final_w for the output
// layer).  A second copy of x can go beside h, for a product that reads several vectors side by side.  All of it is fp32; only h
// and the copy are rounded.
#include "elem.cuh"

namespace pt {
namespace post {

constexpr int kMaxTop = 64;

struct Params {
  int rows, width, h_ld, h_cols, copy_ld, copy_cols, table_ld, vocab, ids_ld, y_ld, pair_ld, top;
  float eps;
  const float *x_in;
  float *x_out;
  const void *table;
  const int *ids, *step;
  int *pos_out, *id_out;
  const int *row_index;
  const float *y, *pair_w;
  const void *pair_y;
  const int *pair_row;
  const float *norm_w, *final_w;
  void *h, *copy;
};

template <int VEC> __device__ __forceinline__ void put_f32(float *p, const float (&v)[VEC]) { store_vec<VEC>(p, v); }

// RESIDUAL: a step whose addend is normalised, without a second copy.  ADD: nothing is normalised before it is added.  ANY: the rest.
enum { RESIDUAL = 0, ADD = 1, ANY = 2 };
template <typename T, typename E, int VEC, int MODE> __global__ void __launch_bounds__(1024, MODE == RESIDUAL ? 2 : 1) post_norm_kernel(const Params p) {
  extern __shared__ __align__(16) float row[];     // [width]: y, then the new x
  __shared__ float red[32], pw[kMaxTop];
  __shared__ int pr[kMaxTop];
  launch_dependents();
  const int r = blockIdx.x, src = p.row_index ? p.row_index[r] : r, tid = threadIdx.x;
  float *xo = p.x_out ? p.x_out + (size_t)r * p.width : nullptr;
  T *hrow = p.h ? reinterpret_cast<T *>(p.h) + (size_t)r * p.h_ld : nullptr, *crow = MODE != RESIDUAL && p.copy ? reinterpret_cast<T *>(p.copy) + (size_t)r * p.copy_ld : nullptr;
  if (hrow)
    for (int i = p.width + tid; i < p.h_cols; i += blockDim.x) hrow[i] = from_f<T>(0.f);     // k padding of the next product
  if (crow)
    for (int i = p.width + tid; i < p.copy_cols; i += blockDim.x) crow[i] = from_f<T>(0.f);
  const T *emb = nullptr;
  if (MODE != RESIDUAL && p.table) {
    const int step = p.step ? *p.step : 0;
    const int id = min(max(p.ids[(size_t)src * p.ids_ld + step], 0), p.vocab - 1);
    emb = reinterpret_cast<const T *>(p.table) + (size_t)id * p.table_ld;
    if (tid == 0) {
      if (p.pos_out) p.pos_out[r] = step;
      if (p.id_out) p.id_out[r] = id;
    }
  }
  if (tid < p.top) {
    const size_t k = (size_t)src * p.top + tid;
    pw[tid] = p.pair_w ? p.pair_w[k] : 1.f;
    pr[tid] = p.pair_row ? p.pair_row[k] : (int)k;
  }
  __syncthreads();
  auto addend = [&](int i, float (&v)[VEC]) {
    if (MODE != RESIDUAL && emb) {
      load_vec<VEC>(emb + i, v);
    } else if (p.y) {
      load_vec<VEC>(p.y + (size_t)src * p.y_ld + i, v);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    }
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      float e[VEC];
      load_vec<VEC>(reinterpret_cast<const E *>(p.pair_y) + (size_t)pr[k] * p.pair_ld + i, e);
      const float w = pw[k];
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = fmaf(w, e[j], v[j]);
    }
  };
  float ss = 0.f, inv = 1.f;
  if (MODE != ADD) {
    for (int i = tid * VEC; i < p.width; i += blockDim.x * VEC) {
      float v[VEC];
      addend(i, v);
      put_f32<VEC>(row + i, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
    }
    inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);     // (every thread reads back what it wrote)
    ss = 0.f;
  }
  const float *x = p.x_in ? p.x_in + (size_t)src * p.width : nullptr;
  for (int i = tid * VEC; i < p.width; i += blockDim.x * VEC) {
    float v[VEC], o[VEC];
    if (MODE == RESIDUAL || x) {
      load_vec<VEC>(x + i, o);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    }
    if (MODE == ADD) {
      addend(i, v);
    } else {
      float w[VEC];
      load_vec<VEC>(row + i, v);
      load_vec<VEC>(p.norm_w + i, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= inv * w[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] += v[j];
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(o[j], o[j], ss);
    if (xo) put_f32<VEC>(xo + i, o);
    if (crow) store_vec<VEC>(crow + i, o);
    if (p.final_w) put_f32<VEC>(row + i, o);
    else if (hrow) store_vec<VEC>(hrow + i, o);
  }
  if (!p.final_w || !hrow) return;
  const float end = 1.0f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);
  for (int i = tid * VEC; i < p.width; i += blockDim.x * VEC) {
    float v[VEC], w[VEC];
    load_vec<VEC>(row + i, v);
    load_vec<VEC>(p.final_w + i, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= end * w[j];
    store_vec<VEC>(hrow + i, v);
  }
}

template <typename T, typename E, int VEC, int MODE> static int launch(const Params &p, cudaStream_t st) {
  const size_t smem = (size_t)p.width * sizeof(float);
  if (smem > 48 * 1024) {
    static bool set = false;
    if (!set) { PT_CUDA(cudaFuncSetAttribute(post_norm_kernel<T, E, VEC, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); set = true; }
  }
  // few rows: as many threads per row as it has work for; many rows: more rows per SM
  const int want = ceil_div(ceil_div(p.width, VEC), 32) * 32, cap = p.rows <= 2 * sm_count() ? 1024 : 256;
  post_norm_kernel<T, E, VEC, MODE><<<p.rows, std::max(64, std::min(want, cap)), smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_post_norm");
  return PT_OK;
}

template <typename T, typename E, int VEC> static int launch(const Params &p, cudaStream_t st) {
  if (!p.norm_w) return launch<T, E, VEC, ADD>(p, st);
  return p.x_in && !p.copy ? launch<T, E, VEC, RESIDUAL>(p, st) : launch<T, E, VEC, ANY>(p, st);
}

}  // namespace post
}  // namespace pt

using namespace pt;

extern "C" int pt_post_norm(const pt_post_norm_args *a, void *stream) {
  PT_REQUIRE(a, "pt_post_norm: null args");
  PT_REQUIRE(a->rows > 0 && a->width > 0 && a->width <= 48 * 1024, "pt_post_norm: bad shape rows=%d width=%d", a->rows, a->width);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_post_norm: activation type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(!a->h || (a->h_ld >= a->width && a->h_cols <= a->h_ld), "pt_post_norm: h_ld=%d h_cols=%d", a->h_ld, a->h_cols);
  PT_REQUIRE(!a->copy || (a->copy_ld >= a->width && a->copy_cols <= a->copy_ld), "pt_post_norm: copy_ld=%d copy_cols=%d", a->copy_ld, a->copy_cols);
  if (a->table) {
    PT_REQUIRE(a->ids && a->vocab > 0 && a->table_ld >= a->width && a->ids_ld >= 1 && a->x_out, "pt_post_norm: an embedding start needs ids, vocab, table_ld and x_out");
  } else {
    PT_REQUIRE(a->x_in || a->y || a->top > 0, "pt_post_norm: nothing to add and nothing to add to");
    PT_REQUIRE(!a->y || a->y_ld >= a->width, "pt_post_norm: y_ld=%d", a->y_ld);
    PT_REQUIRE(a->top >= 0 && a->top <= post::kMaxTop && (!a->top || (a->pair_y && a->pair_ld >= a->width)),
               "pt_post_norm: %d experts per token (at most %d) need pair_y and pair_ld", a->top, post::kMaxTop);
    PT_REQUIRE(!a->top || a->pair_dtype == PT_DT_F32 || (a->pair_dtype == PT_DT_BF16 && a->dtype == PT_DT_BF16), "pt_post_norm: experts' outputs of type %d",
               a->pair_dtype);
  }
  post::Params p{};
  p.rows = a->rows; p.width = a->width; p.h_ld = a->h_ld; p.table_ld = a->table_ld; p.vocab = a->vocab; p.ids_ld = a->ids_ld; p.y_ld = a->y_ld;
  p.pair_ld = a->pair_ld; p.top = a->table ? 0 : a->top; p.eps = a->eps;
  p.h_cols = a->h_cols > 0 ? a->h_cols : a->h_ld; p.copy = a->copy; p.copy_ld = a->copy_ld; p.copy_cols = a->copy_cols;
  p.x_in = a->table ? nullptr : a->x_in; p.x_out = a->x_out; p.table = a->table; p.ids = a->ids; p.step = a->step_dev; p.pos_out = a->pos_out; p.id_out = a->id_out;
  p.row_index = a->row_index; p.y = a->y; p.pair_y = a->pair_y; p.pair_w = a->pair_w; p.pair_row = a->pair_row;
  p.norm_w = a->norm_w; p.final_w = a->final_w; p.h = a->h;
  const int vb = a->dtype == PT_DT_F32 ? 16 : 8;
  const bool v4 = a->width % 4 == 0 && aligned_to(a->x_in, 16) && aligned_to(a->x_out, 16) && aligned_to(a->y, 16) && a->y_ld % 4 == 0 && aligned_to(a->pair_y, a->pair_dtype == PT_DT_F32 ? 16 : 8) &&
                  a->pair_ld % 4 == 0 && aligned_to(a->norm_w, 16) && aligned_to(a->final_w, 16) && aligned_to(a->h, vb) && a->h_ld % 4 == 0 && aligned_to(a->copy, vb) && a->copy_ld % 4 == 0 && aligned_to(a->table, vb) &&
                  a->table_ld % 4 == 0;
  cudaStream_t st = as_stream(stream);
  typedef __nv_bfloat16 B;
  if (a->dtype == PT_DT_F32) return v4 ? post::launch<float, float, 4>(p, st) : post::launch<float, float, 1>(p, st);
  if (p.top > 0 && a->pair_dtype == PT_DT_BF16) return v4 ? post::launch<B, B, 4>(p, st) : post::launch<B, B, 1>(p, st);
  return v4 ? post::launch<B, float, 4>(p, st) : post::launch<B, float, 1>(p, st);
}
