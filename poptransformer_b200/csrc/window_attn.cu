// Masked attention over a paged cache with per-sequence positions: a sliding window, kept first tokens, a softmax sink, grouped
// heads, key and value widths of their own, no rotation.  Position i sees key j when j <= i and (i - j < window or j < keep_first);
// window = 0 means every earlier key.  sink adds exp(sink[h]) to the softmax denominator of head h (no key, no value, not scaled).
//
// The tokens of a launch are packed sequence after sequence (pt_batch_view): row cu[s] + i is position start[s] + i of sequence s,
// whose pages are page_table[slot[s]].  A page holds K [n_kv][page][dim] and then V [n_kv][page][vdim].  New keys and values are
// appended first; a layer that shares another layer's cache passes none and reads what is there.
//
//   attn_plain_kernel   any sizes, fp32 or bf16 caches, CUDA cores: the 32-bit path and the shapes the others do not take
//   attn_prompt_kernel  bf16 prompts: 64 queries of one head per block, Q K^T and P V on the tensor cores, online softmax; only key
//                       tiles that hold a visible key are touched
//   attn_decode_kernel  bf16, one token per sequence: one block per (visible page, kv head, sequence), scores and P V on the tensor
//                       cores, pages combined by the last block to arrive; the append is fused
// Scores, softmax and weights are fp32.  The tensor-core kernels multiply V with weights split into two bf16 parts (hi + lo), which
// keeps 16 significant bits of each weight.
#include "elem.cuh"
#include "tile_math.cuh"

namespace pt {
namespace wa {

constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  int n_seq, n_head, n_kv, qpk, dim, vdim, page, max_pages, window, keep_first;
  int q_ld, kv_ld, out_ld;
  float scale;
  const float *sink;
  const void *q, *k, *v;
  void *pool, *out;
  const int *page_table, *cu, *start, *slot, *tok_seq;
  int *error_flag;
  // decode
  int grid_pages, qsplit;
  float *ws_o;      // [n_seq, n_head, grid_pages, vdim]
  float2 *ws_ml;    // [n_seq, n_head, grid_pages]
  int *counters;    // [n_seq, n_kv, qsplit]
};

__device__ __forceinline__ size_t page_elems(const Params &p) { return (size_t)p.n_kv * p.page * (p.dim + p.vdim); }
template <typename T> __device__ __forceinline__ T *k_page(const Params &p, int phys, int g) {
  return reinterpret_cast<T *>(p.pool) + (size_t)phys * page_elems(p) + (size_t)g * p.page * p.dim;
}
template <typename T> __device__ __forceinline__ T *v_page(const Params &p, int phys, int g) {
  return reinterpret_cast<T *>(p.pool) + (size_t)phys * page_elems(p) + (size_t)p.n_kv * p.page * p.dim + (size_t)g * p.page * p.vdim;
}
__device__ __forceinline__ bool visible(const Params &p, int pos, int key) {
  return key <= pos && (p.window == 0 || pos - key < p.window || key < p.keep_first);
}
// First page whose keys are not all behind the window of position pos.
__device__ __forceinline__ int window_page(const Params &p, int pos) { return p.window == 0 ? 0 : max(0, pos - p.window + 1) / p.page; }
// Pages that hold the kept first tokens (as far as they exist at position pos).
__device__ __forceinline__ int kept_pages(const Params &p, int pos) { return (min(p.keep_first, pos + 1) + p.page - 1) / p.page; }

// ------------------------------------------------------------------------------------------ append
template <typename T> __global__ void kv_append_kernel(const Params p) {
  const int t = blockIdx.x, s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.page * p.max_pages) {
    if (threadIdx.x == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int phys = p.page_table[(size_t)p.slot[s] * p.max_pages + pos / p.page], at = pos % p.page;
  const T *k = reinterpret_cast<const T *>(p.k) + (size_t)t * p.kv_ld, *v = reinterpret_cast<const T *>(p.v) + (size_t)t * p.kv_ld;
  for (int i = threadIdx.x; i < p.n_kv * p.dim; i += blockDim.x) k_page<T>(p, phys, i / p.dim)[(size_t)at * p.dim + i % p.dim] = k[i];
  for (int i = threadIdx.x; i < p.n_kv * p.vdim; i += blockDim.x) v_page<T>(p, phys, i / p.vdim)[(size_t)at * p.vdim + i % p.vdim] = v[i];
}

// ------------------------------------------------------------------------------------------ plain
// Block: one token and one kv head (all of its query heads).  Dynamic shared memory: q [qpk][dim], scores [qpk][page], o [qpk][vdim],
// statistics [qpk][3].
constexpr int PLAIN_THREADS = 128;
template <typename T> __global__ void __launch_bounds__(PLAIN_THREADS) attn_plain_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *q = sm, *sc = q + p.qpk * p.dim, *o = sc + p.qpk * p.page, *st = o + p.qpk * p.vdim;   // st: running max, sum, correction
  const int t = blockIdx.x, g = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.page * p.max_pages) {
    if (tid == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int *table = p.page_table + (size_t)p.slot[s] * p.max_pages;
  const T *qrow = reinterpret_cast<const T *>(p.q) + (size_t)t * p.q_ld + (size_t)g * p.qpk * p.dim;
  for (int i = tid; i < p.qpk * p.dim; i += PLAIN_THREADS) q[i] = to_f(qrow[i]);
  for (int i = tid; i < p.qpk * p.vdim; i += PLAIN_THREADS) o[i] = 0.f;
  for (int h = tid; h < p.qpk; h += PLAIN_THREADS) {
    st[3 * h] = p.sink ? p.sink[g * p.qpk + h] : -INFINITY;
    st[3 * h + 1] = p.sink ? 1.f : 0.f;
  }
  const int kept = kept_pages(p, pos), wpage = window_page(p, pos);
  for (int pg = kept > 0 ? 0 : wpage; pg <= pos / p.page; ++pg) {
    if (pg >= kept && pg < wpage) pg = wpage;
    const int k0 = pg * p.page, nk = min(p.page, pos + 1 - k0);
    const T *K = k_page<T>(p, table[pg], g), *V = v_page<T>(p, table[pg], g);
    __syncthreads();
    for (int i = warp; i < p.qpk * nk; i += PLAIN_THREADS / 32) {
      const int h = i / nk, key = i - h * nk;
      float a = 0.f;
      for (int c = lane; c < p.dim; c += 32) a = fmaf(q[h * p.dim + c], to_f(K[(size_t)key * p.dim + c]), a);
      a = warp_sum(a);
      if (lane == 0) sc[h * p.page + key] = visible(p, pos, k0 + key) ? a * p.scale : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < p.qpk; h += PLAIN_THREADS / 32) {
      float m = st[3 * h];
      for (int i = lane; i < nk; i += 32) m = fmaxf(m, sc[h * p.page + i]);
      m = warp_max(m);
      float l = 0.f;
      for (int i = lane; i < nk; i += 32) {
        const float x = sc[h * p.page + i], e = x == -INFINITY ? 0.f : expf(x - m);
        sc[h * p.page + i] = e;
        l += e;
      }
      l = warp_sum(l);
      __syncwarp();
      if (lane == 0) {
        const float corr = m == -INFINITY ? 1.f : expf(st[3 * h] - m);
        st[3 * h] = m;
        st[3 * h + 1] = st[3 * h + 1] * corr + l;
        st[3 * h + 2] = corr;
      }
    }
    __syncthreads();
    for (int i = tid; i < p.qpk * p.vdim; i += PLAIN_THREADS) {
      const int h = i / p.vdim, c = i - h * p.vdim;
      float a = o[i] * st[3 * h + 2];
      for (int key = 0; key < nk; ++key) a = fmaf(sc[h * p.page + key], to_f(V[(size_t)key * p.vdim + c]), a);
      o[i] = a;
    }
  }
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld + (size_t)g * p.qpk * p.vdim;
  for (int i = tid; i < p.qpk * p.vdim; i += PLAIN_THREADS) out[i] = from_f<T>(o[i] / st[3 * (i / p.vdim) + 1]);
  if (g == p.n_kv - 1)   // k padding of the output product
    for (int i = p.n_head * p.vdim + tid; i < p.out_ld; i += PLAIN_THREADS) reinterpret_cast<T *>(p.out)[(size_t)t * p.out_ld + i] = from_f<T>(0.f);
}

}  // namespace wa
}  // namespace pt

using namespace pt;

// Most pages one decode launch visits per sequence: the kept first tokens and a window that may straddle one page border more.
static int decode_pages(int page_size, int max_len, int window, int keep_first) {
  const int all = ceil_div(max_len, page_size);
  return window == 0 ? all : std::min(all, ceil_div(keep_first, page_size) + ceil_div(window - 1, page_size) + 1);
}
static size_t align256(size_t v) { return (v + 255) / 256 * 256; }

extern "C" size_t pt_window_attn_workspace_bytes(int n_seq, int n_head, int vdim, int page_size, int max_len, int window, int keep_first) {
  const size_t heads = (size_t)n_seq * n_head, pages = decode_pages(page_size, max_len, window, keep_first);
  return align256(heads * sizeof(int)) + align256(heads * pages * sizeof(float2)) + heads * pages * vdim * sizeof(float);
}

extern "C" int pt_window_attn(const pt_window_attn_args *a, void *stream) {
  PT_REQUIRE(a, "pt_window_attn: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.n_tok >= b.n_seq && b.cu && b.start && b.slot && b.tok_seq, "pt_window_attn: bad batch (%d sequences, %d tokens)", b.n_seq, b.n_tok);
  PT_REQUIRE(a->n_head > 0 && a->n_kv > 0 && a->n_head % a->n_kv == 0, "pt_window_attn: n_head=%d must be a positive multiple of n_kv=%d", a->n_head, a->n_kv);
  PT_REQUIRE(a->dim > 0 && a->vdim > 0 && a->page_size > 0 && a->max_pages > 0, "pt_window_attn: bad shape dim=%d vdim=%d page_size=%d max_pages=%d", a->dim,
             a->vdim, a->page_size, a->max_pages);
  PT_REQUIRE(a->window >= 0 && a->keep_first >= 0, "pt_window_attn: window=%d keep_first=%d", a->window, a->keep_first);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_window_attn: type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->q && a->pool && a->page_table && a->out && (!a->k == !a->v), "pt_window_attn: null pointer argument");
  PT_REQUIRE(a->q_ld >= a->n_head * a->dim && a->out_ld >= a->n_head * a->vdim && (!a->k || a->kv_ld >= a->n_kv * std::max(a->dim, a->vdim)),
             "pt_window_attn: row strides q %d, kv %d, out %d too small", a->q_ld, a->kv_ld, a->out_ld);
  wa::Params p{};
  p.n_seq = b.n_seq; p.n_head = a->n_head; p.n_kv = a->n_kv; p.qpk = a->n_head / a->n_kv; p.dim = a->dim; p.vdim = a->vdim;
  p.page = a->page_size; p.max_pages = a->max_pages; p.window = a->window; p.keep_first = a->keep_first;
  p.q_ld = a->q_ld; p.kv_ld = a->kv_ld; p.out_ld = a->out_ld; p.scale = a->scale; p.sink = a->sink;
  p.q = a->q; p.k = a->k; p.v = a->v; p.pool = a->pool; p.out = a->out; p.page_table = a->page_table;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq; p.error_flag = a->error_flag;
  cudaStream_t st = as_stream(stream);
  if (p.k) {
    if (a->dtype == PT_DT_F32) wa::kv_append_kernel<float><<<b.n_tok, 128, 0, st>>>(p);
    else wa::kv_append_kernel<__nv_bfloat16><<<b.n_tok, 128, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_window_attn");
  }
  const size_t smem = (size_t)p.qpk * (p.dim + p.page + p.vdim + 3) * sizeof(float);
  PT_REQUIRE(smem <= 200 * 1024, "pt_window_attn: %d query heads per kv head of widths %d / %d need %zu bytes of shared memory", p.qpk, p.dim, p.vdim, smem);
  if (smem > 48 * 1024) {
    PT_CUDA(cudaFuncSetAttribute(wa::attn_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    PT_CUDA(cudaFuncSetAttribute(wa::attn_plain_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  }
  const dim3 grid(b.n_tok, a->n_kv);
  if (a->dtype == PT_DT_F32) wa::attn_plain_kernel<float><<<grid, wa::PLAIN_THREADS, smem, st>>>(p);
  else wa::attn_plain_kernel<__nv_bfloat16><<<grid, wa::PLAIN_THREADS, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_window_attn");
  return PT_OK;
}
