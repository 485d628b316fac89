// Masked attention over a paged cache with per-sequence positions: a sliding window, kept first tokens, a softmax sink, grouped
// heads, key and value widths of their own, optionally a norm and a rotation of every query and key head.  Position i sees key j when
// j <= i and (i - j < window or j < keep_first); window = 0 means every earlier key.  sink[h] acts as one more logit of head h that brings weight to the denominator only.  With a
// softcap c a score s becomes c tanh(s / c).  The output can be multiplied with the sigmoid of a gate, per element or per head.
// The values can be a part of the cached keys (a latent that all heads share), and prompts can read keys and values from rows of the
// whole context instead of pages (pt_context_rows: a latent that was projected up), with a part of the key shared by all heads.
//
// The tokens of a launch are packed sequence after sequence (pt_batch_view): row cu[s] + i is position start[s] + i of sequence s,
// whose pages are page_table[slot[s]].  A page holds K [n_kv][page][dim] and then V [n_kv][page][vdim].  New keys and values are
// appended first; a layer that shares another layer's cache passes none and reads what is there.
//
//   attn_prep_kernel    norm and rotation of a prompt's queries and keys, and the append
//   attn_plain_kernel   any sizes, fp32 or bf16 caches, CUDA cores: the 32-bit path and the shapes the others do not take
//   attn_prompt_kernel  bf16 prompts: 64 queries of one head per block, Q K^T and P V on the tensor cores, online softmax; only key
//                       tiles that hold a visible key are touched
//   attn_decode_kernel  bf16, one token per sequence: one block per (visible page, kv head, sequence), scores and P V on the tensor
//                       cores, pages combined by the last block to arrive; norm, rotation and append are fused
//   attn_rotate_kernel  rotation alone, of a prompt's bf16 queries
// Softcap and gate are in instantiations of their own (EXT) of the prompt and decode kernels.
// Scores, softmax and weights are fp32.  The tensor-core kernels multiply V with weights split into two bf16 parts (hi + lo), which
// keeps 16 significant bits of each weight.
#include "chunk.cuh"

namespace pt {
namespace wa {

constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  int n_seq, n_head, n_kv, qpk, dim, vdim, page, max_pages, max_len, window, keep_first;
  int q_ld, kv_ld, out_ld;
  float scale;
  const float *sink;
  const void *q, *k, *v;
  void *pool, *out;
  const int *page_table, *cu, *start, *slot, *tok_seq;
  int *error_flag;
  const float *q_norm, *k_norm;
  const float2 *rope;        // [positions][rope_half]
  float norm_eps, out_scale;
  int rope_half, out_cols;
  const void *gate;          // [n_tok][gate_ld]: n_head * vdim columns, or n_head with gate_heads
  int gate_ld;
  bool gate_heads, v_in_k;   // v_in_k: the pool holds keys only, the values are their dimensions v_col ..; row_ld: stride of its rows and of query heads
  int v_col, row_ld, hsplit;         // hsplit: blocks that share a kv head's query heads (plain kernel)
  float softcap;
  // rows of the whole context (prompts)
  const __nv_bfloat16 *ctx_k, *ctx_shared, *ctx_v;
  int ctx_ld, shared_ld, shared_dim;
  const int *ctx_cu;
  bool prep, pair_rows;      // queries and keys are normalised or rotated; their rows can be taken as pairs of neighbours
  // decode
  int grid_pages, qsplit;
  float *ws_o;      // [n_seq, n_head, grid_pages, vdim]
  float2 *ws_ml;    // [n_seq, n_head, grid_pages]
  int *counters;    // [n_seq, n_kv, qsplit]
};

// (ANY: the values may be inside the keys; the tensor-core kernels do not take such pools)
template <bool ANY> __device__ __forceinline__ size_t page_elems(const Params &p) { return (size_t)p.n_kv * p.page * (ANY && p.v_in_k ? p.row_ld : p.dim + p.vdim); }
template <typename T, bool ANY = false> __device__ __forceinline__ T *k_page(const Params &p, int phys, int g) {
  return reinterpret_cast<T *>(p.pool) + (size_t)phys * page_elems<ANY>(p) + (size_t)g * p.page * (ANY && p.v_in_k ? p.row_ld : p.dim);
}
template <typename T, bool ANY = false> __device__ __forceinline__ T *v_page(const Params &p, int phys, int g) {
  if (ANY && p.v_in_k) return k_page<T, ANY>(p, phys, g) + p.v_col;
  return reinterpret_cast<T *>(p.pool) + (size_t)phys * page_elems<ANY>(p) + (size_t)p.n_kv * p.page * p.dim + (size_t)g * p.page * p.vdim;
}
// Scores in the units of exp2 from raw products: scale and softcap.  (tanh z = 1 - 2 / (exp(2 z) + 1))
struct Score {
  float a, b;                // without a cap: a = scale log2(e).  With: b = cap log2(e), a = 2 scale log2(e) / cap
  bool capped;
  __device__ __forceinline__ Score(const Params &p, bool may_cap) {
    capped = may_cap && p.softcap > 0.f;
    a = capped ? 2.0f * p.scale * kLog2e / p.softcap : p.scale * kLog2e;
    b = p.softcap * kLog2e;
  }
  __device__ __forceinline__ float cap(float s) const { return b * (1.0f - __fdividef(2.0f, exp2f(a * s) + 1.0f)); }
  __device__ __forceinline__ float operator()(float s) const { return capped ? cap(s) : a * s; }
};
template <typename T> __device__ __forceinline__ float gate_at(const Params &p, int t, int head, int c) {
  if (!p.gate) return 1.f;
  const float z = to_f(reinterpret_cast<const T *>(p.gate)[(size_t)t * p.gate_ld + (p.gate_heads ? head : head * p.vdim + c)]);
  return 1.0f / (1.0f + expf(-z));
}
__device__ __forceinline__ bool visible(const Params &p, int pos, int key) {
  return key <= pos && (p.window == 0 || pos - key < p.window || key < p.keep_first);
}
// First page whose keys are not all behind the window of position pos.
__device__ __forceinline__ int window_page(const Params &p, int pos) { return p.window == 0 ? 0 : max(0, pos - p.window + 1) / p.page; }
// Pages that hold the kept first tokens (as far as they exist at position pos).
__device__ __forceinline__ int kept_pages(const Params &p, int pos) { return (min(p.keep_first, pos + 1) + p.page - 1) / p.page; }

// ------------------------------------------------------------------------------------------ norm, rotation, append
// One warp, a head's row of a query or key at a time.  put(i, value) may write over src (a lane reads what it writes).
template <typename T, typename Put>
__device__ __forceinline__ void norm_rotate_any(const Params &p, const T *src, const float *norm, int pos, Put put) {
  const int lane = threadIdx.x & 31, half = p.rope_half;
  float inv = 1.f;
  if (norm) {
    float ss = 0.f;
    for (int i = lane; i < p.dim; i += 32) {
      const float x = to_f(src[i]);
      ss = fmaf(x, x, ss);
    }
    inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.norm_eps);
  }
  auto at = [&](int i) { return to_f(src[i]) * inv * (norm ? __ldg(norm + i) : 1.f); };
  const float2 *cs = p.rope + (size_t)pos * half;
  for (int i = lane; i < half; i += 32) {
    const float u = at(i), v = at(i + half);
    const float2 c = __ldg(cs + i);
    put(i, u * c.x - v * c.y);
    put(i + half, v * c.x + u * c.y);
  }
  for (int i = 2 * half + lane; i < p.dim; i += 32) put(i, at(i));
}
// The same in registers for rows of up to 128 dimensions (p.pair_rows): a lane holds the neighbours i, i + 1 and their partners j,
// j + 1.  Behind the rotated dimensions the partners are the next two, and the angle is zero.  Angles and weights serve all heads.
__device__ __forceinline__ float2 load_pair(const float *p) { return *reinterpret_cast<const float2 *>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16 *p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(p)); }
struct HeadLane {
  int i, j;
  bool on;
  float2 c0, c1, wi, wj;
  __device__ __forceinline__ HeadLane(const Params &p, const float *norm, int pos) {
    const int u = 2 * (threadIdx.x & 31), half = p.rope_half;
    on = p.pair_rows && u < p.dim / 2;       // (nothing is loaded for rows that are taken the other way)
    i = u < half ? u : 2 * u;
    j = u < half ? u + half : 2 * u + 2;
    c0 = c1 = make_float2(1.f, 0.f);
    wi = wj = make_float2(1.f, 1.f);
    if (on && u < half) {
      const float4 c = __ldg(reinterpret_cast<const float4 *>(p.rope + (size_t)pos * half + u));
      c0 = make_float2(c.x, c.y);
      c1 = make_float2(c.z, c.w);
    }
    if (on && norm) {
      wi = __ldg(reinterpret_cast<const float2 *>(norm + i));
      wj = __ldg(reinterpret_cast<const float2 *>(norm + j));
    }
  }
  template <typename T> __device__ __forceinline__ void run(const Params &p, const T *src, bool norm, T *dst) const {
    float2 x = make_float2(0.f, 0.f), y = x;
    if (on) {
      x = load_pair(src + i);
      y = load_pair(src + j);
    }
    const float inv = norm ? 1.0f / sqrtf(warp_sum(fmaf(x.x, x.x, x.y * x.y) + fmaf(y.x, y.x, y.y * y.y)) / (float)p.dim + p.norm_eps) : 1.f;
    if (!on) return;
    x.x *= inv * wi.x; x.y *= inv * wi.y;
    y.x *= inv * wj.x; y.y *= inv * wj.y;
    const float a[2] = {x.x * c0.x - y.x * c0.y, x.y * c1.x - y.y * c1.y}, b[2] = {y.x * c0.x + x.x * c0.y, y.y * c1.x + x.y * c1.y};
    store_vec<2>(dst + i, a);
    store_vec<2>(dst + j, b);
  }
};
template <typename T> __device__ __forceinline__ void norm_rotate(const Params &p, const HeadLane &hl, const T *src, const float *norm, int pos, T *dst) {
  if (p.pair_rows) hl.run<T>(p, src, norm != nullptr, dst);
  else norm_rotate_any<T>(p, src, norm, pos, [&](int i, float y) { dst[i] = from_f<T>(y); });
}

constexpr int PREP_WARPS = 4;
template <typename T> __global__ void __launch_bounds__(PREP_WARPS * 32, 5) attn_prep_kernel(const Params p) {   // block: one token, warp: a head at a time
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.max_len) {
    if (lane == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  {
    const HeadLane hl(p, p.q_norm, pos);
#pragma unroll 4
    for (int h = warp; h < p.n_head; h += PREP_WARPS) {
      T *q = reinterpret_cast<T *>(const_cast<void *>(p.q)) + (size_t)t * p.q_ld + (size_t)h * p.dim;
      norm_rotate<T>(p, hl, q, p.q_norm, pos, q);
    }
  }
  if (!p.k) return;
  const HeadLane hl(p, p.k_norm, pos);
  const int phys = p.page_table[(size_t)p.slot[s] * p.max_pages + pos / p.page], at = pos % p.page;
  for (int g = warp; g < p.n_kv; g += PREP_WARPS) {
    const T *k = reinterpret_cast<const T *>(p.k) + (size_t)t * p.kv_ld + (size_t)g * p.dim, *v = reinterpret_cast<const T *>(p.v) + (size_t)t * p.kv_ld + (size_t)g * p.vdim;
    T *kc = k_page<T>(p, phys, g) + (size_t)at * p.dim, *vc = v_page<T>(p, phys, g) + (size_t)at * p.vdim;
    norm_rotate<T>(p, hl, k, p.k_norm, pos, kc);
    for (int i = lane; i < p.vdim; i += 32) vc[i] = v[i];
  }
}

// Rotation alone, of bf16 queries in place: a thread takes eight neighbouring pairs of one head.
__global__ void attn_rotate_kernel(const Params p) {
  const int per = p.rope_half / 8, i = blockIdx.x * blockDim.x + threadIdx.x;
  const int c = (i % per) * 8, h = i / per % p.n_head, t = i / (per * p.n_head);
  if (t >= p.cu[p.n_seq]) return;
  const int s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.max_len) {
    if (p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  __nv_bfloat16 *q = reinterpret_cast<__nv_bfloat16 *>(const_cast<void *>(p.q)) + (size_t)t * p.q_ld + (size_t)h * p.dim + c;
  const float4 *cs = reinterpret_cast<const float4 *>(p.rope + (size_t)pos * p.rope_half + c);
  float u[8], v[8];
  load_vec<8>(q, u);
  load_vec<8>(q + p.rope_half, v);
  uint4 a, b;
  uint32_t *ap = reinterpret_cast<uint32_t *>(&a), *bp = reinterpret_cast<uint32_t *>(&b);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float4 x = __ldg(cs + j);
    ap[j] = pack_bf2(u[2 * j] * x.x - v[2 * j] * x.y, u[2 * j + 1] * x.z - v[2 * j + 1] * x.w);
    bp[j] = pack_bf2(v[2 * j] * x.x + u[2 * j] * x.y, v[2 * j + 1] * x.z + u[2 * j + 1] * x.w);
  }
  *reinterpret_cast<uint4 *>(q) = a;
  *reinterpret_cast<uint4 *>(q + p.rope_half) = b;
}

template <typename T> __global__ void kv_append_kernel(const Params p) {
  const int t = blockIdx.x, s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.max_len) {
    if (threadIdx.x == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int phys = p.page_table[(size_t)p.slot[s] * p.max_pages + pos / p.page], at = pos % p.page;
  const T *k = reinterpret_cast<const T *>(p.k) + (size_t)t * p.kv_ld, *v = reinterpret_cast<const T *>(p.v) + (size_t)t * p.kv_ld;
  for (int i = threadIdx.x; i < p.n_kv * p.dim; i += blockDim.x) k_page<T>(p, phys, i / p.dim)[(size_t)at * p.dim + i % p.dim] = k[i];
  for (int i = threadIdx.x; i < p.n_kv * p.vdim; i += blockDim.x) v_page<T>(p, phys, i / p.vdim)[(size_t)at * p.vdim + i % p.vdim] = v[i];
}

// ------------------------------------------------------------------------------------------ plain
// Block: one token and the query heads of one kv head, or a part of them (nh).  Dynamic shared memory: q [nh][dim], scores [nh][page],
// o [nh][vdim], statistics [nh][3].
constexpr int PLAIN_THREADS = 128;
template <typename T> __global__ void __launch_bounds__(PLAIN_THREADS) attn_plain_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  const int nh = p.qpk / p.hsplit, g = blockIdx.y / p.hsplit, h0 = blockIdx.y * nh, k_ld = p.v_in_k ? p.row_ld : p.dim, v_ld = p.v_in_k ? p.row_ld : p.vdim;   // (heads h0 .. h0 + nh - 1)
  float *q = sm, *sc = q + nh * p.dim, *o = sc + nh * p.page, *st = o + nh * p.vdim;   // st: running max, sum, correction
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.max_len) {
    if (tid == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int *table = p.page_table + (size_t)p.slot[s] * p.max_pages;
  const T *qrow = reinterpret_cast<const T *>(p.q) + (size_t)t * p.q_ld + (size_t)h0 * k_ld;
  for (int i = tid; i < nh * p.dim; i += PLAIN_THREADS) q[i] = to_f(qrow[(size_t)(i / p.dim) * k_ld + i % p.dim]);
  for (int i = tid; i < nh * p.vdim; i += PLAIN_THREADS) o[i] = 0.f;
  for (int h = tid; h < nh; h += PLAIN_THREADS) {
    st[3 * h] = p.sink ? p.sink[h0 + h] : -INFINITY;
    st[3 * h + 1] = p.sink ? 1.f : 0.f;
  }
  const int kept = kept_pages(p, pos), wpage = window_page(p, pos);
  for (int pg = kept > 0 ? 0 : wpage; pg <= pos / p.page; ++pg) {
    if (pg >= kept && pg < wpage) pg = wpage;
    const int k0 = pg * p.page, nk = min(p.page, pos + 1 - k0);
    const T *K = k_page<T, true>(p, table[pg], g), *V = v_page<T, true>(p, table[pg], g);
    __syncthreads();
    for (int i = warp; i < nh * nk; i += PLAIN_THREADS / 32) {
      const int h = i / nk, key = i - h * nk;
      float a = 0.f;
      for (int c = lane; c < p.dim; c += 32) a = fmaf(q[h * p.dim + c], to_f(K[(size_t)key * k_ld + c]), a);
      a = warp_sum(a);
      a *= p.scale;
      if (p.softcap > 0.f) a = p.softcap * tanhf(a / p.softcap);
      if (lane == 0) sc[h * p.page + key] = visible(p, pos, k0 + key) ? a : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < nh; h += PLAIN_THREADS / 32) {
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
    for (int i = tid; i < nh * p.vdim; i += PLAIN_THREADS) {
      const int h = i / p.vdim, c = i - h * p.vdim;
      float a = o[i] * st[3 * h + 2];
      for (int key = 0; key < nk; ++key) a = fmaf(sc[h * p.page + key], to_f(V[(size_t)key * v_ld + c]), a);
      o[i] = a;
    }
  }
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld + (size_t)h0 * p.vdim;
  for (int i = tid; i < nh * p.vdim; i += PLAIN_THREADS)
    out[i] = from_f<T>(o[i] / st[3 * (i / p.vdim) + 1] * p.out_scale * gate_at<T>(p, t, h0 + i / p.vdim, i % p.vdim));
  if (blockIdx.y == gridDim.y - 1)   // k padding of the output product
    for (int i = p.n_head * p.vdim + tid; i < p.out_cols; i += PLAIN_THREADS) reinterpret_cast<T *>(p.out)[(size_t)t * p.out_ld + i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------ tensor cores
constexpr int TC_THREADS = 128, TILE = 64;   // TILE = the page size the tensor-core kernels take

// ------------------------------------------------------------------------------------------ prompts
// Block: 64 new tokens of one sequence, one head; warp w owns queries 16 w .. 16 w + 15, their q fragments stay in registers.  Key
// tiles (one page each) are double-buffered in shared memory; tiles without a visible key are skipped, tiles that every query of
// the warp sees completely take no mask.  DK / DV: dim / vdim rounded up to 32, 64, 128 .. (the padding holds zeros).  CTX: keys and
// values are rows of the context; the first shared_dim dimensions of a key belong to all heads.
template <int DK, int DV, bool CTX, bool EXT> __global__ void __launch_bounds__(TC_THREADS, DK > 128 ? 2 : 3) attn_prompt_kernel(const Params p) {
  constexpr int KLD = DK + 8, VLD = DV + 8;
  extern __shared__ __align__(16) __nv_bfloat16 smb[];
  __nv_bfloat16 *Ks = smb, *Vs = smb + 2 * TILE * KLD;      // [2][TILE][KLD], [2][TILE][VLD]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int s = blockIdx.z, head = blockIdx.y, t0 = (gridDim.x - 1 - blockIdx.x) * TILE, kvh = head / p.qpk;   // (the tiles with most keys first)
  const int row0 = p.cu[s], len = p.cu[s + 1] - row0, start = p.start[s];
  if (t0 >= len) return;
  if (start < 0 || start + len > p.max_len) {
    if (tid == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int *table = p.page_table + (size_t)p.slot[s] * p.max_pages;
  const int q0 = t0 + warp * 16 + g, q1 = q0 + 8;           // this lane's two queries
  const bool ok0 = q0 < len, ok1 = q1 < len;
  const int pos0 = start + q0, pos1 = start + q1;
  const int lo = start + t0, hi = start + min(len, t0 + TILE) - 1;                                  // positions of the block's queries
  const int wlo = start + t0 + warp * 16, whi = start + min(len, t0 + warp * 16 + 16) - 1;          // ... and of the warp's (whi < wlo: none)
  uint32_t qa[DK / 16][4];
  {
    const __nv_bfloat16 *q = reinterpret_cast<const __nv_bfloat16 *>(p.q) + (size_t)head * p.dim + 2 * tig;
    const __nv_bfloat16 *r0 = q + (size_t)(row0 + (ok0 ? q0 : 0)) * p.q_ld, *r1 = q + (size_t)(row0 + (ok1 ? q1 : 0)) * p.q_ld;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      const bool in0 = kk * 16 < p.dim, in1 = kk * 16 + 8 < p.dim;
      qa[kk][0] = (ok0 && in0) ? *reinterpret_cast<const uint32_t *>(r0 + kk * 16) : 0u;
      qa[kk][1] = (ok1 && in0) ? *reinterpret_cast<const uint32_t *>(r1 + kk * 16) : 0u;
      qa[kk][2] = (ok0 && in1) ? *reinterpret_cast<const uint32_t *>(r0 + kk * 16 + 8) : 0u;
      qa[kk][3] = (ok1 && in1) ? *reinterpret_cast<const uint32_t *>(r1 + kk * 16 + 8) : 0u;
    }
  }
  auto load_tile = [&](int kt, int stage) {
    if constexpr (CTX) {
      const size_t row = (size_t)p.ctx_cu[s] + kt * TILE;
      const int own = p.dim - p.shared_dim;
      const __nv_bfloat16 *gS = p.ctx_shared + row * p.shared_ld, *gK = p.ctx_k + row * p.ctx_ld + (size_t)kvh * own - p.shared_dim,
                          *gV = p.ctx_v + row * p.ctx_ld + (size_t)kvh * p.vdim;
      __nv_bfloat16 *k = Ks + stage * TILE * KLD, *v = Vs + stage * TILE * VLD;
      for (int e = tid; e < TILE * (DK / 8); e += TC_THREADS) {
        const int r = e / (DK / 8), c = (e % (DK / 8)) * 8;
        const bool in = kt * TILE + r <= hi && c < p.dim;
        cp16(k + r * KLD + c, !in ? p.ctx_k : c < p.shared_dim ? gS + (size_t)r * p.shared_ld + c : gK + (size_t)r * p.ctx_ld + c, in);
      }
      for (int e = tid; e < TILE * (DV / 8); e += TC_THREADS) {
        const int r = e / (DV / 8), c = (e % (DV / 8)) * 8;
        const bool in = kt * TILE + r <= hi && c < p.vdim;
        cp16(v + r * VLD + c, in ? gV + (size_t)r * p.ctx_ld + c : p.ctx_k, in);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
      return;
    }
    const int phys = table[kt];
    const __nv_bfloat16 *gK = k_page<__nv_bfloat16>(p, phys, kvh), *gV = v_page<__nv_bfloat16>(p, phys, kvh);
    __nv_bfloat16 *k = Ks + stage * TILE * KLD, *v = Vs + stage * TILE * VLD;
    for (int e = tid; e < TILE * (DK / 8); e += TC_THREADS) {
      const int r = e / (DK / 8), c = (e % (DK / 8)) * 8;
      const bool in = kt * TILE + r <= hi && c < p.dim;
      cp16(k + r * KLD + c, gK + (in ? (size_t)r * p.dim + c : 0), in);
    }
    for (int e = tid; e < TILE * (DV / 8); e += TC_THREADS) {
      const int r = e / (DV / 8), c = (e % (DV / 8)) * 8;
      const bool in = kt * TILE + r <= hi && c < p.vdim;
      cp16(v + r * VLD + c, gV + (in ? (size_t)r * p.vdim + c : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int kept = kept_pages(p, hi), wtile = window_page(p, lo), last = hi / TILE;
  auto next_tile = [&](int kt) { return (kt >= kept && kt < wtile) ? wtile : kt; };
  const Score score(p, EXT);
  const float sink2 = p.sink ? p.sink[head] * kLog2e : -INFINITY;
  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_run[2] = {sink2, sink2}, l_run[2] = {0.f, 0.f};
  int kt = next_tile(0), stage = 0;
  load_tile(kt, 0);
  for (; kt <= last; stage ^= 1) {
    const int nt = next_tile(kt + 1);
    if (nt <= last) {
      load_tile(nt, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int k0 = kt * TILE;
    // anything of this tile for this warp?  (uniform over the warp)
    if (wlo <= whi && k0 <= whi && (p.window == 0 || k0 + TILE - 1 > wlo - p.window || k0 < p.keep_first)) {
      const __nv_bfloat16 *K = Ks + stage * TILE * KLD;
      float sc[TILE / 8][4];
      // (matrices of a load: keys 0-7 with channels 0-7 and 8-15, then keys 8-15 likewise)
      const uint32_t k_lane = smem_addr(K + ((lane & 7) + (lane >> 4) * 8) * KLD + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int j = 0; j < TILE / 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk)      // (channels outside: the products of one step are independent)
#pragma unroll
        for (int j = 0; j < TILE / 8; j += 2) {
          uint32_t b0, b1, b2, b3;
          ldsm4(k_lane + (uint32_t)(j * 8 * KLD + kk * 16) * 2u, b0, b1, b2, b3);
          mma16816_bf16(sc[j], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b0, b1);
          mma16816_bf16(sc[j + 1], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b2, b3);
        }
      const bool whole = k0 + TILE - 1 <= wlo && (p.window == 0 || whi - k0 < p.window || k0 + TILE <= p.keep_first);
      if (EXT && score.capped) {                                  // (uniform)
#pragma unroll
        for (int j = 0; j < TILE / 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[j][e] = score.cap(sc[j][e]);
      } else {
#pragma unroll
        for (int j = 0; j < TILE / 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[j][e] *= score.a;
      }
      float m_new[2] = {m_run[0], m_run[1]};
#pragma unroll
      for (int j = 0; j < TILE / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = k0 + j * 8 + 2 * tig + (e & 1);
          float v = sc[j][e];
          if (!whole && !visible(p, e < 2 ? pos0 : pos1, key)) v = -INFINITY;
          sc[j][e] = v;
          m_new[e >> 1] = fmaxf(m_new[e >> 1], v);
        }
      float corr[2], base[2], l_tile[2] = {0.f, 0.f};
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        m_new[r] = fmaxf(m_new[r], __shfl_xor_sync(0xffffffffu, m_new[r], 1));
        m_new[r] = fmaxf(m_new[r], __shfl_xor_sync(0xffffffffu, m_new[r], 2));
        base[r] = m_new[r] == -INFINITY ? 0.f : m_new[r];       // nothing seen yet: every weight below is exp2(-inf) = 0
        corr[r] = exp2f(m_run[r] - base[r]);
        m_run[r] = m_new[r];
      }
#pragma unroll
      for (int j = 0; j < TILE / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sc[j][e] = exp2f(sc[j][e] - base[e >> 1]);
          l_tile[e >> 1] += sc[j][e];
        }
      l_run[0] = l_run[0] * corr[0] + l_tile[0];                // per lane; the four lanes of a row are added at the end
      l_run[1] = l_run[1] * corr[1] + l_tile[1];
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) {
        o[j][0] *= corr[0]; o[j][1] *= corr[0];
        o[j][2] *= corr[1]; o[j][3] *= corr[1];
      }
      const uint32_t v_lane = smem_addr(Vs + stage * TILE * VLD + (lane & 15) * VLD + (lane >> 4) * 8);
#pragma unroll
      for (int k2 = 0; k2 < TILE / 16; ++k2) {
        uint32_t h[4], l[4];                                    // weights as hi + lo: A fragments of two products
        split_bf2(sc[2 * k2][0], sc[2 * k2][1], h[0], l[0]);
        split_bf2(sc[2 * k2][2], sc[2 * k2][3], h[1], l[1]);
        split_bf2(sc[2 * k2 + 1][0], sc[2 * k2 + 1][1], h[2], l[2]);
        split_bf2(sc[2 * k2 + 1][2], sc[2 * k2 + 1][3], h[3], l[3]);
#pragma unroll
        for (int jn = 0; jn < DV / 8; jn += 2) {
          uint32_t b0, b1, b2, b3;
          ldsm4t(v_lane + (uint32_t)(k2 * 16 * VLD + jn * 8) * 2u, b0, b1, b2, b3);
          mma16816_bf16(o[jn], h[0], h[1], h[2], h[3], b0, b1);
          mma16816_bf16(o[jn + 1], h[0], h[1], h[2], h[3], b2, b3);
          mma16816_bf16(o[jn], l[0], l[1], l[2], l[3], b0, b1);
          mma16816_bf16(o[jn + 1], l[0], l[1], l[2], l[3], b2, b3);
        }
      }
    }
    __syncthreads();                                            // the stage may be refilled
    kt = nt;
  }
  float inv[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    if (p.sink) l += exp2f(sink2 - m_run[r]);                   // the sink, in the units of the running maximum
    inv[r] = p.out_scale / l;
  }
  __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(p.out) + (size_t)head * p.vdim + 2 * tig;
  if (EXT && p.gate && p.gate_heads) {
    if (ok0) inv[0] *= gate_at<__nv_bfloat16>(p, row0 + q0, head, 0);
    if (ok1) inv[1] *= gate_at<__nv_bfloat16>(p, row0 + q1, head, 0);
  }
  const bool each = EXT && p.gate && !p.gate_heads;
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) {
    if (j * 8 >= p.vdim) break;
    if (each) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        if (!(r ? ok1 : ok0)) continue;
        const float2 z = load_pair(reinterpret_cast<const __nv_bfloat16 *>(p.gate) + (size_t)(row0 + (r ? q1 : q0)) * p.gate_ld + head * p.vdim + 2 * tig + j * 8);
        o[j][2 * r] *= __fdividef(1.0f, 1.0f + __expf(-z.x));          // (rounded to bf16 below)
        o[j][2 * r + 1] *= __fdividef(1.0f, 1.0f + __expf(-z.y));
      }
    }
    if (ok0) *reinterpret_cast<uint32_t *>(out + (size_t)(row0 + q0) * p.out_ld + j * 8) = pack_bf2(o[j][0] * inv[0], o[j][1] * inv[0]);
    if (ok1) *reinterpret_cast<uint32_t *>(out + (size_t)(row0 + q1) * p.out_ld + j * 8) = pack_bf2(o[j][2] * inv[1], o[j][3] * inv[1]);
  }
  const int pad = p.out_cols - p.n_head * p.vdim;
  if (head == p.n_head - 1)
    for (int i = tid; i < TILE * pad; i += TC_THREADS) {
      const int r = t0 + i / pad;
      if (r < len) reinterpret_cast<__nv_bfloat16 *>(p.out)[(size_t)(row0 + r) * p.out_ld + p.n_head * p.vdim + i % pad] = from_f<__nv_bfloat16>(0.f);
    }
}

// ------------------------------------------------------------------------------------------ one token per sequence
// Block: one visible page of one (sequence, kv head, part of the group's query heads).  scores^T [keys x heads] = K q^T with the K
// rows straight from global memory as A fragments (the k order is a permutation of the channels that q follows); out [heads x vdim]
// = P V with V staged in shared memory.  Rows 0..7 of P's A fragment are the hi parts of up to 8 heads' weights, rows 8..15 the lo
// parts, so the split costs no extra product.  The block of the newest page takes the new key and value from the projection and
// appends them.
constexpr int NQ = 8;
template <int DK, int DV, bool EXT> __global__ void __launch_bounds__(TC_THREADS) attn_decode_kernel(const Params p) {
  constexpr int VLD = DV + 8, QLD = DK + 32, PSLD = TILE + 8;
  typedef __nv_bfloat16 T;
  extern __shared__ __align__(16) unsigned char smd[];
  T *Vs = reinterpret_cast<T *>(smd);                          // [TILE][VLD]
  T *qs = Vs + TILE * VLD;                                     // [NQ][QLD]
  float *ps = reinterpret_cast<float *>(qs + NQ * QLD);        // [NQ][PSLD]
  float *ml = ps + NQ * PSLD;                                  // [NQ][2]
  T *kn = reinterpret_cast<T *>(ml + NQ * 2);                  // [DK] the newest key, normalised and rotated
  float *cw = reinterpret_cast<float *>(kn + DK);              // combine: [NQ][grid_pages] weights
  __shared__ int s_last;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int s = blockIdx.z, kvh = blockIdx.y / p.qsplit, part = blockIdx.y - kvh * p.qsplit;
  const int nq = p.qpk / p.qsplit, h0 = kvh * p.qpk + part * nq;           // this block's query heads h0 .. h0 + nq - 1
  const int pos = p.start[s], t = p.cu[s];
  if (pos < 0 || pos >= p.max_len) {
    if (tid == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int last = pos / TILE, kept = kept_pages(p, pos), wp = window_page(p, pos);
  const int n_act = kept >= wp ? last + 1 : kept + last - wp + 1;
  const int x = blockIdx.x;
  if (x >= n_act) return;
  const int pg = (kept >= wp || x < kept) ? x : wp + x - kept;
  const int phys = p.page_table[(size_t)p.slot[s] * p.max_pages + pg];
  const int k0 = pg * TILE, n_valid = min(TILE, pos + 1 - k0);
  const bool owner = pg == last && p.k != nullptr;
  const int n_load = owner ? n_valid - 1 : n_valid, at = n_valid - 1;      // owner: the newest key is not in the pool yet
  T *gK = k_page<T>(p, phys, kvh), *gV = v_page<T>(p, phys, kvh);
  const T *knew = reinterpret_cast<const T *>(p.k) + (size_t)t * p.kv_ld + (size_t)kvh * p.dim;
  const T *vnew = reinterpret_cast<const T *>(p.v) + (size_t)t * p.kv_ld + (size_t)kvh * p.vdim;

  uint4 kf[2][DK / 32];                                        // K rows 16 warp + g and + 8 of the page
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int key = warp * 16 + g + 8 * r;
#pragma unroll
    for (int pp = 0; pp < DK / 32; ++pp) {
      const int c = pp * 32 + tig * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (c < p.dim) {
        if (key < n_load) v = __ldcg(reinterpret_cast<const uint4 *>(gK + (size_t)key * p.dim + c));
        else if (owner && !p.prep && key == at) v = *reinterpret_cast<const uint4 *>(knew + c);
      }
      kf[r][pp] = v;
    }
  }
  for (int e = tid; e < TILE * (DV / 8); e += TC_THREADS) {
    const int r = e / (DV / 8), c = (e % (DV / 8)) * 8;
    const bool in = c < p.vdim && (r < n_load || (owner && r == at));
    const T *src = (owner && r == at) ? vnew + c : gV + (size_t)r * p.vdim + c;
    cp16(Vs + r * VLD + c, in ? src : gV, in);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.q_ld + (size_t)h0 * p.dim;
  if (p.prep) {
    const HeadLane hq(p, p.q_norm, pos), hk(p, p.k_norm, pos);
    for (int h = warp; h < NQ + 1; h += TC_THREADS / 32) {
      T *dst = h < NQ ? qs + h * QLD : kn;
      const bool have = h < NQ ? h < nq : owner;
      if (have) norm_rotate<T>(p, h < NQ ? hq : hk, h < NQ ? q + (size_t)h * p.dim : knew, h < NQ ? p.q_norm : p.k_norm, pos, dst);
      for (int i = (have ? p.dim : 0) + lane; i < DK; i += 32) dst[i] = from_f<T>(0.f);
    }
  } else for (int i = tid; i < NQ * (DK / 8); i += TC_THREADS) {
    const int h = i / (DK / 8), c = (i % (DK / 8)) * 8;
    *reinterpret_cast<uint4 *>(qs + h * QLD + c) = (h < nq && c < p.dim) ? *reinterpret_cast<const uint4 *>(q + (size_t)h * p.dim + c) : make_uint4(0, 0, 0, 0);
  }
  for (int i = tid; i < NQ * PSLD; i += TC_THREADS) ps[i] = -INFINITY;
  if (owner && part == 0) {
    if (!p.prep)
      for (int c = tid; c < p.dim; c += TC_THREADS) gK[(size_t)at * p.dim + c] = knew[c];
    for (int c = tid; c < p.vdim; c += TC_THREADS) gV[(size_t)at * p.vdim + c] = vnew[c];
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  if (owner && p.prep) {
    if (part == 0)
      for (int c = tid; c < p.dim; c += TC_THREADS) gK[(size_t)at * p.dim + c] = kn[c];
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if (warp * 16 + g + 8 * r == at) {
#pragma unroll
        for (int pp = 0; pp < DK / 32; ++pp) kf[r][pp] = *reinterpret_cast<const uint4 *>(kn + pp * 32 + tig * 8);
      }
  }

  if (warp * 16 < n_valid) {
    float sc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int pp = 0; pp < DK / 32; ++pp) {
      const uint4 qv = *reinterpret_cast<const uint4 *>(qs + g * QLD + pp * 32 + tig * 8);
      mma16816_bf16(sc, kf[0][pp].x, kf[1][pp].x, kf[0][pp].y, kf[1][pp].y, qv.x, qv.y);
      mma16816_bf16(sc, kf[0][pp].z, kf[1][pp].z, kf[0][pp].w, kf[1][pp].w, qv.z, qv.w);
    }
    const Score score(p, EXT);
#pragma unroll
    for (int e = 0; e < 4; ++e) {                              // keys 16 warp + g (+ 8) against heads 2 tig, 2 tig + 1
      const int key = warp * 16 + g + 8 * (e >> 1), h = 2 * tig + (e & 1);
      if (h < nq && key < n_valid && visible(p, pos, k0 + key)) ps[h * PSLD + key] = score(sc[e]);
    }
  }
  __syncthreads();
  for (int h = warp; h < NQ; h += TC_THREADS / 32) {
    float *pr = ps + h * PSLD;
    if (h >= nq) {
      pr[lane] = pr[lane + 32] = 0.f;
      continue;
    }
    const float a = pr[lane], b = pr[lane + 32], m = warp_max(fmaxf(a, b));
    const float base = m == -INFINITY ? 0.f : m, ea = exp2f(a - base), eb = exp2f(b - base);
    pr[lane] = ea;
    pr[lane + 32] = eb;
    const float l = warp_sum(ea + eb);
    if (lane == 0) { ml[2 * h] = m; ml[2 * h + 1] = l; }
  }
  __syncthreads();
  const size_t head0 = (size_t)s * p.n_head + h0;
  {
    constexpr int NT = DV / 32;                                // 8-channel tiles per warp
    float o[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const float *pr = ps + g * PSLD + 2 * tig;
    const uint32_t v_lane = smem_addr(Vs + (lane & 15) * VLD + warp * (DV / 4) + (NT > 1 ? (lane >> 4) * 8 : 0));
    for (int k2 = 0; k2 * 16 < n_valid; ++k2) {
      const float2 p0 = *reinterpret_cast<const float2 *>(pr + k2 * 16), p1 = *reinterpret_cast<const float2 *>(pr + k2 * 16 + 8);
      uint32_t a0, a1, a2, a3;
      split_bf2(p0.x, p0.y, a0, a1);
      split_bf2(p1.x, p1.y, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm4t(v_lane + (uint32_t)(k2 * 16 * VLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(o[j], a0, a1, a2, a3, b0, b1);
        if (j + 1 < NT) mma16816_bf16(o[j + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    if (g < nq) {
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = warp * (DV / 4) + j * 8 + 2 * tig;
        if (c < p.vdim)
          *reinterpret_cast<float2 *>(&p.ws_o[((head0 + g) * p.grid_pages + x) * p.vdim + c]) = make_float2(o[j][0] + o[j][2], o[j][1] + o[j][3]);
      }
    }
  }
  if (tid < nq) p.ws_ml[(head0 + tid) * p.grid_pages + x] = make_float2(ml[2 * tid], ml[2 * tid + 1]);

  // ---- the last block of this (sequence, kv head, part) combines the pages in page order
  __threadfence();
  __syncthreads();
  int *ctr = p.counters + ((size_t)s * p.n_kv + kvh) * p.qsplit + part;
  if (tid == 0) s_last = atomicAdd(ctr, 1) == n_act - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  if (tid == 0) *ctr = 0;
  for (int h = warp; h < nq; h += TC_THREADS / 32) {
    const float2 *src = p.ws_ml + (head0 + h) * p.grid_pages;
    const float sink2 = p.sink ? p.sink[h0 + h] * kLog2e : -INFINITY;
    float m = sink2;
    for (int i = lane; i < n_act; i += 32) m = fmaxf(m, __ldcg(&src[i]).x);
    m = warp_max(m);
    float l = 0.f;
    for (int i = lane; i < n_act; i += 32) {
      const float2 v = __ldcg(&src[i]);
      const float w = exp2f(v.x - m);
      cw[h * p.grid_pages + i] = w;
      l += v.y * w;
    }
    l = warp_sum(l);
    if (lane == 0) ml[2 * h] = p.out_scale / (l + (p.sink ? exp2f(sink2 - m) : 0.f));
  }
  __syncthreads();
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld;
  const int v4 = p.vdim / 4;                                    // (vdim is a multiple of 8 here)
  for (int i = tid; i < nq * v4; i += TC_THREADS) {
    const int h = i / v4, c = (i - h * v4) * 4;
    const float *src = p.ws_o + ((head0 + h) * p.grid_pages) * p.vdim + c, *w = cw + h * p.grid_pages;
    constexpr int PB = 8;                                      // pages in flight
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int i0 = 0; i0 < n_act; i0 += PB) {
      float4 v[PB];
#pragma unroll
      for (int j = 0; j < PB; ++j) v[j] = i0 + j < n_act ? __ldcg(reinterpret_cast<const float4 *>(src + (size_t)(i0 + j) * p.vdim)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < PB; ++j)
        if (i0 + j < n_act) {
          const float x = w[i0 + j];
          acc[0] = fmaf(v[j].x, x, acc[0]);
          acc[1] = fmaf(v[j].y, x, acc[1]);
          acc[2] = fmaf(v[j].z, x, acc[2]);
          acc[3] = fmaf(v[j].w, x, acc[3]);
        }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] *= ml[2 * h];
    if (EXT && p.gate) {
      const T *gate = reinterpret_cast<const T *>(p.gate) + (size_t)t * p.gate_ld + (p.gate_heads ? h0 + h : (h0 + h) * p.vdim + c);
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j] *= __fdividef(1.0f, 1.0f + __expf(-to_f(gate[p.gate_heads ? 0 : j])));
    }
    T *o = out + (size_t)(h0 + h) * p.vdim + c;                // (rows of an even number of elements)
    *reinterpret_cast<__nv_bfloat162 *>(o) = __floats2bfloat162_rn(acc[0], acc[1]);
    *reinterpret_cast<__nv_bfloat162 *>(o + 2) = __floats2bfloat162_rn(acc[2], acc[3]);
  }
  if (h0 + nq == p.n_head)
    for (int i = p.n_head * p.vdim + tid; i < p.out_cols; i += TC_THREADS) out[i] = from_f<T>(0.f);
}

template <int DK, int DV, bool CTX, bool EXT> static int launch_prompt(const Params &p, int longest, cudaStream_t st) {
  constexpr size_t smem = 2 * (size_t)TILE * (DK + 8 + DV + 8) * sizeof(__nv_bfloat16);
  static bool set = false;
  if (!set) { PT_CUDA(cudaFuncSetAttribute(attn_prompt_kernel<DK, DV, CTX, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); set = true; }
  attn_prompt_kernel<DK, DV, CTX, EXT><<<dim3(ceil_div(longest, TILE), p.n_head, p.n_seq), TC_THREADS, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_window_attn");
  return PT_OK;
}
template <int DK, int DV, bool EXT> static int launch_decode(const Params &p, cudaStream_t st) {
  const size_t smem = (size_t)(TILE * (DV + 8) + NQ * (DK + 32) + DK) * sizeof(__nv_bfloat16) + (size_t)(NQ * (TILE + 8) + NQ * 2 + NQ * p.grid_pages) * sizeof(float);
  PT_REQUIRE(smem <= 200 * 1024, "pt_window_attn: %d pages per sequence need %zu bytes of shared memory", p.grid_pages, smem);
  static bool set = false;
  if (!set) { PT_CUDA(cudaFuncSetAttribute(attn_decode_kernel<DK, DV, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); set = true; }
  attn_decode_kernel<DK, DV, EXT><<<dim3(p.grid_pages, p.n_kv * p.qsplit, p.n_seq), TC_THREADS, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_window_attn");
  return PT_OK;
}
template <int DK, int DV> static int dispatch_ext(const Params &p, bool decode, int longest, cudaStream_t st) {
  if (p.softcap > 0.f || p.gate) return decode ? launch_decode<DK, DV, true>(p, st) : launch_prompt<DK, DV, false, true>(p, longest, st);
  return decode ? launch_decode<DK, DV, false>(p, st) : launch_prompt<DK, DV, false, false>(p, longest, st);
}
template <int DK> static int dispatch_v(const Params &p, bool decode, int longest, cudaStream_t st) {
  if (p.vdim <= 32) return dispatch_ext<DK, 32>(p, decode, longest, st);
  if (p.vdim <= 64) return dispatch_ext<DK, 64>(p, decode, longest, st);
  return dispatch_ext<DK, 128>(p, decode, longest, st);
}
template <int DK> static int dispatch_ctx(const Params &p, int longest, cudaStream_t st) {
  return p.vdim <= 64 ? launch_prompt<DK, 64, true, true>(p, longest, st) : launch_prompt<DK, 128, true, true>(p, longest, st);
}
static int dispatch_tc(const Params &p, bool decode, int longest, cudaStream_t st) {
  if (p.dim <= 32) return dispatch_v<32>(p, decode, longest, st);
  if (p.dim <= 64) return dispatch_v<64>(p, decode, longest, st);
  return dispatch_v<128>(p, decode, longest, st);
}
static int dispatch_ctx(const Params &p, int longest, cudaStream_t st) {
  if (p.dim <= 64) return dispatch_ctx<64>(p, longest, st);
  if (p.dim <= 128) return dispatch_ctx<128>(p, longest, st);
  if (p.dim <= 192) return dispatch_ctx<192>(p, longest, st);
  return dispatch_ctx<256>(p, longest, st);
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
// Workspace layout: [arrival counters][(max, sum) per page][outputs per page].  The counter region has ONE size, so that layers and
// batches of different shapes can share a workspace: the statistics of one never land where another expects zeroed counters.
constexpr size_t kCounterBytes = 1u << 18;

extern "C" size_t pt_window_attn_workspace_bytes(int n_seq, int n_head, int vdim, int page_size, int max_len, int window, int keep_first) {
  const size_t heads = (size_t)n_seq * n_head, pages = decode_pages(page_size, max_len, window, keep_first);
  return kCounterBytes + align256(heads * pages * sizeof(float2)) + heads * pages * vdim * sizeof(float);
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
  const pt_context_rows *ctx = a->context;
  PT_REQUIRE(a->q && a->out && (ctx || (a->pool && a->page_table)) && (!a->k == !a->v), "pt_window_attn: null pointer argument");
  PT_REQUIRE(a->q_ld >= a->n_head * a->dim && a->out_ld >= a->n_head * a->vdim && (!a->k || a->kv_ld >= a->n_kv * std::max(a->dim, a->vdim)),
             "pt_window_attn: row strides q %d, kv %d, out %d too small", a->q_ld, a->kv_ld, a->out_ld);
  wa::Params p{};
  p.n_seq = b.n_seq; p.n_head = a->n_head; p.n_kv = a->n_kv; p.qpk = a->n_head / a->n_kv; p.dim = a->dim; p.vdim = a->vdim;
  p.page = a->page_size; p.max_pages = a->max_pages; p.window = a->window; p.keep_first = a->keep_first;
  p.q_ld = a->q_ld; p.kv_ld = a->kv_ld; p.out_ld = a->out_ld; p.scale = a->scale; p.sink = a->sink;
  p.q = a->q; p.k = a->k; p.v = a->v; p.pool = a->pool; p.out = a->out; p.page_table = a->page_table;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq; p.error_flag = a->error_flag;
  p.q_norm = a->q_norm; p.k_norm = a->k_norm; p.norm_eps = a->norm_eps; p.rope = (const float2 *)a->rope; p.rope_half = a->rope_dims / 2;
  PT_REQUIRE(a->softcap >= 0.f && (!a->gate || a->gate_ld >= (a->gate_per_head ? a->n_head : a->n_head * a->vdim)), "pt_window_attn: softcap=%f gate_ld=%d", a->softcap,
             a->gate_ld);
  PT_REQUIRE(!a->values_in_keys || (!a->k && !ctx && a->value_col >= 0 && a->value_col + a->vdim <= a->dim),
             "pt_window_attn: values that are dimensions of the cached keys need value_col + vdim within dim and nothing to append");
  p.softcap = a->softcap; p.gate = a->gate; p.gate_ld = a->gate_ld; p.gate_heads = a->gate_per_head != 0;
  p.v_in_k = a->values_in_keys != 0; p.v_col = a->value_col; p.row_ld = a->row_ld > 0 ? a->row_ld : a->dim;
  PT_REQUIRE(p.row_ld >= a->dim && (!p.v_in_k || a->q_ld >= a->n_head * p.row_ld) && (p.v_in_k || p.row_ld == a->dim), "pt_window_attn: row_ld=%d", a->row_ld);
  p.out_scale = a->out_scale != 0.f ? a->out_scale : 1.0f;
  p.out_cols = a->out_cols > 0 ? a->out_cols : a->out_ld;
  p.prep = a->q_norm || a->k_norm || a->rope_dims;
  {
    const int pair = a->dtype == PT_DT_F32 ? 8 : 4;
    auto al = [](const void *x, int bytes) { return ((uintptr_t)x & (bytes - 1)) == 0; };
    p.pair_rows = a->dim % 4 == 0 && a->dim <= 128 && a->rope_dims % 4 == 0 && a->q_ld % 2 == 0 && a->n_kv * a->page_size * (p.v_in_k ? p.row_ld : a->dim + a->vdim) % 2 == 0 && al(a->q, pair) && al(a->pool, pair) && al(a->rope, 16) && al(a->q_norm, 8) &&
                  al(a->k_norm, 8) && (!a->k || (a->kv_ld % 2 == 0 && al(a->k, pair)));
  }
  PT_REQUIRE(a->rope_dims >= 0 && a->rope_dims % 2 == 0 && a->rope_dims <= a->dim && (!a->rope_dims || a->rope), "pt_window_attn: %d rotated dimensions of %d",
             a->rope_dims, a->dim);
  PT_REQUIRE(p.out_cols >= a->n_head * a->vdim && p.out_cols <= a->out_ld, "pt_window_attn: out_cols=%d", a->out_cols);
  p.max_len = a->max_len > 0 ? a->max_len : a->page_size * a->max_pages;
  PT_REQUIRE(ctx || p.max_len <= a->page_size * a->max_pages, "pt_window_attn: max_len=%d exceeds the %d positions of the page table", p.max_len,
             a->page_size * a->max_pages);
  cudaStream_t st = as_stream(stream);
  // the tensor-core kernels: bf16, 64-position pages, head widths of at most 128 whose rows are whole 16-byte units
  auto al16 = [](const void *x) { return ((uintptr_t)x & 15) == 0; };
  const bool gate_ok = !a->gate || (a->gate_ld % 2 == 0 && aligned_to(a->gate, 4));
  if (ctx) {
    PT_REQUIRE(a->dtype == PT_DT_BF16 && a->n_kv == a->n_head && !a->k && a->dim <= 256 && a->vdim <= 128 && a->dim % 8 == 0 && a->vdim % 8 == 0 && gate_ok && b.n_seq <= 65535,
               "pt_window_attn: context rows take bf16 heads of at most 256 / 128 dimensions in steps of 8, one key head per query head, and nothing to append");
    PT_REQUIRE(ctx->k && ctx->v && ctx->cu && ctx->shared_dim >= 0 && ctx->shared_dim <= a->dim && (!ctx->shared_dim || ctx->shared) && ctx->ld % 8 == 0 && ctx->shared_ld % 8 == 0 &&
                   ctx->shared_dim % 8 == 0 && al16(ctx->k) && al16(ctx->v) && al16(ctx->shared) && al16(a->q) && a->q_ld % 8 == 0 && a->out_ld % 2 == 0 && aligned_to(a->out, 4),
               "pt_window_attn: context rows in units of 16 bytes");
    p.ctx_k = (const __nv_bfloat16 *)ctx->k; p.ctx_v = (const __nv_bfloat16 *)ctx->v; p.ctx_shared = (const __nv_bfloat16 *)ctx->shared;
    p.ctx_ld = ctx->ld; p.shared_ld = ctx->shared_ld; p.shared_dim = ctx->shared_dim; p.ctx_cu = ctx->cu;
  }
  const bool tc = !a->plain && !ctx && !p.v_in_k && gate_ok && a->dtype == PT_DT_BF16 && a->page_size == wa::TILE && a->dim <= 128 && a->vdim <= 128 && a->dim % 8 == 0 && a->vdim % 8 == 0 &&
                  a->q_ld % 8 == 0 && a->out_ld % 2 == 0 && al16(a->q) && al16(a->pool) && (!a->k || (a->kv_ld % 8 == 0 && al16(a->k) && al16(a->v)));
  if (tc && b.n_tok == b.n_seq && b.n_seq <= 65535) {
    const size_t need = pt_window_attn_workspace_bytes(b.n_seq, a->n_head, a->vdim, a->page_size, p.max_len, a->window, a->keep_first);
    PT_REQUIRE(a->workspace && a->workspace_bytes >= need, "pt_window_attn: a decode step needs %zu workspace bytes, got %zu", need, a->workspace_bytes);
    p.grid_pages = decode_pages(a->page_size, p.max_len, a->window, a->keep_first);
    int nq = std::min(p.qpk, wa::NQ);
    while (p.qpk % nq) --nq;
    p.qsplit = p.qpk / nq;
    const size_t heads = (size_t)b.n_seq * a->n_head;
    char *ws = (char *)a->workspace;
    PT_REQUIRE((size_t)b.n_seq * a->n_kv * p.qsplit <= kCounterBytes / sizeof(int), "pt_window_attn: %d sequences x %d heads exceed the arrival counters", b.n_seq,
               a->n_head);
    p.counters = (int *)ws; ws += kCounterBytes;
    p.ws_ml = (float2 *)ws; ws += align256(heads * p.grid_pages * sizeof(float2));
    p.ws_o = (float *)ws;
    return wa::dispatch_tc(p, true, 1, st);
  }
  if (p.prep && !p.k && !a->q_norm && a->dtype == PT_DT_BF16 && p.rope_half % 8 == 0 && p.dim % 8 == 0 && p.q_ld % 8 == 0 && al16(p.q) && al16(p.rope) &&
      (long long)b.n_tok * p.n_head * p.rope_half < (1ll << 31)) {
    wa::attn_rotate_kernel<<<ceil_div(b.n_tok * p.n_head * (p.rope_half / 8), 256), 256, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_window_attn");
  } else if (p.prep) {
    if (a->dtype == PT_DT_F32) wa::attn_prep_kernel<float><<<b.n_tok, wa::PREP_WARPS * 32, 0, st>>>(p);
    else wa::attn_prep_kernel<__nv_bfloat16><<<b.n_tok, wa::PREP_WARPS * 32, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_window_attn");
  } else if (p.k) {
    if (a->dtype == PT_DT_F32) wa::kv_append_kernel<float><<<b.n_tok, 128, 0, st>>>(p);
    else wa::kv_append_kernel<__nv_bfloat16><<<b.n_tok, 128, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_window_attn");
  }
  if (ctx) return wa::dispatch_ctx(p, a->max_tokens_per_seq > 0 ? a->max_tokens_per_seq : b.n_tok, st);
  if (tc && b.n_seq <= 65535)
    return wa::dispatch_tc(p, false, a->max_tokens_per_seq > 0 ? a->max_tokens_per_seq : b.n_tok, st);
  // heads per block: what fits 64 KB of shared memory
  auto bytes = [&](int nh) { return (size_t)nh * (p.dim + p.page + p.vdim + 3) * sizeof(float); };
  p.hsplit = 1;
  while (p.hsplit < p.qpk && (p.qpk % p.hsplit || bytes(p.qpk / p.hsplit) > 64 * 1024)) ++p.hsplit;
  const size_t smem = bytes(p.qpk / p.hsplit);
  PT_REQUIRE(smem <= 200 * 1024, "pt_window_attn: a head of widths %d / %d needs %zu bytes of shared memory", p.dim, p.vdim, smem);
  if (smem > 48 * 1024) {
    PT_CUDA(cudaFuncSetAttribute(wa::attn_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    PT_CUDA(cudaFuncSetAttribute(wa::attn_plain_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  }
  PT_REQUIRE(a->n_kv * p.hsplit <= 65535, "pt_window_attn: %d heads", a->n_head);
  const dim3 grid(b.n_tok, a->n_kv * p.hsplit);
  if (a->dtype == PT_DT_F32) wa::attn_plain_kernel<float><<<grid, wa::PLAIN_THREADS, smem, st>>>(p);
  else wa::attn_plain_kernel<__nv_bfloat16><<<grid, wa::PLAIN_THREADS, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_window_attn");
  return PT_OK;
}
