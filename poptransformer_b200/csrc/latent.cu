// Attention over a latent: the cache holds, per position, one normalised latent of `rank` dimensions and one rotated key part of `rot`
// dimensions that all heads share.  Head h's key is [rotated part | W_uk[h] latent], its value W_uv[h] latent.
//
// Neither is formed for the cached positions of a decode step: q . W_uk c = (W_uk^T q) . c, so every head's query is taken into the
// latent's space, all heads attend over the same cached rows [rotated part | latent] whose latents are also the values, and W_uv is
// applied to the one vector per head that comes out.  Prompts on tensor cores project the whole context up instead
// (pt_latent_context, a matrix product, then pt_window_attn with context rows), which takes a third of the products when a sequence
// brings many queries.
//
//   prep_kernel      both latents' norms, rotation of the shared key part, append
//   context_kernel   the cached rows of every sequence's context, one after the other
//   absorb_kernel    W_uk^T q per head beside the rotated part of q (tensor cores; absorb_plain_kernel: any sizes, fp32 or bf16)
//   decode_kernel    bf16, one token per sequence: 16 or 32 heads x a run of pages, scores and weighted sum on tensor cores from one copy
//                    of the rows in shared memory, which half pages enter through a ring of bulk copies
//   combine_kernel   the runs of pages become one latent vector per head, with a gate per head
//   expand_kernel    W_uv per head, with a gate per output (expand_plain_kernel: any sizes, with either gate)
// A layer may read the latents that another one caches: its own prep then norms the query latent only.
// Prompts in fp32, or of sizes the tensor-core kernels do not take, go through pt_window_attn's any-size kernel with the values inside
// the keys.  Norms, angles, scores, softmax and weights are fp32; weights enter the tensor cores as two bf16 parts (hi + lo).
#include "chunk.cuh"
#include "mbarrier.cuh"

namespace pt {
namespace lat {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int TILE = 64;             // page size of the tensor-core kernel
constexpr int kMaxSplit = 32;

// A launch that may start before the kernel in front of it has ended; the kernel waits before it reads what that one wrote.
template <typename... A, typename... B> static cudaError_t launch_early(void (*kernel)(A...), dim3 grid, int threads, size_t smem, cudaStream_t st, B... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, args...);
}

// ------------------------------------------------------------------------------------------ norms, rotation, append
struct PrepParams {
  int q_rank, rank, rot, row_ld, page, max_pages, max_len, ld, cq_ld;
  float eps;
  const void *q, *kv;                // columns of the projection's rows: the query latent; [latent | key part]
  const float *q_norm, *kv_norm;
  const float2 *rope;                // [positions][rot / 2]
  void *cq, *pool;
  const int *page_table, *cu, *start, *slot, *tok_seq;
  int *error_flag;
};
constexpr int PREP_THREADS = 256;
template <typename T, int VEC> __global__ void __launch_bounds__(PREP_THREADS) prep_kernel(const PrepParams p) {   // block: one token
  __shared__ float red[PREP_THREADS / 32];
  launch_dependents();
  wait_for_prerequisites();
  const int t = blockIdx.x, tid = threadIdx.x, s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  const bool ok = pos >= 0 && pos < p.max_len;
  const int phys = ok ? p.page_table[(size_t)p.slot[s] * p.max_pages + pos / p.page] : 0, half = p.rot / 2;
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.ld, *kv = reinterpret_cast<const T *>(p.kv) + (size_t)t * p.ld;
  // the first half of the block takes the query latent, the second half the cached one
  constexpr int HALF = PREP_THREADS / 2;
  const bool second = tid >= HALF, append = p.kv != nullptr;
  const T *mine = second && append ? kv : q;
  const float *norm = second ? p.kv_norm : p.q_norm;
  const int n = second ? (append ? p.rank : 0) : p.q_rank, lane = tid & 31, warp = tid >> 5, at = tid & (HALF - 1);
  float ss = 0.f;
  for (int i = at * VEC; i < n; i += HALF * VEC) {
    float v[VEC];
    load_vec<VEC>(mine + i, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float sum = 0.f;
  for (int i = 0; i < HALF / 32; ++i) sum += red[(second ? HALF / 32 : 0) + i];
  const float inv = 1.0f / sqrtf(sum / (float)n + p.eps);
  if (second && !append) return;
  if (second && !ok) {
    if (at == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  T *row = reinterpret_cast<T *>(p.pool) + ((size_t)phys * p.page + pos % p.page) * p.row_ld;
  T *out = second ? row + p.rot : reinterpret_cast<T *>(p.cq) + (size_t)t * p.cq_ld;
  for (int i = at * VEC; i < n; i += HALF * VEC) {
    float v[VEC], w[VEC];
    load_vec<VEC>(mine + i, v);
    load_vec<VEC>(norm + i, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= inv * w[j];
    store_vec<VEC>(out + i, v);
  }
  if (!second) {
    for (int i = n + at; i < p.cq_ld; i += HALF) out[i] = from_f<T>(0.f);
    return;
  }
  for (int i = at; i < half; i += HALF) {
    const float u = to_f(kv[p.rank + i]), v = to_f(kv[p.rank + half + i]);
    const float2 c = __ldg(p.rope + (size_t)pos * half + i);
    row[i] = from_f<T>(u * c.x - v * c.y);
    row[half + i] = from_f<T>(v * c.x + u * c.y);
  }
  for (int i = p.rot + p.rank + at; i < p.row_ld - 8; i += HALF) row[i] = from_f<T>(0.f);      // (products go in steps of 16)
}

// ------------------------------------------------------------------------------------------ the whole context
// One warp per context row, 16-byte units.
__global__ void context_kernel(const uint4 *pool, const int *page_table, const int *slot, const int *ctx_cu, int n_seq, int n_ctx, int page, int max_pages,
                               int rot_units, int units, int row_units, uint4 *shared, uint4 *latent, int latent_units) {
  const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= n_ctx) return;
  int lo = 0, hi = n_seq - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (ctx_cu[mid] <= r) lo = mid;
    else hi = mid - 1;
  }
  const int pos = r - ctx_cu[lo];
  const uint4 *src = pool + ((size_t)page_table[(size_t)slot[lo] * max_pages + pos / page] * page + pos % page) * row_units;
  for (int i = lane; i < rot_units + latent_units; i += 32) {
    const uint4 v = i < units ? src[i] : make_uint4(0, 0, 0, 0);
    if (i < rot_units) shared[(size_t)r * rot_units + i] = v;
    else latent[(size_t)r * latent_units + i - rot_units] = v;
  }
}

// ------------------------------------------------------------------------------------------ attention
struct Params {
  int n_tok, n_head, dim, rot, vdim, rank, width, row_ld, q_ld, max_pages, max_len, gate_ld, out_ld, out_cols;   // width = rot + rank, row_ld: cached rows, q_cat rows
  int n_split, slots, ng;            // runs of pages; slots of the ring; expand: groups of 16 outputs per block
  float scale;
  const void *q, *w_k, *w_v, *gate, *pool;
  const float2 *rope;
  const int *page_table, *cu, *start, *slot, *tok_seq;
  void *q_cat, *o_lat, *out;
  float *ws_o;                       // [n_tok][n_head][n_split][rank]
  float2 *ws_ml;                     // [n_tok][n_head][n_split]
  int *error_flag;
  bool gate_values;                  // a gate per output instead of one per head
};

template <typename T> __device__ __forceinline__ float sigmoid_at(const Params &p, int t, int c) {
  return 1.0f / (1.0f + expf(-to_f(reinterpret_cast<const T *>(p.gate)[(size_t)t * p.gate_ld + c])));
}
template <typename T> __device__ __forceinline__ float head_gate(const Params &p, int t, int h) { return p.gate && !p.gate_values ? sigmoid_at<T>(p, t, h) : 1.f; }
template <typename T> __device__ __forceinline__ void rotate_query(const Params &p, int t, int h, int pos, int i, T *dst) {   // pair i
  const int half = p.rot / 2;
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.q_ld + (size_t)h * (p.rot + p.dim);
  const float u = to_f(q[i]), v = to_f(q[half + i]);
  const float2 c = __ldg(p.rope + (size_t)pos * half + i);
  dst[i] = from_f<T>(u * c.x - v * c.y);
  dst[half + i] = from_f<T>(v * c.x + u * c.y);
}

constexpr int PLAIN_THREADS = 128;
template <typename T> __global__ void __launch_bounds__(PLAIN_THREADS) absorb_plain_kernel(const Params p) {   // block: one token and head
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s = p.tok_seq[t], pos = p.start[s] + t - p.cu[s];
  if (pos < 0 || pos >= p.max_len) return;         // (reported where the position is cached)
  T *dst = reinterpret_cast<T *>(p.q_cat) + ((size_t)t * p.n_head + h) * p.row_ld;
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.q_ld + (size_t)h * (p.rot + p.dim) + p.rot;
  const T *w = reinterpret_cast<const T *>(p.w_k) + (size_t)h * p.rank * p.dim;
  for (int i = tid; i < p.rot / 2; i += PLAIN_THREADS) rotate_query<T>(p, t, h, pos, i, dst);
  for (int n = warp; n < p.rank; n += PLAIN_THREADS / 32) {
    float a = 0.f;
    for (int d = lane; d < p.dim; d += 32) a = fmaf(to_f(q[d]), to_f(w[(size_t)n * p.dim + d]), a);
    a = warp_sum(a);
    if (lane == 0) dst[p.rot + n] = from_f<T>(a);
  }
}
template <typename T> __global__ void __launch_bounds__(PLAIN_THREADS) expand_plain_kernel(const Params p) {
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const T *o = reinterpret_cast<const T *>(p.o_lat) + ((size_t)t * p.n_head + h) * p.rank, *w = reinterpret_cast<const T *>(p.w_v) + (size_t)h * p.vdim * p.rank;
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld;
  const float gate = head_gate<T>(p, t, h);
  for (int n = warp; n < p.vdim; n += PLAIN_THREADS / 32) {
    float a = 0.f;
    for (int r = lane; r < p.rank; r += 32) a = fmaf(to_f(o[r]), to_f(w[(size_t)n * p.rank + r]), a);
    a = warp_sum(a);
    if (lane == 0) out[h * p.vdim + n] = from_f<T>(a * (p.gate_values ? sigmoid_at<T>(p, t, h * p.vdim + n) : gate));
  }
  if (h == p.n_head - 1)
    for (int i = p.n_head * p.vdim + tid; i < p.out_cols; i += PLAIN_THREADS) out[i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------ products per head on tensor cores
// y [16 tokens x 16 outputs per warp] += x W^T, 128 k a time, straight from rows with k contiguous: a lane takes eight neighbouring k
// of rows g (and g + 8) as its share of every 32, the same for both operands.
typedef __nv_bfloat16 bf;
struct Frag128 { uint4 v[2][4]; };       // rows g and g + 8
__device__ __forceinline__ void load128(Frag128 &f, const bf *row0, const bf *row1, int k0, int k_end, int tig, bool ok0, bool ok1, bool stream) {
#pragma unroll
  for (int pp = 0; pp < 4; ++pp) {
    const int c = k0 + pp * 32 + tig * 8;
    const uint4 z = make_uint4(0, 0, 0, 0);
    f.v[0][pp] = ok0 && c < k_end ? (stream ? __ldg(reinterpret_cast<const uint4 *>(row0 + c)) : *reinterpret_cast<const uint4 *>(row0 + c)) : z;
    f.v[1][pp] = ok1 && c < k_end ? (stream ? __ldg(reinterpret_cast<const uint4 *>(row1 + c)) : *reinterpret_cast<const uint4 *>(row1 + c)) : z;
  }
}
__device__ __forceinline__ void mma128(float (&acc)[2][4], const Frag128 &x, const Frag128 &w) {
#pragma unroll
  for (int pp = 0; pp < 4; ++pp)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      mma16816_bf16(acc[j], x.v[0][pp].x, x.v[1][pp].x, x.v[0][pp].y, x.v[1][pp].y, w.v[j][pp].x, w.v[j][pp].y);
      mma16816_bf16(acc[j], x.v[0][pp].z, x.v[1][pp].z, x.v[0][pp].w, x.v[1][pp].w, w.v[j][pp].z, w.v[j][pp].w);
    }
}

constexpr int ABSORB_WARPS = 4;
__global__ void __launch_bounds__(ABSORB_WARPS * 32) absorb_kernel(const Params p) {   // grid: (64 outputs, head, 16 tokens)
  launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3, h = blockIdx.y, t0 = blockIdx.z * 16;
  const int n0 = (blockIdx.x * ABSORB_WARPS + warp) * 16;
  const bf *w = reinterpret_cast<const bf *>(p.w_k) + (size_t)h * p.rank * p.dim;
  const bf *w0 = w + (size_t)(n0 + g) * p.dim, *w1 = w + (size_t)(n0 + 8 + g) * p.dim;
  Frag128 wf, xf;
  load128(wf, w0, w1, 0, p.dim, tig, n0 + g < p.rank, n0 + 8 + g < p.rank, true);
  wait_for_prerequisites();
  if (blockIdx.x == 0) {
    const int pad = p.row_ld - 8 - p.width;          // (products go in steps of 16)
    for (int i = tid; i < 16 * pad; i += blockDim.x)
      if (t0 + i / pad < p.n_tok) reinterpret_cast<bf *>(p.q_cat)[((size_t)(t0 + i / pad) * p.n_head + h) * p.row_ld + p.width + i % pad] = from_f<bf>(0.f);
    for (int i = tid; i < 16 * (p.rot / 2); i += blockDim.x) {
      const int m = i / (p.rot / 2), t = t0 + m;
      if (t >= p.n_tok) break;
      const int pos = p.start[t];
      if (pos >= 0 && pos < p.max_len) rotate_query<bf>(p, t, h, pos, i % (p.rot / 2), reinterpret_cast<bf *>(p.q_cat) + ((size_t)t * p.n_head + h) * p.row_ld);
    }
  }
  const bool ok0 = t0 + g < p.n_tok, ok1 = t0 + g + 8 < p.n_tok;
  const bf *x0 = reinterpret_cast<const bf *>(p.q) + (size_t)(t0 + g) * p.q_ld + (size_t)h * (p.rot + p.dim) + p.rot, *x1 = x0 + (size_t)8 * p.q_ld;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < p.dim; k0 += 128) {
    if (k0) load128(wf, w0, w1, k0, p.dim, tig, n0 + g < p.rank, n0 + 8 + g < p.rank, true);
    load128(xf, x0, x1, k0, p.dim, tig, ok0, ok1, false);
    mma128(acc, xf, wf);
  }
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int n = n0 + 8 * j + 2 * tig;
    if (n >= p.rank) continue;               // (rank is a multiple of 8)
    bf *o = reinterpret_cast<bf *>(p.q_cat) + ((size_t)(t0 + g) * p.n_head + h) * p.row_ld + p.rot + n;
    if (ok0) *reinterpret_cast<uint32_t *>(o) = pack_bf2(acc[j][0], acc[j][1]);
    if (ok1) *reinterpret_cast<uint32_t *>(o + (size_t)8 * p.n_head * p.row_ld) = pack_bf2(acc[j][2], acc[j][3]);
  }
}

__device__ __forceinline__ int pages_per_run(int n_pages, int n_split) { return (n_pages + n_split - 1) / n_split; }

// The runs of one token and head become one latent vector (with the gate): a thread takes four neighbouring dimensions, a warp-wide
// softmax over the runs' maxima gives their weights.
constexpr int COMBINE_THREADS = 128;
__global__ void __launch_bounds__(COMBINE_THREADS) combine_kernel(const Params p) {   // grid: (head, token)
  __shared__ float cw[kMaxSplit];
  launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.x, t = blockIdx.y;
  wait_for_prerequisites();
  const int pos = p.start[t];
  const bool ok = pos >= 0 && pos < p.max_len;
  const int n_pages = pos / TILE + 1, per = pages_per_run(n_pages, p.n_split), n_act = ok ? (n_pages + per - 1) / per : 0;
  const size_t head = (size_t)t * p.n_head + h;
  constexpr int PB = 8;
  const float *src = p.ws_o + head * p.n_split * p.rank;
  if (tid < 32) {
    const float2 ml = lane < n_act ? __ldcg(p.ws_ml + head * p.n_split + lane) : make_float2(-INFINITY, 0.f);
    const float top = warp_max(ml.x), e = lane < n_act ? exp2f(ml.x - top) : 0.f, l = warp_sum(ml.y * e);
    cw[lane] = lane < n_act ? e / l * head_gate<bf>(p, t, h) : 0.f;
  }
  float4 v[PB];                                    // (the first runs' loads do not wait for the weights)
  const int c = tid * 4;
#pragma unroll
  for (int j = 0; j < PB; ++j)
    if (j < n_act && c < p.rank) v[j] = __ldcg(reinterpret_cast<const float4 *>(src + (size_t)j * p.rank + c));
  __syncthreads();
  if (c >= p.rank) return;                         // (rank is at most 512)
  float a[4] = {0.f, 0.f, 0.f, 0.f};
  for (int i0 = 0; i0 < n_act; i0 += PB) {
#pragma unroll
    for (int j = 0; j < PB; ++j)
      if (i0 + j < n_act) {
        const float x = cw[i0 + j];
        a[0] = fmaf(v[j].x, x, a[0]);
        a[1] = fmaf(v[j].y, x, a[1]);
        a[2] = fmaf(v[j].z, x, a[2]);
        a[3] = fmaf(v[j].w, x, a[3]);
      }
#pragma unroll
    for (int j = 0; j < PB; ++j)
      if (i0 + PB + j < n_act) v[j] = __ldcg(reinterpret_cast<const float4 *>(src + (size_t)(i0 + PB + j) * p.rank + c));
  }
  *reinterpret_cast<uint2 *>(reinterpret_cast<bf *>(p.o_lat) + head * p.rank + c) = make_uint2(pack_bf2(a[0], a[1]), pack_bf2(a[2], a[3]));
}

constexpr int EXPAND_WARPS = 8;
// Grid: (16 ng outputs, head, 16 tokens).  Warp (n group, k group): 8 / ng warps share an output group's k.
__global__ void __launch_bounds__(EXPAND_WARPS * 32) expand_kernel(const Params p) {
  __shared__ float red[EXPAND_WARPS * 32 * 8];
  launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3, h = blockIdx.y, t0 = blockIdx.z * 16;
  const int ks = EXPAND_WARPS / p.ng, wn = warp % p.ng, wk = warp / p.ng, n0 = (blockIdx.x * p.ng + wn) * 16;
  const int k_per = ((p.rank + ks - 1) / ks + 31) / 32 * 32, kb = wk * k_per, ke = min(p.rank, kb + k_per);
  const bf *w = reinterpret_cast<const bf *>(p.w_v) + (size_t)h * p.vdim * p.rank;
  const bf *w0 = w + (size_t)(n0 + g) * p.rank, *w1 = w + (size_t)(n0 + 8 + g) * p.rank;
  const bool n_ok0 = n0 + g < p.vdim, n_ok1 = n0 + 8 + g < p.vdim, ok0 = t0 + g < p.n_tok, ok1 = t0 + g + 8 < p.n_tok;
  Frag128 wf, xf;
  load128(wf, w0, w1, kb, ke, tig, n_ok0, n_ok1, true);
  wait_for_prerequisites();
  const bf *x0 = reinterpret_cast<const bf *>(p.o_lat) + ((size_t)(t0 + g) * p.n_head + h) * p.rank, *x1 = x0 + (size_t)8 * p.n_head * p.rank;
  float acc[2][4] = {};
  for (int k0 = kb; k0 < ke; k0 += 128) {
    if (k0 > kb) load128(wf, w0, w1, k0, ke, tig, n_ok0, n_ok1, true);
    load128(xf, x0, x1, k0, ke, tig, ok0, ok1, false);
    mma128(acc, xf, wf);
  }
  if (ks > 1) {
    float4 *mine = reinterpret_cast<float4 *>(red + (warp * 32 + lane) * 8);
    mine[0] = make_float4(acc[0][0], acc[0][1], acc[0][2], acc[0][3]);
    mine[1] = make_float4(acc[1][0], acc[1][1], acc[1][2], acc[1][3]);
    __syncthreads();
    if (wk) return;
    for (int k = 1; k < ks; ++k) {
      const float *other = red + ((k * p.ng + wn) * 32 + lane) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j >> 2][j & 3] += other[j];
    }
  }
  bf *out = reinterpret_cast<bf *>(p.out) + (size_t)(t0 + g) * p.out_ld;
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int n = n0 + 8 * j + 2 * tig;
    if (n >= p.vdim) continue;               // (vdim is a multiple of 8)
    if (p.gate_values) {
      const int c = h * p.vdim + n;
      if (ok0) { acc[j][0] *= sigmoid_at<bf>(p, t0 + g, c); acc[j][1] *= sigmoid_at<bf>(p, t0 + g, c + 1); }
      if (ok1) { acc[j][2] *= sigmoid_at<bf>(p, t0 + g + 8, c); acc[j][3] *= sigmoid_at<bf>(p, t0 + g + 8, c + 1); }
    }
    if (ok0) *reinterpret_cast<uint32_t *>(out + h * p.vdim + n) = pack_bf2(acc[j][0], acc[j][1]);
    if (ok1) *reinterpret_cast<uint32_t *>(out + (size_t)8 * p.out_ld + h * p.vdim + n) = pack_bf2(acc[j][2], acc[j][3]);
  }
  if (h == p.n_head - 1 && blockIdx.x == 0 && wn == 0) {    // k padding of the output product (this warp did not leave above)
    const int pad0 = p.n_head * p.vdim, pad = p.out_cols - pad0;
    for (int i = lane; i < 16 * pad; i += 32)
      if (t0 + i / pad < p.n_tok) reinterpret_cast<bf *>(p.out)[(size_t)(t0 + i / pad) * p.out_ld + pad0 + i % pad] = from_f<bf>(0.f);
  }
}

// ------------------------------------------------------------------------------------------ one token per sequence
// Block: one run of pages of one sequence, 16 MT heads.  The rows [rotated part | latent] of a page lie once in shared memory and serve
// as keys and, from column rot on, as values; one bulk copy brings half a page into a slot of a ring (a block computes on two slots while
// the others fill).  Rows are an odd number of 16-byte units long, so that eight of them meet in no bank.  Scores: warp (a quarter of the
// row's dimensions, 8 KT keys), its part of the queries stays in registers (S steps of 32 dimensions); the quarters' sums meet in shared
// memory.  Weighted sum: warp w takes latent dimensions 8 NT w ...
constexpr int PARTS = 4, P_LD = TILE + 8, HALF = TILE / 2, kMaxSlots = 8;
template <int MT> static size_t decode_smem(int row_ld, int slots) {
  return (size_t)slots * HALF * row_ld * sizeof(bf) + (size_t)16 * MT * (P_LD * (PARTS * sizeof(float) + 2 * sizeof(bf)) + sizeof(float));
}
constexpr size_t kSmemLimit = 226 * 1024;
constexpr int kMinSlots = 4;
template <int MT, int NT, int S, int WARPS> __global__ void __launch_bounds__(WARPS * 32, 1) decode_kernel(const Params p) {
  constexpr int HB = 16 * MT, KT = TILE / 8 / (WARPS / PARTS), THREADS = WARPS * 32;   // KT: groups of eight keys per warp
  extern __shared__ __align__(16) unsigned char sm_raw[];
  const int ld = p.row_ld, k_end = ld - 8;        // k_end: the row's dimensions, a multiple of 16
  bf *ks = reinterpret_cast<bf *>(sm_raw);                                  // [slots][HALF][ld]
  float *ps = reinterpret_cast<float *>(ks + p.slots * HALF * ld);          // [PARTS][HB][P_LD]
  bf *ph = reinterpret_cast<bf *>(ps + PARTS * HB * P_LD), *pl = ph + HB * P_LD;   // [HB][P_LD] the weights' two parts
  float *corr = reinterpret_cast<float *>(pl + HB * P_LD);                  // [HB]
  __shared__ uint64_t full[kMaxSlots], q_full;
  __shared__ volatile int abort_flag;
  launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int t = blockIdx.z, h0 = blockIdx.y * HB, nh = min(HB, p.n_head - h0), x = blockIdx.x;
  wait_for_prerequisites();
  const int pos = p.start[t];
  if (pos < 0 || pos >= p.max_len) {
    if (tid == 0 && p.error_flag) atomicExch(p.error_flag, 12);
    return;
  }
  const int n_pages = pos / TILE + 1, per = pages_per_run(n_pages, p.n_split), pg0 = x * per, pg1 = min(n_pages, pg0 + per);
  if (pg0 >= pg1) return;
  const int *table = p.page_table + (size_t)p.slot[t] * p.max_pages;
  const int first = pg0 * TILE, halves = (min(pg1 * TILE, pos + 1) - first + HALF - 1) / HALF;
  int issued = 0, fill_slot = 0, phys = table[pg0];
  auto load_half = [&]() {                        // the next half page of the run into the next slot
    const int rows = min(HALF, pos + 1 - first - issued * HALF);      // rows behind the newest position: zeros (their weights are zero, but what is multiplied must be a number)
    bf *dst = ks + fill_slot * HALF * ld;
    if (tid == 0) {
      const uint32_t bar = smem_addr(&full[fill_slot]), bytes = (uint32_t)(rows * ld * sizeof(bf));
      mbar_expect_tx(bar, bytes);
      bulk_g2s(smem_addr(dst), reinterpret_cast<const bf *>(p.pool) + ((size_t)phys * TILE + (issued & 1) * HALF) * ld, bytes, bar);
      if (issued & 1) phys = table[min(pg0 + (issued + 1) / 2, pg1 - 1)];
    }
    for (int r = rows + warp; r < HALF; r += WARPS)
      for (int i = lane; i < ld / 2; i += 32) reinterpret_cast<uint32_t *>(dst + r * ld)[i] = 0u;
    ++issued;
    if (++fill_slot == p.slots) fill_slot = 0;
  };
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < kMaxSlots; ++i) mbar_init(smem_addr(&full[i]), 1);
    mbar_init(smem_addr(&q_full), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    // the queries pass through the last slot
    const uint32_t bytes = (uint32_t)(nh * ld * sizeof(bf));
    mbar_expect_tx(smem_addr(&q_full), bytes);
    bulk_g2s(smem_addr(ks + (p.slots - 1) * HALF * ld), reinterpret_cast<const bf *>(p.q_cat) + ((size_t)t * p.n_head + h0) * ld, bytes, smem_addr(&q_full));
  }
  __syncthreads();
  while (issued < min(halves, p.slots - 1)) load_half();
  const int part = warp & (PARTS - 1), keys = warp / PARTS * (KT * 8), k0 = part * S * 32;   // this warp's scores: dimensions k0 .., keys keys ..
  auto failed = [&]() {
    if (!abort_flag && p.error_flag) atomicCAS(p.error_flag, 0, 11);
    abort_flag = 1;
  };
  if (!mbar_wait(smem_addr(&q_full), 0, &abort_flag)) failed();
  uint32_t qa[MT][2 * S][4];
  {
    const uint32_t q_lane = smem_addr(ks + ((p.slots - 1) * HALF + (lane & 15)) * ld + k0 + (lane >> 4) * 8);
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int kk = 0; kk < 2 * S; ++kk) {
        qa[mt][kk][0] = qa[mt][kk][1] = qa[mt][kk][2] = qa[mt][kk][3] = 0u;
        if (k0 + kk * 16 < k_end) ldsm4(q_lane + (uint32_t)(mt * 16 * ld + kk * 16) * 2u, qa[mt][kk][0], qa[mt][kk][1], qa[mt][kk][2], qa[mt][kk][3]);
      }
  }
  __syncthreads();
  if (issued < halves) load_half();
  const float sc2 = p.scale * kLog2e;
  constexpr int ROWS = HB / WARPS;
  float m_run[ROWS], l_run[ROWS];                 // heads ROWS warp .. (the same in all lanes)
#pragma unroll
  for (int i = 0; i < ROWS; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  float o[MT][NT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int j = 0; j < NT; ++j) o[mt][j][0] = o[mt][j][1] = o[mt][j][2] = o[mt][j][3] = 0.f;
  const int c0 = warp * NT * 8;                   // this warp's latent dimensions
  int slot0 = 0, turn0 = 0;                       // of the tile's first half: its slot, and how often the ring was used up before
  for (int h = 0; h < halves; h += 2) {
    const int slot1 = slot0 + 1 == p.slots ? 0 : slot0 + 1, turn1 = turn0 + (slot1 == 0);
    const bool two = h + 1 < halves;
    if (!mbar_wait(smem_addr(&full[slot0]), turn0 & 1, &abort_flag) || (two && !mbar_wait(smem_addr(&full[slot1]), turn1 & 1, &abort_flag))) failed();
    const bf *K0 = ks + slot0 * HALF * ld, *K1 = ks + slot1 * HALF * ld;
    if (two || keys < HALF) {
      float sc[MT][KT][4] = {};
      const uint32_t k_lane = smem_addr((keys < HALF ? K0 : K1) + ((keys & (HALF - 1)) + (lane & 7)) * ld + k0 + (lane >> 3) * 8);     // matrices: k 0-7, 8-15, 16-23, 24-31 of eight keys
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (k0 + s * 32 >= k_end) break;          // (uniform over the warp)
        const bool both = k0 + s * 32 + 16 < k_end;
#pragma unroll
        for (int j = 0; j < KT; ++j) {
          uint32_t b0, b1, b2, b3;
          ldsm4(k_lane + (uint32_t)(j * 8 * ld + s * 32) * 2u, b0, b1, b2, b3);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            const uint32_t(&a)[4] = qa[mt][2 * s], (&b)[4] = qa[mt][2 * s + 1];
            mma16816_bf16(sc[mt][j], a[0], a[1], a[2], a[3], b0, b1);
            if (both) mma16816_bf16(sc[mt][j], b[0], b[1], b[2], b[3], b2, b3);
          }
        }
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < KT; ++j)
#pragma unroll
          for (int r = 0; r < 2; ++r)
            *reinterpret_cast<float2 *>(ps + (part * HB + mt * 16 + g + 8 * r) * P_LD + keys + j * 8 + 2 * tig) = make_float2(sc[mt][j][2 * r], sc[mt][j][2 * r + 1]);
    }
    __syncthreads();
    if (abort_flag) {                             // (the same for the whole block) what is still in flight lands before the block ends
      mbar_wait_all(smem_addr(&q_full), 0);
      for (int i = h; i < issued; ++i) mbar_wait_all(smem_addr(&full[i % p.slots]), (i / p.slots) & 1);
      return;
    }
    const int seen = pos - first - h * HALF;      // keys 0 .. seen of this tile
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = warp * ROWS + i;
      float2 v = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < PARTS; ++j) {
        const float2 part_sum = *reinterpret_cast<const float2 *>(ps + (j * HB + r) * P_LD + 2 * lane);
        v.x += part_sum.x;
        v.y += part_sum.y;
      }
      v.x = 2 * lane <= seen ? v.x * sc2 : -INFINITY;
      v.y = 2 * lane + 1 <= seen ? v.y * sc2 : -INFINITY;
      const float m = fmaxf(m_run[i], warp_max(fmaxf(v.x, v.y)));           // (a page of a run holds at least one visible key)
      const float a = exp2f(v.x - m), b = exp2f(v.y - m), c = exp2f(m_run[i] - m);
      uint32_t hi, lo;
      split_bf2(a, b, hi, lo);
      *reinterpret_cast<uint32_t *>(ph + r * P_LD + 2 * lane) = hi;
      *reinterpret_cast<uint32_t *>(pl + r * P_LD + 2 * lane) = lo;
      if (lane == 0) corr[r] = c;
      l_run[i] = l_run[i] * c + warp_sum(a + b);
      m_run[i] = m;
    }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float c_lo = corr[mt * 16 + g], c_hi = corr[mt * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        o[mt][j][0] *= c_lo; o[mt][j][1] *= c_lo;
        o[mt][j][2] *= c_hi; o[mt][j][3] *= c_hi;
      }
    }
    const uint32_t v_off = (uint32_t)((lane & 15) * ld + p.rot + c0 + (lane >> 4) * 8) * 2u, v_lane0 = smem_addr(K0) + v_off, v_lane1 = smem_addr(K1) + v_off;
    const uint32_t h_lane = smem_addr(ph + (lane & 15) * P_LD + (lane >> 4) * 8), l_lane = smem_addr(pl + (lane & 15) * P_LD + (lane >> 4) * 8);
#pragma unroll
    for (int k2 = 0; k2 < TILE / 16; ++k2) {
      if (k2 * 16 >= HALF && !two) break;         // (uniform)
      uint32_t h[MT][4], l[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        ldsm4(h_lane + (uint32_t)(mt * 16 * P_LD + k2 * 16) * 2u, h[mt][0], h[mt][1], h[mt][2], h[mt][3]);
        ldsm4(l_lane + (uint32_t)(mt * 16 * P_LD + k2 * 16) * 2u, l[mt][0], l[mt][1], l[mt][2], l[mt][3]);
      }
#pragma unroll
      for (int jn = 0; jn < NT; jn += 2) {
        if (c0 + jn * 8 >= p.rank) break;         // (uniform over the warp)
        uint32_t b0, b1, b2, b3;
        ldsm4t((k2 * 16 < HALF ? v_lane0 : v_lane1) + (uint32_t)((k2 * 16 & (HALF - 1)) * ld + jn * 8) * 2u, b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma16816_bf16(o[mt][jn], h[mt][0], h[mt][1], h[mt][2], h[mt][3], b0, b1);
          mma16816_bf16(o[mt][jn + 1], h[mt][0], h[mt][1], h[mt][2], h[mt][3], b2, b3);
          mma16816_bf16(o[mt][jn], l[mt][0], l[mt][1], l[mt][2], l[mt][3], b0, b1);
          mma16816_bf16(o[mt][jn + 1], l[mt][0], l[mt][1], l[mt][2], l[mt][3], b2, b3);
        }
      }
    }
    __syncthreads();                              // both slots may be refilled
    if (issued < halves) load_half();
    if (issued < halves) load_half();
    turn0 = turn1 + (slot1 + 1 == p.slots);
    slot0 = slot1 + 1 == p.slots ? 0 : slot1 + 1;
  }
  const size_t head0 = (size_t)t * p.n_head + h0;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = mt * 16 + g + 8 * r;
      if (row >= nh) continue;
      float *dst = p.ws_o + ((head0 + row) * p.n_split + x) * p.rank + c0 + 2 * tig;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        if (c0 + j * 8 < p.rank) *reinterpret_cast<float2 *>(dst + j * 8) = make_float2(o[mt][j][2 * r], o[mt][j][2 * r + 1]);
    }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int row = warp * ROWS + i;
    if (lane == 0 && row < nh) p.ws_ml[(head0 + row) * p.n_split + x] = make_float2(m_run[i], l_run[i]);
  }
}

template <int MT, int NT, int S, int WARPS> static int launch_decode(Params p, cudaStream_t st) {
  p.slots = kMaxSlots;
  while (p.slots > kMinSlots && decode_smem<MT>(p.row_ld, p.slots) > kSmemLimit) --p.slots;
  const size_t smem = decode_smem<MT>(p.row_ld, p.slots);
  static bool set = false;
  if (!set) { PT_CUDA(cudaFuncSetAttribute(decode_kernel<MT, NT, S, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit)); set = true; }
  PT_CUDA(launch_early(decode_kernel<MT, NT, S, WARPS>, dim3(p.n_split, ceil_div(p.n_head, 16 * MT), p.n_tok), WARPS * 32, smem, st, p));
  count_launch();
  return PT_OK;
}
template <int MT, int NT, int WARPS> static int dispatch_width(const Params &p, cudaStream_t st) {
  return p.row_ld - 8 <= PARTS * 32 * 2 ? launch_decode<MT, NT, 2, WARPS>(p, st) : launch_decode<MT, NT, 5, WARPS>(p, st);
}
static int dispatch_decode(const Params &p, bool two_tiles, cudaStream_t st) {
  if (!two_tiles) return p.rank <= 256 ? dispatch_width<1, 2, 16>(p, st) : launch_decode<1, 4, 5, 16>(p, st);
  if (p.rank <= 128) return dispatch_width<2, 2, 8>(p, st);
  return p.rank <= 256 ? dispatch_width<2, 4, 8>(p, st) : launch_decode<2, 8, 5, 8>(p, st);
}

static bool two_tiles(int n_head, int row_ld) { return n_head > 16 && decode_smem<2>(row_ld, kMinSlots) <= kSmemLimit; }
static int splits(int n_tok, int n_head, int row_ld, int max_len) {
  const int blocks = n_tok * ceil_div(n_head, two_tiles(n_head, row_ld) ? 32 : 16);
  return std::max(1, std::min({sm_count() / blocks, kMaxSplit, ceil_div(max_len, TILE)}));
}
static bool decode_takes(int dtype, int page, int dim, int rot, int vdim, int rank) {
  return dtype == PT_DT_BF16 && page == TILE && dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && rank % 8 == 0 && rank <= 512 && pt_latent_row(rot, rank) - 8 <= PARTS * 32 * 5 && decode_smem<1>(pt_latent_row(rot, rank), kMinSlots) <= kSmemLimit;
}
static size_t align256(size_t v) { return (v + 255) / 256 * 256; }

}  // namespace lat
}  // namespace pt

using namespace pt;

extern "C" int pt_latent_row(int rot_dim, int rank) { return (rot_dim + rank + 15) / 16 * 16 + 8; }

extern "C" int pt_latent_prep(const pt_latent_prep_args *a, void *stream) {
  PT_REQUIRE(a, "pt_latent_prep: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.n_tok >= b.n_seq && b.cu && b.start && b.slot && b.tok_seq, "pt_latent_prep: bad batch (%d sequences, %d tokens)", b.n_seq, b.n_tok);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_latent_prep: type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->q_rank > 0 && a->rank > 0 && a->rot_dim >= 0 && a->rot_dim % 2 == 0 && a->page_size > 0 && a->max_pages > 0, "pt_latent_prep: bad shape q_rank=%d rank=%d rot_dim=%d",
             a->q_rank, a->rank, a->rot_dim);
  PT_REQUIRE(a->q && a->q_norm && a->cq && a->page_table && (!a->kv || (a->kv_norm && a->pool && (!a->rot_dim || a->rope))), "pt_latent_prep: null pointer argument");
  PT_REQUIRE(a->ld >= std::max(a->q_rank, a->kv ? a->rank + a->rot_dim : 0) && a->cq_ld >= a->q_rank, "pt_latent_prep: row strides %d, %d", a->ld, a->cq_ld);
  lat::PrepParams p{};
  p.q_rank = a->q_rank; p.rank = a->rank; p.rot = a->rot_dim; p.row_ld = pt_latent_row(a->rot_dim, a->rank); p.page = a->page_size; p.max_pages = a->max_pages; p.ld = a->ld; p.cq_ld = a->cq_ld; p.eps = a->eps;
  p.max_len = a->max_len > 0 ? a->max_len : a->page_size * a->max_pages;
  PT_REQUIRE(p.max_len <= a->page_size * a->max_pages, "pt_latent_prep: max_len=%d exceeds the page table", p.max_len);
  p.q = a->q; p.kv = a->kv; p.q_norm = a->q_norm; p.kv_norm = a->kv_norm; p.rope = (const float2 *)a->rope; p.cq = a->cq; p.pool = a->pool;
  p.page_table = a->page_table; p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq; p.error_flag = a->error_flag;
  const int es = a->dtype == PT_DT_F32 ? 4 : 2;
  auto al = [&](const void *x) { return aligned_to(x, 4 * es); };
  const bool v4 = a->q_rank % 4 == 0 && a->rank % 4 == 0 && a->rot_dim % 4 == 0 && a->ld % 4 == 0 && a->cq_ld % 4 == 0 && al(a->q) && al(a->kv) && al(a->cq) && al(a->pool) &&
                  aligned_to(a->q_norm, 16) && aligned_to(a->kv_norm, 16);
  auto kernel = a->dtype == PT_DT_F32 ? (v4 ? lat::prep_kernel<float, 4> : lat::prep_kernel<float, 1>) : (v4 ? lat::prep_kernel<__nv_bfloat16, 4> : lat::prep_kernel<__nv_bfloat16, 1>);
  PT_CUDA(lat::launch_early(kernel, dim3(b.n_tok), lat::PREP_THREADS, 0, as_stream(stream), p));
  count_launch();
  return PT_OK;
}

extern "C" int pt_latent_context(const pt_latent_context_args *a, void *stream) {
  PT_REQUIRE(a, "pt_latent_context: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.slot && a->ctx_cu && a->n_ctx > 0, "pt_latent_context: bad batch (%d sequences, %d rows)", b.n_seq, a->n_ctx);
  PT_REQUIRE(a->rot_dim > 0 && a->rot_dim % 8 == 0 && a->rank > 0 && a->rank % 8 == 0 && a->latent_ld >= a->rank && a->latent_ld % 8 == 0 && a->page_size > 0 && a->max_pages > 0,
             "pt_latent_context: rows of %d + %d bf16 in units of 8, latent_ld=%d", a->rot_dim, a->rank, a->latent_ld);
  PT_REQUIRE(a->pool && a->page_table && a->shared && a->latent && aligned_to(a->pool, 16) && aligned_to(a->shared, 16) && aligned_to(a->latent, 16),
             "pt_latent_context: null or unaligned pointer");
  lat::context_kernel<<<ceil_div(a->n_ctx, 8), 256, 0, as_stream(stream)>>>((const uint4 *)a->pool, a->page_table, b.slot, a->ctx_cu, b.n_seq, a->n_ctx, a->page_size, a->max_pages,
                                                                            a->rot_dim / 8, (a->rot_dim + a->rank) / 8, pt_latent_row(a->rot_dim, a->rank) / 8, (uint4 *)a->shared, (uint4 *)a->latent,
                                                                            a->latent_ld / 8);
  PT_LAUNCH_CHECK("pt_latent_context");
  return PT_OK;
}

extern "C" size_t pt_latent_attn_workspace_bytes(int n_tok, int n_head, int rot_dim, int rank, int dtype) {
  const size_t heads = (size_t)n_tok * n_head, es = dtype == PT_DT_F32 ? 4 : 2;
  const size_t plain = heads * rank * es, runs = ((size_t)n_tok + sm_count()) * n_head * (rank + 2) * sizeof(float) + 1024;   // (tokens x runs stay below tokens + SMs)
  return lat::align256(heads * pt_latent_row(rot_dim, rank) * es) + plain + (dtype == PT_DT_BF16 ? runs : 0);
}

extern "C" int pt_latent_attn(const pt_latent_attn_args *a, void *stream) {
  PT_REQUIRE(a, "pt_latent_attn: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.n_tok >= b.n_seq && b.cu && b.start && b.slot && b.tok_seq, "pt_latent_attn: bad batch (%d sequences, %d tokens)", b.n_seq, b.n_tok);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_latent_attn: type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->n_head > 0 && a->n_head <= 65535 && a->dim > 0 && a->vdim > 0 && a->rank > 0 && a->rot_dim >= 0 && a->rot_dim % 2 == 0 && a->page_size > 0 && a->max_pages > 0,
             "pt_latent_attn: bad shape heads=%d dim=%d rot_dim=%d vdim=%d rank=%d", a->n_head, a->dim, a->rot_dim, a->vdim, a->rank);
  PT_REQUIRE(a->q && a->w_k && a->w_v && a->pool && a->page_table && a->out && (!a->rot_dim || a->rope), "pt_latent_attn: null pointer argument");
  PT_REQUIRE(a->q_ld >= a->n_head * (a->rot_dim + a->dim) && a->out_ld >= a->n_head * a->vdim && (!a->gate || a->gate_ld >= a->n_head * (a->gate_per_value ? a->vdim : 1)), "pt_latent_attn: row strides q %d, out %d, gate %d",
             a->q_ld, a->out_ld, a->gate_ld);
  const size_t need = pt_latent_attn_workspace_bytes(b.n_tok, a->n_head, a->rot_dim, a->rank, a->dtype);
  PT_REQUIRE(a->workspace && a->workspace_bytes >= need && aligned_to(a->workspace, 16), "pt_latent_attn: %zu workspace bytes needed, got %zu", need, a->workspace_bytes);
  lat::Params p{};
  p.n_tok = b.n_tok; p.n_head = a->n_head; p.dim = a->dim; p.rot = a->rot_dim; p.vdim = a->vdim; p.rank = a->rank; p.width = a->rot_dim + a->rank;
  p.row_ld = pt_latent_row(a->rot_dim, a->rank); p.q_ld = a->q_ld; p.max_pages = a->max_pages; p.gate_ld = a->gate_ld; p.out_ld = a->out_ld;
  p.out_cols = a->out_cols > 0 ? a->out_cols : a->out_ld;
  PT_REQUIRE(p.out_cols >= a->n_head * a->vdim && p.out_cols <= a->out_ld, "pt_latent_attn: out_cols=%d", a->out_cols);
  p.max_len = a->max_len > 0 ? a->max_len : a->page_size * a->max_pages;
  PT_REQUIRE(p.max_len <= a->page_size * a->max_pages, "pt_latent_attn: max_len=%d exceeds the page table", p.max_len);
  p.gate_values = a->gate && a->gate_per_value;
  p.scale = a->scale; p.q = a->q; p.w_k = a->w_k; p.w_v = a->w_v; p.gate = a->gate; p.pool = a->pool; p.rope = (const float2 *)a->rope; p.page_table = a->page_table;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq; p.out = a->out; p.error_flag = a->error_flag;
  const size_t es = a->dtype == PT_DT_F32 ? 4 : 2;
  char *ws = (char *)a->workspace;
  p.q_cat = ws;
  ws += lat::align256((size_t)b.n_tok * a->n_head * p.row_ld * es);
  cudaStream_t st = as_stream(stream);
  const bool tc = !a->plain && b.n_tok == b.n_seq && b.n_seq <= 65535 && lat::decode_takes(a->dtype, a->page_size, a->dim, a->rot_dim, a->vdim, a->rank) && a->q_ld % 8 == 0 &&
                  a->out_ld % 2 == 0 && aligned_to(a->out, 4) && aligned_to(a->q, 16) && aligned_to(a->w_k, 16) && aligned_to(a->w_v, 16) && aligned_to(a->pool, 16);
  if (tc) {
    p.n_split = lat::splits(b.n_tok, a->n_head, p.row_ld, p.max_len);
    p.ws_ml = (float2 *)ws;
    ws += lat::align256((size_t)b.n_tok * a->n_head * p.n_split * sizeof(float2));
    p.ws_o = (float *)ws;
    ws += lat::align256((size_t)b.n_tok * a->n_head * p.n_split * a->rank * sizeof(float));
    p.o_lat = ws;
    const int tokens16 = ceil_div(b.n_tok, 16);
    PT_CUDA(lat::launch_early(lat::absorb_kernel, dim3(ceil_div(a->rank, 16 * lat::ABSORB_WARPS), a->n_head, tokens16), lat::ABSORB_WARPS * 32, 0, st, p));
    count_launch();
    if (int rc = lat::dispatch_decode(p, lat::two_tiles(a->n_head, p.row_ld), st)) return rc;
    PT_CUDA(lat::launch_early(lat::combine_kernel, dim3(a->n_head, b.n_tok), lat::COMBINE_THREADS, 0, st, p));
    count_launch();
    p.ng = 2;
    while (p.ng < lat::EXPAND_WARPS && (long long)ceil_div(a->vdim, 16 * p.ng) * a->n_head * tokens16 > 2 * sm_count()) p.ng *= 2;
    PT_CUDA(lat::launch_early(lat::expand_kernel, dim3(ceil_div(a->vdim, 16 * p.ng), a->n_head, tokens16), lat::EXPAND_WARPS * 32, 0, st, p));
    count_launch();
    return PT_OK;
  }
  const dim3 grid(b.n_tok, a->n_head);
  if (a->dtype == PT_DT_F32) lat::absorb_plain_kernel<float><<<grid, lat::PLAIN_THREADS, 0, st>>>(p);
  else lat::absorb_plain_kernel<__nv_bfloat16><<<grid, lat::PLAIN_THREADS, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_latent_attn");
  p.o_lat = ws;
  pt_window_attn_args w{};
  w.batch = b; w.dtype = a->dtype; w.n_head = a->n_head; w.n_kv = 1; w.dim = p.width; w.vdim = a->rank; w.page_size = a->page_size; w.max_pages = a->max_pages;
  w.scale = a->scale; w.q = p.q_cat; w.q_ld = a->n_head * p.row_ld; w.row_ld = p.row_ld; w.pool = const_cast<void *>(a->pool); w.page_table = a->page_table; w.out = p.o_lat; w.out_ld = a->n_head * a->rank;
  w.max_len = p.max_len; w.plain = 1; w.error_flag = a->error_flag; w.values_in_keys = 1; w.value_col = a->rot_dim;
  if (int rc = pt_window_attn(&w, stream)) return rc;
  if (a->dtype == PT_DT_F32) lat::expand_plain_kernel<float><<<grid, lat::PLAIN_THREADS, 0, st>>>(p);
  else lat::expand_plain_kernel<__nv_bfloat16><<<grid, lat::PLAIN_THREADS, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_latent_attn");
  return PT_OK;
}
