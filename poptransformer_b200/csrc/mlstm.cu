// Matrix memory with exponential gates (the mLSTM cell of xLSTM), per head:
//     i = cap tanh(zi / cap),  f = log sigmoid(cap tanh(zf / cap))                  log input and log forget gate
//     m_t = max(f + m_(t-1), i),  m_0 = 0
//     S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T                     S [N, P], fp32; n [N] likewise with k alone
//     o = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)                              q scaled by N^(-1/2)
//     out = o / rms(o) * norm_w * sigmoid(g) * out_scale                            rms over the P values of the head
// q, k, v and g come from the rows of the input projection; the gates' pre-activations are fp32, and so are the gates, S, n, m and o.
//
// Nothing has to be cleared for a new sequence: at position 0 the old state is ignored.  n and m are kept once per 32 columns of S, so
// that blocks which share a head never wait for one another to read them.
//
//   mlstm_scan_kernel    prompts, any sizes and types: token by token, 32 columns of the state in shared memory
//   mlstm_gate_kernel, mlstm_chunk_* , mlstm_carry_kernel   bf16 prompts: 64 tokens at a time on the tensor cores
//   mlstm_norm_kernel    the last line of the above for prompts
//   mlstm_step_kernel    one token per sequence: everything in one launch, a head's columns over several blocks
#include "chunk.cuh"

namespace pt {
namespace mlstm {

constexpr int COPY_COLS = 32;      // columns of the state that share a copy of n and m

struct Params {
  int n_seq, n_tok, heads, N, P, inner, ld, gate_ld, out_ld, out_cols, copies;
  float cap, eps, q_scale, out_scale;
  const int *cu, *start, *slot, *tok_seq;
  const void *q, *k, *v, *g;
  const float *zi, *zf, *norm_w;
  float *state;                    // [slots][heads][N][P]
  float *nm;                       // [slots][heads][copies][N + 1]: n, then m
  float *y;                        // [n_tok][inner]
  void *out;
  float *chunk_state, *chunk_n, *chunk_m;   // [chunk slots][heads] x ([N][P], [N], 1)
  struct Gates *chunk_gates;
  int *counters;                   // [n_seq][heads] (one token per sequence)
  int tile;                        // columns per block of the step kernel
};

__device__ __forceinline__ float log_input(const Params &p, int t, int h) { return p.cap * tanhf(p.zi[(size_t)t * p.gate_ld + h] / p.cap); }
__device__ __forceinline__ float log_forget(const Params &p, int t, int h) { return -softplus_f(-p.cap * tanhf(p.zf[(size_t)t * p.gate_ld + h] / p.cap)); }
__device__ __forceinline__ float *nm_of(const Params &p, int slot, int h, int copy) {
  return p.nm + (((size_t)slot * p.heads + h) * p.copies + copy) * (p.N + 1);
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// ------------------------------------------------------------------------------------------ any sizes
constexpr int SCAN_WARPS = 8;
// Block: one sequence, one head, 32 columns of the state.  Warp w owns state rows w, w + 8, ...; lane = column.
template <typename T> __global__ void __launch_bounds__(SCAN_WARPS * 32) mlstm_scan_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *S = sm, *n = S + (size_t)p.N * 32, *qs = n + p.N, *ks = qs + p.N, *part = ks + p.N, *red = part + SCAN_WARPS * 32;
  const int s = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * 32, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, col = c0 + lane;
  const bool in = col < p.P, fresh = p.start[s] == 0;
  float *gS = p.state + ((size_t)p.slot[s] * p.heads + h) * p.N * p.P, *gn = nm_of(p, p.slot[s], h, blockIdx.x);
  for (int r = warp; r < p.N; r += SCAN_WARPS) S[r * 32 + lane] = (in && !fresh) ? gS[(size_t)r * p.P + col] : 0.f;
  for (int r = tid; r < p.N; r += blockDim.x) n[r] = fresh ? 0.f : gn[r];
  float m = fresh ? 0.f : gn[p.N];
  for (int t = p.cu[s]; t < p.cu[s + 1]; ++t) {
    const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.ld + (size_t)h * p.N, *k = reinterpret_cast<const T *>(p.k) + (size_t)t * p.ld + (size_t)h * p.N;
    __syncthreads();
    for (int r = tid; r < p.N; r += blockDim.x) {
      qs[r] = to_f(q[r]) * p.q_scale;
      ks[r] = to_f(k[r]);
    }
    const float v = in ? to_f(reinterpret_cast<const T *>(p.v)[(size_t)t * p.ld + (size_t)h * p.P + col]) : 0.f;
    const float li = log_input(p, t, h), fm = log_forget(p, t, h) + m;
    m = fmaxf(fm, li);
    const float keep = expf(fm - m), add = expf(li - m), av = add * v;
    __syncthreads();
    float y = 0.f, d = 0.f;
    for (int r = warp; r < p.N; r += SCAN_WARPS) {
      const float x = fmaf(keep, S[r * 32 + lane], ks[r] * av);
      S[r * 32 + lane] = x;
      y = fmaf(x, qs[r], y);
    }
    for (int r = tid; r < p.N; r += blockDim.x) {
      const float x = fmaf(keep, n[r], add * ks[r]);
      n[r] = x;
      d = fmaf(x, qs[r], d);
    }
    part[warp * 32 + lane] = y;
    d = warp_sum(d);
    if (lane == 0) red[warp] = d;
    __syncthreads();
    if (warp == 0 && in) {
      float num = 0.f, den = 0.f;
#pragma unroll
      for (int w = 0; w < SCAN_WARPS; ++w) { num += part[w * 32 + lane]; den += red[w]; }
      p.y[(size_t)t * p.inner + (size_t)h * p.P + col] = num / (fmaxf(fabsf(den), expf(-m)) + 1e-6f);
    }
  }
  __syncthreads();
  for (int r = warp; r < p.N; r += SCAN_WARPS)
    if (in) gS[(size_t)r * p.P + col] = S[r * 32 + lane];
  for (int r = tid; r < p.N; r += blockDim.x) gn[r] = n[r];
  if (tid == 0) gn[p.N] = m;
}

// ------------------------------------------------------------------------------------------ in chunks of 64 tokens
// With c_t = f_1 + .. + f_t inside a chunk, a_s = i_s - c_s, M_t = max(m before the chunk, a_1 .. a_t) and S, n, m from before it:
//     m_t = c_t + M_t
//     S_t^T q_t = exp(m - M_t) S^T q_t + sum_{s <= t} (k_s . q_t) exp(a_s - M_t) v_s          (n . q likewise with 1 for v)
//     S after the chunk = exp(m - M_last) S + sum_s exp(a_s - M_last) k_s v_s^T
// Four launches, so that all chunks of all sequences work at once and only an elementwise pass runs along the sequence:
//   mlstm_gate_kernel          a, its running maximum and c of every chunk and head
//   mlstm_chunk_state_kernel   the sum of the last line, relative to the chunk's own maximum of a
//   mlstm_carry_kernel         the last line along the chunks: leaves S, n, m BEFORE every chunk
//   mlstm_chunk_out_kernel     the second line
// Operands that are not already bf16 enter the tensor cores as hi + lo pairs.  c, a and the maxima are summed in double and kept as
// pairs of floats: they run into the hundreds while their differences decide.
struct __align__(16) Gates {
  float a_hi[CHUNK], a_lo[CHUNK], mx_hi[CHUNK], mx_lo[CHUNK], c_hi[CHUNK], c_lo[CHUNK], w[CHUNK];   // w = exp(a_s - max a)
  double a_max, c_last;
};
__device__ __forceinline__ void split_d(double x, float &hi, float &lo) {
  hi = (float)x;
  lo = (float)(x - (double)hi);
}
__global__ void mlstm_gate_kernel(const Params p) {   // one warp per (chunk, head)
  const int slot = blockIdx.y, h = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  int s, t0;
  if (h >= p.heads || !chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int row0 = p.cu[s] + t0, valid = min(CHUNK, p.cu[s + 1] - row0);
  double f[2];
  float li[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const bool in = 2 * lane + k < valid;     // beyond the sequence: nothing is forgotten, nothing enters
    f[k] = in ? (double)log_forget(p, row0 + 2 * lane + k, h) : 0.0;
    li[k] = in ? log_input(p, row0 + 2 * lane + k, h) : -1e30f;
  }
  double sum = f[0] + f[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += v;
  }
  const double c[2] = {sum - f[1], sum}, a[2] = {(double)li[0] - c[0], (double)li[1] - c[1]};
  double top = fmax(a[0], a[1]);
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, top, o);
    if (lane >= o) top = fmax(top, v);
  }
  const double before = __shfl_up_sync(0xffffffffu, top, 1), last = __shfl_sync(0xffffffffu, top, 31), c_last = __shfl_sync(0xffffffffu, sum, 31);
  Gates &g = p.chunk_gates[(size_t)slot * p.heads + h];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int r = 2 * lane + k;
    double mx = k ? top : a[0];
    if (k == 0 && lane > 0) mx = fmax(mx, before);
    split_d(a[k], g.a_hi[r], g.a_lo[r]);
    split_d(mx, g.mx_hi[r], g.mx_lo[r]);
    split_d(c[k], g.c_hi[r], g.c_lo[r]);
    g.w[r] = expf((float)(a[k] - last));
  }
  if (lane == 0) {
    g.a_max = last;
    g.c_last = c_last;
    if (t0 == 0) p.chunk_m[(size_t)slot * p.heads + h] = p.start[s] == 0 ? 0.f : nm_of(p, p.slot[s], h, 0)[p.N];
  }
}

template <int NP, int CP> struct StateSmem {
  __nv_bfloat16 K[CHUNK][NP + 8], V[CHUNK][CP + 8], Wh[CHUNK][CP + 8], Wl[CHUNK][CP + 8];
  float w[CHUNK];
};
// Block: one chunk, one head, CP columns.  The warps share the 16-row tiles of the state (and the columns when there are fewer tiles).
template <int NP, int CP> __global__ void __launch_bounds__(CHUNK_THREADS) mlstm_chunk_state_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  constexpr int XLD = CP + 8, MTILES = NP / 16, WPT = MTILES >= 8 ? 1 : 8 / MTILES;      // warps per row tile
  constexpr int MT = MTILES >= 8 ? MTILES / 8 : 1, NJ = CP / 8 / WPT;
  extern __shared__ __align__(16) unsigned char smraw[];
  StateSmem<NP, CP> &sm = *reinterpret_cast<StateSmem<NP, CP> *>(smraw);
  const int slot = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CP;
  int s, t0;
  if (!chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int row0 = p.cu[s] + t0, valid = min(CHUNK, p.cu[s + 1] - row0);
  const T *k = reinterpret_cast<const T *>(p.k) + (size_t)row0 * p.ld + (size_t)h * p.N, *v = reinterpret_cast<const T *>(p.v) + (size_t)row0 * p.ld + (size_t)h * p.P;
  for (int e = tid; e < CHUNK * (NP / 8); e += CHUNK_THREADS) {
    const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
    const bool in = r < valid && c < p.N;
    cp16(&sm.K[r][c], k + (in ? (size_t)r * p.ld + c : 0), in);
  }
  for (int e = tid; e < CHUNK * (CP / 8); e += CHUNK_THREADS) {
    const int r = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = r < valid && col0 + c < p.P;
    cp16(&sm.V[r][c], v + (in ? (size_t)r * p.ld + col0 + c : 0), in);
  }
  if (tid < CHUNK) sm.w[tid] = p.chunk_gates[(size_t)slot * p.heads + h].w[tid];
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
#pragma unroll
  for (int e = tid; e < CHUNK * (CP / 2); e += CHUNK_THREADS) {
    const int r = e / (CP / 2), c = (e % (CP / 2)) * 2;
    const float w = sm.w[r];
    const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162 *>(&sm.V[r][c]);
    uint32_t hi, lo;
    split_bf2(w * __low2float(x2), w * __high2float(x2), hi, lo);
    *reinterpret_cast<uint32_t *>(&sm.Wh[r][c]) = hi;
    *reinterpret_cast<uint32_t *>(&sm.Wl[r][c]) = lo;
  }
  if (blockIdx.x == 0)
    for (int c = tid; c < p.N; c += CHUNK_THREADS) {
      float a = 0.f;
      for (int r = 0; r < valid; ++r) a = fmaf(sm.w[r], __bfloat162float(sm.K[r][c]), a);
      p.chunk_n[((size_t)slot * p.heads + h) * p.N + c] = a;
    }
  __syncthreads();
  const int n0 = (MTILES >= 8 ? warp * MT : warp / WPT) * 16, j0 = MTILES >= 8 ? 0 : (warp % WPT) * NJ;
  float S[MT][NJ][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NJ; ++j) S[i][j][0] = S[i][j][1] = S[i][j][2] = S[i][j][3] = 0.f;
  const uint32_t wh_lane = smem_addr(&sm.Wh[lane & 15][j0 * 8 + (lane >> 4) * 8]), wl_lane = smem_addr(&sm.Wl[lane & 15][j0 * 8 + (lane >> 4) * 8]);
#pragma unroll
  for (int k2 = 0; k2 < CHUNK / 16; ++k2) {
    uint32_t a[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)   // A fragment (rows = state, k = tokens) from the token-major tile, transposed on the way
      ldsm4t(smem_addr(&sm.K[k2 * 16 + (lane & 7) + (lane >> 4) * 8][n0 + i * 16 + ((lane >> 3) & 1) * 8]), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
    for (int j = 0; j < NJ; j += 2) {
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm4t(wh_lane + (uint32_t)(k2 * 16 * XLD + j * 8) * 2u, h0, h1, h2, h3);
      ldsm4t(wl_lane + (uint32_t)(k2 * 16 * XLD + j * 8) * 2u, l0, l1, l2, l3);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        mma16816_bf16(S[i][j], a[i][0], a[i][1], a[i][2], a[i][3], h0, h1);
        mma16816_bf16(S[i][j + 1], a[i][0], a[i][1], a[i][2], a[i][3], h2, h3);
        mma16816_bf16(S[i][j], a[i][0], a[i][1], a[i][2], a[i][3], l0, l1);
        mma16816_bf16(S[i][j + 1], a[i][0], a[i][1], a[i][2], a[i][3], l2, l3);
      }
    }
  }
  float *out = p.chunk_state + ((size_t)slot * p.heads + h) * p.N * p.P;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int n = n0 + i * 16 + g + 8 * r, c = col0 + (j0 + j) * 8 + 2 * tig;
        if (n < p.N && c < p.P) *reinterpret_cast<float2 *>(out + (size_t)n * p.P + c) = make_float2(S[i][j][2 * r], S[i][j][2 * r + 1]);
      }
}

// Thread: eight consecutive elements of one head's S (or of n, behind them), along the chunks of its sequence.  In place: sum of the
// chunk -> value before the chunk; S as eight bf16 hi parts and eight lo parts, n in fp32.
__global__ void mlstm_carry_kernel(const Params p) {
  const int s = blockIdx.z, h = blockIdx.y, i = (blockIdx.x * blockDim.x + threadIdx.x) * 8, n = p.N * p.P;
  if (i >= n + p.N) return;
  const bool vec = i >= n;                      // n instead of S
  const int chunks = (p.cu[s + 1] - p.cu[s] + CHUNK - 1) / CHUNK, slot0 = chunk_slot(p.cu, s);
  const size_t stride = (size_t)p.heads * (vec ? p.N : n);
  float *x = vec ? p.chunk_n + (size_t)slot0 * stride + (size_t)h * p.N + (i - n) : p.chunk_state + (size_t)slot0 * stride + (size_t)h * n + i;
  const Gates *gates = p.chunk_gates + (size_t)slot0 * p.heads + h;
  float *nm = nm_of(p, p.slot[s], h, 0);
  float *state = p.state + ((size_t)p.slot[s] * p.heads + h) * n + i;
  float cur[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) cur[j] = 0.f;
  if (p.start[s] != 0) {
    if (vec) {
#pragma unroll
      for (int j = 0; j < 8; ++j) cur[j] = nm[i - n + j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(cur + j) = *reinterpret_cast<const float4 *>(state + j);
    }
  }
  double m = (double)p.chunk_m[(size_t)slot0 * p.heads + h];
  constexpr int U = 4;
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float v[U][8], keep[U], add[U], before[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < chunks) {
#pragma unroll
        for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(v[u] + j) = *reinterpret_cast<const float4 *>(x + (size_t)(c0 + u) * stride + j);
        const Gates &g = gates[(size_t)(c0 + u) * p.heads];
        const double a_max = g.a_max, top = fmax(m, a_max);
        before[u] = (float)m;
        keep[u] = expf((float)(m - top));
        add[u] = expf((float)(a_max - top));
        m = g.c_last + top;
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < chunks) {
        float *o = x + (size_t)(c0 + u) * stride;
        if (vec) {
#pragma unroll
          for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(o + j) = *reinterpret_cast<const float4 *>(cur + j);
        } else {
          uint4 hi, lo;
          split_bf2(cur[0], cur[1], hi.x, lo.x);
          split_bf2(cur[2], cur[3], hi.y, lo.y);
          split_bf2(cur[4], cur[5], hi.z, lo.z);
          split_bf2(cur[6], cur[7], hi.w, lo.w);
          reinterpret_cast<uint4 *>(o)[0] = hi;
          reinterpret_cast<uint4 *>(o)[1] = lo;
        }
        if (i == 0 && c0 + u > 0) p.chunk_m[(size_t)(slot0 + c0 + u) * p.heads + h] = before[u];
#pragma unroll
        for (int j = 0; j < 8; ++j) cur[j] = fmaf(keep[u], cur[j], add[u] * v[u][j]);
      }
  }
  if (vec) {
    for (int copy = 0; copy < p.copies; ++copy) {
#pragma unroll
      for (int j = 0; j < 8; ++j) nm[(size_t)copy * (p.N + 1) + i - n + j] = cur[j];
      if (i == n) nm[(size_t)copy * (p.N + 1) + p.N] = (float)m;
    }
  } else {
#pragma unroll
    for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(state + j) = *reinterpret_cast<const float4 *>(cur + j);
  }
}

template <int NP, int CP> struct OutSmem {
  __nv_bfloat16 Q[CHUNK][NP + 8], V[CHUNK][CP + 8], Sh[NP][CP + 8], Sl[NP][CP + 8];
  union {
    __nv_bfloat16 K[CHUNK][NP + 8];
    float ypart[4][16][CP + 4];     // the second warp's share of the output rows, once K is no longer needed
  };
  Gates g;
  float n[NP], top_hi[CHUNK], top_lo[CHUNK], ec[CHUNK], dn[3][CHUNK];   // M_t, exp(m - M_t), shares of n . q
};
// Block: one chunk, one head, CP columns.  Two warps share 16 output rows, each with every other 16 state rows (first product) and
// every other 16 tokens s (second product).
template <int NP, int CP> __global__ void __launch_bounds__(CHUNK_THREADS) mlstm_chunk_out_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  constexpr int XLD = CP + 8, KLD = NP + 8;
  extern __shared__ __align__(16) unsigned char smraw[];
  OutSmem<NP, CP> &sm = *reinterpret_cast<OutSmem<NP, CP> *>(smraw);
  const int slot = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CP;
  int s, t0;
  if (!chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int row0 = p.cu[s] + t0, valid = min(CHUNK, p.cu[s + 1] - row0);
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)row0 * p.ld + (size_t)h * p.N, *k = reinterpret_cast<const T *>(p.k) + (size_t)row0 * p.ld + (size_t)h * p.N;
  const T *v = reinterpret_cast<const T *>(p.v) + (size_t)row0 * p.ld + (size_t)h * p.P;
  for (int e = tid; e < CHUNK * (NP / 8); e += CHUNK_THREADS) {
    const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
    const bool in = r < valid && c < p.N;
    const size_t at = in ? (size_t)r * p.ld + c : 0;
    cp16(&sm.K[r][c], k + at, in);
    cp16(&sm.Q[r][c], q + at, in);
  }
  for (int e = tid; e < CHUNK * (CP / 8); e += CHUNK_THREADS) {
    const int r = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = r < valid && col0 + c < p.P;
    cp16(&sm.V[r][c], v + (in ? (size_t)r * p.ld + col0 + c : 0), in);
  }
  {
    const unsigned char *src = reinterpret_cast<const unsigned char *>(p.chunk_gates + (size_t)slot * p.heads + h);
    for (int i = tid; i < (int)(sizeof(Gates) / 16); i += CHUNK_THREADS) cp16(reinterpret_cast<unsigned char *>(&sm.g) + i * 16, src + i * 16, true);
  }
  const float *st = p.chunk_state + ((size_t)slot * p.heads + h) * p.N * p.P;
  for (int e = tid; e < NP * (CP / 8); e += CHUNK_THREADS) {
    const int n = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = n < p.N && col0 + c < p.P;
    const float *src = st + (in ? (size_t)n * p.P + col0 + c : 0);
    cp16(&sm.Sh[n][c], src, in);
    cp16(&sm.Sl[n][c], src + 4, in);
  }
  for (int i = tid; i < NP; i += CHUNK_THREADS) sm.n[i] = i < p.N ? p.chunk_n[((size_t)slot * p.heads + h) * p.N + i] : 0.f;
  const float m_before = p.chunk_m[(size_t)slot * p.heads + h];
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  if (tid < CHUNK) {
    const bool old = (m_before - sm.g.mx_hi[tid]) - sm.g.mx_lo[tid] > 0.f;
    const float hi = old ? m_before : sm.g.mx_hi[tid], lo = old ? 0.f : sm.g.mx_lo[tid];
    sm.top_hi[tid] = hi;
    sm.top_lo[tid] = lo;
    sm.ec[tid] = expf((m_before - hi) - lo);
  }
  {                                        // n . q with the n from before the chunk: four threads per row
    const int r = tid >> 2;
    float a = 0.f;
    for (int c = (tid & 3) * 2; c < NP; c += 8) {
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162 *>(&sm.Q[r][c]);
      a = fmaf(__low2float(x), sm.n[c], fmaf(__high2float(x), sm.n[c + 1], a));
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    if ((tid & 3) == 0) sm.dn[2][r] = a;
  }
  __syncthreads();
  const int rb = warp >> 1, half = warp & 1, tr = rb * 16 + g;      // this lane's output rows tr and tr + 8
  float y[CP / 8][4], G[2][2][4];
#pragma unroll
  for (int j = 0; j < CP / 8; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll
  for (int u = 0; u < 2; ++u)
#pragma unroll
    for (int j = 0; j < 2; ++j) G[u][j][0] = G[u][j][1] = G[u][j][2] = G[u][j][3] = 0.f;
  const uint32_t q_lane = smem_addr(&sm.Q[rb * 16 + (lane & 15)][(lane >> 4) * 8]);
  // (K rows are the n side: matrices (s 0-7, k 0-7), (s 0-7, k 8-15), (s 8-15, k 0-7), (s 8-15, k 8-15))
  const uint32_t k_lane = smem_addr(&sm.K[half * 16 + (lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]);
  const uint32_t sh_lane = smem_addr(&sm.Sh[lane & 15][(lane >> 4) * 8]), sl_lane = smem_addr(&sm.Sl[lane & 15][(lane >> 4) * 8]);
#pragma unroll 2
  for (int kk = 0; kk < NP / 16; ++kk) {
    uint32_t a0, a1, a2, a3;
    ldsm4(q_lane + (uint32_t)kk * 32u, a0, a1, a2, a3);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      if (half + 2 * u > rb) break;     // tokens behind the diagonal only
      uint32_t b0, b1, b2, b3;
      ldsm4(k_lane + (uint32_t)(u * 32 * KLD + kk * 16) * 2u, b0, b1, b2, b3);
      mma16816_bf16(G[u][0], a0, a1, a2, a3, b0, b1);
      mma16816_bf16(G[u][1], a0, a1, a2, a3, b2, b3);
    }
    if ((kk & 1) == half) {
#pragma unroll
      for (int j = 0; j < CP / 8; j += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm4t(sh_lane + (uint32_t)(kk * 16 * XLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(y[j], a0, a1, a2, a3, b0, b1);
        mma16816_bf16(y[j + 1], a0, a1, a2, a3, b2, b3);
        ldsm4t(sl_lane + (uint32_t)(kk * 16 * XLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(y[j], a0, a1, a2, a3, b0, b1);
        mma16816_bf16(y[j + 1], a0, a1, a2, a3, b2, b3);
      }
    }
  }
  const float e0 = sm.ec[tr], e1 = sm.ec[tr + 8];
#pragma unroll
  for (int j = 0; j < CP / 8; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
  const float h0 = sm.top_hi[tr], l0 = sm.top_lo[tr], h1 = sm.top_hi[tr + 8], l1 = sm.top_lo[tr + 8];
  const uint32_t v_lane = smem_addr(&sm.V[half * 16 + (lane & 15)][(lane >> 4) * 8]);
  float d0 = 0.f, d1 = 0.f;
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int k2 = half + 2 * u;
    if (k2 > rb) break;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int sc = k2 * 16 + j * 8 + 2 * tig;
      const float2 ah = *reinterpret_cast<const float2 *>(&sm.g.a_hi[sc]), al = *reinterpret_cast<const float2 *>(&sm.g.a_lo[sc]);
      G[u][j][0] = sc <= tr ? G[u][j][0] * expf((ah.x - h0) + (al.x - l0)) : 0.f;
      G[u][j][1] = sc + 1 <= tr ? G[u][j][1] * expf((ah.y - h0) + (al.y - l0)) : 0.f;
      G[u][j][2] = sc <= tr + 8 ? G[u][j][2] * expf((ah.x - h1) + (al.x - l1)) : 0.f;
      G[u][j][3] = sc + 1 <= tr + 8 ? G[u][j][3] * expf((ah.y - h1) + (al.y - l1)) : 0.f;
      d0 += G[u][j][0] + G[u][j][1];
      d1 += G[u][j][2] + G[u][j][3];
    }
    uint32_t hi[4], lo[4];
    split_bf2(G[u][0][0], G[u][0][1], hi[0], lo[0]);
    split_bf2(G[u][0][2], G[u][0][3], hi[1], lo[1]);
    split_bf2(G[u][1][0], G[u][1][1], hi[2], lo[2]);
    split_bf2(G[u][1][2], G[u][1][3], hi[3], lo[3]);
#pragma unroll
    for (int j = 0; j < CP / 8; j += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm4t(v_lane + (uint32_t)(u * 32 * XLD + j * 8) * 2u, b0, b1, b2, b3);
      mma16816_bf16(y[j], hi[0], hi[1], hi[2], hi[3], b0, b1);
      mma16816_bf16(y[j + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
      mma16816_bf16(y[j], lo[0], lo[1], lo[2], lo[3], b0, b1);
      mma16816_bf16(y[j + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
    }
  }
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    d0 += __shfl_xor_sync(0xffffffffu, d0, o);
    d1 += __shfl_xor_sync(0xffffffffu, d1, o);
  }
  if (tig == 0) {
    sm.dn[half][tr] = d0;
    sm.dn[half][tr + 8] = d1;
  }
  __syncthreads();   // K is no longer needed: its place takes the second warp's rows
  if (half) {
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) *reinterpret_cast<float2 *>(&sm.ypart[rb][g + 8 * r][j * 8 + 2 * tig]) = make_float2(y[j][2 * r], y[j][2 * r + 1]);
  }
  __syncthreads();
  if (half) return;
  float inv[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = tr + 8 * r;
    const float d = (sm.dn[2][t] * sm.ec[t] + sm.dn[0][t] + sm.dn[1][t]) * p.q_scale, m = (sm.g.c_hi[t] + sm.top_hi[t]) + (sm.g.c_lo[t] + sm.top_lo[t]);
    inv[r] = p.q_scale / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
  }
#pragma unroll
  for (int j = 0; j < CP / 8; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = tr + 8 * r, c = j * 8 + 2 * tig;
      if (t >= valid || col0 + c >= p.P) continue;
      const float2 o = *reinterpret_cast<const float2 *>(&sm.ypart[rb][g + 8 * r][c]);
      *reinterpret_cast<float2 *>(p.y + (size_t)(row0 + t) * p.inner + (size_t)h * p.P + col0 + c) =
          make_float2((y[j][2 * r] + o.x) * inv[r], (y[j][2 * r + 1] + o.y) * inv[r]);
    }
}

// ------------------------------------------------------------------------------------------ norm and output gate
// One warp: o of a head (fp32, p.y) -> its outputs.
template <typename T, int VEC> __device__ __forceinline__ void norm_gate_row(const Params &p, int t, int h, int lane) {
  const float *y = p.y + (size_t)t * p.inner + (size_t)h * p.P, *w = p.norm_w + (size_t)h * p.P;
  const T *gate = reinterpret_cast<const T *>(p.g) + (size_t)t * p.ld + (size_t)h * p.P;
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld + (size_t)h * p.P;
  auto load = [&](int i, float (&v)[VEC]) {     // (written by other blocks of this launch in the step kernel: through L2)
    if constexpr (VEC == 4) {
      const float4 r = __ldcg(reinterpret_cast<const float4 *>(y + i));
      v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
    } else {
      v[0] = __ldcg(y + i);
    }
  };
  auto squares = [](const float (&v)[VEC]) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < VEC; ++j) s = fmaf(v[j], v[j], s);
    return s;
  };
  auto scale = [&](float ss) { return p.out_scale / sqrtf(warp_sum(ss) / (float)p.P + p.eps); };
  auto finish = [&](int i, float (&v)[VEC], float (&b)[VEC], float inv) {
    float a[VEC];
    load_vec<VEC>(w + i, a);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= inv * a[j] * sigmoid_f(b[j]);
    store_vec<VEC>(out + i, v);
  };
  constexpr int R = 2;                          // a head of up to 32 R VEC values stays in registers
  if (p.P <= 32 * R * VEC) {
    float v[R][VEC], b[R][VEC], ss = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = (lane + 32 * r) * VEC;
      if (i < p.P) {
        load(i, v[r]);
        load_vec<VEC>(gate + i, b[r]);
        ss += squares(v[r]);
      }
    }
    const float inv = scale(ss);
#pragma unroll
    for (int r = 0; r < R; ++r)
      if ((lane + 32 * r) * VEC < p.P) finish((lane + 32 * r) * VEC, v[r], b[r], inv);
  } else {
    float ss = 0.f;
    for (int i = lane * VEC; i < p.P; i += 32 * VEC) {
      float v[VEC];
      load(i, v);
      ss += squares(v);
    }
    const float inv = scale(ss);
    for (int i = lane * VEC; i < p.P; i += 32 * VEC) {
      float v[VEC], b[VEC];
      load(i, v);
      load_vec<VEC>(gate + i, b);
      finish(i, v, b, inv);
    }
  }
  if (h == p.heads - 1)   // k padding of the output product
    for (int i = p.inner + lane; i < p.out_cols; i += 32) reinterpret_cast<T *>(p.out)[(size_t)t * p.out_ld + i] = from_f<T>(0.f);
}
constexpr int NORM_WARPS = 8;
template <typename T, int VEC> __global__ void __launch_bounds__(NORM_WARPS * 32) mlstm_norm_kernel(const Params p) {   // warp: one token, one head
  const long long i = (long long)blockIdx.x * NORM_WARPS + (threadIdx.x >> 5);
  if (i < (long long)p.n_tok * p.heads) norm_gate_row<T, VEC>(p, (int)(i / p.heads), (int)(i % p.heads), threadIdx.x & 31);
}

// ------------------------------------------------------------------------------------------ one token per sequence
constexpr int STEP_THREADS = 256;
// Block: one sequence, one head, p.tile columns.  Thread (row group, column quad) walks state rows group, + groups, ...; every state
// element is read and written once.  The last block of a head to arrive normalises and gates.
template <typename T, int VEC> __global__ void __launch_bounds__(STEP_THREADS) mlstm_step_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ int s_last;
  float *qs = sm, *ks = qs + p.N, *part = sm + (2 * p.N + 3) / 4 * 4;      // part [row groups][tile]
  const int s = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * p.tile, cols = min(p.tile, p.P - c0), tid = threadIdx.x;
  const int pos = p.start[s], slot = p.slot[s], t = p.cu[s];
  const int pq = (cols + VEC - 1) / VEC, ng = max(1, STEP_THREADS / pq), grp = tid / pq, c = (tid - grp * pq) * VEC;
  float *gS = p.state + ((size_t)slot * p.heads + h) * p.N * p.P + c0;
  const bool fresh = pos == 0;
  constexpr int U = 8;                    // state rows in flight per thread
  float v[U][VEC];
  auto load_rows = [&](int n0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int n = n0 + u * ng;
      if (n < p.N && !fresh) {
        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(v[u]) = __ldcs(reinterpret_cast<const float4 *>(gS + (size_t)n * p.P + c));
        else v[u][0] = gS[(size_t)n * p.P + c];
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[u][j] = 0.f;
      }
    }
  };
  const bool work = grp < ng;
  if (work) load_rows(grp);               // on their way while the gates are computed
  const T *q = reinterpret_cast<const T *>(p.q) + (size_t)t * p.ld + (size_t)h * p.N, *k = reinterpret_cast<const T *>(p.k) + (size_t)t * p.ld + (size_t)h * p.N;
  float *gn = nm_of(p, slot, h, c0 / COPY_COLS);
  float m = fresh ? 0.f : gn[p.N];
  const float li = log_input(p, t, h), fm = log_forget(p, t, h) + m;
  m = fmaxf(fm, li);
  const float keep = expf(fm - m), add = expf(li - m);
  float d = 0.f;
  for (int i = tid; i < p.N; i += STEP_THREADS) {
    const float qv = to_f(q[i]) * p.q_scale, kv = to_f(k[i]), nv = fmaf(keep, fresh ? 0.f : gn[i], add * kv);
    qs[i] = qv;
    ks[i] = kv;
    d = fmaf(nv, qv, d);
    for (int o = 0; o < cols; o += COPY_COLS) gn[(size_t)(o / COPY_COLS) * (p.N + 1) + i] = nv;
  }
  d = block_sum(d, red);                  // (its barriers also publish qs and ks, and every thread has read m)
  if (tid == 0)
    for (int o = 0; o < cols; o += COPY_COLS) gn[(size_t)(o / COPY_COLS) * (p.N + 1) + p.N] = m;
  const float inv = 1.0f / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
  if (work) {
    float y[VEC], av[VEC];
    load_vec<VEC>(reinterpret_cast<const T *>(p.v) + (size_t)t * p.ld + (size_t)h * p.P + c0 + c, av);
#pragma unroll
    for (int j = 0; j < VEC; ++j) { y[j] = 0.f; av[j] *= add; }
    for (int n0 = grp; n0 < p.N; n0 += U * ng) {
      if (n0 != grp) load_rows(n0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * ng;
        if (n >= p.N) break;
        const float kv = ks[n], qv = qs[n];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          v[u][j] = fmaf(keep, v[u][j], kv * av[j]);
          y[j] = fmaf(v[u][j], qv, y[j]);
        }
        store_vec<VEC>(gS + (size_t)n * p.P + c, v[u]);
      }
    }
    store_vec<VEC>(part + (size_t)grp * p.tile + c, y);
  }
  __syncthreads();
  for (int i = tid; i < cols; i += STEP_THREADS) {
    float a = 0.f;
    for (int r = 0; r < ng; ++r) a += part[(size_t)r * p.tile + i];
    p.y[(size_t)t * p.inner + (size_t)h * p.P + c0 + i] = a * inv;
  }
  __threadfence();
  __syncthreads();
  if (gridDim.x > 1) {
    int *ctr = p.counters + (size_t)s * p.heads + h;
    if (tid == 0) s_last = atomicAdd(ctr, 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) *ctr = 0;
  }
  if (tid < 32) norm_gate_row<T, VEC>(p, t, h, tid);
}

template <int NP, int CP> static int launch_chunks(const Params &p, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    PT_CUDA(cudaFuncSetAttribute(mlstm_chunk_state_kernel<NP, CP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(StateSmem<NP, CP>)));
    PT_CUDA(cudaFuncSetAttribute(mlstm_chunk_out_kernel<NP, CP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(OutSmem<NP, CP>)));
    set = true;
  }
  const dim3 grid(ceil_div(p.P, CP), p.heads, p.n_tok / CHUNK + p.n_seq);
  mlstm_gate_kernel<<<dim3(ceil_div(p.heads, 4), grid.z), 128, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_mlstm");
  mlstm_chunk_state_kernel<NP, CP><<<grid, CHUNK_THREADS, sizeof(StateSmem<NP, CP>), st>>>(p);
  PT_LAUNCH_CHECK("pt_mlstm");
  mlstm_carry_kernel<<<dim3(ceil_div((p.N * p.P + p.N) / 8, 64), p.heads, p.n_seq), 64, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_mlstm");
  mlstm_chunk_out_kernel<NP, CP><<<grid, CHUNK_THREADS, sizeof(OutSmem<NP, CP>), st>>>(p);
  PT_LAUNCH_CHECK("pt_mlstm");
  return PT_OK;
}
template <int CP> static int dispatch_chunks(const Params &p, cudaStream_t st) {
  return p.N <= 64 ? launch_chunks<64, CP>(p, st) : (p.N <= 128 ? launch_chunks<128, CP>(p, st) : launch_chunks<256, CP>(p, st));
}

template <typename T> static int run(Params &p, bool plain, cudaStream_t st) {
  const int vb = 4 * sizeof(T);
  const bool v4 = p.P % 4 == 0 && p.ld % 4 == 0 && p.out_ld % 4 == 0 && aligned_to(p.state, 16) && aligned_to(p.y, 16) && aligned_to(p.norm_w, 16) && aligned_to(p.v, vb) &&
                  aligned_to(p.g, vb) && aligned_to(p.out, vb);
  if (p.n_tok == p.n_seq) {
    // few sequences: narrow tiles, so that every SM has a part of some head's state
    p.tile = COPY_COLS;
    while (p.tile < p.P && p.tile < (v4 ? 1024 : 256) && (long long)ceil_div(p.P, 2 * p.tile) * p.heads * p.n_seq >= 4LL * sm_count()) p.tile *= 2;
    const int pq = v4 ? std::min(p.tile, p.P) / 4 : std::min(p.tile, p.P);
    // (the last tile of a head may be narrower and then has more row groups)
    const int rest = p.P % p.tile ? p.P % p.tile : std::min(p.tile, p.P), pq_min = std::min(pq, v4 ? rest / 4 : rest), ng = std::max(1, STEP_THREADS / pq_min);
    const size_t smem = ((size_t)(2 * p.N + 3) / 4 * 4 + (size_t)ng * p.tile) * sizeof(float);
    PT_REQUIRE(smem <= 200 * 1024, "pt_mlstm: head widths %d / %d need %zu bytes of shared memory", p.N, p.P, smem);
    if (smem > 48 * 1024) {
      PT_CUDA(cudaFuncSetAttribute(mlstm_step_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      PT_CUDA(cudaFuncSetAttribute(mlstm_step_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    const dim3 grid(ceil_div(p.P, p.tile), p.heads, p.n_seq);
    if (v4) mlstm_step_kernel<T, 4><<<grid, STEP_THREADS, smem, st>>>(p);
    else mlstm_step_kernel<T, 1><<<grid, STEP_THREADS, smem, st>>>(p);
    PT_LAUNCH_CHECK("pt_mlstm");
    return PT_OK;
  }
  // the chunked form: bf16, rows that are whole 16-byte units, keys of at most 256, with its scratch
  if (!plain && sizeof(T) == 2 && p.chunk_state && p.N <= 256 && p.N % 8 == 0 && p.P % 8 == 0 && p.ld % 8 == 0 && aligned_to(p.state, 16) && aligned_to(p.q, 16) &&
      aligned_to(p.k, 16) && aligned_to(p.v, 16) && aligned_to(p.y, 8)) {
    const int rc = p.P <= 32 ? dispatch_chunks<32>(p, st) : dispatch_chunks<64>(p, st);
    if (rc != PT_OK) return rc;
  } else {
    const size_t smem = ((size_t)p.N * (32 + 3) + SCAN_WARPS * 33) * sizeof(float);
    PT_REQUIRE(smem <= 200 * 1024, "pt_mlstm: keys of %d need %zu bytes of shared memory", p.N, smem);
    if (smem > 48 * 1024) PT_CUDA(cudaFuncSetAttribute(mlstm_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    mlstm_scan_kernel<T><<<dim3(p.copies, p.heads, p.n_seq), SCAN_WARPS * 32, smem, st>>>(p);
    PT_LAUNCH_CHECK("pt_mlstm");
  }
  const int blocks = (int)(((long long)p.n_tok * p.heads + NORM_WARPS - 1) / NORM_WARPS);
  if (v4) mlstm_norm_kernel<T, 4><<<blocks, NORM_WARPS * 32, 0, st>>>(p);
  else mlstm_norm_kernel<T, 1><<<blocks, NORM_WARPS * 32, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_mlstm");
  return PT_OK;
}

}  // namespace mlstm
}  // namespace pt

using namespace pt;

// Workspace layout: [arrival counters][state of every chunk and head][n][gates][m].  The counter region has ONE size, so that layers
// and batches of different shapes can share a workspace.
constexpr size_t kCounterBytes = 1u << 18;
static size_t up16(size_t v) { return (v + 15) / 16 * 16; }

extern "C" size_t pt_mlstm_workspace_bytes(int n_tok, int n_seq, int heads, int dim, int vdim) {
  if (n_tok == n_seq) return kCounterBytes;
  const size_t sh = ((size_t)n_tok / CHUNK + n_seq) * heads;
  return kCounterBytes + up16(sh * dim * vdim * sizeof(float)) + up16(sh * dim * sizeof(float)) + sh * sizeof(mlstm::Gates) + up16(sh * sizeof(float));
}

extern "C" size_t pt_mlstm_state_floats(int heads, int dim, int vdim, int which) {
  return which == 0 ? (size_t)heads * dim * vdim : (size_t)heads * ceil_div(vdim, mlstm::COPY_COLS) * (dim + 1);
}

extern "C" int pt_mlstm(const pt_mlstm_args *a, void *stream) {
  PT_REQUIRE(a, "pt_mlstm: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.n_tok >= b.n_seq && b.n_seq <= 65535 && b.n_tok <= 64 * 65535 && b.cu && b.start && b.slot && b.tok_seq,
             "pt_mlstm: bad batch (%d sequences, %d tokens)", b.n_seq, b.n_tok);
  PT_REQUIRE(a->heads > 0 && a->heads <= 65535 && a->dim > 0 && a->vdim > 0 && a->gate_cap > 0.f, "pt_mlstm: bad shape heads=%d dim=%d vdim=%d cap=%f", a->heads, a->dim,
             a->vdim, a->gate_cap);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_mlstm: type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->q && a->k && a->v && a->gate && a->log_i && a->log_f && a->norm_w && a->state && a->nm && a->y && a->out, "pt_mlstm: null pointer argument");
  const int inner = a->heads * a->vdim;
  PT_REQUIRE(a->ld >= std::max(a->heads * a->dim, inner) && a->gate_ld >= a->heads && a->out_ld >= inner && a->out_cols <= a->out_ld, "pt_mlstm: row strides %d, %d, out %d too small",
             a->ld, a->gate_ld, a->out_ld);
  mlstm::Params p{};
  p.n_seq = b.n_seq; p.n_tok = b.n_tok; p.heads = a->heads; p.N = a->dim; p.P = a->vdim; p.inner = inner; p.ld = a->ld; p.gate_ld = a->gate_ld;
  p.out_ld = a->out_ld; p.out_cols = a->out_cols > 0 ? a->out_cols : a->out_ld; p.copies = ceil_div(a->vdim, mlstm::COPY_COLS);
  p.cap = a->gate_cap; p.eps = a->eps; p.q_scale = a->q_scale; p.out_scale = a->out_scale != 0.f ? a->out_scale : 1.0f;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq;
  p.q = a->q; p.k = a->k; p.v = a->v; p.g = a->gate; p.zi = a->log_i; p.zf = a->log_f; p.norm_w = a->norm_w;
  p.state = a->state; p.nm = a->nm; p.y = a->y; p.out = a->out;
  const size_t need = pt_mlstm_workspace_bytes(b.n_tok, b.n_seq, a->heads, a->dim, a->vdim);
  const bool have = a->workspace && aligned_to(a->workspace, 16) && a->workspace_bytes >= need;
  if (b.n_tok == b.n_seq) {
    PT_REQUIRE(have, "pt_mlstm: a decode step needs %zu workspace bytes, got %zu", need, a->workspace_bytes);
    PT_REQUIRE((size_t)b.n_seq * a->heads <= kCounterBytes / sizeof(int), "pt_mlstm: %d sequences x %d heads exceed the arrival counters", b.n_seq, a->heads);
    p.counters = (int *)a->workspace;
  } else if (have) {
    const size_t sh = ((size_t)b.n_tok / CHUNK + b.n_seq) * a->heads;
    char *ws = (char *)a->workspace + kCounterBytes;
    p.chunk_state = (float *)ws; ws += up16(sh * a->dim * a->vdim * sizeof(float));
    p.chunk_n = (float *)ws; ws += up16(sh * a->dim * sizeof(float));
    p.chunk_gates = (mlstm::Gates *)ws; ws += sh * sizeof(mlstm::Gates);
    p.chunk_m = (float *)ws;
  }
  return a->dtype == PT_DT_F32 ? mlstm::run<float>(p, a->plain != 0, as_stream(stream)) : mlstm::run<__nv_bfloat16>(p, a->plain != 0, as_stream(stream));
}
