// State-space (SSD) mixer with a matrix state per head and a scalar decay:
//     z | x | B | C | dt = row of the input projection           widths inner, inner, G N, G N, heads   (inner = heads * P)
//     x, B, C <- silu(causal conv per channel + bias);  dt <- softplus(dt + dt_bias)
//     S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t            S [N, P] per head, fp32
//     out = rms_norm over norm_groups equal parts of (y * silu(z)), times norm_w
// Everything that enters the recurrence besides the projection and the convolution is fp32, and so are the state and y.
//
// Per sequence slot the mixer keeps S and a ring of the last `taps` raw convolution inputs (position q at ring index q % taps, so
// the ring can be written while others still read the taps - 1 older entries).  Nothing has to be cleared for a new sequence: at
// position 0 the old state is ignored, and convolution taps before position 0 count as zero.
//
//   ssm_conv_kernel    prompts: convolution + silu of all tokens, step sizes
//   ssm_scan_kernel    prompts, any sizes and types: the recurrence token by token, state in shared memory
//   ssm_chunk_* , ssm_carry_kernel   bf16 prompts: the same recurrence 64 tokens at a time on the tensor cores
//   ssm_step_kernel    one token per sequence: convolution, step size, state update and readout in one launch
//   ssm_norm_kernel    gate, group norm, and the ring update
#include <type_traits>

#include "chunk.cuh"

namespace pt {
namespace ssm {

struct Params {
  int n_seq, n_tok, heads, P, N, groups, taps, norm_groups, C, inner, zx_ld, out_ld;
  float eps;
  const int *cu, *start, *slot, *tok_seq;
  const void *zx;
  const float *conv_w, *conv_b, *dt_bias, *A_log, *D, *norm_w;
  void *ring, *xbc, *out;
  float *state, *dt, *y;
  float *chunk_state;                // [n_tok / 64 + n_seq][heads][N][P]
  struct Decays *chunk_decays;       // [n_tok / 64 + n_seq][heads]
};

// ------------------------------------------------------------------------------------------ convolution of a prompt
// Raw convolution input of channel c at position `pos` - back, for row t of a sequence whose portion starts at row t0: from this
// launch's rows, from the ring, or zero before the sequence starts.
template <typename T>
__device__ __forceinline__ float conv_input(const Params &p, const T *zx, const T *ring, int t, int t0, int pos, int back, int c) {
  if (back > pos) return 0.f;
  if (t - back >= t0) return to_f(zx[(size_t)(t - back) * p.zx_ld + p.inner + c]);
  return to_f(ring[(size_t)((pos - back) % p.taps) * p.C + c]);
}

template <typename T> __global__ void ssm_conv_kernel(const Params p) {
  const int t = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int s = p.tok_seq[t], t0 = p.cu[s], pos = p.start[s] + t - t0;
  const T *zx = reinterpret_cast<const T *>(p.zx);
  if (c < p.C) {
    const T *ring = reinterpret_cast<const T *>(p.ring) + (size_t)p.slot[s] * p.taps * p.C;
    float a = p.conv_b[c];
    for (int k = 0; k < p.taps; ++k) a = fmaf(p.conv_w[(size_t)c * p.taps + k], conv_input(p, zx, ring, t, t0, pos, p.taps - 1 - k, c), a);
    reinterpret_cast<T *>(p.xbc)[(size_t)t * p.C + c] = from_f<T>(silu_f(a));
  } else if (c < p.C + p.heads) {
    const int h = c - p.C;
    p.dt[(size_t)t * p.heads + h] = softplus_f(to_f(zx[(size_t)t * p.zx_ld + p.inner + c]) + p.dt_bias[h]);
  }
}

// The same for bf16 rows of whole 16-byte units and at most 4 taps: a thread slides over CONV_TOKENS tokens of 8 channels with the
// window in registers; the last column of blocks computes the step sizes.
constexpr int CONV_TOKENS = 16, CONV_THREADS = 128;
template <int TAPS> __global__ void __launch_bounds__(CONV_THREADS) ssm_conv8_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  const T *zx = reinterpret_cast<const T *>(p.zx);
  const int ta = blockIdx.y * CONV_TOKENS, tb = min(p.n_tok, ta + CONV_TOKENS);
  if (blockIdx.x == gridDim.x - 1) {
    for (int i = threadIdx.x; i < (tb - ta) * p.heads; i += CONV_THREADS) {
      const int t = ta + i / p.heads, h = i % p.heads;
      p.dt[(size_t)t * p.heads + h] = softplus_f(to_f(zx[(size_t)t * p.zx_ld + p.inner + p.C + h]) + p.dt_bias[h]);
    }
    return;
  }
  const int c = (blockIdx.x * CONV_THREADS + threadIdx.x) * 8;
  if (c >= p.C) return;
  float w[8][TAPS], b[8], x[TAPS][8];     // x[k]: the input k tokens back
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    b[j] = p.conv_b[c + j];
    if constexpr (TAPS == 4) load_vec<4>(p.conv_w + (size_t)(c + j) * 4, w[j]);
    else {
#pragma unroll
      for (int k = 0; k < TAPS; ++k) w[j][k] = p.conv_w[(size_t)(c + j) * TAPS + k];
    }
  }
  // the window in front of token t of sequence s
  auto fill_window = [&](int t, int s) {
    const int t0 = p.cu[s], pos = p.start[s] + t - t0;
    const T *ring = reinterpret_cast<const T *>(p.ring) + (size_t)p.slot[s] * TAPS * p.C;
#pragma unroll
    for (int k = 1; k < TAPS; ++k) {
      if (k > pos) {
#pragma unroll
        for (int j = 0; j < 8; ++j) x[k - 1][j] = 0.f;
      } else if (t - k >= t0) {
        load_vec<8>(zx + (size_t)(t - k) * p.zx_ld + p.inner + c, x[k - 1]);
      } else {
        load_vec<8>(ring + (size_t)((pos - k) % TAPS) * p.C + c, x[k - 1]);
      }
    }
  };
  auto one_token = [&](int t, const uint4 &raw) {
#pragma unroll
    for (int k = TAPS - 1; k > 0; --k)
#pragma unroll
      for (int j = 0; j < 8; ++j) x[k][j] = x[k - 1][j];
    const __nv_bfloat162 *r = reinterpret_cast<const __nv_bfloat162 *>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) { x[0][2 * j] = __low2float(r[j]); x[0][2 * j + 1] = __high2float(r[j]); }
    __nv_bfloat162 o[4];
    float y[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      float a = b[j];
#pragma unroll
      for (int k = 0; k < TAPS; ++k) a = fmaf(w[j][k], x[TAPS - 1 - k][j], a);
      y[j] = __fdividef(a, 1.0f + __expf(-a));   // (rounded to bf16 below; for a very negative the quotient is 0 either way)
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = __floats2bfloat162_rn(y[2 * j], y[2 * j + 1]);
    *reinterpret_cast<uint4 *>(reinterpret_cast<T *>(p.xbc) + (size_t)t * p.C + c) = *reinterpret_cast<const uint4 *>(o);
  };
  auto src = [&](int t) { return reinterpret_cast<const uint4 *>(zx + (size_t)t * p.zx_ld + p.inner + c); };
  int seq = p.tok_seq[ta];
  fill_window(ta, seq);
  if (seq == p.tok_seq[tb - 1]) {         // all tokens of one sequence: four loads in flight
    for (int t = ta; t < tb; t += 4) {
      uint4 raw[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) raw[u] = t + u < tb ? *src(t + u) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (t + u < tb) one_token(t + u, raw[u]);
    }
    return;
  }
  for (int t = ta; t < tb; ++t) {
    if (p.tok_seq[t] != seq) {
      seq = p.tok_seq[t];
      fill_window(t, seq);
    }
    one_token(t, *src(t));
  }
}

// ------------------------------------------------------------------------------------------ recurrence, any sizes
constexpr int SCAN_P = 32, SCAN_WARPS = 8;
// Block: one sequence, one head, 32 columns of the state.  Warp w owns state rows w, w + 8, ...; lane = column.
template <typename T> __global__ void __launch_bounds__(SCAN_WARPS * 32) ssm_scan_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *S = sm, *Bs = S + (size_t)p.N * SCAN_P, *Cs = Bs + p.N, *part = Cs + p.N;   // part [SCAN_WARPS][32]
  const int s = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * SCAN_P, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = h / (p.heads / p.groups), col = c0 + lane;
  const bool in = col < p.P;
  float *gS = p.state + ((size_t)p.slot[s] * p.heads + h) * p.N * p.P;
  const bool fresh = p.start[s] == 0;
  for (int n = warp; n < p.N; n += SCAN_WARPS) S[n * SCAN_P + lane] = (in && !fresh) ? gS[(size_t)n * p.P + col] : 0.f;
  const float a = -expf(p.A_log[h]), D = p.D[h];
  for (int t = p.cu[s]; t < p.cu[s + 1]; ++t) {
    const T *row = reinterpret_cast<const T *>(p.xbc) + (size_t)t * p.C;
    __syncthreads();
    for (int n = tid; n < p.N; n += blockDim.x) {
      Bs[n] = to_f(row[p.inner + g * p.N + n]);
      Cs[n] = to_f(row[p.inner + (p.groups + g) * p.N + n]);
    }
    const float x = in ? to_f(row[(size_t)h * p.P + col]) : 0.f;
    const float dt = p.dt[(size_t)t * p.heads + h], decay = expf(a * dt), dx = dt * x;
    __syncthreads();
    float y = 0.f;
    for (int n = warp; n < p.N; n += SCAN_WARPS) {
      const float v = fmaf(decay, S[n * SCAN_P + lane], Bs[n] * dx);
      S[n * SCAN_P + lane] = v;
      y = fmaf(v, Cs[n], y);
    }
    part[warp * 32 + lane] = y;
    __syncthreads();
    if (warp == 0 && in) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < SCAN_WARPS; ++w) sum += part[w * 32 + lane];
      p.y[(size_t)t * p.inner + (size_t)h * p.P + col] = fmaf(D, x, sum);
    }
  }
  for (int n = warp; n < p.N; n += SCAN_WARPS)
    if (in) gS[(size_t)n * p.P + col] = S[n * SCAN_P + lane];
}

// ------------------------------------------------------------------------------------------ recurrence in chunks of 64 tokens
// With c_t = sum_{r <= t} log decay_r inside a chunk and S the state before it, the recurrence is four matrix products:
//     y_t = exp(c_t) C_t S  +  sum_{s <= t} (C_t . B_s) exp(c_t - c_s) dt_s x_s  +  D x_t
//     S  <- exp(c_last) S  +  sum_s B_s (exp(c_last - c_s) dt_s x_s)^T
// Four launches, so that all chunks of all sequences work at once and only an elementwise pass runs along the sequence:
//   ssm_decay_kernel         the decay factors of every chunk and head
//   ssm_chunk_state_kernel   the sum of the second line, per chunk and head
//   ssm_carry_kernel         the second line along the chunks: leaves the state BEFORE every chunk in place of its sum
//   ssm_chunk_out_kernel     the first line, per chunk and head
// Operands that are not already bf16 (the state, the decayed products, the weighted x) enter the tensor cores as hi + lo pairs.  c is kept as a pair
// of floats, so differences of neighbours stay exact however far the sum has run.
// NP: state size rounded up to 64, 128 or 256, CP: columns of a head per block (padding is zero).
struct __align__(16) Decays {
  float c_hi[CHUNK], c_lo[CHUNK], dt[CHUNK], ec[CHUNK], w[CHUNK];   // ec = exp(c_t), w = exp(c_last - c_s) dt_s
  float keep, pad[3];                                               // exp(c_last)
};
// One warp: step sizes of the chunk and what follows from them (tokens beyond the sequence: decay 1, no contribution).
__device__ __forceinline__ void scan_decays(const Params &p, int row0, int valid, int h, Decays &d) {
  const int lane = threadIdx.x & 31;
  const float a = -expf(p.A_log[h]);
  float dt[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) dt[k] = 2 * lane + k < valid ? p.dt[(size_t)(row0 + 2 * lane + k) * p.heads + h] : 0.f;
  const double l1 = (double)(a * dt[1]);
  double sum = (double)(a * dt[0]) + l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += v;
  }
  const double last = __shfl_sync(0xffffffffu, sum, 31);
  const double c[2] = {sum - l1, sum};
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int r = 2 * lane + k;
    d.c_hi[r] = (float)c[k];
    d.c_lo[r] = (float)(c[k] - (double)(float)c[k]);
    d.dt[r] = dt[k];
    d.ec[r] = expf((float)c[k]);
    d.w[r] = expf((float)(last - c[k])) * dt[k];
  }
  if (lane == 0) d.keep = expf((float)last);
}
__global__ void ssm_decay_kernel(const Params p) {   // one warp per (chunk, head)
  const int slot = blockIdx.y, h = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  int s, t0;
  if (h >= p.heads || !chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int row0 = p.cu[s] + t0;
  scan_decays(p, row0, min(CHUNK, p.cu[s + 1] - row0), h, p.chunk_decays[(size_t)slot * p.heads + h]);
}
__device__ __forceinline__ void load_decays(const Params &p, int slot, int h, Decays &d) {
  const unsigned char *src = reinterpret_cast<const unsigned char *>(p.chunk_decays + (size_t)slot * p.heads + h);
  for (int i = threadIdx.x; i < (int)(sizeof(Decays) / 16); i += blockDim.x) cp16(reinterpret_cast<unsigned char *>(&d) + i * 16, src + i * 16, true);
}

template <int NP, int CP> struct StateSmem {
  __nv_bfloat16 B[CHUNK][NP + 8], X[CHUNK][CP + 8], Wh[CHUNK][CP + 8], Wl[CHUNK][CP + 8];
  Decays d;
};
// Block: one chunk, one head, CP columns.  The warps share the 16-row tiles of the state (and the columns when there are fewer tiles).
template <int NP, int CP> __global__ void __launch_bounds__(CHUNK_THREADS) ssm_chunk_state_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  constexpr int XLD = CP + 8, MTILES = NP / 16, WPT = MTILES >= 8 ? 1 : 8 / MTILES;      // warps per row tile
  constexpr int MT = MTILES >= 8 ? MTILES / 8 : 1, NJ = CP / 8 / WPT;
  extern __shared__ __align__(16) unsigned char smraw[];
  StateSmem<NP, CP> &sm = *reinterpret_cast<StateSmem<NP, CP> *>(smraw);
  const int slot = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CP;
  int s, t0;
  if (!chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int grp = h / (p.heads / p.groups), row0 = p.cu[s] + t0, valid = min(CHUNK, p.cu[s + 1] - row0);
  const T *xbc = reinterpret_cast<const T *>(p.xbc) + (size_t)row0 * p.C;
  for (int e = tid; e < CHUNK * (NP / 8); e += CHUNK_THREADS) {
    const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
    const bool in = r < valid && c < p.N;
    cp16(&sm.B[r][c], xbc + (in ? (size_t)r * p.C + p.inner + grp * p.N + c : 0), in);
  }
  for (int e = tid; e < CHUNK * (CP / 8); e += CHUNK_THREADS) {
    const int r = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = r < valid && col0 + c < p.P;
    cp16(&sm.X[r][c], xbc + (in ? (size_t)r * p.C + (size_t)h * p.P + col0 + c : 0), in);
  }
  load_decays(p, slot, h, sm.d);
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
#pragma unroll
  for (int e = tid; e < CHUNK * (CP / 2); e += CHUNK_THREADS) {
    const int r = e / (CP / 2), c = (e % (CP / 2)) * 2;
    const float w = sm.d.w[r];
    const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162 *>(&sm.X[r][c]);
    uint32_t hi, lo;
    split_bf2(w * __low2float(x2), w * __high2float(x2), hi, lo);
    *reinterpret_cast<uint32_t *>(&sm.Wh[r][c]) = hi;
    *reinterpret_cast<uint32_t *>(&sm.Wl[r][c]) = lo;
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
      ldsm4t(smem_addr(&sm.B[k2 * 16 + (lane & 7) + (lane >> 4) * 8][n0 + i * 16 + ((lane >> 3) & 1) * 8]), a[i][0], a[i][1], a[i][2], a[i][3]);
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

// Thread: eight consecutive elements of one head's state, along the chunks of its sequence.  In place: sum of the chunk -> state
// before the chunk, as eight bf16 hi parts and eight lo parts.
__global__ void ssm_carry_kernel(const Params p) {
  const int s = blockIdx.z, h = blockIdx.y, i = (blockIdx.x * blockDim.x + threadIdx.x) * 8, n = p.N * p.P;
  if (i >= n) return;
  const int chunks = (p.cu[s + 1] - p.cu[s] + CHUNK - 1) / CHUNK;
  const size_t stride = (size_t)p.heads * n;
  float *x = p.chunk_state + (size_t)chunk_slot(p.cu, s) * stride + (size_t)h * n + i;
  const Decays *dec = p.chunk_decays + (size_t)chunk_slot(p.cu, s) * p.heads + h;
  float *state = p.state + ((size_t)p.slot[s] * p.heads + h) * n + i;
  float cur[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) cur[j] = 0.f;
  if (p.start[s] != 0) {
#pragma unroll
    for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(cur + j) = *reinterpret_cast<const float4 *>(state + j);
  }
  constexpr int U = 4;
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float v[U][8], k[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < chunks) {
#pragma unroll
        for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(v[u] + j) = *reinterpret_cast<const float4 *>(x + (size_t)(c0 + u) * stride + j);
        k[u] = dec[(size_t)(c0 + u) * p.heads].keep;
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < chunks) {
        uint4 hi, lo;
        split_bf2(cur[0], cur[1], hi.x, lo.x);
        split_bf2(cur[2], cur[3], hi.y, lo.y);
        split_bf2(cur[4], cur[5], hi.z, lo.z);
        split_bf2(cur[6], cur[7], hi.w, lo.w);
        uint4 *o = reinterpret_cast<uint4 *>(x + (size_t)(c0 + u) * stride);
        o[0] = hi;
        o[1] = lo;
#pragma unroll
        for (int j = 0; j < 8; ++j) cur[j] = fmaf(k[u], cur[j], v[u][j]);
      }
  }
#pragma unroll
  for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4 *>(state + j) = *reinterpret_cast<const float4 *>(cur + j);
}

template <int NP, int CP> struct OutSmem {
  __nv_bfloat16 C[CHUNK][NP + 8], X[CHUNK][CP + 8], Sh[NP][CP + 8], Sl[NP][CP + 8];
  union {
    __nv_bfloat16 B[CHUNK][NP + 8];
    float ypart[4][16][CP + 4];     // the second warp's share of the output rows, once B is no longer needed
  };
  Decays d;
};
// Block: one chunk, one head, CP columns.  Two warps share 16 output rows, each with every other 16 state rows (first product) and
// every other 16 tokens s (second product).
template <int NP, int CP> __global__ void __launch_bounds__(CHUNK_THREADS) ssm_chunk_out_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  constexpr int XLD = CP + 8, BLD = NP + 8;
  extern __shared__ __align__(16) unsigned char smraw[];
  OutSmem<NP, CP> &sm = *reinterpret_cast<OutSmem<NP, CP> *>(smraw);
  const int slot = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CP;
  int s, t0;
  if (!chunk_of_slot(p.cu, p.n_seq, slot, s, t0)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int grp = h / (p.heads / p.groups), row0 = p.cu[s] + t0, valid = min(CHUNK, p.cu[s + 1] - row0);
  const T *xbc = reinterpret_cast<const T *>(p.xbc) + (size_t)row0 * p.C;
  for (int e = tid; e < CHUNK * (NP / 8); e += CHUNK_THREADS) {
    const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
    const bool in = r < valid && c < p.N;
    const T *row = xbc + (in ? (size_t)r * p.C + p.inner + grp * p.N + c : 0);
    cp16(&sm.B[r][c], row, in);
    cp16(&sm.C[r][c], row + (in ? p.groups * p.N : 0), in);
  }
  for (int e = tid; e < CHUNK * (CP / 8); e += CHUNK_THREADS) {
    const int r = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = r < valid && col0 + c < p.P;
    cp16(&sm.X[r][c], xbc + (in ? (size_t)r * p.C + (size_t)h * p.P + col0 + c : 0), in);
  }
  load_decays(p, slot, h, sm.d);
  const float *st = p.chunk_state + ((size_t)slot * p.heads + h) * p.N * p.P;
  for (int e = tid; e < NP * (CP / 8); e += CHUNK_THREADS) {
    const int n = e / (CP / 8), c = (e % (CP / 8)) * 8;
    const bool in = n < p.N && col0 + c < p.P;
    const float *src = st + (in ? (size_t)n * p.P + col0 + c : 0);
    cp16(&sm.Sh[n][c], src, in);
    cp16(&sm.Sl[n][c], src + 4, in);
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  const int rb = warp >> 1, half = warp & 1, tr = rb * 16 + g;      // this lane's output rows tr and tr + 8
  float y[CP / 8][4], G[2][2][4];
#pragma unroll
  for (int j = 0; j < CP / 8; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll
  for (int u = 0; u < 2; ++u)
#pragma unroll
    for (int j = 0; j < 2; ++j) G[u][j][0] = G[u][j][1] = G[u][j][2] = G[u][j][3] = 0.f;
  const uint32_t c_lane = smem_addr(&sm.C[rb * 16 + (lane & 15)][(lane >> 4) * 8]);
  // (B rows are the n side: matrices (s 0-7, k 0-7), (s 0-7, k 8-15), (s 8-15, k 0-7), (s 8-15, k 8-15))
  const uint32_t b_lane = smem_addr(&sm.B[half * 16 + (lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]);
  const uint32_t sh_lane = smem_addr(&sm.Sh[lane & 15][(lane >> 4) * 8]), sl_lane = smem_addr(&sm.Sl[lane & 15][(lane >> 4) * 8]);
#pragma unroll 2
  for (int kk = 0; kk < NP / 16; ++kk) {
    uint32_t a0, a1, a2, a3;
    ldsm4(c_lane + (uint32_t)kk * 32u, a0, a1, a2, a3);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      if (half + 2 * u > rb) break;     // tokens behind the diagonal only
      uint32_t b0, b1, b2, b3;
      ldsm4(b_lane + (uint32_t)(u * 32 * BLD + kk * 16) * 2u, b0, b1, b2, b3);
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
  const float e0 = sm.d.ec[tr], e1 = sm.d.ec[tr + 8];
#pragma unroll
  for (int j = 0; j < CP / 8; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
  const float h0 = sm.d.c_hi[tr], l0 = sm.d.c_lo[tr], h1 = sm.d.c_hi[tr + 8], l1 = sm.d.c_lo[tr + 8];
  const uint32_t x_lane = smem_addr(&sm.X[half * 16 + (lane & 15)][(lane >> 4) * 8]);
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int k2 = half + 2 * u;
    if (k2 > rb) break;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int sc = k2 * 16 + j * 8 + 2 * tig;
      const float2 ch = *reinterpret_cast<const float2 *>(&sm.d.c_hi[sc]), cl = *reinterpret_cast<const float2 *>(&sm.d.c_lo[sc]);
      const float2 dt = *reinterpret_cast<const float2 *>(&sm.d.dt[sc]);
      G[u][j][0] = sc <= tr ? G[u][j][0] * expf((h0 - ch.x) + (l0 - cl.x)) * dt.x : 0.f;
      G[u][j][1] = sc + 1 <= tr ? G[u][j][1] * expf((h0 - ch.y) + (l0 - cl.y)) * dt.y : 0.f;
      G[u][j][2] = sc <= tr + 8 ? G[u][j][2] * expf((h1 - ch.x) + (l1 - cl.x)) * dt.x : 0.f;
      G[u][j][3] = sc + 1 <= tr + 8 ? G[u][j][3] * expf((h1 - ch.y) + (l1 - cl.y)) * dt.y : 0.f;
    }
    uint32_t hi[4], lo[4];
    split_bf2(G[u][0][0], G[u][0][1], hi[0], lo[0]);
    split_bf2(G[u][0][2], G[u][0][3], hi[1], lo[1]);
    split_bf2(G[u][1][0], G[u][1][1], hi[2], lo[2]);
    split_bf2(G[u][1][2], G[u][1][3], hi[3], lo[3]);
#pragma unroll
    for (int j = 0; j < CP / 8; j += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm4t(x_lane + (uint32_t)(u * 32 * XLD + j * 8) * 2u, b0, b1, b2, b3);
      mma16816_bf16(y[j], hi[0], hi[1], hi[2], hi[3], b0, b1);
      mma16816_bf16(y[j + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
      mma16816_bf16(y[j], lo[0], lo[1], lo[2], lo[3], b0, b1);
      mma16816_bf16(y[j + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
    }
  }
  __syncthreads();   // B is no longer needed: its place takes the second warp's rows
  if (half) {
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) *reinterpret_cast<float2 *>(&sm.ypart[rb][g + 8 * r][j * 8 + 2 * tig]) = make_float2(y[j][2 * r], y[j][2 * r + 1]);
  }
  __syncthreads();
  if (half) return;
  const float D = p.D[h];
#pragma unroll
  for (int j = 0; j < CP / 8; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = tr + 8 * r, c = j * 8 + 2 * tig;
      if (t >= valid || col0 + c >= p.P) continue;
      const float2 o = *reinterpret_cast<const float2 *>(&sm.ypart[rb][g + 8 * r][c]);
      const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162 *>(&sm.X[t][c]);
      *reinterpret_cast<float2 *>(p.y + (size_t)(row0 + t) * p.inner + (size_t)h * p.P + col0 + c) =
          make_float2(fmaf(D, __low2float(x2), y[j][2 * r] + o.x), fmaf(D, __high2float(x2), y[j][2 * r + 1] + o.y));
    }
}

// ------------------------------------------------------------------------------------------ one token per sequence
constexpr int STEP_THREADS = 256;
// Block: one sequence and one head.  Thread (n group, column quad) walks state rows n group, + n groups, ...; every state element is
// read and written once, coalesced along the columns.
template <typename T, int VEC> __global__ void __launch_bounds__(STEP_THREADS) ssm_step_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  const int s = blockIdx.y, h = blockIdx.x, tid = threadIdx.x, g = h / (p.heads / p.groups);
  const int pos = p.start[s], slot = p.slot[s], t = p.cu[s];
  float *x = sm, *Bs = x + p.P, *Cs = Bs + p.N, *part = sm + (p.P + 2 * p.N + 3) / 4 * 4;   // part [n groups][P]
  const int pq = (p.P + VEC - 1) / VEC, ng = max(1, STEP_THREADS / pq);
  const int ngrp = tid / pq, q = tid - ngrp * pq;
  float *gS = p.state + ((size_t)slot * p.heads + h) * p.N * p.P;
  const T *zx = reinterpret_cast<const T *>(p.zx) + (size_t)t * p.zx_ld;
  const T *ring = reinterpret_cast<const T *>(p.ring) + (size_t)slot * p.taps * p.C;
  constexpr int U = 8;                    // state rows in flight per thread
  float v[U][VEC];
  auto load_rows = [&](int n0, int q0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int n = n0 + u * ng;
      if (n < p.N && pos > 0) {
        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(v[u]) = __ldcs(reinterpret_cast<const float4 *>(gS + (size_t)n * p.P + q0 * 4));
        else v[u][0] = gS[(size_t)n * p.P + q0];
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[u][j] = 0.f;
      }
    }
  };
  if (ngrp < ng && q < pq) load_rows(ngrp, q);   // on their way while the convolution is computed
  for (int i = tid; i < p.P + 2 * p.N; i += STEP_THREADS) {
    const int c = i < p.P ? h * p.P + i : (i < p.P + p.N ? p.inner + g * p.N + i - p.P : p.inner + (p.groups + g) * p.N + i - p.P - p.N);
    float a = p.conv_b[c];
    for (int k = 0; k < p.taps; ++k) {
      const int back = p.taps - 1 - k;
      float v = 0.f;
      if (back == 0) v = to_f(zx[p.inner + c]);
      else if (back <= pos) v = to_f(ring[(size_t)((pos - back) % p.taps) * p.C + c]);
      a = fmaf(p.conv_w[(size_t)c * p.taps + k], v, a);
    }
    sm[i] = silu_f(a);
  }
  const float dt = softplus_f(to_f(zx[p.inner + p.C + h]) + p.dt_bias[h]), decay = expf(-expf(p.A_log[h]) * dt);
  __syncthreads();
  for (int q0 = q; q0 < pq; q0 += STEP_THREADS) {     // (one trip unless a row of the state is wider than the block)
    if (ngrp >= ng) break;
    float y[VEC], dx[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) { y[j] = 0.f; dx[j] = dt * x[q0 * VEC + j]; }
    for (int n0 = ngrp; n0 < p.N; n0 += U * ng) {
      if (n0 != ngrp || q0 != q) load_rows(n0, q0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * ng;
        if (n >= p.N) break;
        const float b = Bs[n], c = Cs[n];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          v[u][j] = fmaf(decay, v[u][j], b * dx[j]);
          y[j] = fmaf(v[u][j], c, y[j]);
        }
        store_vec<VEC>(gS + (size_t)n * p.P + q0 * VEC, v[u]);
      }
    }
    store_vec<VEC>(part + (size_t)ngrp * p.P + q0 * VEC, y);
  }
  __syncthreads();
  const float D = p.D[h];
  for (int i = tid; i < p.P; i += STEP_THREADS) {
    float a = D * x[i];
    for (int k = 0; k < ng; ++k) a += part[(size_t)k * p.P + i];
    p.y[(size_t)t * p.inner + (size_t)h * p.P + i] = a;
  }
}

// ------------------------------------------------------------------------------------------ gate + group norm + ring
template <typename T, int VEC> __global__ void ssm_norm_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *gbuf = sm, *sums = sm + (p.inner + 3) / 4 * 4;     // gated row, then [norm_groups][warps per group]
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
  const int s = p.tok_seq[t], t0 = p.cu[s], t1 = p.cu[s + 1], pos = p.start[s] + t - t0;
  const T *zx = reinterpret_cast<const T *>(p.zx) + (size_t)t * p.zx_ld;
  const float *y = p.y + (size_t)t * p.inner;
  const int len = p.inner / p.norm_groups, wpg = p.norm_groups >= nw ? 1 : nw / p.norm_groups, gstep = nw / wpg;
  for (int g = warp / wpg; g < p.norm_groups; g += gstep) {
    if (warp >= wpg * gstep) break;
    float ss = 0.f;
    for (int i = ((warp % wpg) * 32 + lane) * VEC; i < len; i += wpg * 32 * VEC) {
      float v[VEC], z[VEC];
      load_vec<VEC>(y + g * len + i, v);
      load_vec<VEC>(zx + g * len + i, z);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        v[j] *= silu_f(z[j]);
        ss += v[j] * v[j];
      }
      store_vec<VEC>(gbuf + g * len + i, v);
    }
    ss = warp_sum(ss);
    if (lane == 0) sums[g * wpg + warp % wpg] = ss;
  }
  if (t >= t1 - p.taps) {   // the last `taps` raw convolution inputs of the sequence stay in its ring
    T *ring = reinterpret_cast<T *>(p.ring) + ((size_t)p.slot[s] * p.taps + pos % p.taps) * p.C;
    if constexpr (VEC == 4) {
      typedef typename std::conditional<sizeof(T) == 4, uint4, uint2>::type V;
#pragma unroll 4
      for (int c = tid; c < p.C / 4; c += blockDim.x) reinterpret_cast<V *>(ring)[c] = reinterpret_cast<const V *>(zx + p.inner)[c];
    } else {
      for (int c = tid; c < p.C; c += blockDim.x) ring[c] = zx[p.inner + c];
    }
  }
  __syncthreads();
  for (int g = tid; g < p.norm_groups; g += blockDim.x) {
    float a = 0.f;
    for (int k = 0; k < wpg; ++k) a += sums[g * wpg + k];
    sums[g * wpg] = 1.0f / sqrtf(a / (float)len + p.eps);
  }
  __syncthreads();
  T *out = reinterpret_cast<T *>(p.out) + (size_t)t * p.out_ld;
  for (int i = tid * VEC; i < p.inner; i += blockDim.x * VEC) {
    const float inv = sums[i / len * wpg];
    float v[VEC], w[VEC];
    load_vec<VEC>(gbuf + i, v);
    load_vec<VEC>(p.norm_w + i, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= inv * w[j];
    store_vec<VEC>(out + i, v);
  }
  for (int i = p.inner + tid; i < p.out_ld; i += blockDim.x) out[i] = from_f<T>(0.f);   // k padding of the output product
}

template <int NP, int CP> static int launch_chunks(const Params &p, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    PT_CUDA(cudaFuncSetAttribute(ssm_chunk_state_kernel<NP, CP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(StateSmem<NP, CP>)));
    PT_CUDA(cudaFuncSetAttribute(ssm_chunk_out_kernel<NP, CP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(OutSmem<NP, CP>)));
    set = true;
  }
  const dim3 grid(ceil_div(p.P, CP), p.heads, p.n_tok / CHUNK + p.n_seq);
  ssm_decay_kernel<<<dim3(ceil_div(p.heads, 4), grid.z), 128, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  ssm_chunk_state_kernel<NP, CP><<<grid, CHUNK_THREADS, sizeof(StateSmem<NP, CP>), st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  ssm_carry_kernel<<<dim3(ceil_div(p.N * p.P / 8, 64), p.heads, p.n_seq), 64, 0, st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  ssm_chunk_out_kernel<NP, CP><<<grid, CHUNK_THREADS, sizeof(OutSmem<NP, CP>), st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  return PT_OK;
}
template <int CP> static int dispatch_chunks(const Params &p, cudaStream_t st) {
  return p.N <= 64 ? launch_chunks<64, CP>(p, st) : (p.N <= 128 ? launch_chunks<128, CP>(p, st) : launch_chunks<256, CP>(p, st));
}

template <typename T> static int run(const Params &p, bool plain, cudaStream_t st) {
  if (p.n_tok == p.n_seq) {
    const bool v4 = p.P % 4 == 0 && p.P / 4 <= STEP_THREADS && aligned_to(p.state, 16);
    const int pq = v4 ? p.P / 4 : p.P, ng = std::max(1, STEP_THREADS / pq);
    const size_t smem = ((size_t)(p.P + 2 * p.N + 3) / 4 * 4 + (size_t)ng * p.P) * sizeof(float);
    PT_REQUIRE(smem <= 48 * 1024, "pt_ssm: head width %d and state %d need %zu bytes of shared memory", p.P, p.N, smem);
    const dim3 grid(p.heads, p.n_seq);
    if (v4) ssm_step_kernel<T, 4><<<grid, STEP_THREADS, smem, st>>>(p);
    else ssm_step_kernel<T, 1><<<grid, STEP_THREADS, smem, st>>>(p);
    PT_LAUNCH_CHECK("pt_ssm");
  } else {
    if (!plain && sizeof(T) == 2 && p.taps <= 4 && p.C % 8 == 0 && p.inner % 8 == 0 && p.zx_ld % 8 == 0 && aligned_to(p.zx, 16) && aligned_to(p.xbc, 16) && aligned_to(p.ring, 16) && aligned_to(p.conv_w, 16)) {
      const dim3 grid(ceil_div(p.C / 8, CONV_THREADS) + 1, ceil_div(p.n_tok, CONV_TOKENS));
      switch (p.taps) {
        case 1: ssm_conv8_kernel<1><<<grid, CONV_THREADS, 0, st>>>(p); break;
        case 2: ssm_conv8_kernel<2><<<grid, CONV_THREADS, 0, st>>>(p); break;
        case 3: ssm_conv8_kernel<3><<<grid, CONV_THREADS, 0, st>>>(p); break;
        default: ssm_conv8_kernel<4><<<grid, CONV_THREADS, 0, st>>>(p); break;
      }
    } else {
      ssm_conv_kernel<T><<<dim3(ceil_div(p.C + p.heads, 256), p.n_tok), 256, 0, st>>>(p);
    }
    PT_LAUNCH_CHECK("pt_ssm");
    // the chunked form: bf16, rows that are whole 16-byte units, state of at most 256, with its scratch
    if (!plain && sizeof(T) == 2 && p.chunk_state && aligned_to(p.state, 16) && p.N <= 256 && p.N % 8 == 0 && p.P % 8 == 0 && aligned_to(p.xbc, 16) && aligned_to(p.y, 8)) {
      const int rc = p.P <= 32 ? dispatch_chunks<32>(p, st) : dispatch_chunks<64>(p, st);
      if (rc != PT_OK) return rc;
    } else {
      const size_t smem = ((size_t)p.N * SCAN_P + 2 * p.N + SCAN_WARPS * 32) * sizeof(float);
      PT_REQUIRE(smem <= 200 * 1024, "pt_ssm: state %d needs %zu bytes of shared memory", p.N, smem);
      if (smem > 48 * 1024) PT_CUDA(cudaFuncSetAttribute(ssm_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      ssm_scan_kernel<T><<<dim3(ceil_div(p.P, SCAN_P), p.heads, p.n_seq), SCAN_WARPS * 32, smem, st>>>(p);
      PT_LAUNCH_CHECK("pt_ssm");
    }
  }
  const int len = p.inner / p.norm_groups;
  const bool v4 = len % 4 == 0 && p.C % 4 == 0 && p.zx_ld % 4 == 0 && p.out_ld % 4 == 0 && aligned_to(p.out, 4 * sizeof(T)) && aligned_to(p.zx, 4 * sizeof(T)) &&
                  aligned_to(p.ring, 4 * sizeof(T)) && aligned_to(p.y, 16) && aligned_to(p.norm_w, 16);
  // few rows: as many threads per row as it has work for (the launch is one chain of latencies); many rows: more rows per SM
  const int threads = p.n_tok <= 2 * sm_count() ? std::min(1024, std::max(128, ceil_div(p.inner / (v4 ? 4 : 1), 32) * 32)) : 256;
  const size_t smem = ((size_t)(p.inner + 3) / 4 * 4 + (size_t)std::max(p.norm_groups, threads / 32)) * sizeof(float);
  PT_REQUIRE(smem <= 200 * 1024, "pt_ssm: inner width %d needs %zu bytes of shared memory", p.inner, smem);
  if (smem > 48 * 1024) {
    PT_CUDA(cudaFuncSetAttribute(ssm_norm_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    PT_CUDA(cudaFuncSetAttribute(ssm_norm_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  }
  if (v4) ssm_norm_kernel<T, 4><<<p.n_tok, threads, smem, st>>>(p);
  else ssm_norm_kernel<T, 1><<<p.n_tok, threads, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  return PT_OK;
}

}  // namespace ssm
}  // namespace pt

using namespace pt;

extern "C" size_t pt_ssm_workspace_bytes(int n_tok, int n_seq, int heads, int vdim, int state_dim) {
  const size_t slots = (size_t)n_tok / CHUNK + n_seq;
  return slots * heads * ((size_t)state_dim * vdim * sizeof(float) + sizeof(ssm::Decays)) + 16;
}

extern "C" int pt_ssm(const pt_ssm_args *a, void *stream) {
  PT_REQUIRE(a, "pt_ssm: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(b.n_seq > 0 && b.n_tok >= b.n_seq && b.n_tok <= 65535 && b.cu && b.start && b.slot && b.tok_seq, "pt_ssm: bad batch (%d sequences, %d tokens)",
             b.n_seq, b.n_tok);
  PT_REQUIRE(a->heads > 0 && a->vdim > 0 && a->state_dim > 0 && a->groups > 0 && a->heads % a->groups == 0 && a->taps >= 1,
             "pt_ssm: bad shape heads=%d vdim=%d state=%d groups=%d taps=%d", a->heads, a->vdim, a->state_dim, a->groups, a->taps);
  const int inner = a->heads * a->vdim, C = inner + 2 * a->groups * a->state_dim;
  PT_REQUIRE(a->norm_groups > 0 && inner % a->norm_groups == 0, "pt_ssm: norm_groups=%d does not divide inner=%d", a->norm_groups, inner);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_ssm: type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->zx && a->conv_w && a->conv_b && a->dt_bias && a->A_log && a->D && a->norm_w && a->ring && a->state && a->y && a->out,
             "pt_ssm: null pointer argument");
  PT_REQUIRE(b.n_tok == b.n_seq || (a->xbc && a->dt), "pt_ssm: a prompt needs the xbc and dt scratch");
  PT_REQUIRE(a->zx_ld >= inner + C + a->heads && a->out_ld >= inner, "pt_ssm: row strides zx %d, out %d too small", a->zx_ld, a->out_ld);
  ssm::Params p{};
  p.n_seq = b.n_seq; p.n_tok = b.n_tok; p.heads = a->heads; p.P = a->vdim; p.N = a->state_dim; p.groups = a->groups; p.taps = a->taps;
  p.norm_groups = a->norm_groups; p.C = C; p.inner = inner; p.zx_ld = a->zx_ld; p.out_ld = a->out_ld; p.eps = a->eps;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq;
  p.zx = a->zx; p.conv_w = a->conv_w; p.conv_b = a->conv_b; p.dt_bias = a->dt_bias; p.A_log = a->A_log; p.D = a->D; p.norm_w = a->norm_w;
  p.ring = a->ring; p.xbc = a->xbc; p.out = a->out; p.state = a->state; p.dt = a->dt; p.y = a->y;
  if (a->workspace && ((uintptr_t)a->workspace & 15) == 0 && a->workspace_bytes >= pt_ssm_workspace_bytes(b.n_tok, b.n_seq, a->heads, a->vdim, a->state_dim)) {
    p.chunk_state = (float *)a->workspace;
    const size_t n = ((size_t)b.n_tok / CHUNK + b.n_seq) * a->heads * a->state_dim * a->vdim;
    p.chunk_decays = (ssm::Decays *)(p.chunk_state + (n + 3) / 4 * 4);
  }
  return a->dtype == PT_DT_F32 ? ssm::run<float>(p, a->plain != 0, as_stream(stream)) : ssm::run<__nv_bfloat16>(p, a->plain != 0, as_stream(stream));
}
