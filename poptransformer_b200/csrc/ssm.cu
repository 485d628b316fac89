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
//   ssm_chunk_kernel   bf16 prompts: the same recurrence 64 tokens at a time on the tensor cores
//   ssm_step_kernel    one token per sequence: convolution, step size, state update and readout in one launch
//   ssm_norm_kernel    gate, group norm, and the ring update
#include "elem.cuh"
#include "tile_math.cuh"

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
// Block: 32 columns of one head's state, one sequence; it walks the chunks in order with the state in fp32 accumulators.  Operands
// that are not already bf16 (the state, the decayed products, the weighted x) enter the tensor cores as hi + lo pairs.  c is kept
// as a pair of floats, so differences of neighbours stay exact however far the sum has run.
// NP: state size rounded up to 64, 128 or 256 (padding is zero).
constexpr int CHUNK = 64, CP = 32, CHUNK_THREADS = 128;
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void cp16(void *dst, const void *src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
template <int NP> struct ChunkSmem {
  static constexpr int BLD = NP + 8, XLD = CP + 8;
  __nv_bfloat16 B[2][CHUNK][BLD], C[2][CHUNK][BLD], X[2][CHUNK][XLD];
  __nv_bfloat16 Sh[NP][XLD], Sl[NP][XLD];      // state before the chunk, hi and lo
  __nv_bfloat16 Wh[CHUNK][XLD], Wl[CHUNK][XLD];   // exp(c_last - c_s) dt_s x_s
  float c_hi[CHUNK], c_lo[CHUNK], dt[CHUNK];
};

template <int NP> __global__ void __launch_bounds__(CHUNK_THREADS) ssm_chunk_kernel(const Params p) {
  typedef __nv_bfloat16 T;
  constexpr int MT = NP / 64;                       // 16-row tiles of the state per warp
  extern __shared__ __align__(16) unsigned char smraw[];
  ChunkSmem<NP> &sm = *reinterpret_cast<ChunkSmem<NP> *>(smraw);
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CP;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tig = lane & 3;
  const int grp = h / (p.heads / p.groups);
  const int row0 = p.cu[s], len = p.cu[s + 1] - row0;
  const T *xbc = reinterpret_cast<const T *>(p.xbc) + (size_t)row0 * p.C;
  const float a = -expf(p.A_log[h]), D = p.D[h];
  float *gS = p.state + ((size_t)p.slot[s] * p.heads + h) * p.N * p.P;

  auto load_chunk = [&](int t0, int stage) {
    for (int e = tid; e < CHUNK * (NP / 8); e += CHUNK_THREADS) {
      const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
      const bool in = t0 + r < len && c < p.N;
      const T *row = xbc + (in ? (size_t)(t0 + r) * p.C + p.inner + grp * p.N + c : 0);
      cp16(&sm.B[stage][r][c], row, in);
      cp16(&sm.C[stage][r][c], row + (in ? p.groups * p.N : 0), in);
    }
    for (int e = tid; e < CHUNK * (CP / 8); e += CHUNK_THREADS) {
      const int r = e / (CP / 8), c = (e % (CP / 8)) * 8;
      const bool in = t0 + r < len && col0 + c < p.P;
      cp16(&sm.X[stage][r][c], xbc + (in ? (size_t)(t0 + r) * p.C + (size_t)h * p.P + col0 + c : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_chunk(0, 0);

  // state accumulators: warp w owns rows w NP / 4 ..; tile i, column tile j, lane (g, tig): rows g and g + 8, columns 2 tig, + 1
  float S[MT][CP / 8][4];
  const int srow = warp * (NP / 4) + g;
  const bool fresh = p.start[s] == 0;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = srow + i * 16 + 8 * (e >> 1), c = col0 + j * 8 + 2 * tig + (e & 1);
        S[i][j][e] = (!fresh && n < p.N && c < p.P) ? gS[(size_t)n * p.P + c] : 0.f;
      }
  auto publish_state = [&]() {
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split_bf2(S[i][j][2 * r], S[i][j][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t *>(&sm.Sh[srow + i * 16 + 8 * r][j * 8 + 2 * tig]) = hi;
          *reinterpret_cast<uint32_t *>(&sm.Sl[srow + i * 16 + 8 * r][j * 8 + 2 * tig]) = lo;
        }
  };
  publish_state();

  int stage = 0;
  for (int t0 = 0; t0 < len; t0 += CHUNK, stage ^= 1) {
    if (t0 + CHUNK < len) {
      load_chunk(t0 + CHUNK, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    if (warp == 0) {   // step sizes and running log decays of the chunk (zero beyond the sequence: decay 1, no contribution)
      const int r0 = t0 + 2 * lane, r1 = r0 + 1;
      const float d0 = r0 < len ? p.dt[(size_t)(row0 + r0) * p.heads + h] : 0.f, d1 = r1 < len ? p.dt[(size_t)(row0 + r1) * p.heads + h] : 0.f;
      const double l0 = (double)(a * d0), l1 = (double)(a * d1);
      double sum = l0 + l1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
      }
      const double c1 = sum, c0 = sum - l1;
      sm.dt[2 * lane] = d0; sm.dt[2 * lane + 1] = d1;
      sm.c_hi[2 * lane] = (float)c0; sm.c_lo[2 * lane] = (float)(c0 - (double)(float)c0);
      sm.c_hi[2 * lane + 1] = (float)c1; sm.c_lo[2 * lane + 1] = (float)(c1 - (double)(float)c1);
    }
    __syncthreads();   // operands, step sizes and the published state are in shared memory
    const float ce_hi = sm.c_hi[CHUNK - 1], ce_lo = sm.c_lo[CHUNK - 1];
    for (int e = tid; e < CHUNK * (CP / 2); e += CHUNK_THREADS) {   // weighted x for the state update
      const int r = e / (CP / 2), c = (e % (CP / 2)) * 2;
      const float w = expf((ce_hi - sm.c_hi[r]) + (ce_lo - sm.c_lo[r])) * sm.dt[r];
      const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162 *>(&sm.X[stage][r][c]);
      uint32_t hi, lo;
      split_bf2(w * __low2float(x2), w * __high2float(x2), hi, lo);
      *reinterpret_cast<uint32_t *>(&sm.Wh[r][c]) = hi;
      *reinterpret_cast<uint32_t *>(&sm.Wl[r][c]) = lo;
    }
    // ---- rows 16 warp .. + 15 of the chunk's output
    const int tr = warp * 16 + g;
    float y[CP / 8][4], G[CHUNK / 8][4];
#pragma unroll
    for (int j = 0; j < CP / 8; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < CHUNK / 8; ++j) G[j][0] = G[j][1] = G[j][2] = G[j][3] = 0.f;
    const uint32_t sh_lane = smem_addr(&sm.Sh[lane & 15][(lane >> 4) * 8]), sl_lane = smem_addr(&sm.Sl[lane & 15][(lane >> 4) * 8]);
#pragma unroll 2
    for (int kk = 0; kk < NP / 16; ++kk) {
      const T *c0 = &sm.C[stage][tr][kk * 16 + 2 * tig], *c1 = &sm.C[stage][tr + 8][kk * 16 + 2 * tig];
      const uint32_t a0 = *reinterpret_cast<const uint32_t *>(c0), a1 = *reinterpret_cast<const uint32_t *>(c1);
      const uint32_t a2 = *reinterpret_cast<const uint32_t *>(c0 + 8), a3 = *reinterpret_cast<const uint32_t *>(c1 + 8);
#pragma unroll
      for (int j = 0; j < CHUNK / 8; ++j) {
        if (j > 2 * warp + 1) break;      // columns behind the diagonal only
        const T *b = &sm.B[stage][j * 8 + g][kk * 16 + 2 * tig];
        mma16816_bf16(G[j], a0, a1, a2, a3, *reinterpret_cast<const uint32_t *>(b), *reinterpret_cast<const uint32_t *>(b + 8));
      }
#pragma unroll
      for (int j = 0; j < CP / 8; j += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm4t(sh_lane + (uint32_t)(kk * 16 * ChunkSmem<NP>::XLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(y[j], a0, a1, a2, a3, b0, b1);
        mma16816_bf16(y[j + 1], a0, a1, a2, a3, b2, b3);
        ldsm4t(sl_lane + (uint32_t)(kk * 16 * ChunkSmem<NP>::XLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(y[j], a0, a1, a2, a3, b0, b1);
        mma16816_bf16(y[j + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    const float h0 = sm.c_hi[tr], l0 = sm.c_lo[tr], h1 = sm.c_hi[tr + 8], l1 = sm.c_lo[tr + 8];
    const float e0 = expf(h0 + l0), e1 = expf(h1 + l1);
#pragma unroll
    for (int j = 0; j < CP / 8; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
#pragma unroll
    for (int j = 0; j < CHUNK / 8; ++j) {
      if (j > 2 * warp + 1) break;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int sc = j * 8 + 2 * tig + (e & 1), t = e < 2 ? tr : tr + 8;
        const float d = e < 2 ? (h0 - sm.c_hi[sc]) + (l0 - sm.c_lo[sc]) : (h1 - sm.c_hi[sc]) + (l1 - sm.c_lo[sc]);
        G[j][e] = sc <= t ? G[j][e] * expf(d) * sm.dt[sc] : 0.f;
      }
    }
    const uint32_t x_lane = smem_addr(&sm.X[stage][lane & 15][(lane >> 4) * 8]);
#pragma unroll
    for (int k2 = 0; k2 < CHUNK / 16; ++k2) {
      if (k2 > warp) break;
      uint32_t hi[4], lo[4];
      split_bf2(G[2 * k2][0], G[2 * k2][1], hi[0], lo[0]);
      split_bf2(G[2 * k2][2], G[2 * k2][3], hi[1], lo[1]);
      split_bf2(G[2 * k2 + 1][0], G[2 * k2 + 1][1], hi[2], lo[2]);
      split_bf2(G[2 * k2 + 1][2], G[2 * k2 + 1][3], hi[3], lo[3]);
#pragma unroll
      for (int j = 0; j < CP / 8; j += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm4t(x_lane + (uint32_t)(k2 * 16 * ChunkSmem<NP>::XLD + j * 8) * 2u, b0, b1, b2, b3);
        mma16816_bf16(y[j], hi[0], hi[1], hi[2], hi[3], b0, b1);
        mma16816_bf16(y[j + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
        mma16816_bf16(y[j], lo[0], lo[1], lo[2], lo[3], b0, b1);
        mma16816_bf16(y[j + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
      }
    }
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = tr + 8 * r, c = j * 8 + 2 * tig;
        if (t0 + t >= len || col0 + c >= p.P) continue;
        const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162 *>(&sm.X[stage][t][c]);
        *reinterpret_cast<float2 *>(p.y + (size_t)(row0 + t0 + t) * p.inner + (size_t)h * p.P + col0 + c) =
            make_float2(fmaf(D, __low2float(x2), y[j][2 * r]), fmaf(D, __high2float(x2), y[j][2 * r + 1]));
      }
    __syncthreads();   // the weighted x is complete; nobody reads the old state any more
    // ---- state update: B^T [state rows x tokens] times the weighted x
    const float keep = expf(ce_hi + ce_lo);
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= keep;
    const uint32_t wh_lane = smem_addr(&sm.Wh[lane & 15][(lane >> 4) * 8]), wl_lane = smem_addr(&sm.Wl[lane & 15][(lane >> 4) * 8]);
#pragma unroll
    for (int k2 = 0; k2 < CHUNK / 16; ++k2) {
      uint32_t wh[CP / 8][2], wl[CP / 8][2];
#pragma unroll
      for (int j = 0; j < CP / 8; j += 2) {
        ldsm4t(wh_lane + (uint32_t)(k2 * 16 * ChunkSmem<NP>::XLD + j * 8) * 2u, wh[j][0], wh[j][1], wh[j + 1][0], wh[j + 1][1]);
        ldsm4t(wl_lane + (uint32_t)(k2 * 16 * ChunkSmem<NP>::XLD + j * 8) * 2u, wl[j][0], wl[j][1], wl[j + 1][0], wl[j + 1][1]);
      }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        // A fragment (rows = state, k = tokens) from the token-major tile: matrices (tokens 0-7 | 8-15) x (state 0-7 | 8-15), transposed
        uint32_t a0, a1, a2, a3;
        ldsm4t(smem_addr(&sm.B[stage][k2 * 16 + (lane & 7) + (lane >> 4) * 8][warp * (NP / 4) + i * 16 + ((lane >> 3) & 1) * 8]), a0, a1, a2, a3);
#pragma unroll
        for (int j = 0; j < CP / 8; ++j) {
          mma16816_bf16(S[i][j], a0, a1, a2, a3, wh[j][0], wh[j][1]);
          mma16816_bf16(S[i][j], a0, a1, a2, a3, wl[j][0], wl[j][1]);
        }
      }
    }
    publish_state();
    __syncthreads();   // this stage of the operands may be refilled
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = srow + i * 16 + 8 * (e >> 1), c = col0 + j * 8 + 2 * tig + (e & 1);
        if (n < p.N && c < p.P) gS[(size_t)n * p.P + c] = S[i][j][e];
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
    constexpr int U = 4;
    for (int n0 = ngrp; n0 < p.N; n0 += U * ng) {
      float v[U][VEC];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * ng;
        if (n < p.N && pos > 0) {
          if constexpr (VEC == 4) *reinterpret_cast<float4 *>(v[u]) = *reinterpret_cast<const float4 *>(gS + (size_t)n * p.P + q0 * 4);
          else v[u][0] = gS[(size_t)n * p.P + q0];
        } else {
#pragma unroll
          for (int j = 0; j < VEC; ++j) v[u][j] = 0.f;
        }
      }
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
      float v[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        v[j] = y[g * len + i + j] * silu_f(to_f(zx[g * len + i + j]));
        ss += v[j] * v[j];
      }
      store_vec<VEC>(gbuf + g * len + i, v);
    }
    ss = warp_sum(ss);
    if (lane == 0) sums[g * wpg + warp % wpg] = ss;
  }
  if (t >= t1 - p.taps) {   // the last `taps` raw convolution inputs of the sequence stay in its ring
    T *ring = reinterpret_cast<T *>(p.ring) + ((size_t)p.slot[s] * p.taps + pos % p.taps) * p.C;
    for (int c = tid; c < p.C; c += blockDim.x) ring[c] = zx[p.inner + c];
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
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = gbuf[i + j] * inv * p.norm_w[i + j];
    store_vec<VEC>(out + i, v);
  }
  for (int i = p.inner + tid; i < p.out_ld; i += blockDim.x) out[i] = from_f<T>(0.f);   // k padding of the output product
}

static bool al(const void *q, int bytes) { return ((uintptr_t)q & (bytes - 1)) == 0; }

template <int NP> static int launch_chunk(const Params &p, cudaStream_t st) {
  static bool set = false;
  if (!set) { PT_CUDA(cudaFuncSetAttribute(ssm_chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(ChunkSmem<NP>))); set = true; }
  ssm_chunk_kernel<NP><<<dim3(ceil_div(p.P, CP), p.heads, p.n_seq), CHUNK_THREADS, sizeof(ChunkSmem<NP>), st>>>(p);
  PT_LAUNCH_CHECK("pt_ssm");
  return PT_OK;
}

template <typename T> static int run(const Params &p, bool plain, cudaStream_t st) {
  if (p.n_tok == p.n_seq) {
    const bool v4 = p.P % 4 == 0 && p.P / 4 <= STEP_THREADS && al(p.state, 16);
    const int pq = v4 ? p.P / 4 : p.P, ng = std::max(1, STEP_THREADS / pq);
    const size_t smem = ((size_t)(p.P + 2 * p.N + 3) / 4 * 4 + (size_t)ng * p.P) * sizeof(float);
    PT_REQUIRE(smem <= 48 * 1024, "pt_ssm: head width %d and state %d need %zu bytes of shared memory", p.P, p.N, smem);
    const dim3 grid(p.heads, p.n_seq);
    if (v4) ssm_step_kernel<T, 4><<<grid, STEP_THREADS, smem, st>>>(p);
    else ssm_step_kernel<T, 1><<<grid, STEP_THREADS, smem, st>>>(p);
    PT_LAUNCH_CHECK("pt_ssm");
  } else {
    ssm_conv_kernel<T><<<dim3(ceil_div(p.C + p.heads, 256), p.n_tok), 256, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_ssm");
    // the chunked form: bf16, rows that are whole 16-byte units, state of at most 256
    if (!plain && sizeof(T) == 2 && p.N <= 256 && p.N % 8 == 0 && p.P % 8 == 0 && al(p.xbc, 16) && al(p.y, 8)) {
      const int rc = p.N <= 64 ? launch_chunk<64>(p, st) : (p.N <= 128 ? launch_chunk<128>(p, st) : launch_chunk<256>(p, st));
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
  const bool v4 = len % 4 == 0 && al(p.out, 4 * sizeof(T)) && p.out_ld % 4 == 0;
  const int threads = 256;
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
  return a->dtype == PT_DT_F32 ? ssm::run<float>(p, a->plain != 0, as_stream(stream)) : ssm::run<__nv_bfloat16>(p, a->plain != 0, as_stream(stream));
}
