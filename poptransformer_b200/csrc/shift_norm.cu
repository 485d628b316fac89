// Residual step of layers that read two norms of the stream, one of them mixed with the token before:
//     x <- x + y            n(x) = x / rms of its group             h1 = a + (a' - a) * shift,  a = n(x) w1        h2 = n(x) w2
// a' is the a of the same sequence's token before: the row above, or the sequence's state (zeros at position 0), which takes the a of
// the last new token.  y is a dense output plus the weighted outputs of the experts a token went to; an expert without a row gave the
// feed-forward's input back.  The kernel also starts a token (x = n(embedding row) w) and ends the model (h2 only).
//
// A block takes a run of rows.  For the row above the first one it computes the sum again from the same inputs (which is why x_out is
// another buffer than x_in), so no block waits for another.  All of it is fp32; only h1 and h2 are rounded.
//   rows_kernel        four columns per thread: a row lives in registers while the next one's loads are on their way, the a of the row
//                      above stays where it is, and weights are read once per run.  Groups in units of 128 columns (a warp's share)
//   shift_norm_kernel  any width and groups: the run's rows in shared memory, a warp sums the squares of a part of a group at a time
#include <type_traits>

#include "elem.cuh"

namespace pt {
namespace shift {

constexpr int kMaxTop = 64, kMaxRun = 4, kRows = kMaxRun + 1, kMaxFastRun = 16;

struct Params {
  int rows, width, groups, part, run, segs, h1_ld, h2_ld, table_ld, vocab, ids_ld, y_ld, pair_ld, top, self_ld;   // part: columns of a group; segs: warps' shares of one
  float eps;
  const float *x_in;
  float *x_out;
  const void *table;
  const int *ids, *step;
  int *pos_out;
  const float *embed_w;
  const int *row_index;
  const float *y, *pair_w;
  const void *pair_y, *self;
  const int *pair_row;
  const float *w1, *shift, *w2, *state_in;
  float *state_out;
  bool by_seq;
  void *h1, *h2;
  const int *cu, *start, *slot, *tok_seq;
};

// 1 / rms of every group of the n rows in shared memory, into inv [n][groups]; `red` holds n * groups * segs sums.
template <int VEC> __device__ __forceinline__ void group_rms(const Params &p, int n, const float *x, float *red, float *inv) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5, units = n * p.groups * p.segs;
  const int per = ((p.part + p.segs - 1) / p.segs + VEC - 1) / VEC * VEC;
  __syncthreads();
  for (int u = warp; u < units; u += warps) {
    const int seg = u % p.segs, rg = u / p.segs, b = seg * per, e = min(p.part, b + per);       // rg: row and group
    const float *src = x + (size_t)(rg / p.groups) * p.width + (rg % p.groups) * p.part;
    float ss = 0.f;
    for (int i = b + lane * VEC; i < e; i += 32 * VEC) {
      float v[VEC];
      load_vec<VEC>(src + i, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[u] = ss;
  }
  __syncthreads();
  for (int rg = threadIdx.x; rg < n * p.groups; rg += blockDim.x) {
    float ss = 0.f;
    for (int s = 0; s < p.segs; ++s) ss += red[rg * p.segs + s];
    inv[rg] = 1.0f / sqrtf(ss / (float)p.part + p.eps);
  }
  __syncthreads();
}

enum { ABOVE = 0, STATE = 1, NOTHING = 2 };      // where a row's a' comes from
template <typename T, typename E, int VEC, bool START> __global__ void __launch_bounds__(1024) shift_norm_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float pw[kRows * kMaxTop];
  __shared__ int pr[kRows * kMaxTop], before[kRows], from[kRows], to[kRows];
  launch_dependents();
  const int tid = threadIdx.x, r0 = blockIdx.x * p.run, r1 = min(p.rows, r0 + p.run);
  const bool mix = p.h1 != nullptr;
  const int lead = mix && r0 > p.cu[p.tok_seq[r0]] ? 1 : 0, base = r0 - lead, n = r1 - base;   // rows base .. base + n - 1, the first of them for its a only
  float *x = sm, *inv = x + (size_t)(p.run + (mix ? 1 : 0)) * p.width, *red = inv + (p.run + (mix ? 1 : 0)) * p.groups;
  for (int i = tid; i < n * p.top; i += blockDim.x) {
    const int r = base + i / p.top;
    const size_t k = (size_t)(p.row_index ? p.row_index[r] : r) * p.top + i % p.top;
    pw[i] = p.pair_w ? p.pair_w[k] : 1.f;
    pr[i] = p.pair_row ? p.pair_row[k] : (int)k;
  }
  if (mix && tid < n) {
    const int r = base + tid, s = p.tok_seq[r];
    const int first = p.cu[s], at = START && p.step ? *p.step : p.start[s];
    before[tid] = r > first ? ABOVE : at > 0 ? STATE : NOTHING;
    from[tid] = p.slot[s];
    to[tid] = r >= r0 && r + 1 == p.cu[s + 1] ? (p.by_seq ? s : p.slot[s]) : -1;
  }
  __syncthreads();
  auto id_of = [&](int r) { return min(max(p.ids[(size_t)r * p.ids_ld + (p.step ? *p.step : 0)], 0), p.vocab - 1); };
  for (int i = 0; i < n; ++i) {
    const int r = base + i, src = p.row_index ? p.row_index[r] : r;
    const T *emb = START ? reinterpret_cast<const T *>(p.table) + (size_t)id_of(r) * p.table_ld : nullptr;
    if (START && tid == 0 && r >= r0 && p.pos_out) p.pos_out[r] = p.step ? *p.step : 0;
    for (int c = tid * VEC; c < p.width; c += blockDim.x * VEC) {
      float v[VEC];
      if (START) {
        load_vec<VEC>(emb + c, v);
      } else {
        load_vec<VEC>(p.x_in + (size_t)src * p.width + c, v);
        if (p.y) {
          float a[VEC];
          load_vec<VEC>(p.y + (size_t)src * p.y_ld + c, a);
#pragma unroll 4
          for (int k = 0; k < p.top; ++k) {
            float e[VEC];
            const int row = pr[i * p.top + k];
            if (row < 0 && !p.self) continue;
            if (row < 0) load_vec<VEC>(reinterpret_cast<const T *>(p.self) + (size_t)src * p.self_ld + c, e);
            else load_vec<VEC>(reinterpret_cast<const E *>(p.pair_y) + (size_t)row * p.pair_ld + c, e);
            const float w = pw[i * p.top + k];
#pragma unroll
            for (int j = 0; j < VEC; ++j) a[j] = fmaf(w, e[j], a[j]);
          }
#pragma unroll
          for (int j = 0; j < VEC; ++j) v[j] += a[j];
        }
        if (p.x_out && r >= r0) store_vec<VEC>(p.x_out + (size_t)r * p.width + c, v);
      }
      store_vec<VEC>(x + (size_t)i * p.width + c, v);
    }
  }
  if (START) {
    group_rms<VEC>(p, n, x, red, inv);
    for (int i = 0; i < n; ++i)
      for (int c = tid * VEC; c < p.width; c += blockDim.x * VEC) {
        float v[VEC], w[VEC];
        load_vec<VEC>(x + (size_t)i * p.width + c, v);
        load_vec<VEC>(p.embed_w + c, w);
        const float f = inv[i * p.groups + c / p.part];
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] *= f * w[j];
        store_vec<VEC>(x + (size_t)i * p.width + c, v);
        if (p.x_out && base + i >= r0) store_vec<VEC>(p.x_out + (size_t)(base + i) * p.width + c, v);
      }
  }
  if (!mix && !p.h2) return;
  group_rms<VEC>(p, n, x, red, inv);
  for (int c = tid * VEC; c < p.width; c += blockDim.x * VEC) {
    const int g = c / p.part;
    float w1[VEC], w2[VEC], share[VEC], above[VEC];
    if (mix) {
      load_vec<VEC>(p.w1 + c, w1);
      load_vec<VEC>(p.shift + c, share);
    }
    if (p.h2) load_vec<VEC>(p.w2 + c, w2);
#pragma unroll
    for (int j = 0; j < VEC; ++j) above[j] = 0.f;
    for (int i = 0; i < n; ++i) {
      const int r = base + i;
      const float f = inv[i * p.groups + g];
      float v[VEC], o[VEC];
      load_vec<VEC>(x + (size_t)i * p.width + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= f;
      if (p.h2 && r >= r0) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) o[j] = v[j] * w2[j];
        store_vec<VEC>(reinterpret_cast<T *>(p.h2) + (size_t)r * p.h2_ld + c, o);
      }
      if (!mix) continue;
      if (before[i] == STATE) {
        load_vec<VEC>(p.state_in + (size_t)from[i] * p.width + c, above);
      } else if (before[i] == NOTHING) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) above[j] = 0.f;
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= w1[j];
      if (r >= r0) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) o[j] = fmaf(above[j] - v[j], share[j], v[j]);
        store_vec<VEC>(reinterpret_cast<T *>(p.h1) + (size_t)r * p.h1_ld + c, o);
        if (to[i] >= 0) store_vec<VEC>(p.state_out + (size_t)to[i] * p.width + c, v);
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) above[j] = v[j];
    }
  }
  for (int r = r0; r < r1; ++r) {                // k padding of the next products
    if (mix)
      for (int c = p.width + tid; c < p.h1_ld; c += blockDim.x) reinterpret_cast<T *>(p.h1)[(size_t)r * p.h1_ld + c] = from_f<T>(0.f);
    if (p.h2)
      for (int c = p.width + tid; c < p.h2_ld; c += blockDim.x) reinterpret_cast<T *>(p.h2)[(size_t)r * p.h2_ld + c] = from_f<T>(0.f);
  }
}

__device__ __forceinline__ void fetch4(const float *p, float4 &v) { v = *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ void fetch4(const __nv_bfloat16 *p, uint2 &v) { v = *reinterpret_cast<const uint2 *>(p); }
__device__ __forceinline__ void add4(float (&a)[4], float w, const float4 &v) {
  a[0] = fmaf(w, v.x, a[0]); a[1] = fmaf(w, v.y, a[1]); a[2] = fmaf(w, v.z, a[2]); a[3] = fmaf(w, v.w, a[3]);
}
__device__ __forceinline__ void add4(float (&a)[4], float w, const uint2 &v) {
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&v.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&v.y));
  a[0] = fmaf(w, lo.x, a[0]); a[1] = fmaf(w, lo.y, a[1]); a[2] = fmaf(w, hi.x, a[2]); a[3] = fmaf(w, hi.y, a[3]);
}
template <typename T> struct Raw4 { typedef float4 type; };
template <> struct Raw4<__nv_bfloat16> { typedef uint2 type; };

constexpr int CHUNK = 128;                       // columns of a warp
template <typename T, bool START> __global__ void __launch_bounds__(1024) rows_kernel(const Params p) {
  __shared__ __align__(16) float pw[(kMaxFastRun + 1) * kMaxTop];      // every row's pairs, in fours (of the last four the rest repeats a row with weight 0)
  __shared__ __align__(16) int pr[(kMaxFastRun + 1) * kMaxTop];
  __shared__ float red[2][32];
  __shared__ int before[kMaxFastRun + 1], from[kMaxFastRun + 1], to[kMaxFastRun + 1];
  launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, c = tid * 4, r0 = blockIdx.x * p.run, r1 = min(p.rows, r0 + p.run);
  const bool mix = p.h1 != nullptr;
  const int lead = mix && p.run > 1 && r0 > p.cu[p.tok_seq[r0]] ? 1 : 0, base = r0 - lead, n = r1 - base;      // (a run of one row: every sequence brings one token)
  auto source = [&](int i) { return p.row_index ? p.row_index[base + i] : base + i; };
  // ---- loads of one row, and their sum once they are there
  typedef typename Raw4<T>::type Raw;
  float4 xv, yv;
  Raw ev[4], tv;                                 // four experts' rows, the embedding's row
  const int quads = (p.top + 3) / 4;
  auto request = [&](int i) {
    const int src = source(i);
    if (START) {
      const int r = base + i, id = min(max(p.ids[(size_t)r * p.ids_ld + (p.step ? *p.step : 0)], 0), p.vocab - 1);
      fetch4(reinterpret_cast<const T *>(p.table) + (size_t)id * p.table_ld + c, tv);
      return;
    }
    fetch4(p.x_in + (size_t)src * p.width + c, xv);
    if (p.y) fetch4(p.y + (size_t)src * p.y_ld + c, yv);
  };
  auto request_pairs = [&](int i, int quad) {    // (after the block's pr are in place)
    const int4 rows = *reinterpret_cast<const int4 *>(pr + (i * quads + quad) * 4);
    const T *self = reinterpret_cast<const T *>(p.self) + (size_t)source(i) * p.self_ld + c, *pair = reinterpret_cast<const T *>(p.pair_y) + c;
    fetch4(rows.x < 0 ? self : pair + (size_t)rows.x * p.pair_ld, ev[0]);
    fetch4(rows.y < 0 ? self : pair + (size_t)rows.y * p.pair_ld, ev[1]);
    fetch4(rows.z < 0 ? self : pair + (size_t)rows.z * p.pair_ld, ev[2]);
    fetch4(rows.w < 0 ? self : pair + (size_t)rows.w * p.pair_ld, ev[3]);
  };
  auto add_pairs = [&](int i, int quad, float (&v)[4]) {
    const float4 w = *reinterpret_cast<const float4 *>(pw + (i * quads + quad) * 4);
    add4(v, w.x, ev[0]);
    add4(v, w.y, ev[1]);
    add4(v, w.z, ev[2]);
    add4(v, w.w, ev[3]);
  };
  auto sum = [&](int i, float (&v)[4]) {
    v[0] = v[1] = v[2] = v[3] = 0.f;
    if (START) {
      add4(v, 1.f, tv);
      return;
    }
    if (p.y) {
      add4(v, 1.f, yv);
      if (quads) add_pairs(i, 0, v);
      for (int q = 1; q < quads; ++q) {
        request_pairs(i, q);
        add_pairs(i, q, v);
      }
    }
    v[0] += xv.x; v[1] += xv.y; v[2] += xv.z; v[3] += xv.w;
  };
  request(0);
  float above[4] = {0.f, 0.f, 0.f, 0.f}, w1[4], w2[4], share[4], we[4];
  int first_to = -1;
  if (mix && p.run == 1) {                       // sequence r0: its state is on its way at once
    const int at = START && p.step ? *p.step : p.start[r0], slot = p.slot[r0];
    if (at > 0) load_vec<4>(p.state_in + (size_t)slot * p.width + c, above);
    first_to = p.by_seq ? r0 : slot;
  }
  if (mix) {
    load_vec<4>(p.w1 + c, w1);
    load_vec<4>(p.shift + c, share);
  }
  if (p.h2) load_vec<4>(p.w2 + c, w2);
  if (START) load_vec<4>(p.embed_w + c, we);
  for (int i = tid; i < n * quads * 4; i += blockDim.x) {
    const int row = i / (quads * 4), j = i % (quads * 4);
    const size_t k = (size_t)source(row) * p.top + min(j, p.top - 1);
    const int at = p.pair_row ? p.pair_row[k] : (int)k;
    const bool none = j >= p.top || (at < 0 && !p.self);
    pw[i] = none ? 0.f : p.pair_w ? p.pair_w[k] : 1.f;
    pr[i] = at < 0 && !p.self ? 0 : at;
  }
  if (mix && p.run > 1 && tid < n) {
    const int r = base + tid, s = p.tok_seq[r], at = START && p.step ? *p.step : p.start[s];
    before[tid] = r > p.cu[s] ? ABOVE : at > 0 ? STATE : NOTHING;
    from[tid] = p.slot[s];
    to[tid] = r >= r0 && r + 1 == p.cu[s + 1] ? (p.by_seq ? s : p.slot[s]) : -1;
  }
  const int per = p.part / CHUNK, g0 = c / p.part * per;         // the warps of this column's group
  int turn = 0;
  auto inv_rms = [&](const float (&v)[4]) {
    const float ss = warp_sum(fmaf(v[0], v[0], fmaf(v[1], v[1], fmaf(v[2], v[2], v[3] * v[3]))));
    if (lane == 0) red[turn][warp] = ss;
    __syncthreads();
    float all = 0.f;
    for (int i = 0; i < per; ++i) all += red[turn][g0 + i];
    turn ^= 1;                                   // (the next sums land in the other half: one barrier per row)
    return 1.0f / sqrtf(all / (float)p.part + p.eps);
  };
  if (quads || p.run > 1) __syncthreads();
  if (!START && quads) request_pairs(0, 0);
  for (int i = 0; i < n; ++i) {
    const int r = base + i;
    const bool mine = r >= r0;
    float v[4], o[4];
    sum(i, v);
    if (i + 1 < n) {
      request(i + 1);
      if (!START && quads) request_pairs(i + 1, 0);
    }
    const int kind = mix && p.run > 1 ? before[i] : ABOVE;
    if (kind == STATE) load_vec<4>(p.state_in + (size_t)from[i] * p.width + c, above);
    if (START) {
      if (tid == 0 && mine && p.pos_out) p.pos_out[r] = p.step ? *p.step : 0;
      const float f = inv_rms(v);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] *= f * we[j];
    }
    if (p.x_out && mine) store_vec<4>(p.x_out + (size_t)r * p.width + c, v);
    if (!mix && !p.h2) continue;
    const float f = inv_rms(v);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] *= f;
    if (p.h2 && mine) {
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = v[j] * w2[j];
      store_vec<4>(reinterpret_cast<T *>(p.h2) + (size_t)r * p.h2_ld + c, o);
    }
    if (!mix) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      v[j] *= w1[j];
      o[j] = fmaf((kind == NOTHING ? 0.f : above[j]) - v[j], share[j], v[j]);
      above[j] = v[j];
    }
    if (mine) {
      store_vec<4>(reinterpret_cast<T *>(p.h1) + (size_t)r * p.h1_ld + c, o);
      const int dst = p.run > 1 ? to[i] : first_to;
      if (dst >= 0) store_vec<4>(p.state_out + (size_t)dst * p.width + c, v);
    }
  }
  for (int r = r0; r < r1; ++r) {                // k padding of the next products
    if (mix)
      for (int k = p.width + tid; k < p.h1_ld; k += blockDim.x) reinterpret_cast<T *>(p.h1)[(size_t)r * p.h1_ld + k] = from_f<T>(0.f);
    if (p.h2)
      for (int k = p.width + tid; k < p.h2_ld; k += blockDim.x) reinterpret_cast<T *>(p.h2)[(size_t)r * p.h2_ld + k] = from_f<T>(0.f);
  }
}

constexpr size_t kSmemLimit = 200 * 1024;
static size_t smem_bytes(const Params &p, int run) {
  const size_t rows = run + (p.h1 ? 1 : 0);
  return rows * (p.width + p.groups + (size_t)p.groups * p.segs) * sizeof(float);
}

template <typename T, typename E, int VEC, bool START> static int launch(Params p, bool single, cudaStream_t st) {
  if (VEC == 4 && p.part % CHUNK == 0 && p.width <= 4096 && (!p.top || std::is_same<T, E>::value)) {
    const int threads = p.width / 4, resident = std::max(1, 1024 / threads) * sm_count();        // blocks on the GPU at a time
    p.run = single ? 1 : std::min(kMaxFastRun, std::max(2, ceil_div(p.rows, resident)));
    rows_kernel<T, START><<<ceil_div(p.rows, p.run), threads, 0, st>>>(p);
    PT_LAUNCH_CHECK("pt_shift_norm");
    return PT_OK;
  }
  // few rows: as many threads as a row has work for; many: several rows of a sequence per block, so that few are computed twice
  const int want = ceil_div(ceil_div(p.width, VEC), 32) * 32, cap = p.rows <= 2 * sm_count() ? 1024 : 256, threads = std::max(64, std::min(want, cap));
  p.run = single ? 1 : p.rows >= 8 * sm_count() ? kMaxRun : p.rows >= 4 * sm_count() ? 2 : 1;
  p.segs = std::max(1, std::min(threads / 32 / ((p.run + (p.h1 ? 1 : 0)) * p.groups), ceil_div(p.part, 32 * VEC)));
  while (p.run > 1 && smem_bytes(p, p.run) > kSmemLimit) --p.run;
  const size_t smem = smem_bytes(p, p.run);
  PT_REQUIRE(smem <= kSmemLimit, "pt_shift_norm: rows of %d in %d groups need %zu bytes of shared memory", p.width, p.groups, smem);
  if (smem > 40 * 1024) {
    static bool set = false;
    if (!set) { PT_CUDA(cudaFuncSetAttribute(shift_norm_kernel<T, E, VEC, START>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit)); set = true; }
  }
  shift_norm_kernel<T, E, VEC, START><<<ceil_div(p.rows, p.run), threads, smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_shift_norm");
  return PT_OK;
}
template <typename T, typename E, int VEC> static int launch(const Params &p, bool single, cudaStream_t st) {
  return p.table ? launch<T, E, VEC, true>(p, single, st) : launch<T, E, VEC, false>(p, single, st);
}

}  // namespace shift
}  // namespace pt

using namespace pt;

extern "C" int pt_shift_norm(const pt_shift_norm_args *a, void *stream) {
  PT_REQUIRE(a, "pt_shift_norm: null args");
  const pt_batch_view &b = a->batch;
  PT_REQUIRE(a->rows > 0 && a->width > 0 && a->groups > 0 && a->width % a->groups == 0, "pt_shift_norm: %d rows of %d in %d groups", a->rows, a->width, a->groups);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_shift_norm: activation type %d (fp32 or bf16)", a->dtype);
  if (a->table) {
    PT_REQUIRE(a->ids && a->vocab > 0 && a->table_ld >= a->width && a->ids_ld >= 1 && a->embed_w && !a->row_index, "pt_shift_norm: an embedding start needs ids, vocab, table_ld and embed_w");
  } else {
    PT_REQUIRE(a->x_in && (!a->y || a->y_ld >= a->width) && a->top >= 0 && a->top <= shift::kMaxTop, "pt_shift_norm: y_ld=%d, %d experts per token (at most %d)", a->y_ld, a->top,
               shift::kMaxTop);
    PT_REQUIRE(!a->top || (a->y && a->pair_y && a->pair_ld >= a->width), "pt_shift_norm: experts' outputs need y, pair_y and pair_ld");
    PT_REQUIRE(!a->top || a->pair_dtype == PT_DT_F32 || (a->pair_dtype == PT_DT_BF16 && a->dtype == PT_DT_BF16), "pt_shift_norm: experts' outputs of type %d", a->pair_dtype);
    PT_REQUIRE(!a->top || !a->pair_row || !a->self || a->self_ld >= a->width, "pt_shift_norm: self_ld=%d", a->self_ld);
  }
  const bool single = !a->h1 || b.n_tok == b.n_seq;
  if (a->h1) {
    PT_REQUIRE(b.n_seq > 0 && b.n_tok == a->rows && b.n_tok >= b.n_seq && b.cu && b.start && b.slot && b.tok_seq && !a->row_index, "pt_shift_norm: bad batch (%d sequences, %d tokens)", b.n_seq,
               b.n_tok);
    PT_REQUIRE(a->w1 && a->shift && a->state_in && a->state_out && a->h1_ld >= a->width, "pt_shift_norm: h1 needs w1, shift, states and h1_ld");
    PT_REQUIRE(single || (a->state_in != a->state_out && (!a->x_in || a->x_in != a->x_out)), "pt_shift_norm: several tokens per sequence need other buffers for x_out and state_out than for x_in and state_in");
  }
  PT_REQUIRE(!a->h2 || (a->w2 && a->h2_ld >= a->width), "pt_shift_norm: h2 needs w2 and h2_ld");
  shift::Params p{};
  p.rows = a->rows; p.width = a->width; p.groups = a->groups; p.part = a->width / a->groups; p.h1_ld = a->h1_ld; p.h2_ld = a->h2_ld; p.table_ld = a->table_ld; p.vocab = a->vocab;
  p.ids_ld = a->ids_ld; p.y_ld = a->y_ld; p.pair_ld = a->pair_ld; p.top = a->table ? 0 : a->top; p.self_ld = a->self_ld; p.eps = a->eps;
  p.x_in = a->table ? nullptr : a->x_in; p.x_out = a->x_out; p.table = a->table; p.ids = a->ids; p.step = a->step_dev; p.pos_out = a->pos_out; p.embed_w = a->embed_w;
  p.row_index = a->row_index; p.y = a->table ? nullptr : a->y; p.pair_y = a->pair_y; p.pair_w = a->pair_w; p.pair_row = a->pair_row; p.self = a->self;
  p.w1 = a->w1; p.shift = a->shift; p.w2 = a->w2; p.state_in = a->state_in; p.state_out = a->state_out; p.by_seq = a->state_by_seq != 0; p.h1 = a->h1; p.h2 = a->h2;
  p.cu = b.cu; p.start = b.start; p.slot = b.slot; p.tok_seq = b.tok_seq;
  const int tb = a->dtype == PT_DT_F32 ? 16 : 8;      // bytes of four elements
  auto f4 = [](const void *q) { return aligned_to(q, 16); };
  auto t4 = [&](const void *q, int ld) { return !q || (aligned_to(q, tb) && ld % 4 == 0); };
  const bool v4 = p.part % 4 == 0 && f4(p.x_in) && f4(p.x_out) && (!p.y || (f4(p.y) && p.y_ld % 4 == 0)) && f4(p.embed_w) && f4(p.w1) && f4(p.shift) && f4(p.w2) && f4(p.state_in) && f4(p.state_out) &&
                  t4(p.table, p.table_ld) && t4(p.self, p.self_ld) && t4(p.h1, p.h1_ld) && t4(p.h2, p.h2_ld) &&
                  (!p.top || (aligned_to(p.pair_y, a->pair_dtype == PT_DT_F32 ? 16 : 8) && p.pair_ld % 4 == 0));
  cudaStream_t st = as_stream(stream);
  typedef __nv_bfloat16 B;
  if (a->dtype == PT_DT_F32) return v4 ? shift::launch<float, float, 4>(p, single, st) : shift::launch<float, float, 1>(p, single, st);
  if (p.top > 0 && a->pair_dtype == PT_DT_BF16) return v4 ? shift::launch<B, B, 4>(p, single, st) : shift::launch<B, B, 1>(p, single, st);
  return v4 ? shift::launch<B, float, 4>(p, single, st) : shift::launch<B, float, 1>(p, single, st);
}
