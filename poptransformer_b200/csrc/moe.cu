// Mixture of experts: which experts a token goes to, and where its rows lie for the grouped products.
//   choose   per token the `top` experts with the largest router logits (the lowest index first among equals), and as weights the
//            softmax over those logits or their sigmoids.  fp32.
//            Or: scores are the softmax over all logits, corrected scores decide, only the best groups of neighbours take part, and the
//            weights are the chosen scores over their sum.  Experts at the end may have no matrices (their output is the input).
//   place    pair i = token i / top with its choice i % top gets a row of its own among its expert's rows.  The rows of an expert are
//            padded to whole tiles; tile_expert names the expert of every tile (-1: unused) and tile_rows its rows in use, so a grouped
//            product can look its weights up per tile.  Pairs keep their order within an expert.
//   gather   the tokens' activations are copied to their pairs' rows.  (Rows of the padding keep what they held: rows of a product do
//            not touch one another, and nothing reads theirs.)
// With few tokens every pair is a tile of one row and nothing is placed or copied.
#include <limits.h>

#include "elem.cuh"

namespace pt {
namespace moe {

constexpr int kMaxExperts = 1024, kMaxTop = 64, PLACE_THREADS = 1024;

struct Params {
  int n_tok, experts, top, logits_ld, tile, max_tiles, hist_copies;
  const float *logits;
  int *expert, *pair_row, *tile_expert, *tile_rows, *row_token;   // [n_tok][top] x 2, [max_tiles] x 2, [max_tiles * tile]
  float *weight, *row_weight;                         // [n_tok][top], [max_tiles * tile] or null: the weight of every placed row
  int sigmoid;                                        // weights: sigmoid(logit) instead of the softmax over the chosen
  const int *counts;                                  // [experts], or null: counted while placing
  int all, groups, keep;                              // logits: experts and identity experts
  const float *correction;
};

// One warp per token; lane l holds the logits of experts l, l + 32, ...
__global__ void choose_kernel(const Params p) {
  launch_dependents();
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.n_tok) return;
  const float *z = p.logits + (size_t)t * p.logits_ld;
  __shared__ float zs[4][kMaxExperts];
  float *mine = zs[threadIdx.x >> 5];
  for (int e = lane; e < p.experts; e += 32) mine[e] = z[e];
  __syncwarp();
  float first = 0.f, sum = 0.f, w0 = 0.f, w1 = 0.f;     // lane k keeps the weights of choices k and k + 32
  for (int k = 0; k < p.top; ++k) {
    float best = -INFINITY;
    int at = INT_MAX;
    for (int e = lane; e < p.experts; e += 32)
      if (mine[e] > best) { best = mine[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, best, o);
      const int a = __shfl_xor_sync(0xffffffffu, at, o);
      if (b > best || (b == best && a < at)) { best = b; at = a; }
    }
    if (at == INT_MAX) at = k;                          // only infinities or NaN are left
    if (k == 0) first = best;
    const float w = p.sigmoid ? 1.0f / (1.0f + expf(-best)) : expf(best - first);
    sum += w;
    if (lane == (k & 31)) {
      (k < 32 ? w0 : w1) = w;
      p.expert[(size_t)t * p.top + k] = at;
      mine[at] = -INFINITY;
    }
    __syncwarp();
  }
  if (p.sigmoid) sum = 1.f;
  if (lane < p.top) p.weight[(size_t)t * p.top + lane] = w0 / sum;
  if (lane + 32 < p.top) p.weight[(size_t)t * p.top + lane + 32] = w1 / sum;
}

// Corrected scores, groups and identity experts.  One warp per token; shared memory per warp: [all] scores, [all] corrected, [groups].
constexpr int CHOOSE_WARPS = 4;
__global__ void __launch_bounds__(CHOOSE_WARPS * 32) choose_corrected_kernel(const Params p) {
  extern __shared__ float choose_sm[];
  launch_dependents();
  const int t = blockIdx.x * CHOOSE_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.n_tok) return;
  float *s = choose_sm + (size_t)(threadIdx.x >> 5) * (2 * p.all + p.groups), *c = s + p.all, *best = c + p.all;
  const float *z = p.logits + (size_t)t * p.logits_ld;
  float top = -INFINITY, sum = 0.f;
  for (int e = lane; e < p.all; e += 32) top = fmaxf(top, z[e]);
  top = warp_max(top);
  for (int e = lane; e < p.all; e += 32) {
    s[e] = expf(z[e] - top);
    sum += s[e];
  }
  sum = warp_sum(sum);
  for (int e = lane; e < p.all; e += 32) {
    s[e] /= sum;
    c[e] = s[e] + (p.correction ? __ldg(p.correction + e) : 0.f);
  }
  __syncwarp();
  if (p.keep < p.groups) {
    const int size = p.all / p.groups;
    for (int g = lane; g < p.groups; g += 32) {
      float m = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, c[e]);
      best[g] = m;
    }
    __syncwarp();
    for (int g = lane; g < p.groups; g += 32) {
      const float mine = best[g];
      int before = 0;                                   // groups in front of this one (the lowest index first among equals)
      for (int o = 0; o < p.groups; ++o) before += best[o] > mine || (best[o] == mine && o < g);
      if (before >= p.keep)
        for (int e = g * size; e < (g + 1) * size; ++e) c[e] = -INFINITY;
    }
    __syncwarp();
  }
  sum = 0.f;
  float w0 = 0.f, w1 = 0.f;                             // lane k keeps the weights of choices k and k + 32
  for (int k = 0; k < p.top; ++k) {
    float most = -INFINITY;
    int at = INT_MAX;
    for (int e = lane; e < p.all; e += 32)
      if (c[e] > most) { most = c[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, most, o);
      const int a = __shfl_xor_sync(0xffffffffu, at, o);
      if (b > most || (b == most && a < at)) { most = b; at = a; }
    }
    if (at == INT_MAX) at = k;                          // only infinities or NaN are left
    const float w = s[at];
    sum += w;
    __syncwarp();
    if (lane == (k & 31)) {
      (k < 32 ? w0 : w1) = w;
      const size_t i = (size_t)t * p.top + k;
      p.expert[i] = at < p.experts ? at : -1;
      if (p.pair_row) p.pair_row[i] = at < p.experts ? (int)i : -1;      // (placed experts get their rows later)
      c[at] = -INFINITY;
    }
    __syncwarp();
  }
  sum += 1e-20f;
  if (lane < p.top) p.weight[(size_t)t * p.top + lane] = w0 / sum;
  if (lane + 32 < p.top) p.weight[(size_t)t * p.top + lane + 32] = w1 / sum;
}

// Pairs per expert, for many pairs: block e counts those of expert e.
__global__ void __launch_bounds__(PLACE_THREADS) count_kernel(const int *expert, int pairs, int *counts) {
  __shared__ int warps[PLACE_THREADS / 32];
  const int e = blockIdx.x, tid = threadIdx.x, n4 = pairs / 4;
  int hits = 0;
  for (int i = tid; i < n4; i += PLACE_THREADS) {
    const int4 x = reinterpret_cast<const int4 *>(expert)[i];
    hits += (x.x == e) + (x.y == e) + (x.z == e) + (x.w == e);
  }
  for (int i = 4 * n4 + tid; i < pairs; i += PLACE_THREADS) hits += expert[i] == e;
  for (int o = 16; o > 0; o >>= 1) hits += __shfl_xor_sync(0xffffffffu, hits, o);
  if ((tid & 31) == 0) warps[tid >> 5] = hits;
  __syncthreads();
  if (tid == 0) {
    int n = 0;
    for (int w = 0; w < PLACE_THREADS / 32; ++w) n += warps[w];
    counts[e] = n;
  }
}

// Block e places the pairs of expert e: the pairs of all experts are counted (or come from count_kernel) for the tiles in front of its
// own, then its own pairs get their rows.  Thread i looks at a run of consecutive pairs, so the order within an expert is the order of the pairs.
__global__ void __launch_bounds__(PLACE_THREADS) place_kernel(const Params p) {
  extern __shared__ int hist[];                   // [copies][experts]: warps count into copies of their own while they fit
  __shared__ int warps[PLACE_THREADS / 32];
  __shared__ int first, total;
  const int e = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, pairs = p.n_tok * p.top;
  const int per = ((pairs + PLACE_THREADS - 1) / PLACE_THREADS + 3) & ~3, i0 = min(pairs, tid * per), i1 = min(pairs, i0 + per);
  int *mine = hist + (warp % p.hist_copies) * p.experts;
  for (int i = tid; i < p.hist_copies * p.experts; i += PLACE_THREADS) hist[i] = 0;
  __syncthreads();
  int hits = 0;
  auto count_one = [&](int x) {
    if (!p.counts && x >= 0) atomicAdd(mine + x, 1);
    hits += x == e;
  };
  int i = i0;
  if (((uintptr_t)p.expert & 15) == 0)
    for (; i + 4 <= i1; i += 4) {
      const int4 x = *reinterpret_cast<const int4 *>(p.expert + i);
      count_one(x.x);
      count_one(x.y);
      count_one(x.z);
      count_one(x.w);
    }
  for (; i < i1; ++i) count_one(p.expert[i]);
  __syncthreads();
  for (int i = tid; i < p.experts; i += PLACE_THREADS) {
    int n = 0;
    if (p.counts) n = p.counts[i];
    else
      for (int c = 0; c < p.hist_copies; ++c) n += hist[c * p.experts + i];
    hist[i] = n;                                  // (the same thread read copy 0 of this expert just before)
  }
  int scan = hits;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, scan, o);
    if (lane >= o) scan += v;
  }
  if (lane == 31) warps[warp] = scan;
  __syncthreads();
  if (warp == 0) {
    int before = 0, all = 0;
    for (int i = lane; i < p.experts; i += 32) {
      const int tiles = (hist[i] + p.tile - 1) / p.tile;
      all += tiles;
      if (i < e) before += tiles;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      before += __shfl_xor_sync(0xffffffffu, before, o);
      all += __shfl_xor_sync(0xffffffffu, all, o);
    }
    if (lane == 0) { first = before; total = all; }
  } else if (warp == 1) {
    const int own = warps[lane];
    int sum = own;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += v;
    }
    warps[lane] = sum - own;
  }
  __syncthreads();
  const int count = hist[e], tiles = (count + p.tile - 1) / p.tile, row0 = first * p.tile;
  for (int i = tid; i < tiles; i += PLACE_THREADS) {
    p.tile_expert[first + i] = e;
    p.tile_rows[first + i] = min(p.tile, count - i * p.tile);
  }
  for (int i = count + tid; i < tiles * p.tile; i += PLACE_THREADS) p.row_token[row0 + i] = -1;
  if (e == 0) {
    for (int i = total + tid; i < p.max_tiles; i += PLACE_THREADS) { p.tile_expert[i] = -1; p.tile_rows[i] = 0; }
    for (int i = total * p.tile + tid; i < p.max_tiles * p.tile; i += PLACE_THREADS) p.row_token[i] = -1;
  }
  int row = row0 + warps[warp] + scan - hits;
  for (int i = i0; hits > 0 && i < i1; ++i)
    if (p.expert[i] == e) {
      p.pair_row[i] = row;
      if (p.row_weight) p.row_weight[row] = p.weight[i];
      p.row_token[row++] = i / p.top;
    }
}

// Rows of h (whole 16-byte units) to where row_token says.
__global__ void gather_kernel(const uint4 *h, uint4 *out, int units, const int *row_token) {
  launch_dependents();
  const int tok = row_token[blockIdx.x];
  if (tok < 0) return;
  for (int i = threadIdx.x; i < units; i += blockDim.x) out[(size_t)blockIdx.x * units + i] = h[(size_t)tok * units + i];
}
__global__ void gather4_kernel(const uint32_t *h, uint32_t *out, int units, const int *row_token) {
  const int tok = row_token[blockIdx.x];
  if (tok < 0) return;
  for (int i = threadIdx.x; i < units; i += blockDim.x) out[(size_t)blockIdx.x * units + i] = h[(size_t)tok * units + i];
}

}  // namespace moe
}  // namespace pt

using namespace pt;

extern "C" int pt_moe_max_tiles(int n_tok, int experts, int top, int tile) {
  const int pairs = n_tok * top, used = std::min(experts, pairs);     // every expert in use pads less than a tile
  return (pairs + used * (tile - 1)) / tile;
}

extern "C" int pt_moe_route(const pt_moe_route_args *a, void *stream) {
  PT_REQUIRE(a, "pt_moe_route: null args");
  const int all = a->experts + a->identity;       // logits
  PT_REQUIRE(a->identity >= 0 && (!a->identity || a->score == PT_MOE_SOFTMAX_ALL), "pt_moe_route: %d identity experts", a->identity);
  PT_REQUIRE(a->n_tok > 0 && a->experts > 0 && all <= moe::kMaxExperts && a->top > 0 && a->top <= std::min(all, moe::kMaxTop),
             "pt_moe_route: %d tokens, %d of %d experts (at most %d of %d)", a->n_tok, a->top, all, moe::kMaxTop, moe::kMaxExperts);
  PT_REQUIRE((long long)a->n_tok * a->top < (1 << 28), "pt_moe_route: %d tokens x %d choices", a->n_tok, a->top);
  PT_REQUIRE(a->logits && a->logits_ld >= all && a->expert && a->weight, "pt_moe_route: null pointer argument");
  moe::Params p{};
  p.n_tok = a->n_tok; p.experts = a->experts; p.top = a->top; p.logits_ld = a->logits_ld; p.logits = a->logits; p.expert = a->expert; p.weight = a->weight;
  PT_REQUIRE(a->score == PT_MOE_SOFTMAX || a->score == PT_MOE_SIGMOID || a->score == PT_MOE_SOFTMAX_ALL, "pt_moe_route: weights of kind %d", a->score);
  p.sigmoid = a->score == PT_MOE_SIGMOID;
  cudaStream_t st = as_stream(stream);
  if (a->score == PT_MOE_SOFTMAX_ALL) {
    p.all = all; p.groups = std::max(1, a->groups); p.keep = a->groups ? a->keep : 1; p.correction = a->correction; p.pair_row = a->pair_row;
    PT_REQUIRE(all % p.groups == 0 && p.keep >= 1 && p.keep <= p.groups && a->top <= all / p.groups * p.keep, "pt_moe_route: %d of %d groups of %d experts, %d choices", p.keep,
               p.groups, all, a->top);
    PT_REQUIRE(!a->identity || a->pair_row, "pt_moe_route: identity experts need pair_row");
    moe::choose_corrected_kernel<<<ceil_div(p.n_tok, moe::CHOOSE_WARPS), moe::CHOOSE_WARPS * 32, (size_t)moe::CHOOSE_WARPS * (2 * all + p.groups) * sizeof(float), st>>>(p);
  } else {
    moe::choose_kernel<<<ceil_div(p.n_tok, 4), 128, 0, st>>>(p);
  }
  PT_LAUNCH_CHECK("pt_moe_route");
  if (!a->tile) return PT_OK;
  PT_REQUIRE(a->tile > 0 && a->pair_row && a->tile_expert && a->tile_rows && a->row_token && a->max_tiles >= pt_moe_max_tiles(a->n_tok, a->experts, a->top, a->tile),
             "pt_moe_route: tiles of %d rows need pair_row, row_token and %d entries of tile_expert", a->tile, pt_moe_max_tiles(a->n_tok, a->experts, a->top, a->tile));
  p.tile = a->tile; p.max_tiles = a->max_tiles; p.pair_row = a->pair_row; p.tile_expert = a->tile_expert; p.tile_rows = a->tile_rows; p.row_token = a->row_token;
  p.row_weight = a->row_weight;
  if (p.n_tok * p.top > 4096 && a->counts && aligned_to(p.expert, 16)) {
    moe::count_kernel<<<p.experts, moe::PLACE_THREADS, 0, st>>>(p.expert, p.n_tok * p.top, a->counts);
    PT_LAUNCH_CHECK("pt_moe_route");
    p.counts = a->counts;
  }
  p.hist_copies = p.counts ? 1 : std::max(1, std::min(32, 8192 / p.experts));
  moe::place_kernel<<<p.experts, moe::PLACE_THREADS, (size_t)p.hist_copies * p.experts * sizeof(int), st>>>(p);
  PT_LAUNCH_CHECK("pt_moe_route");
  if (a->h) {
    PT_REQUIRE(a->gathered && a->h_bytes > 0 && a->h_bytes % 4 == 0, "pt_moe_route: rows of %d bytes", a->h_bytes);
    const int rows = a->max_tiles * a->tile;
    if (a->h_bytes % 16 == 0 && aligned_to(a->h, 16) && aligned_to(a->gathered, 16))
      moe::gather_kernel<<<rows, 128, 0, st>>>((const uint4 *)a->h, (uint4 *)a->gathered, a->h_bytes / 16, p.row_token);
    else
      moe::gather4_kernel<<<rows, 128, 0, st>>>((const uint32_t *)a->h, (uint32_t *)a->gathered, a->h_bytes / 4, p.row_token);
    PT_LAUNCH_CHECK("pt_moe_route");
  }
  return PT_OK;
}
