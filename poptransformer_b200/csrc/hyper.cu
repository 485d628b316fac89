// Hyper-connections: several fp32 residual streams per token instead of one, with learned read, write and mixing weights.
//
// A sublayer reads u = sum_s in[s] x_s, computes y = f(rms_norm(u)), and then every stream becomes a mix of the previous streams plus its share of y:
//     x_t <- sum_s mix[s, t] x_s + mult * out[t] * y .
// One launch does everything that lies between two sublayers' matrix products: the write of the finished sublayer, the read of
// the next one and its RMS norm, so the streams cross HBM once in each direction per sublayer.  The same kernel starts a token
// (every stream is the embedding row) and ends the model (the streams are summed and normalised for the output layer).
// streams = 1 with in = out = mix = 1 is the ordinary pre-norm residual.  All of it is fp32; only h, the input of the matrix
// product that follows, is rounded to the activation type.
#include "elem.cuh"

namespace pt {
namespace hyper {

constexpr int kMaxStreams = 16;

struct Params {
  int rows, width, streams, h_ld, table_ld, vocab, ids_ld, y_ld;
  float eps, mult;
  float *xs;                  // [rows, streams, width]
  const void *table;          // start of a token: embedding rows
  const int *ids, *step;
  int *pos_out;
  const int *row_index;       // rows of xs / y this launch works on (null: 0 .. rows - 1)
  const float *y;             // output of the finished sublayer (null: nothing to write)
  const float *mix, *w_out;   // [streams, streams] indexed [from, to], [streams]
  const float *w_in;          // read weights of the next sublayer (null: plain sum, streams not written back)
  const float *norm_w;
  void *h;
  float *sum_out;             // optional [rows, width]: sum of the new streams
};

template <int VEC> struct Vec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Vec<VEC> ld(const float *p) {
  Vec<VEC> r;
  if constexpr (VEC == 4) *reinterpret_cast<float4 *>(r.v) = *reinterpret_cast<const float4 *>(p);
  else r.v[0] = *p;
  return r;
}
template <int VEC> __device__ __forceinline__ void st(float *p, const Vec<VEC> &r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = *reinterpret_cast<const float4 *>(r.v);
  else *p = r.v[0];
}

// S > 0: that many streams, unrolled.  S == 0: p.streams (at most kMaxStreams).
template <typename T, int S, int VEC> __global__ void hyper_kernel(const Params p) {
  constexpr int SM = S > 0 ? S : kMaxStreams;
  extern __shared__ __align__(16) float u_row[];   // [width]
  __shared__ float c_mix[SM * SM], c_out[SM], c_in[SM], red[32];
  const int ns = S > 0 ? S : p.streams;
  const int r = blockIdx.x, src = p.row_index ? p.row_index[r] : r;
  const bool start = p.table != nullptr, write = p.y != nullptr, last = p.w_in == nullptr;
  for (int i = threadIdx.x; i < ns * ns; i += blockDim.x) c_mix[i] = write ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < ns; i += blockDim.x) {
    c_out[i] = write ? p.mult * p.w_out[i] : 0.f;
    c_in[i] = last ? 1.f : p.w_in[i];
  }
  const T *emb = nullptr;
  if (start) {
    const int step = p.step ? *p.step : 0;
    int id = p.ids[(size_t)src * p.ids_ld + step];
    id = min(max(id, 0), p.vocab - 1);
    emb = reinterpret_cast<const T *>(p.table) + (size_t)id * p.table_ld;
    if (threadIdx.x == 0 && p.pos_out) p.pos_out[r] = step;
  }
  __syncthreads();
  float *xrow = p.xs + (size_t)src * ns * p.width;
  const float *yrow = write ? p.y + (size_t)src * p.y_ld : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < p.width; i += blockDim.x * VEC) {
    Vec<VEC> x[SM], y, u, sum;
    if (start) {
      Vec<VEC> e;
#pragma unroll
      for (int j = 0; j < VEC; ++j) e.v[j] = to_f(emb[i + j]);
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < ns) x[s] = e;
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < ns) x[s] = ld<VEC>(xrow + (size_t)s * p.width + i);
    }
    if (write) y = ld<VEC>(yrow + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u.v[j] = sum.v[j] = 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) {
      if (t >= ns) break;
      Vec<VEC> n;
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        float a;
        if (write) {
          a = c_out[t] * y.v[j];
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (s < ns) a += c_mix[s * ns + t] * x[s].v[j];
        } else {
          a = x[t].v[j];
        }
        n.v[j] = a;
        u.v[j] += c_in[t] * a;
        sum.v[j] += a;
      }
      if (!last && (start || write)) st<VEC>(xrow + (size_t)t * p.width + i, n);
    }
    if (p.sum_out) st<VEC>(p.sum_out + (size_t)r * p.width + i, sum);
    st<VEC>(u_row + i, u);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += u.v[j] * u.v[j];
  }
  if (!p.h) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);
  T *hrow = reinterpret_cast<T *>(p.h) + (size_t)r * p.h_ld;
  for (int i = threadIdx.x * VEC; i < p.width; i += blockDim.x * VEC) {
    const Vec<VEC> u = ld<VEC>(u_row + i), w = ld<VEC>(p.norm_w + i);
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = u.v[j] * inv * w.v[j];
    store_vec<VEC>(hrow + i, o);
  }
  for (int i = p.width + threadIdx.x; i < p.h_ld; i += blockDim.x) hrow[i] = from_f<T>(0.f);   // k padding of the next product
}

template <typename T, int S, int VEC> static int launch(const Params &p, cudaStream_t st) {
  const size_t smem = (size_t)p.width * sizeof(float);
  if (smem > 48 * 1024) {
    static bool set = false;
    if (!set) { PT_CUDA(cudaFuncSetAttribute(hyper_kernel<T, S, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); set = true; }
  }
  const int want = ceil_div(ceil_div(p.width, VEC), 32) * 32, cap = p.rows <= 2 * sm_count() ? 1024 : 256;
  const int regs_cap = S == 0 ? 256 : 1024;
  hyper_kernel<T, S, VEC><<<p.rows, std::min(std::min(want, cap), regs_cap), smem, st>>>(p);
  PT_LAUNCH_CHECK("pt_hyper");
  return PT_OK;
}
template <typename T> static int dispatch(const Params &p, bool vec4, cudaStream_t st) {
  if (vec4) switch (p.streams) {
      case 1: return launch<T, 1, 4>(p, st);
      case 2: return launch<T, 2, 4>(p, st);
      case 3: return launch<T, 3, 4>(p, st);
      case 4: return launch<T, 4, 4>(p, st);
      default: break;
    }
  return launch<T, 0, 1>(p, st);
}

}  // namespace hyper
}  // namespace pt

using namespace pt;

extern "C" int pt_hyper(const pt_hyper_args *a, void *stream) {
  PT_REQUIRE(a, "pt_hyper: null args");
  PT_REQUIRE(a->rows > 0 && a->width > 0 && a->width <= 48 * 1024 && a->streams >= 1 && a->streams <= hyper::kMaxStreams,
             "pt_hyper: bad shape rows=%d width=%d streams=%d (streams 1..%d)", a->rows, a->width, a->streams, hyper::kMaxStreams);
  PT_REQUIRE(a->dtype == PT_DT_F32 || a->dtype == PT_DT_BF16, "pt_hyper: activation type %d (fp32 or bf16)", a->dtype);
  PT_REQUIRE(a->xs, "pt_hyper: null streams");
  PT_REQUIRE(!a->table || (a->ids && a->vocab > 0 && a->table_ld >= a->width && a->ids_ld >= 1), "pt_hyper: an embedding start needs ids, vocab and table_ld");
  PT_REQUIRE(!(a->table && a->y), "pt_hyper: an embedding start has no sublayer output to write");
  PT_REQUIRE(!a->table || a->w_in, "pt_hyper: an embedding start needs the read weights of the first sublayer");
  PT_REQUIRE(!a->y || (a->mix && a->w_out && a->y_ld >= a->width), "pt_hyper: a write needs mix, w_out and y_ld");
  PT_REQUIRE(!a->h || (a->norm_w && a->h_ld >= a->width), "pt_hyper: a norm output needs its weight and h_ld");
  hyper::Params p{};
  p.rows = a->rows; p.width = a->width; p.streams = a->streams; p.h_ld = a->h_ld; p.table_ld = a->table_ld; p.vocab = a->vocab;
  p.ids_ld = a->ids_ld; p.y_ld = a->y_ld; p.eps = a->eps; p.mult = a->mult;
  p.xs = a->xs; p.table = a->table; p.ids = a->ids; p.step = a->step_dev; p.pos_out = a->pos_out; p.row_index = a->row_index;
  p.y = a->y; p.mix = a->mix; p.w_out = a->w_out; p.w_in = a->w_in; p.norm_w = a->norm_w; p.h = a->h; p.sum_out = a->sum_out;
  auto al16 = [](const void *q) { return ((uintptr_t)q & 15) == 0; };
  const int esz = a->dtype == PT_DT_F32 ? 4 : 2;
  const bool vec4 = a->width % 4 == 0 && al16(a->xs) && (!a->y || (al16(a->y) && a->y_ld % 4 == 0)) && (!a->norm_w || al16(a->norm_w)) &&
                    (!a->sum_out || al16(a->sum_out)) && (!a->h || (((uintptr_t)a->h & (4 * esz - 1)) == 0 && a->h_ld % 4 == 0));
  if (a->dtype == PT_DT_F32) return hyper::dispatch<float>(p, vec4, as_stream(stream));
  return hyper::dispatch<__nv_bfloat16>(p, vec4, as_stream(stream));
}
