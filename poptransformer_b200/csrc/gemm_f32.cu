// Matrix product in true fp32 for models that run in 32-bit: y[m, n] = epilogue(alpha * sum_k x[m, k] w[n, k] + bias[n]).
// 64 x 64 output tiles, 16 k per step through shared memory, 4 x 4 outputs per thread, fused multiply-adds in k order.  Every step
// is summed on its own and then added, so the rounding error grows with the number of steps, not with k.
// Grouped products (experts): every tile of 64 rows names the weight matrix it is multiplied with.
#include "dense_out.cuh"

namespace pt {
namespace f32 {

constexpr int BM = 64, BN = 64, BK = 16, THREADS = 256;

__global__ void __launch_bounds__(THREADS) gemm_f32_kernel(const float *__restrict__ x, int x_ld, const float *__restrict__ w, int w_ld, int M, int N,
                                                           int K, const int *__restrict__ group_of, const DenseOut o) {
  __shared__ float xs[BK][BM + 4], ws[BK][BN + 4];
  if (group_of) {
    const int grp = group_of[blockIdx.y];
    if (grp < 0) return;
    w += (size_t)grp * N * w_ld;
  }
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN, tid = threadIdx.x, tm = tid / 16, tn = tid % 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int i = tid; i < BM * BK; i += THREADS) {
      const int r = i / BK, k = i % BK;
      const bool in = k0 + k < K;
      xs[k][r] = (in && m0 + r < M) ? x[(size_t)(m0 + r) * x_ld + k0 + k] : 0.f;
      ws[k][r] = (in && n0 + r < N) ? w[(size_t)(n0 + r) * w_ld + k0 + k] : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) { a[j] = xs[k][tm * 4 + j]; b[j] = ws[k][tn * 4 + j]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(a[i], b[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + tm * 4 + i, n = n0 + tn * 4 + j;
      // gated features: the up row n + 8 is this thread's neighbour two to the right
      const float other = o.epilogue == PT_EPI_GLU ? __shfl_xor_sync(0xffffffffu, acc[i][j], 2) : 0.f;
      if (m >= M || n >= N) continue;
      if (o.epilogue == PT_EPI_GLU && n < o.split_n) {
        if (n % 16 < 8) dense_store_glu<true, true>(o, m, n, acc[i][j], other);
      } else {
        dense_store<true, true>(o, m, n, acc[i][j]);
      }
    }
}

}  // namespace f32
}  // namespace pt

using namespace pt;

extern "C" int pt_gemm_f32(const float *x, int x_ld, const float *w, int w_ld, int m, int n, int k, float alpha, int epilogue, float *y, int y_ld,
                           const pt_dense_ext *ext, void *stream) {
  PT_REQUIRE(x && w && y, "pt_gemm_f32: null pointer argument");
  const int n_y = epilogue == PT_EPI_GLU ? 0 : (ext && ext->out2 ? ext->split_n : n);
  PT_REQUIRE(m > 0 && n > 0 && k > 0 && x_ld >= k && w_ld >= k && y_ld >= n_y, "pt_gemm_f32: bad shape m=%d n=%d k=%d (row strides %d %d %d)", m, n, k, x_ld,
             w_ld, y_ld);
  PT_REQUIRE(dense_epilogue_known(epilogue), "pt_gemm_f32: epilogue %d (store, relu2, glu, gelu-mul, softcap or xielu)", epilogue);
  const char *bad = dense_ext_error(epilogue, n, ext);
  PT_REQUIRE(!bad, "pt_gemm_f32: %s", bad);
  const bool grouped = ext && ext->n_groups > 0;
  PT_REQUIRE(!grouped || (ext->group_rows == f32::BM && m % f32::BM == 0), "pt_gemm_f32: groups come in tiles of %d rows", f32::BM);
  PT_REQUIRE(ceil_div(m, f32::BM) <= 65535, "pt_gemm_f32: m=%d too large", m);
  f32::gemm_f32_kernel<<<dim3(ceil_div(n, f32::BN), ceil_div(m, f32::BM)), f32::THREADS, 0, as_stream(stream)>>>(
      x, x_ld, w, w_ld, m, n, k, grouped ? ext->group_of : nullptr, make_dense_out(y, y_ld, PT_DT_F32, epilogue, alpha, ext));
  PT_LAUNCH_CHECK("pt_gemm_f32");
  return PT_OK;
}
