// Products in f32 only: y[m, n] = sum_k x[m, k] w[n, k] with plain weights widened exactly, f32
// multiplies and f32 accumulation in ascending k. Serves sessions that compute in 32-bit, and plain
// weights whose shapes the tensor-core and streaming kernels do not take (any K, any alignment).
//
// One CTA = 64 rows x 64 outputs, 256 threads of 4 x 4, K in slices of 16 through shared memory.
#include "codec.cuh"
#include "mixers.cuh"

namespace dyn {
namespace {

constexpr int GF_T = 64, GF_K = 16, GF_P = GF_T + 4;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const uint8_t* __restrict__ w, int w_type, int64_t N, int64_t K, const uint8_t* __restrict__ x,
                int x_type, int64_t M, float* y, const float* residual) {
  __shared__ __align__(16) float xs[GF_K][GF_P], ws[GF_K][GF_P];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int64_t n0 = (int64_t)blockIdx.x * GF_T, m0 = (int64_t)blockIdx.y * GF_T;
  float acc[4][4] = {};
  pdl_trigger();
  for (int64_t k0 = 0; k0 < K; k0 += GF_K) {
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int i = tid + 256 * j, r = i / GF_K, k = i % GF_K;
      const bool kin = k0 + k < K;
      xs[k][r] = kin && m0 + r < M ? aux_load(x, x_type, (m0 + r) * K + k0 + k) : 0.f;
      ws[k][r] = kin && n0 + r < N ? aux_load(w, w_type, (n0 + r) * K + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GF_K; k++) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][4 * ty]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][4 * tx]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int64_t m = m0 + 4 * ty + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int64_t n = n0 + 4 * tx + j;
      if (n < N) y[m * N + n] = residual ? acc[i][j] + residual[m * N + n] : acc[i][j];
    }
  }
}

}  // namespace

int launch_gemm_f32(const WRef& w, const void* x, int x_type, int64_t m, float* y, const float* residual,
                    cudaStream_t s) {
  DYN_CHECK(w.enc == E_F32 || w.enc == E_F16 || w.enc == E_BF16, "f32 product: encoding %d is not a plain type", w.enc);
  if (m == 0 || w.rows == 0) return 0;
  const int64_t mt = (m + GF_T - 1) / GF_T;
  DYN_CHECK(mt <= 65535, "f32 product: %lld rows are too many for one launch", (long long)m);
  gemm_f32_kernel<<<dim3((unsigned)((w.rows + GF_T - 1) / GF_T), (unsigned)mt), 256, 0, s>>>(
      w.data, w.enc, w.rows, w.cols, reinterpret_cast<const uint8_t*>(x), x_type, m, y, residual);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace dyn
