// Streaming GEMV for plain bf16 / f16 weights and one to four activation rows (f32 accumulate).
//
// The dense path of the reference widens bf16 / f16 to f32 exactly and multiplies in f32
// (crates/dyninfer-compiler/src/lowering/kernels.rs:741-772,1157-1173). The matrices are read once per
// step, so this kernel is HBM-bound: 2 bytes per weight, one widening and one FMA per weight and row.
//
// Sixteen warps per CTA, two CTAs per SM (one for several activation rows); a warp owns whole weight rows,
// dealt so that consecutive rows go to different SMs (a projection has fewer rows than the GPU has warps).
// A warp's rows are one run of pieces of 256 weights (16 bytes per lane), fetched eight at a time; the first
// eight are under way before the kernel waits for its predecessor: weights depend on nothing in the stream.
// (Refilling each piece as it is used looks deeper but is not: loads share scoreboards, so the wait for the
// oldest piece waits for younger ones; 61 instead of 31 us on 32768 x 2048.) The activation row is held in
// shared memory as f32, split in two planes of four so that a lane's two reads are conflict-free.
//
// The activations may be formed on the way in: RMSNorm of the rows, or silu(gate) * up of [gate | up]
// rows. Every CTA repeats that for itself, which costs less than a launch of its own.
#include <algorithm>

#include "common.cuh"

namespace dyn {
namespace {

constexpr int GP_WARPS = 16;
constexpr int GP_DEPTH = 8;  // pieces in flight per warp

template <bool BF16>
__device__ __forceinline__ void widen8(const uint4& w, float (&f)[8]) {
  const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
  for (int i = 0; i < 4; i++) {
    if (BF16) {
      f[2 * i] = __uint_as_float(u[i] << 16);
      f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    } else {
      f[2 * i] = __half2float(__ushort_as_half((unsigned short)(u[i] & 0xffffu)));
      f[2 * i + 1] = __half2float(__ushort_as_half((unsigned short)(u[i] >> 16)));
    }
  }
}

// y[m][n] = sum_k x[m][k] * w[n][k] (+ residual). K % 256 == 0, M <= 4.
template <bool BF16, int M>
__global__ void __launch_bounds__(GP_WARPS * 32, M == 1 ? 2 : 1) gemv_plain_kernel(const uint8_t* __restrict__ w, int64_t N, int K,
                                                                   const void* __restrict__ x, int x_bf16, GemvInput in,
                                                                   float* y, const float* residual) {
  extern __shared__ __align__(16) float gp_xs[];  // [M][2][K / 8] float4
  __shared__ float red[GP_WARPS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_trigger();
  const int64_t warps = (int64_t)gridDim.x * GP_WARPS, wid = (int64_t)warp * gridDim.x + blockIdx.x;
  const int64_t lo = N * wid / warps, hi = N * (wid + 1) / warps;
  const int pieces = K / 256;
  const int64_t total = (hi - lo) * pieces;
  const uint4* src = reinterpret_cast<const uint4*>(w + (size_t)lo * K * 2) + lane;  // rows of the run are contiguous
  uint4 buf[GP_DEPTH];
  auto fetch = [&](int64_t i0) {
#pragma unroll
    for (int j = 0; j < GP_DEPTH; j++)
      if (i0 + j < total) buf[j] = __ldcs(src + (i0 + j) * 32);
  };
  fetch(0);
  // the weights do not depend on earlier kernels of the stream; the activations do
  pdl_wait();
  float4* xs = reinterpret_cast<float4*>(gp_xs);
  const int K8 = K / 8;
  auto at = [&](int m, int k) -> float& { return gp_xs[(((m * 2 + ((k >> 2) & 1)) * K8 + (k >> 3)) << 2) + (k & 3)]; };
  if (in.mode == GEMV_NORM) {
    const float* xf = reinterpret_cast<const float*>(x);
    for (int m = 0; m < M; m++) {
      float ss = 0.f;
      for (int i = tid; i < K; i += GP_WARPS * 32) {
        const float v = xf[(int64_t)m * K + i];
        at(m, i) = v;
        ss = fmaf(v, v, ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) red[warp] = ss;
      __syncthreads();
      ss = 0.f;
#pragma unroll
      for (int i = 0; i < GP_WARPS; i++) ss += red[i];
      const float inv = 1.0f / sqrtf(ss / (float)K + in.eps);
      for (int i = tid; i < K; i += GP_WARPS * 32)  // the thread's own elements
        at(m, i) = __fmul_rn(__fmul_rn(at(m, i), inv), aux_load(reinterpret_cast<const uint8_t*>(in.norm_w), in.norm_type, i));
      __syncthreads();
    }
  } else if (in.mode == GEMV_SWIGLU) {
    const float* gu = reinterpret_cast<const float*>(x);
    for (int i = tid; i < M * K; i += GP_WARPS * 32) {
      const int m = M == 1 ? 0 : i / K, k = i - m * K;
      const float g = gu[(int64_t)m * 2 * K + k];
      at(m, k) = (g / (1.0f + expf(-g))) * gu[(int64_t)m * 2 * K + K + k];
    }
    __syncthreads();
  } else {
    for (int i = tid; i < M * K; i += GP_WARPS * 32) {
      const int m = M == 1 ? 0 : i / K, k = i - m * K;
      at(m, k) = x_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(x)[i]) : reinterpret_cast<const float*>(x)[i];
    }
    __syncthreads();
  }
  float acc[M][2];
#pragma unroll
  for (int m = 0; m < M; m++) acc[m][0] = acc[m][1] = 0.f;
  int64_t row = lo;
  int piece = 0;
  for (int64_t i0 = 0; i0 < total; i0 += GP_DEPTH) {
    if (i0) fetch(i0);
#pragma unroll
    for (int j = 0; j < GP_DEPTH; j++) {
      if (i0 + j >= total) break;
      float f[8];
      widen8<BF16>(buf[j], f);
      const int k8 = piece * 32 + lane;
#pragma unroll
      for (int m = 0; m < M; m++) {
        const float4 a = xs[(m * 2) * K8 + k8], b = xs[(m * 2 + 1) * K8 + k8];
        acc[m][0] = fmaf(a.x, f[0], acc[m][0]), acc[m][1] = fmaf(b.x, f[4], acc[m][1]);
        acc[m][0] = fmaf(a.y, f[1], acc[m][0]), acc[m][1] = fmaf(b.y, f[5], acc[m][1]);
        acc[m][0] = fmaf(a.z, f[2], acc[m][0]), acc[m][1] = fmaf(b.z, f[6], acc[m][1]);
        acc[m][0] = fmaf(a.w, f[3], acc[m][0]), acc[m][1] = fmaf(b.w, f[7], acc[m][1]);
      }
      if (++piece == pieces) {
#pragma unroll
        for (int m = 0; m < M; m++) {
          const float v = warp_sum(acc[m][0] + acc[m][1]);
          if (lane == 0) y[(int64_t)m * N + row] = residual ? v + residual[(int64_t)m * N + row] : v;
          acc[m][0] = acc[m][1] = 0.f;
        }
        piece = 0, row++;
      }
    }
  }
}

template <bool BF16, int M>
int run_plain(const WRef& w, const void* x, int x_type, const GemvInput& in, float* y, const float* residual, cudaStream_t s) {
  const int K = (int)w.cols;
  const size_t smem = (size_t)M * K * 4;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(gemv_plain_kernel<BF16, M>), (int)std::max<size_t>(smem, 48 * 1024)))
    return 1;
  const int grid = (int)std::min<int64_t>((M == 1 && smem <= 96 * 1024 ? 2 : 1) * std::max(1, sm_count()), w.rows);
  DYN_CUDA(launch_pdl(gemv_plain_kernel<BF16, M>, dim3(grid), dim3(GP_WARPS * 32), smem, s, w.data, (int64_t)w.rows, K,
                      x, x_type == E_BF16 ? 1 : 0, in, y, residual));
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace

bool gemv_plain_takes(const WRef& w, int64_t M) {
  return (w.enc == E_BF16 || w.enc == E_F16) && M >= 1 && M <= 4 && w.cols % 256 == 0 && w.rows >= 1 &&
         (size_t)M * w.cols * 4 <= 160 * 1024 && (reinterpret_cast<uintptr_t>(w.data) & 15) == 0;
}

// *handled = false when the encoding or shape does not qualify (the caller uses another kernel).
int launch_gemv_plain(const WRef& w, const void* x, int x_type, int M, float* y, const float* residual,
                      cudaStream_t s, bool* handled, const GemvInput& in) {
  *handled = false;
  if (!gemv_plain_takes(w, M)) return 0;
  DYN_CHECK(in.mode == GEMV_PLAIN || x_type == E_F32, "gemv: normalised or gated input must be f32");
  int rc;
  const bool bf = w.enc == E_BF16;
  switch (M) {
    case 1: rc = bf ? run_plain<true, 1>(w, x, x_type, in, y, residual, s) : run_plain<false, 1>(w, x, x_type, in, y, residual, s); break;
    case 2: rc = bf ? run_plain<true, 2>(w, x, x_type, in, y, residual, s) : run_plain<false, 2>(w, x, x_type, in, y, residual, s); break;
    case 3: rc = bf ? run_plain<true, 3>(w, x, x_type, in, y, residual, s) : run_plain<false, 3>(w, x, x_type, in, y, residual, s); break;
    default: rc = bf ? run_plain<true, 4>(w, x, x_type, in, y, residual, s) : run_plain<false, 4>(w, x, x_type, in, y, residual, s); break;
  }
  if (rc) return rc;
  *handled = true;
  return 0;
}

}  // namespace dyn
