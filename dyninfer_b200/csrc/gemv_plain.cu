// Streaming GEMV for plain bf16 / f16 weights and one to four activation rows (f32 accumulate).
//
// The dense path of the reference widens bf16 / f16 to f32 exactly and multiplies in f32
// (crates/dyninfer-compiler/src/lowering/kernels.rs:741-772,1157-1173). The matrices are read once per
// step, so this kernel is HBM-bound: 2 bytes per weight, one widening and one FMA per weight and row.
//
// One CTA per SM, 32 warps (sixteen for several activation rows). A CTA owns a block of outputs; its weight rows,
// each cut into `parts` equal spans of K when there are fewer rows than warps, are dealt to the warps as
// contiguous runs of pieces of 256 weights (16 bytes per lane), fetched eight at a time; the first
// eight are under way before the kernel waits for its predecessor: weights depend on nothing in the stream.
// (Refilling each piece as it is used looks deeper but is not: loads share scoreboards, so the wait for the
// oldest piece waits for younger ones; 61 instead of 31 us on 32768 x 2048.) The activation row is held in
// shared memory as f32, split in two planes of four so that a lane's two reads are conflict-free. The sums meet
// in shared memory and leave as coalesced stores.
//
// The activations may be formed on the way in (RMSNorm of the rows: every CTA repeats it for itself, which
// costs less than a launch of its own), and the outputs on the way out: of a matrix [gate; up] a CTA takes
// the rows of its outputs from both halves and writes silu(gate) * up.
#include <limits.h>

#include <algorithm>

#include "common.cuh"

namespace dyn {
namespace {

__host__ __device__ constexpr int gp_warps(int m) { return m == 1 ? 32 : 16; }
constexpr int GP_DEPTH = 8;  // pieces in flight per warp
constexpr int GP_SMEM = 208 * 1024;

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

// y[m][n] = sum_k x[m][k] * w[n][k] (+ residual), or with PAIRS y[m][n] = silu(w[n] . x) * (w[N / 2 + n] . x) for
// n < N / 2. K % 256 == 0, M <= 4.
template <bool BF16, int M, bool PAIRS>
__global__ void __launch_bounds__(gp_warps(M) * 32, 1) gemv_plain_kernel(const uint8_t* __restrict__ w, int64_t N, int K, int parts,
                                                                         const void* __restrict__ x, int x_bf16, GemvForm form,
                                                                         float* y, const float* residual) {
  constexpr int WARPS = gp_warps(M), THREADS = WARPS * 32;
  extern __shared__ __align__(16) float gp_xs[];  // [M][2][K / 8] float4, then sums [M][units]
  __shared__ float red[WARPS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_trigger();
  const int64_t outs = PAIRS ? N / 2 : N;
  const int64_t out0 = outs * blockIdx.x / gridDim.x;
  const int own = (int)(outs * (blockIdx.x + 1) / gridDim.x - out0);
  const int units = own * (PAIRS ? 2 : 1) * parts, span = K / 256 / parts;  // unit = span of one row
  const int ulo = units * warp / WARPS, uhi = units * (warp + 1) / WARPS;
  const int total = (uhi - ulo) * span;
  // with PAIRS the CTA's rows are two blocks, out0.. and N / 2 + out0..: the run jumps where the second begins
  const int jump = PAIRS ? (own * parts - ulo) * span : 0;
  const int64_t across = PAIRS ? (outs - own) * (int64_t)(K / 8) : 0;
  const uint4* src = reinterpret_cast<const uint4*>(w + (size_t)out0 * K * 2) + (int64_t)ulo * span * 32 + lane;
  uint4 buf[GP_DEPTH];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int j = 0; j < GP_DEPTH; j++)
      if (i0 + j < total) buf[j] = __ldcs(src + (int64_t)(i0 + j) * 32 + (PAIRS && i0 + j >= jump ? across : 0));
  };
  fetch(0);
  // the weights do not depend on earlier kernels of the stream; the activations do
  pdl_wait();
  float4* xs = reinterpret_cast<float4*>(gp_xs);
  const int K8 = K / 8;
  auto at = [&](int m, int k) -> float& { return gp_xs[(((m * 2 + ((k >> 2) & 1)) * K8 + (k >> 3)) << 2) + (k & 3)]; };
  if (form.norm_w) {
    const float* xf = reinterpret_cast<const float*>(x);
    for (int m = 0; m < M; m++) {
      float ss = 0.f;
      for (int i = tid; i < K; i += THREADS) {
        const float v = xf[(int64_t)m * K + i];
        at(m, i) = v;
        ss = fmaf(v, v, ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) red[warp] = ss;
      __syncthreads();
      ss = warp_sum(lane < WARPS ? red[lane] : 0.f);
      const float inv = 1.0f / sqrtf(ss / (float)K + form.eps);
      for (int i = tid; i < K; i += THREADS)  // the thread's own elements
        at(m, i) = __fmul_rn(__fmul_rn(at(m, i), inv), aux_load(reinterpret_cast<const uint8_t*>(form.norm_w), form.norm_type, i));
      __syncthreads();
    }
  } else {
    for (int i = tid; i < M * K; i += THREADS) {
      const int m = M == 1 ? 0 : i / K, k = i - m * K;
      at(m, k) = x_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(x)[i]) : reinterpret_cast<const float*>(x)[i];
    }
    __syncthreads();
  }
  float* sums = gp_xs + M * K;
  float acc[M][2];
#pragma unroll
  for (int m = 0; m < M; m++) acc[m][0] = acc[m][1] = 0.f;
  int unit = ulo, piece = 0, part = parts > 1 ? ulo % parts : 0;
  for (int i0 = 0; i0 < total; i0 += GP_DEPTH) {
    if (i0) fetch(i0);
#pragma unroll
    for (int j = 0; j < GP_DEPTH; j++) {
      if (i0 + j >= total) break;
      float f[8];
      widen8<BF16>(buf[j], f);
      const int k8 = (part * span + piece) * 32 + lane;
#pragma unroll
      for (int m = 0; m < M; m++) {
        const float4 a = xs[(m * 2) * K8 + k8], b = xs[(m * 2 + 1) * K8 + k8];
        acc[m][0] = fmaf(a.x, f[0], acc[m][0]), acc[m][1] = fmaf(b.x, f[4], acc[m][1]);
        acc[m][0] = fmaf(a.y, f[1], acc[m][0]), acc[m][1] = fmaf(b.y, f[5], acc[m][1]);
        acc[m][0] = fmaf(a.z, f[2], acc[m][0]), acc[m][1] = fmaf(b.z, f[6], acc[m][1]);
        acc[m][0] = fmaf(a.w, f[3], acc[m][0]), acc[m][1] = fmaf(b.w, f[7], acc[m][1]);
      }
      if (++piece == span) {
#pragma unroll
        for (int m = 0; m < M; m++) {
          const float v = warp_sum(acc[m][0] + acc[m][1]);
          if (lane == 0) sums[m * units + unit] = v;
          acc[m][0] = acc[m][1] = 0.f;
        }
        piece = 0, unit++;
        if (++part == parts) part = 0;
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < M * own; i += THREADS) {
    const int m = M == 1 ? 0 : i / own, o = i - m * own;
    auto row_sum = [&](int r) {
      const float* p = sums + m * units + r * parts;
      float v = p[0];
      for (int k = 1; k < parts; k++) v += p[k];
      return v;
    };
    const int64_t at = (int64_t)m * outs + out0 + o;
    const float v = row_sum(o);
    if (PAIRS)
      y[at] = (v / (1.0f + expf(-v))) * row_sum(own + o);
    else {
      const float b = form.bias ? v + aux_load(reinterpret_cast<const uint8_t*>(form.bias), form.bias_type, out0 + o) : v;
      y[at] = residual ? b + residual[at] : b;
    }
  }
}

// How many spans to cut the rows into: the fewest pieces, plus one for the sum of each span, of any warp.
int plan_parts(int rows, int pieces, int warps) {
  int best = 1, cost = INT_MAX;
  for (int p : {1, 2, 4, 8}) {
    if (pieces % p) continue;
    const int c = (rows * p + warps - 1) / warps * (pieces / p + 1);
    if (c < cost) cost = c, best = p;
  }
  return best;
}

template <bool BF16, int M, bool PAIRS>
int run_plain(const WRef& w, const void* x, int x_type, const GemvForm& form, float* y, const float* residual, cudaStream_t s) {
  const int K = (int)w.cols;
  const int64_t outs = PAIRS ? w.rows / 2 : w.rows;
  const int grid = (int)std::min<int64_t>(std::max(1, sm_count()), outs);
  const int rows = (int)((outs + grid - 1) / grid) * (PAIRS ? 2 : 1);  // of the fullest CTA
  const int parts = plan_parts(rows, K / 256, gp_warps(M));
  const size_t smem = ((size_t)M * K + (size_t)M * rows * parts) * 4;
  const auto kernel = gemv_plain_kernel<BF16, M, PAIRS>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), GP_SMEM)) return 1;
  DYN_CUDA(launch_pdl(kernel, dim3(grid), dim3(gp_warps(M) * 32), smem, s, w.data, (int64_t)w.rows, K, parts, x,
                      x_type == E_BF16 ? 1 : 0, form, y, residual));
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

template <bool BF16, int M>
int run_form(const WRef& w, const void* x, int x_type, const GemvForm& form, float* y, const float* residual, cudaStream_t s) {
  return form.pairs ? run_plain<BF16, M, true>(w, x, x_type, form, y, residual, s)
                    : run_plain<BF16, M, false>(w, x, x_type, form, y, residual, s);
}

}  // namespace

bool gemv_plain_takes(const WRef& w, int64_t M) {
  // activation rows and the sums of a CTA's rows (at most eight spans each) in shared memory
  const int64_t rows = w.rows / std::max(1, sm_count()) + 2;
  return (w.enc == E_BF16 || w.enc == E_F16) && M >= 1 && M <= 4 && w.cols % 256 == 0 && w.rows >= 1 &&
         M * (w.cols + rows * 8) * 4 <= GP_SMEM && (reinterpret_cast<uintptr_t>(w.data) & 15) == 0;
}

// *handled = false when the encoding or shape does not qualify (the caller uses another kernel).
int launch_gemv_plain(const WRef& w, const void* x, int x_type, int M, float* y, const float* residual,
                      cudaStream_t s, bool* handled, const GemvForm& form) {
  *handled = false;
  if (!gemv_plain_takes(w, M)) return 0;
  DYN_CHECK(!form.norm_w || x_type == E_F32, "gemv: normalised input must be f32");
  DYN_CHECK(!form.pairs || !form.bias, "gemv: pairs have no bias");
  DYN_CHECK(!form.pairs || (w.rows % 2 == 0 && !residual), "gemv: pairs need an even row count and no residual");
  int rc;
  const bool bf = w.enc == E_BF16;
  switch (M) {
    case 1: rc = bf ? run_form<true, 1>(w, x, x_type, form, y, residual, s) : run_form<false, 1>(w, x, x_type, form, y, residual, s); break;
    case 2: rc = bf ? run_form<true, 2>(w, x, x_type, form, y, residual, s) : run_form<false, 2>(w, x, x_type, form, y, residual, s); break;
    case 3: rc = bf ? run_form<true, 3>(w, x, x_type, form, y, residual, s) : run_form<false, 3>(w, x, x_type, form, y, residual, s); break;
    default: rc = bf ? run_form<true, 4>(w, x, x_type, form, y, residual, s) : run_form<false, 4>(w, x, x_type, form, y, residual, s); break;
  }
  if (rc) return rc;
  *handled = true;
  return 0;
}

}  // namespace dyn
