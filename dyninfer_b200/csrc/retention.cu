// Retention: linear attention with a fixed decay per head, no softmax and no denominator.
//
// Decode rows: one cluster per (head, row). A CTA of the cluster owns a slice of the value columns of
// the head's state: it rotates q and k, updates its part of S in place (one read, one write of the f32
// state: the kernel is bound by that traffic) and forms its part of o = S^T q; the squared sums of the
// slices meet through distributed shared memory, so norm and gate are applied in the same launch.
//
// Portions: chunks of 64 tokens, all chunks at once.
//   U_c = sum_{t in c} decay^{last - t} k_t v_t^T        (retention_chunk_state_kernel)
//   P_c = state before chunk c, by a scan over the U_c     (retention_scan_kernel; leaves the new state)
//   o_t = sum_{s <= t, s in c} decay^{t-s} (q_t . k_s) v_s + decay^{t+1-first} P_c^T q_t, then norm and
//   gate                                                   (retention_chunk_out_kernel)
// Scores, decays and states are 32-bit quantities. Heads of up to 128 x 128 run these products on the tensor
// cores with every f32 operand as a pair of tf32 terms (x = hi + lo to 2^-21; hi hi + hi lo + lo hi, the
// "3xTF32" scheme of CUTLASS's examples); sessions that compute in f32 and other head sizes run them on the
// vector pipes.
#include <cooperative_groups.h>

#include <algorithm>

#include "mixers.cuh"
#include "tf32x3.cuh"

namespace cg = cooperative_groups;

namespace dyn {
namespace {

constexpr int RT_C = 64;      // tokens per chunk
constexpr int RT_PITCH = RT_C + 4;
constexpr int RT_SLICE = 32;  // reduction elements staged at a time
constexpr int RT_PRE = 16;    // state rows a decode thread fetches ahead

__device__ __forceinline__ void load4(float* dst, const float* src) {  // src 16-byte aligned
  const float4 v = *reinterpret_cast<const float4*>(src);
  dst[0] = v.x, dst[1] = v.y, dst[2] = v.z, dst[3] = v.w;
}

// ---- decode: independent rows ----------------------------------------------------------------
__global__ void __launch_bounds__(256) retention_step_kernel(RetentionArgs a, const int64_t* row_pos,
                                                             const int64_t* row_seq, int64_t pos0, int64_t seq0,
                                                             int64_t row0) {
  extern __shared__ float rs_smem[];
  __shared__ float part_ss, red_ss[8];
  const cg::cluster_group cl = cg::this_cluster();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = a.dim, E = a.vdim, nsplit = gridDim.x;
  const int h = blockIdx.y;
  const int64_t r = row0 + blockIdx.z;
  const int per = (E + nsplit - 1) / nsplit, e0 = min((int)blockIdx.x * per, E), ne = min(per, E - e0);
  float* qs = rs_smem;           // [D]
  float* ks = qs + D;            // [D]
  float* red = ks + D;           // [8][per]
  float* os = red + 8 * per;     // [per]
  pdl_trigger();
  const int64_t pos = row_pos ? row_pos[r] : pos0, seq = row_seq ? row_seq[r] : seq0;
  // the state was written one token ago, with ordinary launches in between, so its first 128 rows are fetched
  // before the kernel waits for this token's products
  float* S = a.state + ((seq * a.heads + h) * D) * (int64_t)E + e0;
  float pre[RT_PRE];
#pragma unroll
  for (int j = 0; j < RT_PRE; j++) pre[j] = warp + 8 * j < D && lane < ne && pos > 0 ? S[(int64_t)(warp + 8 * j) * E + lane] : 0.f;
  pdl_wait();
  const float decay = a.decay[h], kscale = 1.0f / sqrtf((float)D);
  const float* q = a.q.ptr + r * a.q.ld + (int64_t)h * D;
  const float* k = a.k.ptr + r * a.k.ld + (int64_t)h * D;
  const float* v = a.v.ptr + r * a.v.ld + (int64_t)h * E + e0;
  const int half = a.rot_dims / 2;
  for (int i = tid; i < D; i += 256) {
    if (i < half) {
      float sv, cv;
      sincos_position(pos, a.freq[i], &sv, &cv);
      const float q0 = q[i], q1 = q[i + half], k0 = k[i], k1 = k[i + half];
      qs[i] = q0 * cv - q1 * sv, qs[i + half] = q1 * cv + q0 * sv;
      ks[i] = (k0 * cv - k1 * sv) * kscale, ks[i + half] = (k1 * cv + k0 * sv) * kscale;
    } else if (i >= 2 * half) {
      qs[i] = q[i], ks[i] = k[i] * kscale;
    }
  }
  __syncthreads();
  for (int c = lane; c < ne; c += 32) {
    const float vv = v[c];
    float acc = 0.f;
    int first = warp;
    if (c == lane) {
#pragma unroll
      for (int j = 0; j < RT_PRE; j++) {
        const int d = warp + 8 * j;
        if (d < D) {
          const float n = fmaf(decay, pre[j], ks[d] * vv);
          S[(int64_t)d * E + c] = n;
          acc = fmaf(n, qs[d], acc);
        }
      }
      first += 8 * RT_PRE;
    }
    for (int d0 = first; d0 < D; d0 += 64) {  // eight rows of the state in flight per thread
      float s[8];
#pragma unroll
      for (int j = 0; j < 8; j++) s[j] = (d0 + 8 * j < D && pos > 0) ? S[(int64_t)(d0 + 8 * j) * E + c] : 0.f;
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const int d = d0 + 8 * j;
        if (d < D) {
          const float n = fmaf(decay, s[j], ks[d] * vv);
          S[(int64_t)d * E + c] = n;
          acc = fmaf(n, qs[d], acc);
        }
      }
    }
    red[warp * per + c] = acc;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < ne; c += 256) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) o += red[w * per + c];
    os[c] = o;
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red_ss[warp] = ss;
  __syncthreads();
  if (tid == 0) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) t += red_ss[w];
    part_ss = t;
  }
  cl.sync();
  float total = 0.f;
  for (int i = 0; i < nsplit; i++) total += *cl.map_shared_rank(&part_ss, i);
  cl.sync();  // nobody leaves while another CTA still reads its sum
  const float inv = 1.0f / sqrtf(total / (float)E + a.eps);
  const float* g = a.g.ptr + r * a.g.ld + (int64_t)h * E + e0;
  float* out = a.out + r * (int64_t)a.heads * E + (int64_t)h * E + e0;
  for (int c = tid; c < ne; c += 256) out[c] = os[c] * inv * silu_of(g[c]);
}

int step_rows(const RetentionArgs& a, const int64_t* pos, const int64_t* seq, int64_t pos0, int64_t seq0, int64_t row0,
              int64_t rows, cudaStream_t st) {
  int nsplit = 1;
  while (nsplit < 8 && a.vdim / (nsplit * 2) >= 32) nsplit *= 2;
  const int per = (a.vdim + nsplit - 1) / nsplit;
  const size_t smem = (size_t)(2 * a.dim + 9 * per) * 4;
  DYN_CHECK(smem <= 48 * 1024, "retention: head of %d x %d is too large", a.dim, a.vdim);
  for (int64_t r0 = 0; r0 < rows; r0 += 65535) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)nsplit, (unsigned)a.heads, (unsigned)std::min<int64_t>(65535, rows - r0));
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2] = {};
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = (unsigned)nsplit, attr[0].val.clusterDim.y = 1, attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    // a portion run token by token has no ordinary launch between its states: no early start there
    cfg.attrs = attr, cfg.numAttrs = pos && pdl_enabled() ? 2 : 1;
    DYN_CUDA(cudaLaunchKernelEx(&cfg, retention_step_kernel, a, pos, seq, pos0, seq0, row0 + r0));
    count_launch();
  }
  return 0;
}

// ---- portions ---------------------------------------------------------------------------------
// q and k of a portion rotated in place (k also scaled): thread = (row, head, pair or passed dim).
__global__ void __launch_bounds__(256) retention_rotate_kernel(RetentionArgs a, int64_t rows, int64_t base) {
  const int half = a.rot_dims / 2, per = a.dim - half;  // pairs, then the dims that pass
  const int64_t total = rows * a.heads * per;
  const float kscale = 1.0f / sqrtf((float)a.dim);
  for (int64_t it = blockIdx.x * 256ll + threadIdx.x; it < total; it += (int64_t)gridDim.x * 256) {
    const int i = (int)(it % per);
    const int64_t rh = it / per, h = rh % a.heads, r = rh / a.heads;
    float* q = a.q.ptr + r * a.q.ld + h * a.dim;
    float* k = a.k.ptr + r * a.k.ld + h * a.dim;
    if (i < half) {
      float sv, cv;
      sincos_position(base + r, a.freq[i], &sv, &cv);
      const float q0 = q[i], q1 = q[i + half], k0 = k[i], k1 = k[i + half];
      q[i] = q0 * cv - q1 * sv, q[i + half] = q1 * cv + q0 * sv;
      k[i] = (k0 * cv - k1 * sv) * kscale, k[i + half] = (k1 * cv + k0 * sv) * kscale;
    } else {
      k[i + half] *= kscale;
    }
  }
}

// U[c][h][d][e], one 64 x 64 tile of (d, e) per CTA.
__global__ void __launch_bounds__(64) retention_chunk_state_kernel(RetentionArgs a, int64_t rows) {
  __shared__ __align__(16) float ks[RT_C][64], vs[RT_C][64];
  const int tid = threadIdx.x, tx = tid & 7, ty = tid >> 3;
  const int D = a.dim, E = a.vdim, et = (E + 63) / 64;
  const int64_t c = blockIdx.x, t0 = c * RT_C;
  const int h = blockIdx.y, d0 = (int)(blockIdx.z / et) * 64, e0 = (int)(blockIdx.z % et) * 64;
  const int n = (int)min((int64_t)RT_C, rows - t0);
  const float decay = a.decay[h];
  for (int t = 0; t < n; t++) {
    const float wt = powf(decay, (float)(n - 1 - t));
    const float* kr = a.k.ptr + (t0 + t) * a.k.ld + (int64_t)h * D + d0;
    const float* vr = a.v.ptr + (t0 + t) * a.v.ld + (int64_t)h * E + e0;
    ks[t][tid] = d0 + tid < D ? kr[tid] * wt : 0.f;
    vs[t][tid] = e0 + tid < E ? vr[tid] : 0.f;
  }
  __syncthreads();
  float acc[8][8] = {};
  for (int t = 0; t < n; t++) {
    float kv[8], vv[8];
    load4(kv, &ks[t][4 * ty]);
    load4(kv + 4, &ks[t][32 + 4 * ty]);
    load4(vv, &vs[t][4 * tx]);
    load4(vv + 4, &vs[t][32 + 4 * tx]);
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
      for (int j = 0; j < 8; j++) acc[i][j] = fmaf(kv[i], vv[j], acc[i][j]);
  }
  float* U = a.scratch + ((c * a.heads + h) * D) * (int64_t)E;
#pragma unroll
  for (int i = 0; i < 8; i++) {
    const int d = d0 + (i < 4 ? 4 * ty + i : 28 + 4 * ty + i);
    if (d >= D) continue;
#pragma unroll
    for (int j = 0; j < 8; j++) {
      const int e = e0 + (j < 4 ? 4 * tx + j : 28 + 4 * tx + j);
      if (e < E) U[(int64_t)d * E + e] = acc[i][j];
    }
  }
}

// U[c] -> state before chunk c; the slot's state -> state after the portion.
__global__ void __launch_bounds__(256) retention_scan_kernel(RetentionArgs a, int64_t rows, int64_t base, int64_t slot) {
  const int64_t per = (int64_t)a.dim * a.vdim, plane = a.heads * per;
  const int64_t idx = blockIdx.x * 256ll + threadIdx.x;
  if (idx >= plane) return;
  const float decay = a.decay[idx / per];
  const float full = powf(decay, (float)RT_C);
  float* st = a.state + slot * plane + idx;
  float S = base > 0 ? *st : 0.f;
  const int64_t nc = (rows + RT_C - 1) / RT_C;
  for (int64_t c0 = 0; c0 < nc; c0 += 8) {
    float u[8];
#pragma unroll
    for (int j = 0; j < 8; j++) u[j] = c0 + j < nc ? a.scratch[(c0 + j) * plane + idx] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; j++) {
      const int64_t c = c0 + j;
      if (c >= nc) break;
      a.scratch[c * plane + idx] = S;
      const int64_t n = min((int64_t)RT_C, rows - c * RT_C);
      S = fmaf(n == RT_C ? full : powf(decay, (float)n), S, u[j]);
    }
  }
  *st = S;
}

// One (chunk, head) per CTA: scores, products with the values and with the state before the chunk,
// norm and gate. EC = 64-column groups of the value dim.
template <int EC>
__global__ void __launch_bounds__(256) retention_chunk_out_kernel(RetentionArgs a, int64_t rows, int64_t base) {
  extern __shared__ __align__(16) float ro_smem[];
  constexpr int BP = EC * 64 + 4;
  float(*Qt)[RT_PITCH] = reinterpret_cast<float(*)[RT_PITCH]>(ro_smem);                       // [slice][t]
  float(*Kt)[RT_PITCH] = Qt + RT_SLICE;                                                        // [slice][s]
  float(*At)[RT_PITCH] = Kt + RT_SLICE;                                                        // [s][t]
  float(*Bs)[BP] = reinterpret_cast<float(*)[BP]>(At + RT_C);                                 // [slice][e]
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int D = a.dim, E = a.vdim;
  const int64_t c = blockIdx.x, t0 = c * RT_C;
  const int h = blockIdx.y;
  const int n = (int)min((int64_t)RT_C, rows - t0);
  const float decay = a.decay[h];
  const float* qp = a.q.ptr + t0 * a.q.ld + (int64_t)h * D;
  const float* kp = a.k.ptr + t0 * a.k.ld + (int64_t)h * D;
  const float* vp = a.v.ptr + t0 * a.v.ld + (int64_t)h * E;
  // ---- scores of the chunk, decayed and causal
  {
    float s[4][4] = {};
    for (int d0 = 0; d0 < D; d0 += RT_SLICE) {
#pragma unroll
      for (int j = 0; j < RT_C * RT_SLICE / 256; j++) {
        const int i = tid + 256 * j, t = i / RT_SLICE, d = i % RT_SLICE;
        const bool live = t < n && d0 + d < D;
        Qt[d][t] = live ? qp[t * a.q.ld + d0 + d] : 0.f;
        Kt[d][t] = live ? kp[t * a.k.ld + d0 + d] : 0.f;
      }
      __syncthreads();
#pragma unroll 8
      for (int d = 0; d < RT_SLICE; d++) {
        float qv[4], kv[4];
        load4(qv, &Qt[d][4 * ty]);
        load4(kv, &Kt[d][4 * tx]);
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
          for (int j = 0; j < 4; j++) s[i][j] = fmaf(qv[i], kv[j], s[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const int t = 4 * ty + i, u = 4 * tx + j;
        At[u][t] = u <= t ? s[i][j] * powf(decay, (float)(t - u)) : 0.f;
      }
  }
  float o[4][EC * 4] = {};
  auto accumulate = [&](float (*L)[RT_PITCH]) {
#pragma unroll 8
    for (int k = 0; k < RT_SLICE; k++) {
      float av[4];
      load4(av, &L[k][4 * ty]);
#pragma unroll
      for (int g = 0; g < EC; g++) {
        float bv[4];
        load4(bv, &Bs[k][64 * g + 4 * tx]);
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
          for (int j = 0; j < 4; j++) o[i][4 * g + j] = fmaf(av[i], bv[j], o[i][4 * g + j]);
      }
    }
  };
  // ---- scores x values
  for (int s0 = 0; s0 < n; s0 += RT_SLICE) {
    for (int i = tid; i < RT_SLICE * EC * 64; i += 256) {
      const int k = i / (EC * 64), e = i % (EC * 64);
      Bs[k][e] = s0 + k < n && e < E ? vp[(s0 + k) * a.v.ld + e] : 0.f;
    }
    __syncthreads();  // also covers the scores' stores before the first use
    accumulate(At + s0);
    __syncthreads();
  }
  // ---- the state before the chunk
  if (c > 0 || base > 0) {
    const float* P = a.scratch + ((c * a.heads + h) * D) * (int64_t)E;
    for (int d0 = 0; d0 < D; d0 += RT_SLICE) {
#pragma unroll
      for (int j = 0; j < RT_C * RT_SLICE / 256; j++) {
        const int i = tid + 256 * j, t = i / RT_SLICE, d = i % RT_SLICE;
        Qt[d][t] = t < n && d0 + d < D ? qp[t * a.q.ld + d0 + d] * powf(decay, (float)(t + 1)) : 0.f;
      }
      for (int i = tid; i < RT_SLICE * EC * 64; i += 256) {
        const int k = i / (EC * 64), e = i % (EC * 64);
        Bs[k][e] = d0 + k < D && e < E ? P[(int64_t)(d0 + k) * E + e] : 0.f;
      }
      __syncthreads();
      accumulate(Qt);
      __syncthreads();
    }
  }
  // ---- norm over the head's value dims (columns past E hold zeros), gate
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int t = 4 * ty + i;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < EC * 4; j++) ss = fmaf(o[i][j], o[i][j], ss);
#pragma unroll
    for (int m = 8; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if (t >= n) continue;
    const float inv = 1.0f / sqrtf(ss / (float)E + a.eps);
    const float* g = a.g.ptr + (t0 + t) * a.g.ld + (int64_t)h * E;
    float* out = a.out + (t0 + t) * (int64_t)a.heads * E + (int64_t)h * E;
#pragma unroll
    for (int j = 0; j < EC * 4; j++) {
      const int e = 64 * (j / 4) + 4 * tx + j % 4;
      if (e < E) out[e] = o[i][j] * inv * silu_of(g[e]);
    }
  }
}

template <int EC>
int chunk_out(const RetentionArgs& a, int64_t rows, int64_t base, cudaStream_t st) {
  const int smem = (int)((2 * RT_SLICE + RT_C) * RT_PITCH + RT_SLICE * (EC * 64 + 4)) * 4;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(retention_chunk_out_kernel<EC>), smem)) return 1;
  retention_chunk_out_kernel<EC><<<dim3((unsigned)((rows + RT_C - 1) / RT_C), (unsigned)a.heads), 256, smem, st>>>(a, rows, base);
  count_launch();
  return 0;
}

// ---- the same two products on the tensor cores -----------------------------------------------------------
constexpr int TC_D = 128;  // widest head (dim and vdim)
constexpr int TC_AP = TC_D + 4, TC_BP = TC_D + 8, TC_SP = RT_C + 4;  // pitches: A-side and B-side fragment reads conflict-free

// rows x cols floats (cols <= 128, both 16-byte aligned) into shared memory, zeros to `fill_rows` x 128
__device__ __forceinline__ void stage_rows(float* dst, int pitch, const float* src, int64_t ld, int rows, int cols, int fill_rows,
                                           int tid, int threads) {
  for (int i = tid; i < fill_rows * (TC_D / 4); i += threads) {
    const int r = i / (TC_D / 4), c = (i % (TC_D / 4)) * 4;
    const bool live = r < rows && c < cols;
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst + r * pitch + c);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(live ? src + r * ld + c : src), "r"(live ? 16 : 0)
                 : "memory");
  }
}

constexpr int TCS_SMEM = RT_C * (TC_BP + 72) * 4;
constexpr int TC_THREADS = 512;  // sixteen warps: four groups of 16 rows x four of 32 columns
// U of one (chunk, head, 64 rows of the state): A = (decayed k)^T, B = v. Columns past vdim hold zeros.
__global__ void __launch_bounds__(TC_THREADS) retention_chunk_state_tc_kernel(RetentionArgs a, int64_t rows) {
  extern __shared__ __align__(16) float ts_smem[];
  float* vs = ts_smem;                 // [t][TC_BP]
  float* ks = vs + RT_C * TC_BP;       // [t][72]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int D = a.dim, E = a.vdim, h = blockIdx.y, d0 = blockIdx.z * 64;
  const int64_t c = blockIdx.x, t0 = c * RT_C;
  const int n = (int)min((int64_t)RT_C, rows - t0);
  stage_rows(vs, TC_BP, a.v.ptr + t0 * a.v.ld + (int64_t)h * E, a.v.ld, n, E, RT_C, tid, TC_THREADS);
  for (int i = tid; i < RT_C * 16; i += TC_THREADS) {
    const int t = i / 16, d = (i % 16) * 4;
    const bool live = t < n && d0 + d < D;
    const float* src = a.k.ptr + t0 * a.k.ld + (int64_t)h * D;
    const unsigned dst = (unsigned)__cvta_generic_to_shared(ks + t * 72 + d);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(live ? src + t * a.k.ld + d0 + d : src),
                 "r"(live ? 16 : 0) : "memory");
  }
  const float decay = a.decay[h];
  const int mt = warp & 3, nq = warp >> 2;
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  float acc[4][4] = {};
#pragma unroll
  for (int kk = 0; kk < RT_C / 8; kk++) {
    const int ta = 8 * kk + t4, tb = ta + 4;
    const float wa = ta < n ? powf(decay, (float)(n - 1 - ta)) : 0.f, wb = tb < n ? powf(decay, (float)(n - 1 - tb)) : 0.f;
    const float *ka = ks + ta * 72 + 16 * mt + g, *kb = ks + tb * 72 + 16 * mt + g;
    AFrag f;
    split_into(f, 0, ka[0] * wa), split_into(f, 1, ka[8] * wa), split_into(f, 2, kb[0] * wb), split_into(f, 3, kb[8] * wb);
    mma3<4>(acc, f, [&](int nt, int half) { return vs[(half ? tb : ta) * TC_BP + nq * 32 + 8 * nt + g]; });
  }
  float* U = a.scratch + ((c * a.heads + h) * D) * (int64_t)E;
#pragma unroll
  for (int nt = 0; nt < 4; nt++) {
    const int e = nq * 32 + 8 * nt + 2 * t4;
    if (e >= E) continue;
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int d = d0 + 16 * mt + g + 8 * i;
      if (d < D) *reinterpret_cast<float2*>(U + (int64_t)d * E + e) = make_float2(acc[nt][2 * i], acc[nt][2 * i + 1]);
    }
  }
}

constexpr int TCO_SMEM = (2 * RT_C * TC_AP + RT_C * TC_BP + TC_D * TC_BP + RT_C * TC_SP + 4 * RT_C) * 4;
// Outputs of one (chunk, head). Warp: 16 tokens x a quarter of the keys, then x a quarter of the value columns.
__global__ void __launch_bounds__(TC_THREADS) retention_chunk_out_tc_kernel(RetentionArgs a, int64_t rows, int64_t base) {
  extern __shared__ __align__(16) float to_smem[];
  float* qs = to_smem;                 // [t][TC_AP]
  float* ks = qs + RT_C * TC_AP;       // [s][TC_AP]
  float* vs = ks + RT_C * TC_AP;       // [s][TC_BP]
  float* ps = vs + RT_C * TC_BP;       // [d][TC_BP]
  float* ss = ps + TC_D * TC_BP;       // [t][TC_SP]
  float* sums = ss + RT_C * TC_SP;     // [column quarter][t]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int D = a.dim, E = a.vdim, h = blockIdx.y;
  const int64_t c = blockIdx.x, t0 = c * RT_C;
  const int n = (int)min((int64_t)RT_C, rows - t0);
  const int mt = warp & 3, nq = warp >> 2;
  const bool past = c > 0 || base > 0;
  stage_rows(qs, TC_AP, a.q.ptr + t0 * a.q.ld + (int64_t)h * D, a.q.ld, n, D, RT_C, tid, TC_THREADS);
  stage_rows(ks, TC_AP, a.k.ptr + t0 * a.k.ld + (int64_t)h * D, a.k.ld, n, D, RT_C, tid, TC_THREADS);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (past) stage_rows(ps, TC_BP, a.scratch + ((c * a.heads + h) * D) * (int64_t)E, E, D, E, (D + 7) / 8 * 8, tid, TC_THREADS);
  stage_rows(vs, TC_BP, a.v.ptr + t0 * a.v.ld + (int64_t)h * E, a.v.ld, n, E, RT_C, tid, TC_THREADS);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const float decay = a.decay[h];
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  // ---- decayed causal scores
  {
    float s[2][4] = {};
    if (nq <= mt) {  // keys 16 nq .. are not all later than the tokens
#pragma unroll 4
      for (int d = 0; d < D; d += 8) {
        AFrag f;
        const float* q = qs + (16 * mt + g) * TC_AP + d + t4;
        split_into(f, 0, q[0]), split_into(f, 1, q[8 * TC_AP]), split_into(f, 2, q[4]), split_into(f, 3, q[8 * TC_AP + 4]);
        mma3<2>(s, f, [&](int nt, int half) { return ks[(nq * 16 + 8 * nt + g) * TC_AP + d + t4 + 4 * half]; });
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; nt++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = 16 * mt + g + 8 * (e >> 1), u = nq * 16 + 8 * nt + 2 * t4 + (e & 1);
        ss[t * TC_SP + u] = u <= t ? s[nt][e] * powf(decay, (float)(t - u)) : 0.f;
      }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  float o[4][4] = {};
  auto accumulate = [&](const float* A, int pitch, int depth, const float* B) {
#pragma unroll 2
    for (int k = 0; k < depth; k += 8) {
      AFrag f;
      const float* p = A + (16 * mt + g) * pitch + k + t4;
      split_into(f, 0, p[0]), split_into(f, 1, p[8 * pitch]), split_into(f, 2, p[4]), split_into(f, 3, p[8 * pitch + 4]);
      mma3<4>(o, f, [&](int nt, int half) { return B[(k + t4 + 4 * half) * TC_BP + nq * 32 + 8 * nt + g]; });
    }
  };
  if (past) {  // the state before the chunk, decayed to each token
    accumulate(qs, TC_AP, D, ps);
    const float w0 = powf(decay, (float)(16 * mt + g + 1)), w1 = powf(decay, (float)(16 * mt + g + 9));
#pragma unroll
    for (int nt = 0; nt < 4; nt++) o[nt][0] *= w0, o[nt][1] *= w0, o[nt][2] *= w1, o[nt][3] *= w1;
  }
  accumulate(ss, TC_SP, 16 * (mt + 1), vs);  // later keys score zero
  // ---- norm over the head's value dims (columns past E hold zeros), gate
  float q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int nt = 0; nt < 4; nt++) {
    q0 = fmaf(o[nt][0], o[nt][0], q0), q0 = fmaf(o[nt][1], o[nt][1], q0);
    q1 = fmaf(o[nt][2], o[nt][2], q1), q1 = fmaf(o[nt][3], o[nt][3], q1);
  }
  q0 += __shfl_xor_sync(0xffffffffu, q0, 1), q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
  q1 += __shfl_xor_sync(0xffffffffu, q1, 1), q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
  if (t4 == 0) sums[nq * RT_C + 16 * mt + g] = q0, sums[nq * RT_C + 16 * mt + g + 8] = q1;
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int t = 16 * mt + g + 8 * i;
    if (t >= n) continue;
    const float inv = 1.0f / sqrtf(((sums[t] + sums[RT_C + t]) + (sums[2 * RT_C + t] + sums[3 * RT_C + t])) / (float)E + a.eps);
    const float* gate = a.g.ptr + (t0 + t) * a.g.ld + (int64_t)h * E;
    float* out = a.out + (t0 + t) * (int64_t)a.heads * E + (int64_t)h * E;
#pragma unroll
    for (int nt = 0; nt < 4; nt++) {
      const int e = nq * 32 + 8 * nt + 2 * t4;
      if (e >= E) continue;
      const float2 z = *reinterpret_cast<const float2*>(gate + e);
      *reinterpret_cast<float2*>(out + e) = make_float2(o[nt][2 * i] * inv * silu_of(z.x), o[nt][2 * i + 1] * inv * silu_of(z.y));
    }
  }
}

// Heads the tensor-core kernels take: whole MMA steps, rows that 16-byte copies can read.
bool tensor_core_shape(const RetentionArgs& a) {
  auto ok = [](const Rows& r) { return r.ld % 4 == 0 && (reinterpret_cast<uintptr_t>(r.ptr) & 15) == 0; };
  return !a.exact && a.dim <= TC_D && a.vdim <= TC_D && a.dim % 8 == 0 && a.vdim % 8 == 0 && ok(a.q) && ok(a.k) && ok(a.v) && ok(a.g);
}

bool chunked_shape(const RetentionArgs& a) { return a.vdim <= 256; }

}  // namespace

size_t retention_scratch_floats(const RetentionArgs& a, int64_t rows) {
  return chunked_shape(a) ? (size_t)((rows + RT_C - 1) / RT_C) * a.heads * a.dim * a.vdim : 0;
}

int launch_retention(const RetentionArgs& a, const StepRows& r, cudaStream_t st) {
  if (r.rows == 0) return 0;
  if (r.base < 0) return step_rows(a, r.pos, r.seq, 0, 0, 0, r.rows, st);
  if (r.rows == 1) return step_rows(a, nullptr, nullptr, r.base, r.slot, 0, 1, st);
  if (!chunked_shape(a)) {  // wide value heads: token by token
    for (int64_t i = 0; i < r.rows; i++)
      if (step_rows(a, nullptr, nullptr, r.base + i, r.slot, i, 1, st)) return 1;
    return 0;
  }
  const unsigned nc = (unsigned)((r.rows + RT_C - 1) / RT_C);
  {
    const int64_t total = r.rows * a.heads * (a.dim - a.rot_dims / 2);
    retention_rotate_kernel<<<(unsigned)std::min<int64_t>((total + 255) / 256, 148 * 16), 256, 0, st>>>(a, r.rows, r.base);
    const unsigned dt = (unsigned)((a.dim + 63) / 64), et = (unsigned)((a.vdim + 63) / 64);
    if (tensor_core_shape(a)) {
      if (ensure_dynamic_smem(reinterpret_cast<const void*>(retention_chunk_state_tc_kernel), TCS_SMEM)) return 1;
      retention_chunk_state_tc_kernel<<<dim3(nc, (unsigned)a.heads, dt), TC_THREADS, TCS_SMEM, st>>>(a, r.rows);
    } else {
      retention_chunk_state_kernel<<<dim3(nc, (unsigned)a.heads, dt * et), 64, 0, st>>>(a, r.rows);
    }
    const int64_t plane = (int64_t)a.heads * a.dim * a.vdim;
    retention_scan_kernel<<<(unsigned)((plane + 255) / 256), 256, 0, st>>>(a, r.rows, r.base, r.slot);
    count_launch(3);
  }
  if (tensor_core_shape(a)) {
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(retention_chunk_out_tc_kernel), TCO_SMEM)) return 1;
    retention_chunk_out_tc_kernel<<<dim3(nc, (unsigned)a.heads), TC_THREADS, TCO_SMEM, st>>>(a, r.rows, r.base);
    count_launch();
    DYN_CUDA(cudaGetLastError());
    return 0;
  }
  const int ec = (a.vdim + 63) / 64;
  if (ec == 1 ? chunk_out<1>(a, r.rows, r.base, st) : ec == 2 ? chunk_out<2>(a, r.rows, r.base, st)
                                                            : chunk_out<4>(a, r.rows, r.base, st))
    return 1;
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace dyn
