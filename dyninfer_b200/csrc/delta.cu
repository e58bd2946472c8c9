// Gated delta rule: linear attention whose state is corrected towards each value,
//   S <- g_t S;  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t,
// behind short causal convolutions of q, k and v, with a norm per head and an output gate.
//
// The convolutions' inputs live in a ring of `taps` rows per slot, position p in row p mod taps, so a decode
// step writes its own row while other CTAs still read the rows before it.
//
// Decode rows: one cluster per (head, row), a CTA per slice of the value columns. The state arrives in shared
// memory while the step's products are still under way; convolution, unit norms, decay and step size are formed
// by every CTA for itself; one pass over the state gives S^T k and S^T q, because o = g S^T q + (k . q) u; the squared
// sums of the slices meet through distributed shared memory.
//
// Portions: convolution, gates and unit norms of all rows at once; then
//   * a few rows, f32 sessions and unusual heads: one CTA per (head, value slice) walks the tokens, state in
//     shared memory (delta_tokens_kernel);
//   * otherwise chunks of 64 tokens. With b_t the decay from the chunk's start through t, the corrections of a chunk
//     solve (I + A) u = beta v - beta b (K S_0), A_ts = beta_t b_t / b_s (k_t . k_s) for s < t. delta_chunk_kernel forms
//     T = (I + A)^-1 by 16 x 16 blocks, U = T (beta v), W = T (beta b k) and P_ts = b_t / b_s (q_t . k_s) for every chunk at
//     once; delta_scan_kernel walks the chunks: V = U - W S, o = b (Q S) + P V, S <- b_C S + (K b_C / b)^T V, a
//     CTA per (head, 32 or 16 value columns): half of its warps hold the state in registers and form corrections and updates,
//     the other half the outputs. All products with pairs of tf32 terms.
// delta_finish_kernel applies norm and gate to a portion's rows; delta_finish_operand_kernel leaves them as the dequant
// GEMM's activation operand.
#include <cooperative_groups.h>

#include <algorithm>

#include "mixers.cuh"
#include "tf32x3.cuh"

namespace cg = cooperative_groups;

namespace dyn {
namespace {

constexpr int DL_C = 64;        // tokens per chunk
constexpr int DL_THREADS = 256;
constexpr int DL_FEW = 16;      // portions up to this long walk their tokens

__host__ __device__ inline int64_t channels_of(const DeltaArgs& a) {
  return 2ll * a.kv_heads * a.dim + (int64_t)a.heads * a.vdim;
}
__device__ __forceinline__ float decay_log(const DeltaArgs& a, int h, float z) {
  return -expf(vec_at(a.a_log, h)) * softplus_of(z + vec_at(a.dt, h));
}
__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src),
               "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// One head of q, k or v: where its inputs, weights and ring channels are. Slots 0 .. 2 kv_heads + heads - 1.
struct HeadIn {
  const float* x;   // row 0
  int64_t ld, ch;   // floats between rows; first ring channel
  Vec w;
  int64_t w0;       // first channel of its weights
  int n;
};
__device__ __forceinline__ HeadIn head_in(const DeltaArgs& a, int slot) {
  HeadIn s;
  const int G = a.kv_heads, part = slot < G ? 0 : slot < 2 * G ? 1 : 2, h = slot - part * G;
  const Rows& r = part == 0 ? a.q : part == 1 ? a.k : a.v;
  s.n = part < 2 ? a.dim : a.vdim;
  s.w0 = (int64_t)h * s.n;
  s.x = r.ptr + s.w0, s.ld = r.ld;
  s.ch = (int64_t)min(part, 2) * G * a.dim + s.w0;
  s.w = part == 0 ? a.conv_q : part == 1 ? a.conv_k : a.conv_v;
  return s;
}

__device__ __forceinline__ float block_total(float v, float* red) {  // red: 8 floats; all 256 threads
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) t += red[w];
  return t;
}

// One token of one (head, slice): S [D][per] in shared memory is updated, os[c] = o.
// red: [2][8][per]; us: [per]. q and k final, kq = k . q.
__device__ __forceinline__ void delta_token(float* S, int D, int per, int ne, const float* ks, const float* qs, const float* vs,
                                            float g, float beta, float kq, float* red, float* us, float* os) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int c = lane; c < ne; c += 32) {
    float rk = 0.f, rq = 0.f;
    for (int d = warp; d < D; d += 8) {
      const float s = S[d * per + c];
      rk = fmaf(s, ks[d], rk), rq = fmaf(s, qs[d], rq);
    }
    red[warp * per + c] = rk, red[(8 + warp) * per + c] = rq;
  }
  __syncthreads();
  for (int c = tid; c < ne; c += DL_THREADS) {
    float rk = 0.f, rq = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) rk += red[w * per + c], rq += red[(8 + w) * per + c];
    const float u = beta * (vs[c] - g * rk);
    us[c] = u;
    os[c] = fmaf(kq, u, g * rq);
  }
  __syncthreads();
  for (int c = lane; c < ne; c += 32) {
    const float u = us[c];
    for (int d = warp; d < D; d += 8) S[d * per + c] = fmaf(g, S[d * per + c], ks[d] * u);
  }
}

// ---- decode: independent rows ----------------------------------------------------------------
// Everything that earlier tokens left (state, convolution history) is gathered before the wait for this token's
// products. Sums over the state run on the convolved q and k as they are; their lengths enter afterwards, as factors.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire;" ::: "memory"); }

__global__ void __launch_bounds__(DL_THREADS) delta_step_kernel(DeltaArgs a, const int64_t* row_pos, const int64_t* row_seq,
                                                                int64_t pos0, int64_t seq0, int64_t row0, int wide) {
  extern __shared__ __align__(16) float dl_smem[];
  __shared__ float part_ss, red[3];
  const cg::cluster_group cl = cg::this_cluster();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = a.dim, E = a.vdim, nsplit = gridDim.x, h = blockIdx.y;
  const int64_t r = row0 + blockIdx.z, C = channels_of(a);
  const int per = (E + nsplit - 1) / nsplit, e0 = min((int)blockIdx.x * per, E), ne = min(per, E - e0);
  float* S = dl_smem;             // [D][per]
  float* us = S + D * per;        // [per]
  float* os = us + per;           // [per]
  float* sums = os + per;         // [2][8][per]
  float* qs = sums + 16 * per;    // [D]
  float* ks = qs + D;             // [D]
  float* vs = ks + D;             // [per]
  float* w0s = vs + per;          // [2 D + per] weights of the current input
  pdl_trigger();
  const int64_t pos = row_pos ? row_pos[r] : pos0, seq = row_seq ? row_seq[r] : seq0;
  // the state was written one token ago, with ordinary launches in between
  float* Sg = a.state + ((seq * a.heads + h) * D) * (int64_t)E + e0;
  if (pos > 0 && wide) {  // whole pieces of four columns
    const int q4 = per / 4;
    for (int i = tid; i < D * q4; i += DL_THREADS) {
      const int d = i / q4, c = (i - d * q4) * 4;
      if (c < ne) cp_async16(S + d * per + c, Sg + (int64_t)d * E + c, true);
    }
  } else {
    for (int d = warp; d < D; d += 8)
      for (int c = lane; c < ne; c += 32) {
        if (pos > 0) cp_async4(S + d * per + c, Sg + (int64_t)d * E + c);
        else S[d * per + c] = 0.f;
      }
  }
  cp_commit();
  const int group = a.heads / a.kv_heads, j = h / group;
  const HeadIn hq = head_in(a, j), hk = head_in(a, a.kv_heads + j), hv = head_in(a, 2 * a.kv_heads + h);
  float* ring = a.ring + seq * (int64_t)a.taps * C;
  const int now = (int)(pos % a.taps), back = (int)min(pos, (int64_t)(a.taps - 1)), channels = 2 * D + ne;
  // channel i of this CTA: q, k, its columns of v. First what the earlier inputs add to its convolution.
  auto locate = [&](int i, int* c) -> const HeadIn& {
    *c = i < D ? i : i < 2 * D ? i - D : e0 + i - 2 * D;
    return i < D ? hq : i < 2 * D ? hk : hv;
  };
  for (int i = tid; i < channels; i += DL_THREADS) {
    int c;
    const HeadIn& s = locate(i, &c);
    const int64_t w = (s.w0 + c) * a.taps + a.taps - 1, ch = s.ch + c;
    float wt[3], x[3], u = 0.f;
#pragma unroll
    for (int t = 1; t <= 3; t++) {  // in flight together
      wt[t - 1] = t <= back ? vec_at(s.w, w - t) : 0.f;
      x[t - 1] = t <= back ? ring[(now >= t ? now - t : now - t + a.taps) * C + ch] : 0.f;
    }
#pragma unroll
    for (int t = 0; t < 3; t++) u = fmaf(wt[t], x[t], u);
    for (int t = 4; t <= back; t++) u = fmaf(vec_at(s.w, w - t), ring[(now >= t ? now - t : now - t + a.taps) * C + ch], u);
    qs[i] = u;  // a thread's own channels until the block meets
    w0s[i] = vec_at(s.w, w);
  }
  const float A = expf(vec_at(a.a_log, h)), dt = vec_at(a.dt, h);
  pdl_wait();
  const bool keeps = blockIdx.x == 0 && h % group == 0;  // this CTA writes the head's ring rows of q and k
  float* row = ring + now * C;
  const float zb = a.b.ptr[r * a.b.ld + h], za = a.a.ptr[r * a.a.ld + h];
  const float* gate = a.g.ptr + r * a.g.ld + (int64_t)h * E + e0;
  const float gate0 = tid < ne ? gate[tid] : 0.f;
  for (int i = tid; i < channels; i += DL_THREADS) {
    int c;
    const HeadIn& s = locate(i, &c);
    const float x = s.x[r * s.ld + c];
    qs[i] = silu_of(fmaf(w0s[i], x, qs[i]));
    if (keeps || i >= 2 * D) row[s.ch + c] = x;
  }
  cp_wait<0>();
  __syncthreads();
  if (warp < 3) {  // squared lengths and the product of q and k
    const float *x = warp == 1 ? ks : qs, *y = warp == 0 ? qs : ks;
    float t = 0.f;
    for (int d = lane; d < D; d += 32) t = fmaf(x[d], y[d], t);
    t = warp_sum(t);
    if (lane == 0) red[warp] = t;
  }
  for (int c = lane; c < ne; c += 32) {
    float rk = 0.f, rq = 0.f;
#pragma unroll 8
    for (int d = warp; d < D; d += 8) {
      const float s = S[d * per + c];
      rk = fmaf(s, ks[d], rk), rq = fmaf(s, qs[d], rq);
    }
    sums[warp * per + c] = rk, sums[(8 + warp) * per + c] = rq;
  }
  const float beta = sigmoid_of(zb), g = expf(-A * softplus_of(za + dt));
  __syncthreads();
  if (warp == 0) {
    const float iq = 1.0f / sqrtf(red[0] + a.unit_eps) * (1.0f / sqrtf((float)D)), ik = 1.0f / sqrtf(red[1] + a.unit_eps);
    float ss = 0.f;
    for (int c = lane; c < ne; c += 32) {
      float rk = 0.f, rq = 0.f;
#pragma unroll
      for (int w = 0; w < 8; w++) rk += sums[w * per + c], rq += sums[(8 + w) * per + c];
      const float u = beta * (vs[c] - g * (rk * ik)), o = fmaf(red[2] * iq * ik, u, g * (rq * iq));
      us[c] = u * ik, os[c] = o;
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) part_ss = ss;
  }
  __syncthreads();
  cluster_arrive();  // the slices' sums meet while the state is written back
  for (int c = lane; c < ne; c += 32) {
    const float u = us[c];
#pragma unroll 8
    for (int d = warp; d < D; d += 8) Sg[(int64_t)d * E + c] = fmaf(g, S[d * per + c], ks[d] * u);
  }
  cluster_wait();
  float total = 0.f;
  for (int i = 0; i < nsplit; i++) total += *cl.map_shared_rank(&part_ss, i);
  cluster_arrive();
  const float inv = 1.0f / sqrtf(total / (float)E + a.eps);
  float* out = a.out + r * (int64_t)a.heads * E + (int64_t)h * E + e0;
  for (int c = tid; c < ne; c += DL_THREADS) out[c] = os[c] * inv * vec_at(a.norm, e0 + c) * silu_of(c == tid ? gate0 : gate[c]);
  cluster_wait();  // nobody leaves while another CTA still reads its sum
}

constexpr int DL_MAX_SMEM = 200 * 1024;

int step_rows(const DeltaArgs& a, const int64_t* pos, const int64_t* seq, int64_t pos0, int64_t seq0, int64_t rows,
              cudaStream_t st) {
  int nsplit = 1;
  while (nsplit < 8 && (a.vdim + nsplit - 1) / nsplit > 32) nsplit *= 2;
  const int per = (a.vdim + nsplit - 1) / nsplit;
  const size_t smem = ((size_t)a.dim * per + 4 * a.dim + 20 * per) * 4;
  DYN_CHECK(smem <= DL_MAX_SMEM, "delta rule: head of %d x %d is too large", a.dim, a.vdim);
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(delta_step_kernel), DL_MAX_SMEM)) return 1;
  const int wide = per % 4 == 0 && a.vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
  for (int64_t r0 = 0; r0 < rows; r0 += 65535) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)nsplit, (unsigned)a.heads, (unsigned)std::min<int64_t>(65535, rows - r0));
    cfg.blockDim = dim3(DL_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2] = {};
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = (unsigned)nsplit, attr[0].val.clusterDim.y = 1, attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr, cfg.numAttrs = pos && pdl_enabled() ? 2 : 1;
    DYN_CUDA(cudaLaunchKernelEx(&cfg, delta_step_kernel, a, pos, seq, pos0, seq0, r0, wide));
    count_launch();
  }
  return 0;
}

// ---- portions ---------------------------------------------------------------------------------
// Scratch of a portion: convolved rows [rows][q | k | v], gates [rows][beta | log g], then per chunk and head W, U, P and
// decays [b_t | b_C / b_t].
struct DeltaScratch {
  float *cv, *gates, *w, *u, *p, *decay, *end;
};
__host__ __device__ inline DeltaScratch carve(const DeltaArgs& a, int64_t rows) {
  const int64_t nc = (rows + DL_C - 1) / DL_C, ch = nc * a.heads;
  DeltaScratch s;
  s.cv = a.scratch;
  s.gates = s.cv + (rows * channels_of(a) + 3) / 4 * 4;
  s.w = s.gates + (rows * 2 * a.heads + 3) / 4 * 4;
  s.u = s.w + ch * DL_C * ((a.dim + 3) / 4 * 4);
  s.p = s.u + ch * DL_C * ((a.vdim + 3) / 4 * 4);
  s.decay = s.p + ch * DL_C * DL_C;
  s.end = s.decay + ch * 2 * DL_C;
  return s;
}

constexpr int DV_ROWS = 8;  // consecutive rows a warp convolves
// Warp = (eight rows, one head of q, k or v). TAPS: compile-time window (taps <= TAPS), 0: any.
template <int TAPS>
__global__ void __launch_bounds__(DL_THREADS) delta_conv_kernel(DeltaArgs a, int64_t rows, int64_t base, int64_t slot) {
  const DeltaScratch sc = carve(a, rows);
  const int lane = threadIdx.x & 31;
  const int slots = 2 * a.kv_heads + a.heads;
  const int64_t item = blockIdx.x * 8ll + (threadIdx.x >> 5), groups = (rows + DV_ROWS - 1) / DV_ROWS;
  if (item >= groups * slots) return;
  const int s = (int)(item % slots);
  const int64_t r0 = item / slots * DV_ROWS, C = channels_of(a);
  const HeadIn in = head_in(a, s);
  const float* ring = a.ring + slot * (int64_t)a.taps * C;
  const int live = (int)min((int64_t)DV_ROWS, rows - r0);
  const bool unit = s < 2 * a.kv_heads;
  float ss[DV_ROWS] = {};
  for (int c = lane; c < in.n; c += 32) {
    auto input = [&](int64_t row) -> float {  // row < 0: before the portion
      if (row >= 0) return in.x[row * in.ld + c];
      const int64_t p = base + row;
      return p >= 0 ? ring[(p % a.taps) * C + in.ch + c] : 0.f;
    };
    float* out = sc.cv + r0 * C + in.ch + c;
    if constexpr (TAPS > 0) {
      float w[TAPS], x[TAPS + DV_ROWS - 1];
#pragma unroll
      for (int t = 0; t < TAPS; t++) w[t] = t >= TAPS - a.taps ? vec_at(in.w, (in.w0 + c) * a.taps + t - (TAPS - a.taps)) : 0.f;
#pragma unroll
      for (int t = 0; t < TAPS + DV_ROWS - 1; t++) {
        const int64_t row = r0 + t - (TAPS - 1);
        x[t] = t >= TAPS - a.taps && row < rows ? input(row) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < DV_ROWS; i++) {
        if (i < live) {
          float u = w[TAPS - 1] * x[i + TAPS - 1];
#pragma unroll
          for (int j = 1; j < TAPS; j++) u = fmaf(w[TAPS - 1 - j], x[i + TAPS - 1 - j], u);
          u = silu_of(u);
          out[i * C] = u;
          ss[i] = fmaf(u, u, ss[i]);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < DV_ROWS; i++) {
        if (i < live) {
          float u = 0.f;
          for (int j = 0; j < a.taps; j++) u = fmaf(vec_at(in.w, (in.w0 + c) * a.taps + a.taps - 1 - j), input(r0 + i - j), u);
          u = silu_of(u);
          out[i * C] = u;
          ss[i] = fmaf(u, u, ss[i]);
        }
      }
    }
  }
  if (unit) {
    const float extra = s < a.kv_heads ? 1.0f / sqrtf((float)a.dim) : 1.0f;
#pragma unroll
    for (int i = 0; i < DV_ROWS; i++) ss[i] = 1.0f / sqrtf(warp_sum(ss[i]) + a.unit_eps) * extra;
    for (int c = lane; c < in.n; c += 32) {  // the lane's own elements
      float* out = sc.cv + r0 * C + in.ch + c;
#pragma unroll
      for (int i = 0; i < DV_ROWS; i++)
        if (i < live) out[i * C] *= ss[i];
    }
  } else if (lane < live) {
    const int h = s - 2 * a.kv_heads;
    const int64_t r = r0 + lane;
    sc.gates[r * 2 * a.heads + h] = sigmoid_of(a.b.ptr[r * a.b.ld + h]);
    sc.gates[r * 2 * a.heads + a.heads + h] = decay_log(a, h, a.a.ptr[r * a.a.ld + h]);
  }
}

constexpr int DX_ROWS = 4;  // consecutive rows a warp convolves below
// The same for windows of up to four taps and heads of whole groups of four channels, NV * 128 at most: a lane holds four
// neighbouring channels, every input is in flight before the first is used, and rows leave once, in final form.
template <int NV>
__global__ void __launch_bounds__(DL_THREADS) delta_conv_wide_kernel(DeltaArgs a, int64_t rows, int64_t base, int64_t slot) {
  constexpr int T = 4, NX = T + DX_ROWS - 1;
  const DeltaScratch sc = carve(a, rows);
  const int lane = threadIdx.x & 31;
  const int slots = 2 * a.kv_heads + a.heads;
  const unsigned item = blockIdx.x * 8u + (threadIdx.x >> 5), groups = (unsigned)((rows + DX_ROWS - 1) / DX_ROWS);
  if (item >= groups * slots) return;
  const int s = (int)(item % slots);
  const int64_t r0 = (int64_t)(item / slots) * DX_ROWS, C = channels_of(a);
  const HeadIn in = head_in(a, s);
  const float* ring = a.ring + slot * (int64_t)a.taps * C;
  const int live = (int)min((int64_t)DX_ROWS, rows - r0);
  float4 x[NV][NX], y[NV][DX_ROWS];
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 128 * v + 4 * lane;
#pragma unroll
    for (int t = 0; t < NX; t++) {
      const int64_t row = r0 + t - (T - 1), p = base + row;
      x[v][t] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < in.n && t >= T - a.taps && row < rows) {
        if (row >= 0) x[v][t] = *reinterpret_cast<const float4*>(in.x + row * in.ld + c);
        else if (p >= 0) x[v][t] = *reinterpret_cast<const float4*>(ring + (p % a.taps) * C + in.ch + c);
      }
    }
  }
  float ss[DX_ROWS] = {};
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 128 * v + 4 * lane;
    float w[4][T];
#pragma unroll
    for (int k = 0; k < 4; k++)
#pragma unroll
      for (int t = 0; t < T; t++)
        w[k][t] = c < in.n && t >= T - a.taps ? vec_at(in.w, (in.w0 + c + k) * a.taps + t - (T - a.taps)) : 0.f;
#pragma unroll
    for (int i = 0; i < DX_ROWS; i++) {
      float u[4];
#pragma unroll
      for (int k = 0; k < 4; k++) {
        u[k] = 0.f;
#pragma unroll
        for (int t = T - 1; t >= 0; t--) {
          const float4& q = x[v][i + t];
          u[k] = fmaf(w[k][t], k == 0 ? q.x : k == 1 ? q.y : k == 2 ? q.z : q.w, u[k]);
        }
        u[k] = __fdividef(u[k], 1.0f + __expf(-u[k]));  // silu
        ss[i] = fmaf(u[k], u[k], ss[i]);
      }
      y[v][i] = make_float4(u[0], u[1], u[2], u[3]);
    }
  }
  if (s < 2 * a.kv_heads) {
    const float extra = s < a.kv_heads ? 1.0f / sqrtf((float)a.dim) : 1.0f;
#pragma unroll
    for (int i = 0; i < DX_ROWS; i++) {
      const float f = 1.0f / sqrtf(warp_sum(ss[i]) + a.unit_eps) * extra;
#pragma unroll
      for (int v = 0; v < NV; v++) y[v][i].x *= f, y[v][i].y *= f, y[v][i].z *= f, y[v][i].w *= f;
    }
  } else if (lane < live) {
    const int h = s - 2 * a.kv_heads;
    const int64_t r = r0 + lane;
    sc.gates[r * 2 * a.heads + h] = sigmoid_of(a.b.ptr[r * a.b.ld + h]);
    sc.gates[r * 2 * a.heads + a.heads + h] = decay_log(a, h, a.a.ptr[r * a.a.ld + h]);
  }
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 128 * v + 4 * lane;
    if (c >= in.n) continue;
#pragma unroll
    for (int i = 0; i < DX_ROWS; i++)
      if (i < live) *reinterpret_cast<float4*>(sc.cv + (r0 + i) * C + in.ch + c) = y[v][i];
  }
}

bool conv_wide(const DeltaArgs& a) {
  auto ok = [](const Rows& r) { return r.ld % 4 == 0 && (reinterpret_cast<uintptr_t>(r.ptr) & 15) == 0; };
  return a.taps <= 4 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.dim <= 256 && a.vdim <= 256 && ok(a.q) && ok(a.k) && ok(a.v) &&
         (reinterpret_cast<uintptr_t>(a.ring) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.scratch) & 15) == 0;
}

// The ring after the portion; a launch after the convolutions' (they read the rows before it).
__device__ __forceinline__ void keep_inputs(const DeltaArgs& a, int64_t rows, int64_t base, int64_t slot, int block, int blocks) {
  const int64_t C = channels_of(a), qk = (int64_t)a.kv_heads * a.dim, from = max((int64_t)0, rows - a.taps);
  float* ring = a.ring + slot * (int64_t)a.taps * C;
  const int64_t total = (rows - from) * C;
  for (int64_t i = block * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)blocks * blockDim.x) {
    const int64_t row = from + i / C, c = i % C;
    const float x = c < qk ? a.q.ptr[row * a.q.ld + c] : c < 2 * qk ? a.k.ptr[row * a.k.ld + c - qk] : a.v.ptr[row * a.v.ld + c - 2 * qk];
    ring[((base + row) % a.taps) * C + c] = x;
  }
}

// Token by token: CTA = (value slice, head). Leaves o without norm and gate in a.out.
__global__ void __launch_bounds__(DL_THREADS) delta_tokens_kernel(DeltaArgs a, int64_t rows, int64_t base, int64_t slot) {
  extern __shared__ __align__(16) float dt_smem[];
  const DeltaScratch sc = carve(a, rows);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = a.dim, E = a.vdim, h = blockIdx.y, j = h / (a.heads / a.kv_heads);
  const int per = (E + gridDim.x - 1) / gridDim.x, e0 = min((int)blockIdx.x * per, E), ne = min(per, E - e0);
  const int64_t C = channels_of(a), qk = (int64_t)a.kv_heads * D;
  float* S = dt_smem;              // [D][per]
  float* qs = S + D * per;         // [D]
  float* ks = qs + D;              // [D]
  float* vs = ks + D;              // [per]
  float* us = vs + per;            // [per]
  float* os = us + per;            // [per]
  float* red = os + per;           // [2][8][per]
  __shared__ float red8[8];
  keep_inputs(a, rows, base, slot, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
  float* Sg = a.state + ((slot * a.heads + h) * D) * (int64_t)E + e0;
  for (int d = warp; d < D; d += 8)
    for (int c = lane; c < ne; c += 32) S[d * per + c] = base > 0 ? Sg[(int64_t)d * E + c] : 0.f;
  for (int64_t t = 0; t < rows; t++) {
    const float* cv = sc.cv + t * C;
    float kq = 0.f;
    for (int d = tid; d < D; d += DL_THREADS) {
      const float q = cv[(int64_t)j * D + d], k = cv[qk + (int64_t)j * D + d];
      qs[d] = q, ks[d] = k;
      kq = fmaf(k, q, kq);
    }
    for (int c = tid; c < ne; c += DL_THREADS) vs[c] = cv[2 * qk + (int64_t)h * E + e0 + c];
    const float beta = sc.gates[t * 2 * a.heads + h], g = expf(sc.gates[t * 2 * a.heads + a.heads + h]);
    kq = block_total(kq, red8);
    delta_token(S, D, per, ne, ks, qs, vs, g, beta, kq, red, us, os);
    for (int c = tid; c < ne; c += DL_THREADS) a.out[t * (int64_t)a.heads * E + (int64_t)h * E + e0 + c] = os[c];
    __syncthreads();  // the token's vectors are read
  }
  for (int d = warp; d < D; d += 8)
    for (int c = lane; c < ne; c += 32) Sg[(int64_t)d * E + c] = S[d * per + c];
}

// rows x cols floats (16-byte aligned, cols % 4 == 0) into shared memory, zeros up to fill_rows x fill_cols (at most 128)
template <int THREADS = DL_THREADS>
__device__ __forceinline__ void stage(float* dst, int pitch, const float* src, int64_t ld, int rows, int cols, int fill_rows,
                                      int fill_cols) {
  const int c = (threadIdx.x & 31) * 4;  // a warp per row
  if (c >= fill_cols) return;
  int r = threadIdx.x >> 5;
  const float* p = src + r * ld + c;
  float* d = dst + r * pitch + c;
#pragma unroll 4
  for (; r < fill_rows; r += THREADS / 32, p += (THREADS / 32) * ld, d += (THREADS / 32) * pitch) {
    const bool live = r < rows && c < cols;
    cp_async16(d, live ? p : src, live);
  }
}
__device__ __forceinline__ void load_a(AFrag& f, const float* p, int pitch) {  // rows g, g + 8; columns t4, t4 + 4
  split_into(f, 0, p[0]), split_into(f, 1, p[8 * pitch]), split_into(f, 2, p[4]), split_into(f, 3, p[8 * pitch + 4]);
}

// Decays of a chunk, by one warp, two tokens a lane: with G_t the sum of log g through t (in double, kept as two floats, so
// that differences of large sums are exact), d = [G hi | G lo | beta | beta b_t | b_t | b_C / b_t] of 64 each, b_t = exp(G_t).
__device__ __forceinline__ void chunk_decay(const DeltaArgs& a, const float* gates, int64_t t0, int n, int h, float* d) {
  const int lane = threadIdx.x & 31;
  double v[2];
  float beta[2];
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int t = 2 * lane + i;
    v[i] = t < n ? (double)gates[(t0 + t) * 2 * a.heads + a.heads + h] : 0.0;
    beta[i] = t < n ? gates[(t0 + t) * 2 * a.heads + h] : 0.f;
  }
  double s = v[0] + v[1];
#pragma unroll
  for (int o = 1; o < 32; o *= 2) {
    const double other = __shfl_up_sync(0xffffffffu, s, o);
    if (lane >= o) s += other;
  }
  const double last = __shfl_sync(0xffffffffu, s, 31);
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int t = 2 * lane + i;
    const double G = i ? s : s - v[1];
    const float hi = (float)G, b = expf(hi);
    d[t] = hi, d[DL_C + t] = (float)(G - (double)hi), d[2 * DL_C + t] = beta[i], d[3 * DL_C + t] = beta[i] * b;
    d[4 * DL_C + t] = b, d[5 * DL_C + t] = expf((float)(last - G));
  }
}

constexpr int DC_D = 128;                   // widest q/k head of the chunk kernels
constexpr int DC_P = DC_D + 4, DC_S = DL_C + 4;
constexpr int DC_SMEM = (2 * DL_C * DC_P + 2 * DL_C * DC_S + 6 * DL_C) * 4;

constexpr int DC_THREADS = 512;
// W, U and P of one (chunk, head).
__global__ void __launch_bounds__(DC_THREADS, 2) delta_chunk_kernel(DeltaArgs a, int64_t rows) {
  extern __shared__ __align__(16) float dc_smem[];
  const DeltaScratch sc = carve(a, rows);
  float* ks = dc_smem;                 // [t][DC_P]
  float* qs = ks + DL_C * DC_P;        // [t][DC_P]; then blocks of v
  float* A = qs + DL_C * DC_P;         // [t][DC_S]
  float* T = A + DL_C * DC_S;          // [t][DC_S]
  float* dec = T + DL_C * DC_S;        // decays
  const float *beta = dec + 2 * DL_C, *beta_b = beta + DL_C;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int D = a.dim, E = a.vdim, h = blockIdx.y, j = h / (a.heads / a.kv_heads);
  const int64_t c = blockIdx.x, t0 = c * DL_C, C = channels_of(a), qk = (int64_t)a.kv_heads * D;
  const int n = (int)min((int64_t)DL_C, rows - t0);
  const float* cv = sc.cv + t0 * C;
  stage<DC_THREADS>(ks, DC_P, cv + qk + (int64_t)j * D, C, n, D, DL_C, D);
  stage<DC_THREADS>(qs, DC_P, cv + (int64_t)j * D, C, n, D, DL_C, D);
  cp_commit();
  if (warp == 0) chunk_decay(a, sc.gates, t0, n, h, dec);
  cp_wait<0>();
  __syncthreads();
  const int mt = warp & 3, nq = warp >> 2;   // 16 tokens x a quarter of the keys (or of the columns)
  {
    float s[2][4] = {}, p[2][4] = {};
    const int depth = nq <= mt ? D : 0;  // the other blocks' keys are all later than the tokens
#pragma unroll 2
    for (int d = 0; d < depth; d += 8) {
      AFrag fk, fq;
      load_a(fk, ks + (16 * mt + g) * DC_P + d + t4, DC_P);
      load_a(fq, qs + (16 * mt + g) * DC_P + d + t4, DC_P);
      Tf32Pair b0[2], b1[2];
#pragma unroll
      for (int nt = 0; nt < 2; nt++) {
        const float* b = ks + (nq * 16 + 8 * nt + g) * DC_P + d + t4;
        b0[nt] = tf32_split(b[0]), b1[nt] = tf32_split(b[4]);
      }
      mma3_split<2>(s, fk, b0, b1);
      mma3_split<2>(p, fq, b0, b1);
    }
    if (tid < 2 * DL_C) sc.decay[(c * a.heads + h) * 2 * DL_C + tid] = dec[4 * DL_C + tid];
    float* P = sc.p + (c * a.heads + h) * DL_C * DL_C;
#pragma unroll
    for (int nt = 0; nt < 2; nt++)
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int t = 16 * mt + g + 8 * i, u = nq * 16 + 8 * nt + 2 * t4;
        float2 pv;
        float av[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const float w = u + e <= t ? expf((dec[t] - dec[u + e]) + (dec[DL_C + t] - dec[DL_C + u + e])) : 0.f;
          (e ? pv.y : pv.x) = p[nt][2 * i + e] * w;
          av[e] = u + e < t ? beta[t] * w * s[nt][2 * i + e] : 0.f;
        }
        A[t * DC_S + u] = av[0], A[t * DC_S + u + 1] = av[1];
        *reinterpret_cast<float2*>(P + t * DL_C + u) = pv;
      }
  }
  __syncthreads();
  // ---- T = (I + A)^-1. Diagonal blocks by forward substitution, thread = (block, column); qs is free
  for (int i = tid; i < DL_C * DC_S; i += DC_THREADS) T[i] = 0.f;
  __syncthreads();
  if (tid < DL_C) {
    const int b = tid & ~15, col = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; i++) {
      float v = i == col ? 1.f : 0.f;
#pragma unroll
      for (int k = 0; k < 16; k++)
        if (k < i) v = fmaf(-A[(b + i) * DC_S + b + k], x[k], v);
      x[i] = i >= col ? v : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 16; i++) T[(b + i) * DC_S + b + col] = x[i];
  }
  __syncthreads();
  // blocks below: T_ij = -T_ii sum_{k = j .. i-1} A_ik T_kj, one block diagonal after the other
  {
    float* M = qs;  // [block][16][17]
    const int rr = (tid >> 4) & 15, cc = tid & 15, half = tid >> 8;  // two blocks at a time
    for (int dist = 1; dist < 4; dist++) {
      for (int jb = half; jb + dist < 4; jb += 2) {
        const int ib = jb + dist;
        float v = 0.f;
        for (int k0 = jb * 16; k0 < ib * 16; k0 += 16) {
#pragma unroll
          for (int k = k0; k < k0 + 16; k++) v = fmaf(A[(ib * 16 + rr) * DC_S + k], T[k * DC_S + jb * 16 + cc], v);
        }
        M[jb * 272 + rr * 17 + cc] = v;
      }
      __syncthreads();
      for (int jb = half; jb + dist < 4; jb += 2) {
        const int ib = jb + dist;
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < 16; k++) v = fmaf(-T[(ib * 16 + rr) * DC_S + ib * 16 + k], M[jb * 272 + k * 17 + cc], v);
        T[(ib * 16 + rr) * DC_S + jb * 16 + cc] = v;
      }
      __syncthreads();
    }
  }
  // ---- U = T (beta v), W = T (beta b k): 64 rows x up to 128 columns at a time, a warp 16 rows x a quarter of them
  auto product = [&](const float* B, int cols, const float* w, float* out, int64_t ld) {
    float acc[4][4] = {};
    for (int k = 0; k < 16 * (mt + 1); k += 8) {  // T is lower triangular
      AFrag f;
      load_a(f, T + (16 * mt + g) * DC_S + k + t4, DC_S);
      const int ka = k + t4, kb = ka + 4;
      const float wa = w[ka], wb = w[kb];
      mma3<4>(acc, f, [&](int nt, int half) {
        const int col = nq * 32 + 8 * nt + g;
        return col < cols ? (half ? wb * B[kb * DC_P + col] : wa * B[ka * DC_P + col]) : 0.f;
      });
    }
#pragma unroll
    for (int nt = 0; nt < 4; nt++) {
      const int col = nq * 32 + 8 * nt + 2 * t4;
      if (col >= cols) continue;
#pragma unroll
      for (int i = 0; i < 2; i++)
        *reinterpret_cast<float2*>(out + (16 * mt + g + 8 * i) * ld + col) = make_float2(acc[nt][2 * i], acc[nt][2 * i + 1]);
    }
  };
  for (int e0 = 0; e0 < E; e0 += DC_D) {
    const int cols = min(DC_D, E - e0);
    if (e0) __syncthreads();
    stage<DC_THREADS>(qs, DC_P, cv + 2 * qk + (int64_t)h * E + e0, C, n, cols, DL_C, cols);
    cp_commit();
    if (e0 == 0) product(ks, D, beta_b, sc.w + (c * a.heads + h) * DL_C * (int64_t)D, D);
    cp_wait<0>();
    __syncthreads();
    product(qs, cols, beta, sc.u + (c * a.heads + h) * DL_C * (int64_t)E + e0, E);
  }
}

constexpr int DS_THREADS = 512;                // warps 0-7: corrections and state; 8-15: outputs
constexpr int DS_KP = DC_D + 8;
constexpr int ds_pitch(int n) { return n % 16 == 8 ? n : n + 8; }  // of the split operands: conflict-free B fragments
constexpr int ds_smem(int n) {
  return (2 * DL_C * DC_P + DL_C * DS_KP + DL_C * DC_S + 2 * DC_D * ds_pitch(n) + 2 * DL_C * ds_pitch(n) + 4 * DL_C) * 4;
}

// The walk over the chunks for one (slice of 16 NT value columns, head).
template <int NT>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(DeltaArgs a, int64_t rows, int64_t base, int64_t slot) {
  constexpr int DS_N = 16 * NT, DS_B = ds_pitch(DS_N);
  extern __shared__ __align__(16) float dn_smem[];
  const DeltaScratch sc = carve(a, rows);
  float* Ws = dn_smem;                    // [t][DC_P]
  float* Qs = Ws + DL_C * DC_P;           // [t][DC_P]
  float* Ks = Qs + DL_C * DC_P;           // [t][DS_KP]
  float* Ps = Ks + DL_C * DS_KP;          // [t][DC_S]
  float* Sh = Ps + DL_C * DC_S;           // [d][DS_B] tf32 terms of the state
  float* Sl = Sh + DC_D * DS_B;
  float* Vh = Sl + DC_D * DS_B;           // [t][DS_B] of the corrections
  float* Vl = Vh + DL_C * DS_B;
  float* dec = Vl + DL_C * DS_B;          // [chunk parity][b_t | b_C / b_t]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int D = a.dim, E = a.vdim, h = blockIdx.y, j = h / (a.heads / a.kv_heads), e0 = blockIdx.x * DS_N;
  const int64_t C = channels_of(a), qk = (int64_t)a.kv_heads * D;
  const int nc = (int)((rows + DL_C - 1) / DL_C);
  auto stage_wq = [&](int c) {
    const int n = (int)min((int64_t)DL_C, rows - (int64_t)c * DL_C);
    const int64_t ch = (int64_t)c * a.heads + h;
    stage<DS_THREADS>(Ws, DC_P, sc.w + ch * DL_C * D, D, DL_C, D, DL_C, D);
    stage<DS_THREADS>(Qs, DC_P, sc.cv + (int64_t)c * DL_C * C + (int64_t)j * D, C, n, D, DL_C, D);
    if (tid < 2 * DL_C / 4) cp_async16(dec + (c & 1) * 2 * DL_C + 4 * tid, sc.decay + ch * 2 * DL_C + 4 * tid, true);
    cp_commit();
  };
  auto stage_kp = [&](int c) {
    const int n = (int)min((int64_t)DL_C, rows - (int64_t)c * DL_C);
    stage<DS_THREADS>(Ks, DS_KP, sc.cv + (int64_t)c * DL_C * C + qk + (int64_t)j * D, C, n, D, DL_C, D);
    stage<DS_THREADS>(Ps, DC_S, sc.p + ((int64_t)c * a.heads + h) * DL_C * DL_C, DL_C, DL_C, DL_C, DL_C, DL_C);
    cp_commit();
  };
  stage_wq(0);
  stage_kp(0);
  keep_inputs(a, rows, base, slot, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
  const int mt = warp & 3, nh = (warp >> 2) & 1;  // 16 tokens x half of the value columns
  const bool states = warp < 8;
  // warps 0-7: 16 rows of the state as accumulators
  float* Sg = a.state + ((slot * a.heads + h) * D) * (int64_t)E + e0;
  const int d0 = 16 * (warp & 7);
  const bool owns = states && d0 < D;
  float S[2 * NT][4] = {};
  if (owns && base > 0) {
#pragma unroll
    for (int nt = 0; nt < 2 * NT; nt++)
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const int d = d0 + g + 8 * (i >> 1), e = 8 * nt + 2 * t4 + (i & 1);
        if (d < D && e0 + e < E) S[nt][i] = Sg[(int64_t)d * E + e];
      }
  }
  auto publish = [&]() {
#pragma unroll
    for (int nt = 0; nt < 2 * NT; nt++)
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        const int d = d0 + g + 4 * i, e = 8 * nt + 2 * t4;
        const Tf32Pair p = tf32_split(S[nt][i]), q = tf32_split(S[nt][i + 1]);
        *reinterpret_cast<float2*>(Sh + d * DS_B + e) = make_float2(__uint_as_float(p.hi), __uint_as_float(q.hi));
        *reinterpret_cast<float2*>(Sl + d * DS_B + e) = make_float2(__uint_as_float(p.lo), __uint_as_float(q.lo));
      }
  };
  if (owns) publish();
  float uv[NT][4] = {};  // U of the warp's tile, fetched a chunk ahead
  auto fetch_u = [&](int c) {
    const float* U = sc.u + ((int64_t)c * a.heads + h) * DL_C * E + e0;
#pragma unroll
    for (int nt = 0; nt < NT; nt++)
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int t = 16 * mt + g + 8 * i, e = nh * 8 * NT + 8 * nt + 2 * t4;
        const float2 v = e0 + e < E ? *reinterpret_cast<const float2*>(U + t * (int64_t)E + e) : make_float2(0.f, 0.f);
        uv[nt][2 * i] = v.x, uv[nt][2 * i + 1] = v.y;
      }
  };
  if (states) fetch_u(0);
  auto split_at = [&](const float* hi, const float* lo, int k, int col, Tf32Pair& b0, Tf32Pair& b1) {
    const int at = (k + t4) * DS_B + col;
    b0.hi = __float_as_uint(hi[at]), b0.lo = __float_as_uint(lo[at]);
    b1.hi = __float_as_uint(hi[at + 4 * DS_B]), b1.lo = __float_as_uint(lo[at + 4 * DS_B]);
  };
  for (int c = 0; c < nc; c++) {
    const int64_t t0 = (int64_t)c * DL_C;
    const int n = (int)min((int64_t)DL_C, rows - t0);
    const float* bt = dec + (c & 1) * 2 * DL_C;
    cp_wait<1>();
    __syncthreads();  // W, Q, the decays and the state's terms are there
    // ---- W S, Q S
    float acc[NT][4] = {};
    {
      const float* A = (states ? Ws : Qs) + (16 * mt + g) * DC_P + t4;
#pragma unroll 4
      for (int d = 0; d < D; d += 8) {
        AFrag f;
        load_a(f, A + d, DC_P);
        Tf32Pair b0[NT], b1[NT];
#pragma unroll
        for (int nt = 0; nt < NT; nt++) split_at(Sh, Sl, d, nh * 8 * NT + 8 * nt + g, b0[nt], b1[nt]);
        mma3_split<NT>(acc, f, b0, b1);
      }
    }
    if (states) {
#pragma unroll
      for (int nt = 0; nt < NT; nt++)
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
          const int t = 16 * mt + g + 4 * i, e = nh * 8 * NT + 8 * nt + 2 * t4;
          const Tf32Pair p = tf32_split(uv[nt][i] - acc[nt][i]), q = tf32_split(uv[nt][i + 1] - acc[nt][i + 1]);
          *reinterpret_cast<float2*>(Vh + t * DS_B + e) = make_float2(__uint_as_float(p.hi), __uint_as_float(q.hi));
          *reinterpret_cast<float2*>(Vl + t * DS_B + e) = make_float2(__uint_as_float(p.lo), __uint_as_float(q.lo));
        }
      if (c + 1 < nc) fetch_u(c + 1);
    }
    cp_wait<0>();
    __syncthreads();  // corrections, K and P are there; W, Q and the state's terms are read
    if (c + 1 < nc) stage_wq(c + 1);
    if (owns) {
      // ---- S <- b_C S + (K b_C / b)^T V
      const float full = bt[DL_C - 1];
      const bool second = d0 + 8 < D;
#pragma unroll
      for (int nt = 0; nt < 2 * NT; nt++)
#pragma unroll
        for (int i = 0; i < 4; i++) S[nt][i] *= full;
#pragma unroll 2
      for (int k = 0; k < DL_C; k += 8) {
        const float wa = bt[DL_C + k + t4], wb = bt[DL_C + k + t4 + 4];
        const float *ka = Ks + (k + t4) * DS_KP + d0 + g, *kb = ka + 4 * DS_KP;
        AFrag f;
        split_into(f, 0, ka[0] * wa), split_into(f, 1, second ? ka[8] * wa : 0.f);
        split_into(f, 2, kb[0] * wb), split_into(f, 3, second ? kb[8] * wb : 0.f);
        Tf32Pair b0[2 * NT], b1[2 * NT];
#pragma unroll
        for (int nt = 0; nt < 2 * NT; nt++) split_at(Vh, Vl, k, 8 * nt + g, b0[nt], b1[nt]);
        mma3_split<2 * NT>(S, f, b0, b1);
      }
      publish();
    } else if (!states) {
      // ---- o = b Q S + P V (P is lower triangular)
      const float w0 = bt[16 * mt + g], w1 = bt[16 * mt + g + 8];
#pragma unroll
      for (int nt = 0; nt < NT; nt++) acc[nt][0] *= w0, acc[nt][1] *= w0, acc[nt][2] *= w1, acc[nt][3] *= w1;
#pragma unroll 2
      for (int k = 0; k < 16 * (mt + 1); k += 8) {
        AFrag f;
        load_a(f, Ps + (16 * mt + g) * DC_S + k + t4, DC_S);
        Tf32Pair b0[NT], b1[NT];
#pragma unroll
        for (int nt = 0; nt < NT; nt++) split_at(Vh, Vl, k, nh * 8 * NT + 8 * nt + g, b0[nt], b1[nt]);
        mma3_split<NT>(acc, f, b0, b1);
      }
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int t = 16 * mt + g + 8 * i;
        if (t >= n) continue;
        float* out = a.out + (t0 + t) * (int64_t)a.heads * E + (int64_t)h * E + e0;
#pragma unroll
        for (int nt = 0; nt < NT; nt++) {
          const int e = nh * 8 * NT + 8 * nt + 2 * t4;
          if (e0 + e < E) *reinterpret_cast<float2*>(out + e) = make_float2(acc[nt][2 * i], acc[nt][2 * i + 1]);
        }
      }
    }
    __syncthreads();  // K, P and the corrections are read
    if (c + 1 < nc) stage_kp(c + 1);
  }
  if (!owns) return;
#pragma unroll
  for (int nt = 0; nt < 2 * NT; nt++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int d = d0 + g + 8 * (i >> 1), e = 8 * nt + 2 * t4 + (i & 1);
      if (d < D && e0 + e < E) Sg[(int64_t)d * E + e] = S[nt][i];
    }
}

// Norm and gate of a portion's rows, in place: warp = (row, head).
__global__ void __launch_bounds__(DL_THREADS) delta_finish_kernel(DeltaArgs a, int64_t rows) {
  const int lane = threadIdx.x & 31, E = a.vdim;
  const int64_t item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (item >= rows * a.heads) return;
  const int64_t r = item / a.heads, h = item % a.heads;
  float* out = a.out + item * E;
  const float* gate = a.g.ptr + r * a.g.ld + h * E;
  float ss = 0.f;
  for (int e = lane; e < E; e += 32) ss = fmaf(out[e], out[e], ss);
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)E + a.eps);
  for (int e = lane; e < E; e += 32) out[e] = out[e] * inv * vec_at(a.norm, e) * silu_of(gate[e]);
}

// CTA = row; a warp takes heads in turn. f16 values scaled by a power of two that puts the row's largest magnitude in
// [2^12, 2^13), as the GEMM's own activation pass does.
__global__ void __launch_bounds__(DL_THREADS) delta_finish_operand_kernel(DeltaArgs a) {
  extern __shared__ __align__(16) float df_row[];  // [heads * vdim]
  __shared__ float red[8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = a.vdim, total = a.heads * E;
  const int64_t r = blockIdx.x;
  const float* o = a.out + r * total;
  const float* gate = a.g.ptr + r * a.g.ld;
  float mx = 0.f;
  for (int h = warp; h < a.heads; h += 8) {
    float v[8], z[8], ss = 0.f;  // vdim <= 256
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int e = lane + 32 * i;
      v[i] = e < E ? o[h * E + e] : 0.f, z[i] = e < E ? gate[h * E + e] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; i++) ss = fmaf(v[i], v[i], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)E + a.eps);
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int e = lane + 32 * i;
      if (e >= E) continue;
      const float y = v[i] * inv * vec_at(a.norm, e) * silu_of(z[i]);
      df_row[h * E + e] = y;
      mx = fmaxf(mx, fabsf(y));
    }
  }
  mx = warp_max(mx);
  if (lane == 0) red[warp] = mx;
  __syncthreads();
  mx = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) mx = fmaxf(mx, red[w]);
  int e = 0;
  if (mx > 0.f && mx < 3.0e38f) frexpf(mx, &e);
  const float sc = ldexpf(1.0f, 13 - e);
  if (tid == 0) a.xinv[r] = ldexpf(1.0f, e - 13);
  for (int i = tid * 2; i < total; i += DL_THREADS * 2)
    *reinterpret_cast<__half2*>(a.xh + r * total + i) = __floats2half2_rn(df_row[i] * sc, df_row[i + 1] * sc);
}

bool chunk_shape(const DeltaArgs& a, int64_t rows) {
  return !a.exact && rows > DL_FEW && a.dim <= DC_D && a.dim % 8 == 0 && a.vdim % 8 == 0;
}

}  // namespace

size_t delta_scratch_floats(const DeltaArgs& a, int64_t rows) {
  DeltaArgs z = a;
  z.scratch = nullptr;
  const DeltaScratch s = carve(z, rows);
  return (chunk_shape(a, rows) ? s.end : s.w) - s.cv;
}

bool delta_writes_operand(const DeltaArgs& a) {
  return a.vdim <= 256 && a.heads * a.vdim % 2 == 0 && (size_t)a.heads * a.vdim * 4 <= DL_MAX_SMEM;
}

int launch_delta(const DeltaArgs& a, const StepRows& r, cudaStream_t st) {
  if (r.rows == 0) return 0;
  DYN_CHECK(a.kv_heads > 0 && a.heads % a.kv_heads == 0, "delta rule: %d heads over %d q/k heads", a.heads, a.kv_heads);
  if (r.base < 0) return step_rows(a, r.pos, r.seq, 0, 0, r.rows, st);
  if (r.rows == 1) return step_rows(a, nullptr, nullptr, r.base, r.slot, 1, st);
  const bool wide = conv_wide(a);
  const int64_t per = wide ? DX_ROWS : DV_ROWS, items = (r.rows + per - 1) / per * (2 * a.kv_heads + a.heads);
  const unsigned grid = (unsigned)((items + 7) / 8);
  const auto conv = wide          ? (std::max(a.dim, a.vdim) <= 128 ? delta_conv_wide_kernel<1> : delta_conv_wide_kernel<2>)
                    : a.taps <= 4 ? delta_conv_kernel<4>
                                  : delta_conv_kernel<0>;
  conv<<<grid, DL_THREADS, 0, st>>>(a, r.rows, r.base, r.slot);
  if (chunk_shape(a, r.rows)) {
    const unsigned nc = (unsigned)((r.rows + DL_C - 1) / DL_C);
    // narrow slices where wide ones would leave half of the GPU idle: the walk's time is its latency then
    const bool narrow = 2 * a.heads * ((a.vdim + 31) / 32) <= std::max(1, sm_count());
    const auto scan = narrow ? delta_scan_kernel<1> : delta_scan_kernel<2>;
    const int cols = narrow ? 16 : 32, smem = ds_smem(cols);
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(delta_chunk_kernel), DC_SMEM) ||
        ensure_dynamic_smem(reinterpret_cast<const void*>(scan), smem))
      return 1;
    delta_chunk_kernel<<<dim3(nc, (unsigned)a.heads), DC_THREADS, DC_SMEM, st>>>(a, r.rows);
    scan<<<dim3((unsigned)((a.vdim + cols - 1) / cols), (unsigned)a.heads), DS_THREADS, smem, st>>>(a, r.rows, r.base, r.slot);
    count_launch(2);
  } else {
    int nsplit = std::max(1, (a.vdim + 31) / 32);
    const int per = (a.vdim + nsplit - 1) / nsplit;
    const size_t smem = ((size_t)a.dim * per + 2 * a.dim + 19 * per) * 4;
    DYN_CHECK(smem <= DL_MAX_SMEM, "delta rule: head of %d x %d is too large", a.dim, a.vdim);
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(delta_tokens_kernel), DL_MAX_SMEM)) return 1;
    delta_tokens_kernel<<<dim3((unsigned)nsplit, (unsigned)a.heads), DL_THREADS, smem, st>>>(a, r.rows, r.base, r.slot);
    count_launch();
  }
  if (a.xh) {
    DYN_CHECK(delta_writes_operand(a), "delta rule: no operand of %d heads of %d", a.heads, a.vdim);
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(delta_finish_operand_kernel), DL_MAX_SMEM)) return 1;
    delta_finish_operand_kernel<<<(unsigned)r.rows, DL_THREADS, (size_t)a.heads * a.vdim * 4, st>>>(a);
  } else {
    delta_finish_kernel<<<(unsigned)((r.rows * a.heads + 7) / 8), DL_THREADS, 0, st>>>(a, r.rows);
  }
  count_launch(2);
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace dyn
