// Softmax attention over cached keys and values as a session mixer: biases, rotation of any part of a head,
// a score factor of the model's own, capped scores, values of another width than keys.
//
// softmax_prepare_kernel adds the biases, rotates q in place and k into the cache, and stores v. Then
//   * many rows of one sequence on a 16-bit cache: the tensor-core prefill kernel (attention_prefill.cu);
//   * other rows on a 16-bit cache: softmax_split_kernel, a CTA per (kv head, up to four of its query heads, row, slice
//     of the keys). Eight lanes share a key, so a warp scores four keys at once for all of the CTA's heads and each
//     cached row is read once for them; slices are merged by attention_merge_kernel;
//   * f32 caches and unusual heads: softmax_rows_kernel, a CTA per (head, row).
#include <algorithm>

#include "mixers.cuh"

namespace dyn {
namespace {

constexpr int SA_THREADS = 128, SA_WARPS = SA_THREADS / 32;

template <int KV>
struct Cached;
template <>
struct Cached<E_F32> {
  using T = float;
  __device__ static __forceinline__ T enc(float v) { return v; }
  __device__ static __forceinline__ float dec(T v) { return v; }
};
template <>
struct Cached<E_F16> {
  using T = __half;
  __device__ static __forceinline__ T enc(float v) { return __float2half_rn(v); }
  __device__ static __forceinline__ float dec(T v) { return __half2float(v); }
};
template <>
struct Cached<E_BF16> {
  using T = __nv_bfloat16;
  __device__ static __forceinline__ T enc(float v) { return __float2bfloat16_rn(v); }
  __device__ static __forceinline__ float dec(T v) { return __bfloat162float(v); }
};

__device__ __forceinline__ int64_t pos_of(const StepRows& s, int64_t r) { return s.base >= 0 ? s.base + r : s.pos[r]; }
__device__ __forceinline__ int64_t slot_of(const StepRows& s, int64_t r) { return s.base >= 0 ? s.slot : s.seq[r]; }
__device__ __forceinline__ float bias_at(const Vec& v, int64_t i) { return v.ptr ? vec_at(v, i) : 0.f; }
__device__ __forceinline__ float score_of(const SoftmaxArgs& a, float dot) {
  const float s = dot * a.scale;
  return a.softcap > 0.f ? a.softcap * tanhf(s / a.softcap) : s;
}

// One row per CTA: angles once in shared memory, then all heads.
template <int KV>
__global__ void __launch_bounds__(256) softmax_prepare_kernel(SoftmaxArgs a, StepRows s) {
  using T = typename Cached<KV>::T;
  extern __shared__ float sp_angles[];  // [half][sin, cos]
  const int64_t r = blockIdx.x;
  const int half = a.rot_dims / 2, per = a.dim - half;  // pairs, then the dims that pass
  pdl_trigger();
  pdl_wait();
  const int64_t pos = pos_of(s, r), seq = slot_of(s, r);
  for (int i = threadIdx.x; i < half; i += 256) sincos_position(pos, a.freq[i], &sp_angles[2 * i], &sp_angles[2 * i + 1]);
  __syncthreads();
  const int nq = a.heads * per, nk = a.kv_heads * per, nv = a.kv_heads * a.vdim;
  for (int it = threadIdx.x + blockIdx.y * 256; it < nq + nk + nv; it += 256 * gridDim.y) {
    if (it >= nq + nk) {
      const int c = it - nq - nk, h = c / a.vdim, e = c - h * a.vdim;
      reinterpret_cast<T*>(a.vcache)[((seq * a.kv_heads + h) * a.cap + pos) * a.vdim + e] =
          Cached<KV>::enc(a.v.ptr[r * a.v.ld + c] + bias_at(a.vb, c));
      continue;
    }
    const bool is_q = it < nq;
    const int j = is_q ? it : it - nq, h = j / per, i = j - h * per;
    const Vec& b = is_q ? a.qb : a.kb;
    float* x = is_q ? a.q.ptr + r * a.q.ld + h * a.dim : a.k.ptr + r * a.k.ld + h * a.dim;
    T* kc = reinterpret_cast<T*>(a.kcache) + ((seq * a.kv_heads + h) * a.cap + pos) * a.dim;
    if (i < half) {
      const float sv = sp_angles[2 * i], cv = sp_angles[2 * i + 1];
      const float u = x[i] + bias_at(b, h * a.dim + i), v = x[i + half] + bias_at(b, h * a.dim + i + half);
      const float y0 = u * cv - v * sv, y1 = v * cv + u * sv;
      if (is_q) x[i] = y0, x[i + half] = y1;
      else kc[i] = Cached<KV>::enc(y0), kc[i + half] = Cached<KV>::enc(y1);
    } else {
      const float u = x[i + half] + bias_at(b, h * a.dim + i + half);
      if (is_q) x[i + half] = u;
      else kc[i + half] = Cached<KV>::enc(u);
    }
  }
}

// ---- any head size, f32 caches -----------------------------------------------------------------
constexpr int SR_KEYS = 64, SR_MAX_E = 8;  // keys at a time; value dims per thread (vdim <= 1024)
template <int KV>
__global__ void __launch_bounds__(SA_THREADS) softmax_rows_kernel(SoftmaxArgs a, StepRows s) {
  using T = typename Cached<KV>::T;
  extern __shared__ float sr_q[];  // [dim]
  __shared__ float p[SR_KEYS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = a.dim, E = a.vdim;
  const int64_t h = blockIdx.x, r = blockIdx.y, kvh = h / (a.heads / a.kv_heads);
  const int64_t pos = pos_of(s, r), seq = slot_of(s, r);
  const T* kb = reinterpret_cast<const T*>(a.kcache) + (seq * a.kv_heads + kvh) * a.cap * D;
  const T* vb = reinterpret_cast<const T*>(a.vcache) + (seq * a.kv_heads + kvh) * a.cap * E;
  for (int d = tid; d < D; d += SA_THREADS) sr_q[d] = a.q.ptr[r * a.q.ld + h * D + d];
  __syncthreads();
  float m = -3.40282347e38f, l = 0.f, acc[SR_MAX_E] = {};
  for (int64_t k0 = 0; k0 <= pos; k0 += SR_KEYS) {
    const int n = (int)min((int64_t)SR_KEYS, pos + 1 - k0);
    for (int k = warp; k < n; k += SA_WARPS) {
      float dot = 0.f;
      for (int d = lane; d < D; d += 32) dot = fmaf(sr_q[d], Cached<KV>::dec(kb[(k0 + k) * D + d]), dot);
      dot = warp_sum(dot);
      if (lane == 0) p[k] = score_of(a, dot);
    }
    __syncthreads();
    float mx = m;
    for (int k = lane; k < n; k += 32) mx = fmaxf(mx, p[k]);
    mx = warp_max(mx);
    const float f = expf(m - mx);
    m = mx, l *= f;
    __syncthreads();
    for (int k = tid; k < n; k += SA_THREADS) p[k] = expf(p[k] - m);
    __syncthreads();
#pragma unroll
    for (int j = 0; j < SR_MAX_E; j++) acc[j] *= f;
    for (int k = 0; k < n; k++) {
      const float w = p[k];
      l += w;
#pragma unroll
      for (int j = 0; j < SR_MAX_E; j++) {
        const int e = tid + SA_THREADS * j;
        if (e < E) acc[j] = fmaf(w, Cached<KV>::dec(vb[(k0 + k) * E + e]), acc[j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < SR_MAX_E; j++) {
    const int e = tid + SA_THREADS * j;
    if (e < E) a.out[(r * a.heads + h) * E + e] = acc[j] / l;
  }
}

// ---- 16-bit caches, few rows per sequence ---------------------------------------------------------
// N: elements of a key or value per lane (8 lanes x N >= dim, vdim); piece c of a lane = elements 64 c + 8 lane8 ..
template <int KV, int N, int HB>
__global__ void __launch_bounds__(SA_THREADS) softmax_split_kernel(SoftmaxArgs a, StepRows s, float* __restrict__ part, int nsplit) {
  using T = typename Cached<KV>::T;
  constexpr int P = N / 8;
  __shared__ float s_m[SA_WARPS][HB], s_l[SA_WARPS][HB], s_acc[SA_WARPS][HB][8 * N];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l8 = lane & 7, kg = lane >> 3;
  const int group = a.heads / a.kv_heads, blocks = (group + HB - 1) / HB;
  const int kvh = blockIdx.x / blocks, hb0 = (int)(blockIdx.x % blocks) * HB, nh = min(HB, group - hb0);
  const int64_t h0 = (int64_t)kvh * group + hb0, r = blockIdx.y, sp = blockIdx.z;
  const int D = a.dim, E = a.vdim;
  pdl_trigger();
  pdl_wait();
  const int64_t pos = pos_of(s, r), seq = slot_of(s, r);
  const int64_t n = pos + 1, per = (n + nsplit - 1) / nsplit, k_lo = sp * per, k_hi = min(k_lo + per, n);
  const T* kb = reinterpret_cast<const T*>(a.kcache) + (seq * a.kv_heads + kvh) * a.cap * D;
  const T* vb = reinterpret_cast<const T*>(a.vcache) + (seq * a.kv_heads + kvh) * a.cap * E;
  float q[HB][N], acc[HB][N], m[HB], l[HB];
#pragma unroll
  for (int b = 0; b < HB; b++) {
    m[b] = -3.40282347e38f, l[b] = 0.f;
#pragma unroll
    for (int i = 0; i < N; i++) {
      const int d = 64 * (i / 8) + 8 * l8 + i % 8;
      q[b][i] = b < nh && d < D ? a.q.ptr[r * a.q.ld + (h0 + b) * D + d] : 0.f;
      acc[b][i] = 0.f;
    }
  }
  constexpr int U = N <= 16 ? 2 : 1;  // keys per lane group in flight
  for (int64_t key0 = k_lo + warp * 4 + kg; key0 - kg < k_hi; key0 += 4 * SA_WARPS * U) {
    uint4 kr[U][P], vr[U][P];
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int64_t key = key0 + (int64_t)u * 4 * SA_WARPS;
#pragma unroll
      for (int c = 0; c < P; c++) {
        const int d = 64 * c + 8 * l8;
        kr[u][c] = key < k_hi && d < D ? *reinterpret_cast<const uint4*>(kb + key * D + d) : make_uint4(0, 0, 0, 0);
        vr[u][c] = key < k_hi && d < E ? *reinterpret_cast<const uint4*>(vb + key * E + d) : make_uint4(0, 0, 0, 0);
      }
    }
#pragma unroll
    for (int u = 0; u < U; u++) {
      const bool live = key0 + (int64_t)u * 4 * SA_WARPS < k_hi;
      const T* kt = reinterpret_cast<const T*>(kr[u]);
      const T* vt = reinterpret_cast<const T*>(vr[u]);
#pragma unroll
      for (int b = 0; b < HB; b++) {
        float dot = 0.f;
#pragma unroll
        for (int i = 0; i < N; i++) dot = fmaf(q[b][i], Cached<KV>::dec(kt[i]), dot);
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        dot += __shfl_xor_sync(0xffffffffu, dot, 2);
        dot += __shfl_xor_sync(0xffffffffu, dot, 4);
        if (!live) continue;
        const float sc = score_of(a, dot), mn = fmaxf(m[b], sc), f = expf(m[b] - mn), p = expf(sc - mn);
        m[b] = mn;
        l[b] = l[b] * f + p;
#pragma unroll
        for (int i = 0; i < N; i++) acc[b][i] = fmaf(acc[b][i], f, p * Cached<KV>::dec(vt[i]));
      }
    }
  }
  // the warp's four key groups, then the warps
#pragma unroll
  for (int b = 0; b < HB; b++) {
#pragma unroll
    for (int o = 8; o < 32; o *= 2) {
      const float mo = __shfl_xor_sync(0xffffffffu, m[b], o), lo = __shfl_xor_sync(0xffffffffu, l[b], o);
      const float mn = fmaxf(m[b], mo), f = expf(m[b] - mn), fo = expf(mo - mn);
      m[b] = mn, l[b] = l[b] * f + lo * fo;
#pragma unroll
      for (int i = 0; i < N; i++) {
        const float ao = __shfl_xor_sync(0xffffffffu, acc[b][i], o);
        acc[b][i] = acc[b][i] * f + ao * fo;
      }
    }
    if (kg == 0) {
      if (l8 == 0) s_m[warp][b] = m[b], s_l[warp][b] = l[b];
#pragma unroll
      for (int i = 0; i < N; i++) s_acc[warp][b][64 * (i / 8) + 8 * l8 + i % 8] = acc[b][i];
    }
  }
  __syncthreads();
  for (int i = tid; i < nh * E; i += SA_THREADS) {
    const int b = i / E, e = i - b * E;
    float gm = s_m[0][b], gl = 0.f, o = 0.f;
#pragma unroll
    for (int w = 1; w < SA_WARPS; w++) gm = fmaxf(gm, s_m[w][b]);
#pragma unroll
    for (int w = 0; w < SA_WARPS; w++) {
      const float f = expf(s_m[w][b] - gm);
      gl += s_l[w][b] * f, o += s_acc[w][b][e] * f;
    }
    float* out = part + ((r * a.heads + h0 + b) * nsplit + sp) * (E + 2);
    out[e] = o;
    if (e == 0) out[E] = gm, out[E + 1] = gl;
  }
}

bool split_shape(const SoftmaxArgs& a) {
  auto ok = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return !a.exact && a.kv_type != E_F32 && a.dim <= 256 && a.vdim <= 256 && a.dim % 8 == 0 && a.vdim % 8 == 0 && ok(a.kcache) && ok(a.vcache);
}
int heads_per_cta(const SoftmaxArgs& a) {
  const int group = a.heads / a.kv_heads, most = std::max(a.dim, a.vdim) <= 128 ? 4 : 2;
  return group >= most ? most : group >= 2 ? 2 : 1;
}
// A function of shapes and capacity only: a captured graph stays valid as positions grow.
int split_count(const SoftmaxArgs& a, int64_t rows) {
  const int hb = heads_per_cta(a), group = a.heads / a.kv_heads;
  const int64_t ctas = rows * a.kv_heads * ((group + hb - 1) / hb);
  return (int)std::max<int64_t>(1, std::min<int64_t>({592 / ctas, a.cap / 64, 32}));
}

template <int KV, int N>
int run_split(const SoftmaxArgs& a, const StepRows& s, float* part, int nsplit, cudaStream_t st) {
  const int hb = heads_per_cta(a), group = a.heads / a.kv_heads;
  const dim3 grid((unsigned)(a.kv_heads * ((group + hb - 1) / hb)), (unsigned)s.rows, (unsigned)nsplit);
  cudaError_t e;
  if constexpr (N <= 16) {
    e = hb == 4   ? launch_pdl(softmax_split_kernel<KV, N, 4>, grid, dim3(SA_THREADS), 0, st, a, s, part, nsplit)
        : hb == 2 ? launch_pdl(softmax_split_kernel<KV, N, 2>, grid, dim3(SA_THREADS), 0, st, a, s, part, nsplit)
                  : launch_pdl(softmax_split_kernel<KV, N, 1>, grid, dim3(SA_THREADS), 0, st, a, s, part, nsplit);
  } else {
    e = hb == 2 ? launch_pdl(softmax_split_kernel<KV, N, 2>, grid, dim3(SA_THREADS), 0, st, a, s, part, nsplit)
                : launch_pdl(softmax_split_kernel<KV, N, 1>, grid, dim3(SA_THREADS), 0, st, a, s, part, nsplit);
  }
  DYN_CUDA(e);
  count_launch();
  return launch_attention_merge(part, nsplit, a.out, s.rows, a.heads, a.vdim, st);
}

template <int KV>
int run_rows(const SoftmaxArgs& a, const StepRows& s, cudaStream_t st) {
  DYN_CHECK(a.vdim <= SA_THREADS * SR_MAX_E && a.dim * 4 <= 48 * 1024, "softmax attention: head of %d / %d is too large", a.dim, a.vdim);
  for (int64_t r0 = 0; r0 < s.rows; r0 += 65535) {
    StepRows p = s;
    SoftmaxArgs b = a;
    p.rows = std::min<int64_t>(65535, s.rows - r0);
    if (s.base >= 0) p.base += r0;
    else p.pos += r0, p.seq += r0;
    b.q.ptr += r0 * a.q.ld, b.out += r0 * a.heads * a.vdim;
    softmax_rows_kernel<KV><<<dim3((unsigned)a.heads, (unsigned)p.rows), SA_THREADS, (size_t)a.dim * 4, st>>>(b, p);
    count_launch();
  }
  DYN_CUDA(cudaGetLastError());
  return 0;
}

template <int KV>
int prepare(const SoftmaxArgs& a, const StepRows& s, cudaStream_t st) {
  DYN_CHECK(a.rot_dims * 4 <= 48 * 1024, "softmax attention: rotation of %d dims is too large", a.rot_dims);
  // few rows: several CTAs share one
  const int items = (a.heads + a.kv_heads) * (a.dim - a.rot_dims / 2) + a.kv_heads * a.vdim;
  const unsigned shares = (unsigned)std::max<int64_t>(1, std::min<int64_t>((items + 255) / 256, 148 / s.rows));
  DYN_CUDA(launch_pdl(softmax_prepare_kernel<KV>, dim3((unsigned)s.rows, shares), dim3(256), (size_t)a.rot_dims * 4, st, a, s));
  count_launch();
  return 0;
}

}  // namespace

size_t softmax_scratch_floats(const SoftmaxArgs& a, int64_t rows) {
  size_t need = 0;
  if (split_shape(a))
    for (int64_t r = 1; r <= rows; r = r < rows ? std::min(2 * r, rows) : r + 1) {
      // the count of slices falls as rows grow: take the larger of both ends of a doubling
      need = std::max(need, (size_t)std::min(2 * r, rows) * a.heads * split_count(a, r) * (a.vdim + 2));
    }
  return need;
}

int launch_softmax_attention(const SoftmaxArgs& a, const StepRows& s, cudaStream_t st) {
  if (s.rows == 0) return 0;
  DYN_CHECK(a.kv_heads > 0 && a.heads % a.kv_heads == 0, "softmax attention: %d heads over %d kv heads", a.heads, a.kv_heads);
  const int kv = a.kv_type;
  if (kv == E_F32 ? prepare<E_F32>(a, s, st) : kv == E_F16 ? prepare<E_F16>(a, s, st) : prepare<E_BF16>(a, s, st)) return 1;
  if (s.base >= 0 && !a.exact) {
    AttnArgs f{};
    f.q = a.q.ptr, f.ldq = a.q.ld, f.kcache = a.kcache, f.vcache = a.vcache, f.ctx = a.out, f.rows = s.rows, f.nh = a.heads;
    f.nkv = a.kv_heads, f.d = a.dim, f.dv = a.vdim, f.cap = a.cap, f.kv_type = kv, f.scale = a.scale, f.softcap = a.softcap;
    bool handled = false;
    if (launch_attention_prefill(f, s.base, s.slot, st, &handled)) return 1;
    if (handled) return 0;
  }
  if (!split_shape(a)) return kv == E_F32 ? run_rows<E_F32>(a, s, st) : kv == E_F16 ? run_rows<E_F16>(a, s, st) : run_rows<E_BF16>(a, s, st);
  DYN_CHECK(s.rows <= 65535, "softmax attention: %lld rows in one launch", (long long)s.rows);
  const int nsplit = split_count(a, s.rows), wide = std::max(a.dim, a.vdim);
  if (kv == E_F16)
    return wide <= 64    ? run_split<E_F16, 8>(a, s, a.scratch, nsplit, st)
           : wide <= 128 ? run_split<E_F16, 16>(a, s, a.scratch, nsplit, st)
                         : run_split<E_F16, 32>(a, s, a.scratch, nsplit, st);
  return wide <= 64    ? run_split<E_BF16, 8>(a, s, a.scratch, nsplit, st)
         : wide <= 128 ? run_split<E_BF16, 16>(a, s, a.scratch, nsplit, st)
                       : run_split<E_BF16, 32>(a, s, a.scratch, nsplit, st);
}

}  // namespace dyn
