// Attention whose cache holds one latent vector per token (shared by all heads) instead of keys and
// values, without positions.
//
// Few rows, or f32: the up-projections are absorbed. score = q . (W_uk c) = (W_uk^T q) . c, so a row's
// queries are mapped into the latent space once per head, the keys of a slice of the cache are scored
// and summed there (one read of the latents serves eight heads), and the merge kernel maps the
// weighted latent back through W_uv, normalises and gates.
//
// Many rows of one sequence on a bf16 cache: the latents up to the portion's end are expanded to keys
// and values (one product per block of tokens, rounded to bf16 as ordinary cached keys are) and the
// tensor-core prefill attention runs on them. Heads narrower than its 128 dims are padded with zeros.
#include <algorithm>

#include "mixers.cuh"

namespace dyn {
namespace {

__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }

template <int KV>
struct Lat;
template <>
struct Lat<E_F32> {
  using T = float;
  __device__ static __forceinline__ T enc(float v) { return v; }
  __device__ static __forceinline__ float dec(T v) { return v; }
};
template <>
struct Lat<E_F16> {
  using T = __half;
  __device__ static __forceinline__ T enc(float v) { return __float2half_rn(v); }
  __device__ static __forceinline__ float dec(T v) { return __half2float(v); }
};
template <>
struct Lat<E_BF16> {
  using T = __nv_bfloat16;
  __device__ static __forceinline__ T enc(float v) { return __float2bfloat16_rn(v); }
  __device__ static __forceinline__ float dec(T v) { return __bfloat162float(v); }
};

__device__ __forceinline__ int64_t pos_of(const StepRows& s, int64_t r) { return s.base >= 0 ? s.base + r : s.pos[r]; }
__device__ __forceinline__ int64_t slot_of(const StepRows& s, int64_t r) { return s.base >= 0 ? s.slot : s.seq[r]; }

// ---- normalised latents into the cache: one block per row ---------------------------------------
template <int KV>
__global__ void __launch_bounds__(128) latent_store_kernel(LatentArgs a, StepRows s) {
  __shared__ float red[4];
  const int tid = threadIdx.x;
  const int64_t r = blockIdx.x;
  const float* d = a.d.ptr + r * a.d.ld;
  pdl_trigger();
  float ss = 0.f;
  for (int i = tid; i < a.rank; i += 128) ss = fmaf(d[i], d[i], ss);
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  const float inv = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)a.rank + a.eps);
  typename Lat<KV>::T* dst = reinterpret_cast<typename Lat<KV>::T*>(a.cache) + (slot_of(s, r) * a.cap + pos_of(s, r)) * a.rank;
  for (int i = tid; i < a.rank; i += 128) dst[i] = Lat<KV>::enc(d[i] * inv * aux_load(a.norm.ptr, a.norm.type, i));
}

// ---- queries into the latent space: qa[row][head][rank] = scale * W_uk^T q ----------------------------
// CTA = 64 latent dims of one (head, row); eight warps share the head's dims.
constexpr int AB_R = 64;
__global__ void __launch_bounds__(256) latent_absorb_kernel(LatentArgs a, float* __restrict__ qa) {
  extern __shared__ float ab_q[];  // [dim]
  __shared__ float part[8][AB_R];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, r0 = blockIdx.x * AB_R;
  const int64_t row = blockIdx.z;
  const float* q = a.q.ptr + row * a.q.ld + (int64_t)h * a.dim;
  pdl_trigger();
  for (int i = tid; i < a.dim; i += 256) ab_q[i] = q[i];
  __syncthreads();
  float s0 = 0.f, s1 = 0.f;
  const int c0 = r0 + lane, c1 = c0 + 32;
#pragma unroll 8
  for (int d = warp; d < a.dim; d += 8) {
    const int64_t at = ((int64_t)h * a.dim + d) * a.rank;
    if (c0 < a.rank) s0 = fmaf(ab_q[d], aux_load(a.uk.data, a.uk.enc, at + c0), s0);
    if (c1 < a.rank) s1 = fmaf(ab_q[d], aux_load(a.uk.data, a.uk.enc, at + c1), s1);
  }
  part[warp][lane] = s0, part[warp][lane + 32] = s1;
  __syncthreads();
  if (tid < AB_R && r0 + tid < a.rank) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) t += part[w][tid];
    qa[(row * a.heads + h) * a.rank + r0 + tid] = t * a.scale;
  }
}

// ---- scores and weighted latents of one slice of a row's keys ---------------------------------------
// Eight heads per CTA, a warp each; lane owns latent dims lane + 32 j. Latents pass through shared
// memory as f32. part[row][head][slice]: weighted sum [rank], maximum, weight sum.
constexpr int LA_H = 8, LA_KEYS = 8;
template <int KV, int RL>
__global__ void __launch_bounds__(256) latent_split_kernel(LatentArgs a, StepRows s, const float* __restrict__ qa,
                                                           float* __restrict__ part) {
  __shared__ float cs[LA_KEYS][RL * 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nsplit = gridDim.x, h = blockIdx.y * LA_H + warp;
  const int64_t row = blockIdx.z, n = pos_of(s, row) + 1, per = (n + nsplit - 1) / nsplit;
  const int64_t lo = blockIdx.x * per, hi = min(lo + per, n);
  const typename Lat<KV>::T* cache = reinterpret_cast<const typename Lat<KV>::T*>(a.cache) + slot_of(s, row) * a.cap * a.rank;
  const bool head = h < a.heads;
  pdl_trigger();
  float q[RL], acc[RL];
#pragma unroll
  for (int j = 0; j < RL; j++) {
    const int c = lane + 32 * j;
    q[j] = head && c < a.rank ? qa[(row * a.heads + h) * a.rank + c] : 0.f;
    acc[j] = 0.f;
  }
  float m = -3.40282347e38f, l = 0.f;
  for (int64_t k0 = lo; k0 < hi; k0 += LA_KEYS) {
    const int nk = (int)min((int64_t)LA_KEYS, hi - k0);
    __syncthreads();
    for (int i = tid; i < LA_KEYS * RL * 32; i += 256) {
      const int k = i / (RL * 32), c = i % (RL * 32);
      cs[k][c] = k < nk && c < a.rank ? Lat<KV>::dec(cache[(k0 + k) * a.rank + c]) : 0.f;
    }
    __syncthreads();
    if (!head) continue;
    float sc[LA_KEYS], mn = m;
#pragma unroll
    for (int k = 0; k < LA_KEYS; k++) {
      float d = 0.f;
#pragma unroll
      for (int j = 0; j < RL; j++) d = fmaf(q[j], cs[k][lane + 32 * j], d);
      sc[k] = warp_sum(d);
      if (k < nk) mn = fmaxf(mn, sc[k]);
    }
    const float f = expf(m - mn);
    m = mn, l *= f;
#pragma unroll
    for (int j = 0; j < RL; j++) acc[j] *= f;
#pragma unroll
    for (int k = 0; k < LA_KEYS; k++) {
      const float p = k < nk ? expf(sc[k] - m) : 0.f;
      l += p;
#pragma unroll
      for (int j = 0; j < RL; j++) acc[j] = fmaf(p, cs[k][lane + 32 * j], acc[j]);
    }
  }
  if (!head) return;
  float* out = part + ((row * a.heads + h) * nsplit + blockIdx.x) * (a.rank + 2);
#pragma unroll
  for (int j = 0; j < RL; j++)
    if (lane + 32 * j < a.rank) out[lane + 32 * j] = acc[j];
  if (lane == 0) out[a.rank] = m, out[a.rank + 1] = l;
}

// ---- slices merged, W_uv, output gate: CTA = 32 value dims of one (head, row) ----------------------------
constexpr int LV_E = 32;
__global__ void __launch_bounds__(256) latent_value_kernel(LatentArgs a, const float* __restrict__ part, int nsplit) {
  extern __shared__ float lv_c[];  // [rank]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, e0 = blockIdx.x * LV_E;
  const int64_t row = blockIdx.z;
  const float* p0 = part + (row * a.heads + h) * (int64_t)nsplit * (a.rank + 2);
  pdl_trigger();
  float gm = -3.40282347e38f, gl = 0.f;
  for (int i = 0; i < nsplit; i++) gm = fmaxf(gm, p0[(int64_t)i * (a.rank + 2) + a.rank]);
  for (int i = 0; i < nsplit; i++) {
    const float* ps = p0 + (int64_t)i * (a.rank + 2);
    gl += ps[a.rank + 1] * expf(ps[a.rank] - gm);  // an empty slice has sum 0
  }
  for (int c = tid; c < a.rank; c += 256) {
    float t = 0.f;
    for (int i = 0; i < nsplit; i++) {
      const float* ps = p0 + (int64_t)i * (a.rank + 2);
      t = fmaf(ps[c], expf(ps[a.rank] - gm), t);
    }
    lv_c[c] = t / gl;
  }
  __syncthreads();
  for (int e = e0 + warp; e < min(a.vdim, e0 + LV_E); e += 8) {
    const int64_t at = ((int64_t)h * a.vdim + e) * a.rank;
    float t = 0.f;
    for (int c = lane; c < a.rank; c += 32) t = fmaf(aux_load(a.uv.data, a.uv.enc, at + c), lv_c[c], t);
    t = warp_sum(t);
    if (lane == 0)
      a.out[(row * a.heads + h) * a.vdim + e] = t * sigmoid_of(a.g.ptr[row * a.g.ld + (int64_t)h * a.vdim + e]);
  }
}

// The slice count depends only on shapes and capacity, so a captured graph stays valid as positions grow.
int slices(const LatentArgs& a, int64_t rows) {
  const int64_t groups = rows * ((a.heads + LA_H - 1) / LA_H);
  return (int)std::max<int64_t>(1, std::min<int64_t>({16, a.cap / 64, 296 / groups}));
}

template <int KV>
int run_absorbed(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  const int64_t rows = s.rows;
  float* qa = a.scratch;
  float* part = qa + rows * a.heads * a.rank;
  const int ns = slices(a, rows);
  DYN_CHECK(a.rank <= 1024 && a.dim <= 8192, "latent attention: rank %d or head dim %d is too large", a.rank, a.dim);
  DYN_CHECK(rows <= 65535 && a.heads <= 65535, "latent attention: %lld rows in one step", (long long)rows);
  latent_absorb_kernel<<<dim3((unsigned)((a.rank + AB_R - 1) / AB_R), (unsigned)a.heads, (unsigned)rows), 256, (size_t)a.dim * 4, st>>>(a, qa);
  const dim3 grid((unsigned)ns, (unsigned)((a.heads + LA_H - 1) / LA_H), (unsigned)rows);
  if (a.rank <= 128)
    latent_split_kernel<KV, 4><<<grid, 256, 0, st>>>(a, s, qa, part);
  else if (a.rank <= 256)
    latent_split_kernel<KV, 8><<<grid, 256, 0, st>>>(a, s, qa, part);
  else if (a.rank <= 512)
    latent_split_kernel<KV, 16><<<grid, 256, 0, st>>>(a, s, qa, part);
  else
    latent_split_kernel<KV, 32><<<grid, 256, 0, st>>>(a, s, qa, part);
  latent_value_kernel<<<dim3((unsigned)((a.vdim + LV_E - 1) / LV_E), (unsigned)a.heads, (unsigned)rows), 256, (size_t)a.rank * 4, st>>>(a, part, ns);
  count_launch(3);
  DYN_CUDA(cudaGetLastError());
  return 0;
}

// ---- expanded keys and values ---------------------------------------------------------------------
constexpr int EX_D = 128;  // head width of the prefill attention

// y rows [k heads | v heads] of tokens t0.. -> K, V planes [head][cap][128] bf16, zero padded
__global__ void __launch_bounds__(256)
latent_expand_kernel(const float* __restrict__ k, int64_t ldk, const float* __restrict__ v, int64_t ldv, int heads, int dim, int vdim,
                     int64_t t0, int64_t tokens, int64_t cap, __nv_bfloat162* __restrict__ kx, __nv_bfloat162* __restrict__ vx) {
  const int64_t total = tokens * heads * (EX_D / 2);
  for (int64_t it = blockIdx.x * 256ll + threadIdx.x; it < total; it += (int64_t)gridDim.x * 256) {
    const int c = (int)(it % (EX_D / 2)) * 2;
    const int64_t th = it / (EX_D / 2), h = th % heads, t = th / heads;
    const float* kr = k + t * ldk + h * dim;
    const float* vr = v + t * ldv + h * vdim;
    const int64_t at = ((h * cap + t0 + t) * EX_D + c) / 2;
    kx[at] = __floats2bfloat162_rn(c < dim ? kr[c] : 0.f, c + 1 < dim ? kr[c + 1] : 0.f);
    vx[at] = __floats2bfloat162_rn(c < vdim ? vr[c] : 0.f, c + 1 < vdim ? vr[c + 1] : 0.f);
  }
}

__global__ void __launch_bounds__(256) latent_pad_q_kernel(LatentArgs a, int64_t rows, float* __restrict__ q) {
  const int64_t total = rows * a.heads * EX_D;
  for (int64_t it = blockIdx.x * 256ll + threadIdx.x; it < total; it += (int64_t)gridDim.x * 256) {
    const int c = (int)(it % EX_D);
    const int64_t rh = it / EX_D, h = rh % a.heads, r = rh / a.heads;
    q[it] = c < a.dim ? a.q.ptr[r * a.q.ld + h * a.dim + c] : 0.f;
  }
}

__global__ void __launch_bounds__(256) latent_gate_kernel(LatentArgs a, int64_t rows, const float* __restrict__ ctx) {
  const int64_t total = rows * a.heads * a.vdim;
  for (int64_t it = blockIdx.x * 256ll + threadIdx.x; it < total; it += (int64_t)gridDim.x * 256) {
    const int e = (int)(it % a.vdim);
    const int64_t rh = it / a.vdim, h = rh % a.heads, r = rh / a.heads;
    a.out[it] = ctx[(r * a.heads + h) * EX_D + e] * sigmoid_of(a.g.ptr[r * a.g.ld + h * a.vdim + e]);
  }
}

bool expands(const LatentArgs& a) {
  return !a.exact && a.kv_type == E_BF16 && a.dim <= EX_D && a.vdim <= EX_D && a.cap % 64 == 0 && a.rank % 4 == 0;
}
constexpr int64_t EXPAND_MIN_ROWS = 32;  // the prefill attention's own lower limit

unsigned ew_grid(int64_t total) { return (unsigned)std::max<int64_t>(1, std::min<int64_t>((total + 255) / 256, 148 * 16)); }

int run_expanded(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  const int64_t rows = s.rows, H = a.heads, end = s.base + rows;
  const int64_t kd = H * a.dim, vd = H * a.vdim;
  __nv_bfloat16* kx = reinterpret_cast<__nv_bfloat16*>(a.scratch);
  __nv_bfloat16* vx = kx + H * a.cap * EX_D;
  float* y = reinterpret_cast<float*>(vx + H * a.cap * EX_D);  // [max_rows, kd + vd]
  float* qp = y + a.max_rows * (kd + vd);                      // [rows, H * 128]
  float* ctx = qp + a.max_rows * H * EX_D;
  const __nv_bfloat16* lat = reinterpret_cast<const __nv_bfloat16*>(a.cache) + s.slot * a.cap * a.rank;
  for (int64_t t0 = 0; t0 < end; t0 += a.max_rows) {
    const int64_t n = std::min(a.max_rows, end - t0);
    const float *k = y, *v = y + kd;
    int64_t ldk = kd + vd, ldv = kd + vd;
    if (a.ukv.data) {
      if (launch_linear(a.ukv, lat + t0 * a.rank, E_BF16, n, y, nullptr, st)) return 1;
    } else {
      v = y + n * kd, ldk = kd, ldv = vd;
      if (launch_linear(a.uk, lat + t0 * a.rank, E_BF16, n, y, nullptr, st) ||
          launch_linear(a.uv, lat + t0 * a.rank, E_BF16, n, y + n * kd, nullptr, st))
        return 1;
    }
    latent_expand_kernel<<<ew_grid(n * H * (EX_D / 2)), 256, 0, st>>>(k, ldk, v, ldv, a.heads, a.dim, a.vdim, t0, n, a.cap,
                                                                      reinterpret_cast<__nv_bfloat162*>(kx),
                                                                      reinterpret_cast<__nv_bfloat162*>(vx));
    count_launch();
  }
  AttnArgs f{};
  f.q = a.q.ptr, f.ldq = a.q.ld;
  if (a.dim != EX_D || a.q.ld % 2) {
    latent_pad_q_kernel<<<ew_grid(rows * H * EX_D), 256, 0, st>>>(a, rows, qp);
    count_launch();
    f.q = qp, f.ldq = H * EX_D;
  }
  f.kcache = kx, f.vcache = vx, f.ctx = ctx, f.rows = rows, f.nh = H, f.nkv = H, f.d = EX_D, f.cap = a.cap;
  f.kv_type = E_BF16, f.base_pos = s.base, f.scale = a.scale;
  bool handled = false;
  if (launch_attention_prefill(f, s.base, 0, st, &handled)) return 1;
  DYN_CHECK(handled, "prefill attention refused an expanded latent portion");
  latent_gate_kernel<<<ew_grid(rows * vd), 256, 0, st>>>(a, rows, ctx);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace

size_t latent_scratch_floats(const LatentArgs& a, int64_t rows) {
  // part of an absorbed step: the slice count falls as the rows grow
  size_t need = 0;
  for (int64_t r = 1; r <= rows; r++)
    need = std::max(need, (size_t)r * a.heads * (a.rank + (size_t)slices(a, r) * (a.rank + 2)));
  if (expands(a) && rows >= EXPAND_MIN_ROWS)
    need = std::max(need, (size_t)a.heads * a.cap * EX_D +
                              (size_t)a.max_rows * a.heads * (a.dim + a.vdim + 2 * EX_D) + 64);
  return need;
}

int launch_latent_attention(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  if (s.rows == 0) return 0;
  switch (a.kv_type) {
    case E_F32: latent_store_kernel<E_F32><<<(unsigned)s.rows, 128, 0, st>>>(a, s); break;
    case E_F16: latent_store_kernel<E_F16><<<(unsigned)s.rows, 128, 0, st>>>(a, s); break;
    case E_BF16: latent_store_kernel<E_BF16><<<(unsigned)s.rows, 128, 0, st>>>(a, s); break;
    default: DYN_CHECK(false, "kv_type %d unsupported", a.kv_type);
  }
  count_launch();
  if (s.base >= 0 && s.rows >= EXPAND_MIN_ROWS && expands(a)) return run_expanded(a, s, st);
  switch (a.kv_type) {
    case E_F32: return run_absorbed<E_F32>(a, s, st);
    case E_F16: return run_absorbed<E_F16>(a, s, st);
    default: return run_absorbed<E_BF16>(a, s, st);
  }
}

}  // namespace dyn
