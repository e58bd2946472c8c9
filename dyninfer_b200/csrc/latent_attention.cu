// Attention whose cache holds one latent vector per token (shared by all heads) instead of keys and
// values, without positions.
//
// Few rows, or f32: the up-projections are absorbed. score = q . (W_uk c) = (W_uk^T q) . c, so a row's
// queries are mapped into the latent space once per head, the keys of a slice of the cache are scored
// and summed there (one read of the latents serves sixteen heads on the tensor cores, eight in f32), and
// the merge kernel maps the weighted latent back through W_uv, normalises and gates.
//
// Many rows of one sequence on a bf16 cache: the latents up to the portion's end are expanded to keys
// and values (one product per block of tokens, rounded to bf16 as ordinary cached keys are) and the
// tensor-core prefill attention runs on them. Heads narrower than its 128 dims are padded with zeros.
#include <algorithm>

#include "mixers.cuh"

namespace dyn {
namespace {


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

// ---- entry: normalised latents into the cache, queries into the latent space --------------------------
// qa[row][head][rank] = scale * W_uk^T q. CTA = 64 latent dims of one (head, row), eight warps share the
// head's dims; the first sixteen weight rows of a warp are fetched before the kernel waits for the
// products. One more CTA per row normalises and stores the row's latent.
constexpr int AB_R = 64, AB_PRE = 16;
template <int KV, bool PAIR>  // PAIR: bf16 weights, even rank
__global__ void __launch_bounds__(256) latent_enter_kernel(LatentArgs a, StepRows s, float* __restrict__ qa) {
  extern __shared__ float ab_q[];  // [dim]
  __shared__ float part[8][AB_R];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, r0 = blockIdx.x * AB_R;
  const int64_t row = blockIdx.z;
  pdl_trigger();
  if (h == a.heads) {
    pdl_wait();
    if (blockIdx.x) return;
    const float* d = a.d.ptr + row * a.d.ld;
    float ss = 0.f;
    for (int i = tid; i < a.rank; i += 256) ss = fmaf(d[i], d[i], ss);
    ss = warp_sum(ss);
    if (lane == 0) part[warp][0] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) ss += part[w][0];
    const float inv = 1.0f / sqrtf(ss / (float)a.rank + a.eps);
    typename Lat<KV>::T* dst = reinterpret_cast<typename Lat<KV>::T*>(a.cache) + (slot_of(s, row) * a.cap + pos_of(s, row)) * a.rank;
    for (int i = tid; i < a.rank; i += 256) dst[i] = Lat<KV>::enc(d[i] * inv * aux_load(a.norm.ptr, a.norm.type, i));
    return;
  }
  const int64_t w0 = (int64_t)h * a.dim * a.rank;
  const int c = PAIR ? r0 + 2 * lane : r0 + lane;  // PAIR: dims c, c + 1; else c, c + 32
  uint32_t pre[AB_PRE];
  if (PAIR) {
#pragma unroll
    for (int j = 0; j < AB_PRE; j++) {
      const int d = warp + 8 * j;
      pre[j] = d < a.dim && c < a.rank ? *reinterpret_cast<const uint32_t*>(a.uk.data + (w0 + (int64_t)d * a.rank + c) * 2) : 0u;
    }
  }
  pdl_wait();
  const float* q = a.q.ptr + row * a.q.ld + (int64_t)h * a.dim;
  for (int i = tid; i < a.dim; i += 256) ab_q[i] = q[i];
  __syncthreads();
  float s0 = 0.f, s1 = 0.f;
  if (PAIR) {
#pragma unroll
    for (int j = 0; j < AB_PRE; j++) {
      const int d = warp + 8 * j;
      if (d < a.dim) s0 = fmaf(ab_q[d], __uint_as_float(pre[j] << 16), s0), s1 = fmaf(ab_q[d], __uint_as_float(pre[j] & 0xffff0000u), s1);
    }
    for (int d = warp + 8 * AB_PRE; d < a.dim; d += 8) {
      if (c >= a.rank) break;
      const uint32_t u = *reinterpret_cast<const uint32_t*>(a.uk.data + (w0 + (int64_t)d * a.rank + c) * 2);
      s0 = fmaf(ab_q[d], __uint_as_float(u << 16), s0), s1 = fmaf(ab_q[d], __uint_as_float(u & 0xffff0000u), s1);
    }
    part[warp][2 * lane] = s0, part[warp][2 * lane + 1] = s1;
  } else {
#pragma unroll 8
    for (int d = warp; d < a.dim; d += 8) {
      const int64_t at = w0 + (int64_t)d * a.rank;
      if (c < a.rank) s0 = fmaf(ab_q[d], aux_load(a.uk.data, a.uk.enc, at + c), s0);
      if (c + 32 < a.rank) s1 = fmaf(ab_q[d], aux_load(a.uk.data, a.uk.enc, at + c + 32), s1);
    }
    part[warp][lane] = s0, part[warp][lane + 32] = s1;
  }
  __syncthreads();
  if (tid < AB_R && r0 + tid < a.rank) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) t += part[w][tid];
    qa[(row * a.heads + h) * a.rank + r0 + tid] = t * a.scale;
  }
}

// ---- scores and weighted latents of one slice of a row's keys ---------------------------------------
// part[row][head][slice]: weighted sum [rank], maximum, weight sum, two unused floats. A row's n keys are cut
// into slices of whole blocks of 64; slices past the last key write nothing.
constexpr int LA_BLOCK = 64;
__device__ __forceinline__ int64_t part_stride(const LatentArgs& a) { return a.rank + 4; }
__device__ __forceinline__ int64_t slice_keys(int64_t n, int nsplit) {
  return ((n + nsplit - 1) / nsplit + LA_BLOCK - 1) / LA_BLOCK * LA_BLOCK;
}

// Any rank, f32 arithmetic: eight heads per CTA, a warp each; lane owns latent dims lane + 32 j. Latents pass
// through shared memory as f32.
constexpr int LA_H = 8, LA_KEYS = 8;
template <int KV, int RL>
__global__ void __launch_bounds__(256) latent_split_kernel(LatentArgs a, StepRows s, const float* __restrict__ qa,
                                                           float* __restrict__ part) {
  __shared__ float cs[LA_KEYS][RL * 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nsplit = gridDim.x, h = blockIdx.y * LA_H + warp;
  const int64_t row = blockIdx.z;
  pdl_trigger();
  pdl_wait();
  const int64_t n = pos_of(s, row) + 1, per = slice_keys(n, nsplit);
  const int64_t lo = blockIdx.x * per, hi = min(lo + per, n);
  if (lo >= n) return;
  const typename Lat<KV>::T* cache = reinterpret_cast<const typename Lat<KV>::T*>(a.cache) + slot_of(s, row) * a.cap * a.rank;
  const bool head = h < a.heads;
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
  float* out = part + ((row * a.heads + h) * nsplit + blockIdx.x) * part_stride(a);
#pragma unroll
  for (int j = 0; j < RL; j++)
    if (lane + 32 * j < a.rank) out[lane + 32 * j] = acc[j];
  if (lane == 0) out[a.rank] = m, out[a.rank + 1] = l;
}

// 2-byte caches, ranks of whole 16-byte pieces up to 512: sixteen heads per CTA are the rows of an MMA, blocks of
// 64 latents stream through shared memory with cp.async, the next block in flight while the current one is
// used -- read once for scores and values. Latents enter as stored; the f32 queries and weights as hi + lo pairs
// of the cache's type, accumulators are f32. Warp w scores keys 8 w .. of a block and owns 1/8 of the latent dims of the
// weighted sums. NT = padded rank / 64.
template <int KV>
__device__ __forceinline__ void lat_mma(float (&c)[4], const uint4& a, uint32_t b0, uint32_t b1) {
  if constexpr (KV == E_BF16)
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a.x), "r"(a.y), "r"(a.z), "r"(a.w), "r"(b0), "r"(b1));
  else
    asm("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a.x), "r"(a.y), "r"(a.z), "r"(a.w), "r"(b0), "r"(b1));
}

template <int KV>
__device__ __forceinline__ uint32_t bits_of(float v) {
  const typename Lat<KV>::T t = Lat<KV>::enc(v);
  return *reinterpret_cast<const uint16_t*>(&t);
}
template <int KV>
__device__ __forceinline__ void split_pair(float x, float y, uint32_t* hi, uint32_t* lo) {
  const float hx = Lat<KV>::dec(Lat<KV>::enc(x)), hy = Lat<KV>::dec(Lat<KV>::enc(y));
  *hi = bits_of<KV>(x) | (bits_of<KV>(y) << 16);
  *lo = bits_of<KV>(x - hx) | (bits_of<KV>(y - hy) << 16);
}

constexpr int LT_H = 16;
template <int NT>
struct LtSmem {
  static constexpr int RP = NT * 64, PITCH = RP + 8, SP = LA_BLOCK + 4, PP = LA_BLOCK + 8;
  static constexpr int CS = 2 * LA_BLOCK * PITCH * 2, QF = RP / 16 * 2 * 32 * 16, SS = LT_H * SP * 4, PH = LT_H * PP * 2;
  static constexpr int BYTES = CS + QF + SS + 2 * PH + 3 * LT_H * 4;
};

template <int KV, int NT>
__global__ void __launch_bounds__(256) latent_split_tc_kernel(LatentArgs a, StepRows s, const float* __restrict__ qa,
                                                              float* __restrict__ part) {
  using T = typename Lat<KV>::T;
  using L = LtSmem<NT>;
  extern __shared__ __align__(16) uint8_t lt_smem[];
  T* cs = reinterpret_cast<T*>(lt_smem);                                  // [buffer][key][PITCH]
  uint4* qf = reinterpret_cast<uint4*>(lt_smem + L::CS);                  // [k-step][hi, lo][lane]
  float* ss = reinterpret_cast<float*>(lt_smem + L::CS + L::QF);          // [head][SP]
  T* ph = reinterpret_cast<T*>(lt_smem + L::CS + L::QF + L::SS);          // [head][PP]
  T* pl = ph + LT_H * L::PP;
  float* row_m = reinterpret_cast<float*>(lt_smem + L::CS + L::QF + L::SS + 2 * L::PH);
  float *row_l = row_m + LT_H, *row_f = row_l + LT_H;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int nsplit = gridDim.x, h0 = blockIdx.y * LT_H;
  const int64_t row = blockIdx.z;
  pdl_trigger();
  pdl_wait();
  const int64_t n = pos_of(s, row) + 1, per = slice_keys(n, nsplit);
  const int64_t lo = blockIdx.x * per, hi = min(lo + per, n);
  if (lo >= n) return;
  const T* cache = reinterpret_cast<const T*>(a.cache) + slot_of(s, row) * a.cap * a.rank;
  auto load = [&](int64_t k0, int b) {  // keys past the slice and dims past the rank arrive as zeros
    for (int i = tid; i < LA_BLOCK * (L::RP / 8); i += 256) {
      const int k = i / (L::RP / 8), p = i % (L::RP / 8);
      const bool live = k0 + k < hi && p * 8 < a.rank;
      const T* src = cache + (live ? (k0 + k) * a.rank + p * 8 : 0);
      const unsigned dst = (unsigned)__cvta_generic_to_shared(cs + ((size_t)b * LA_BLOCK + k) * L::PITCH + p * 8);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(lo, 0);
  for (int i = tid; i < L::RP / 16 * 32; i += 256) {
    const int kk = i / 32, ln = i % 32, r = ln >> 2, c = 16 * kk + 2 * (ln & 3);
    auto at = [&](int hr, int cc) {
      return h0 + hr < a.heads && cc < a.rank ? qa[(row * a.heads + h0 + hr) * a.rank + cc] : 0.f;
    };
    uint4 hq, lq;
    split_pair<KV>(at(r, c), at(r, c + 1), &hq.x, &lq.x);
    split_pair<KV>(at(r + 8, c), at(r + 8, c + 1), &hq.y, &lq.y);
    split_pair<KV>(at(r, c + 8), at(r, c + 9), &hq.z, &lq.z);
    split_pair<KV>(at(r + 8, c + 8), at(r + 8, c + 9), &hq.w, &lq.w);
    qf[(2 * kk) * 32 + ln] = hq, qf[(2 * kk + 1) * 32 + ln] = lq;
  }
  if (tid < LT_H) row_m[tid] = -3.40282347e38f, row_l[tid] = 0.f;
  float o[NT][4] = {};
  int b = 0;
  for (int64_t k0 = lo; k0 < hi; k0 += LA_BLOCK, b ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the block has arrived for everyone, nobody reads the other buffer any more
    if (k0 + LA_BLOCK < hi) load(k0 + LA_BLOCK, b ^ 1);
    const T* cb = cs + (size_t)b * LA_BLOCK * L::PITCH;
    {
      float acc[4][4] = {};
      const T* key = cb + (8 * warp + g) * L::PITCH;
#pragma unroll
      for (int kk = 0; kk < L::RP / 16; kk++) {
        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(key + 16 * kk + 2 * t);
        const uint32_t b1 = *reinterpret_cast<const uint32_t*>(key + 16 * kk + 8 + 2 * t);
        lat_mma<KV>(acc[kk & 1], qf[(2 * kk) * 32 + lane], b0, b1);
        lat_mma<KV>(acc[2 + (kk & 1)], qf[(2 * kk + 1) * 32 + lane], b0, b1);
      }
#pragma unroll
      for (int e = 0; e < 4; e++)
        ss[(g + 8 * (e >> 1)) * L::SP + 8 * warp + 2 * t + (e & 1)] = (acc[0][e] + acc[1][e]) + (acc[2][e] + acc[3][e]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int r = 2 * warp + i;
      const bool in0 = k0 + lane < hi, in1 = k0 + lane + 32 < hi;
      const float x0 = in0 ? ss[r * L::SP + lane] : -3.40282347e38f, x1 = in1 ? ss[r * L::SP + lane + 32] : -3.40282347e38f;
      const float m0 = row_m[r], mn = fmaxf(m0, warp_max(fmaxf(x0, x1)));
      const float p0 = in0 ? expf(x0 - mn) : 0.f, p1 = in1 ? expf(x1 - mn) : 0.f;
      const float f = expf(m0 - mn), sum = warp_sum(p0 + p1);
      const T q0 = Lat<KV>::enc(p0), q1 = Lat<KV>::enc(p1);
      ph[r * L::PP + lane] = q0, ph[r * L::PP + lane + 32] = q1;
      pl[r * L::PP + lane] = Lat<KV>::enc(p0 - Lat<KV>::dec(q0)), pl[r * L::PP + lane + 32] = Lat<KV>::enc(p1 - Lat<KV>::dec(q1));
      __syncwarp();
      if (lane == 0) row_m[r] = mn, row_l[r] = row_l[r] * f + sum, row_f[r] = f;
    }
    __syncthreads();
    const float f0 = row_f[g], f1 = row_f[g + 8];
#pragma unroll
    for (int nt = 0; nt < NT; nt++) o[nt][0] *= f0, o[nt][1] *= f0, o[nt][2] *= f1, o[nt][3] *= f1;
#pragma unroll
    for (int j = 0; j < LA_BLOCK / 16; j++) {
      auto frag = [&](const T* p) {
        uint4 v;
        v.x = *reinterpret_cast<const uint32_t*>(p + g * L::PP + 16 * j + 2 * t);
        v.y = *reinterpret_cast<const uint32_t*>(p + (g + 8) * L::PP + 16 * j + 2 * t);
        v.z = *reinterpret_cast<const uint32_t*>(p + g * L::PP + 16 * j + 8 + 2 * t);
        v.w = *reinterpret_cast<const uint32_t*>(p + (g + 8) * L::PP + 16 * j + 8 + 2 * t);
        return v;
      };
      const uint4 hf = frag(ph), lf = frag(pl);
#pragma unroll
      for (int nt = 0; nt < NT; nt++) {
        uint32_t b0, b1;
        const T* src = cb + (16 * j + (lane & 15)) * L::PITCH + (warp * NT + nt) * 8;
        asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];"
                     : "=r"(b0), "=r"(b1) : "r"((uint32_t)__cvta_generic_to_shared(src)));
        lat_mma<KV>(o[nt], hf, b0, b1);
        lat_mma<KV>(o[nt], lf, b0, b1);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; e++) {
    const int h = h0 + g + 8 * e;
    if (h >= a.heads) continue;
    float* out = part + ((row * a.heads + h) * nsplit + blockIdx.x) * part_stride(a);
#pragma unroll
    for (int nt = 0; nt < NT; nt++) {
      const int c = (warp * NT + nt) * 8 + 2 * t;
      if (c < a.rank) out[c] = o[nt][2 * e];
      if (c + 1 < a.rank) out[c + 1] = o[nt][2 * e + 1];
    }
    if (warp == 0 && t == 0) out[a.rank] = row_m[g + 8 * e], out[a.rank + 1] = row_l[g + 8 * e];
  }
}

// ---- slices merged, W_uv, output gate: CTA = 32 value dims of one (head, row) ----------------------------
// The merge is shared by groups of threads that take slices in turn; with WIDE (bf16 rows of whole 16-byte
// pieces up to 512) the CTA's weight rows are fetched before the kernel waits for the slices.
constexpr int LV_E = 32, LV_SLICES = 64;
template <bool WIDE>
__global__ void __launch_bounds__(256) latent_value_kernel(LatentArgs a, StepRows s, const float* __restrict__ part, int nsplit) {
  extern __shared__ __align__(16) float lv_smem[];
  __shared__ float wts[LV_SLICES];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, e0 = blockIdx.x * LV_E, R = a.rank;
  const int64_t row = blockIdx.z;
  pdl_trigger();
  uint4 wv[4][2];
  if (WIDE) {
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int p = 0; p < 2; p++) {
        const int e = e0 + warp + 8 * i, c = (p * 32 + lane) * 8;
        wv[i][p] = e < a.vdim && c < R ? *reinterpret_cast<const uint4*>(a.uv.data + (((int64_t)h * a.vdim + e) * R + c) * 2)
                                       : make_uint4(0, 0, 0, 0);
      }
  }
  pdl_wait();
  const int64_t n = pos_of(s, row) + 1, per = slice_keys(n, nsplit);
  const int ns = (int)((n + per - 1) / per);
  const int64_t stride = part_stride(a);
  const float* p0 = part + (row * a.heads + h) * (int64_t)nsplit * stride;
  if (warp == 0) {
    float m0 = lane < ns ? p0[lane * stride + R] : -3.40282347e38f, m1 = lane + 32 < ns ? p0[(lane + 32) * stride + R] : -3.40282347e38f;
    const float gm = warp_max(fmaxf(m0, m1));
    m0 = lane < ns ? expf(m0 - gm) : 0.f, m1 = lane + 32 < ns ? expf(m1 - gm) : 0.f;
    const float gl = warp_sum((lane < ns ? m0 * p0[lane * stride + R + 1] : 0.f) +
                              (lane + 32 < ns ? m1 * p0[(lane + 32) * stride + R + 1] : 0.f));
    wts[lane] = m0 / gl, wts[lane + 32] = m1 / gl;
  }
  __syncthreads();
  float* lat = lv_smem;  // [groups][R]
  const int quads = (R + 3) / 4, groups = R % 4 == 0 && quads <= 128 ? 256 / quads : 1;
  if (R % 4 == 0) {
    for (int i = tid; i < groups * quads; i += 256) {
      const int grp = i / quads, c = (i % quads) * 4;
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int k = grp; k < ns; k += groups) {
        const float4 v = *reinterpret_cast<const float4*>(p0 + k * stride + c);
        const float w = wts[k];
        t.x = fmaf(v.x, w, t.x), t.y = fmaf(v.y, w, t.y), t.z = fmaf(v.z, w, t.z), t.w = fmaf(v.w, w, t.w);
      }
      *reinterpret_cast<float4*>(lat + grp * R + c) = t;
    }
  } else {
    for (int c = tid; c < R; c += 256) {
      float t = 0.f;
      for (int k = 0; k < ns; k++) t = fmaf(p0[k * stride + c], wts[k], t);
      lat[c] = t;
    }
  }
  __syncthreads();
  if (groups > 1) {
    for (int c = tid; c < R; c += 256) {
      float t = lat[c];
      for (int k = 1; k < groups; k++) t += lat[k * R + c];
      lat[c] = t;  // the thread's own column
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int e = e0 + warp + 8 * i;
    if (e >= a.vdim) break;
    float t = 0.f;
    if (WIDE) {
#pragma unroll
      for (int p = 0; p < 2; p++) {
        const int c = (p * 32 + lane) * 8;
        if (c >= R) continue;
        const uint32_t u[4] = {wv[i][p].x, wv[i][p].y, wv[i][p].z, wv[i][p].w};
#pragma unroll
        for (int k = 0; k < 4; k++)
          t = fmaf(__uint_as_float(u[k] << 16), lat[c + 2 * k], t), t = fmaf(__uint_as_float(u[k] & 0xffff0000u), lat[c + 2 * k + 1], t);
      }
    } else {
      const int64_t at = ((int64_t)h * a.vdim + e) * R;
      for (int c = lane; c < R; c += 32) t = fmaf(aux_load(a.uv.data, a.uv.enc, at + c), lat[c], t);
    }
    t = warp_sum(t);
    if (lane == 0)
      a.out[(row * a.heads + h) * a.vdim + e] = t * sigmoid_of(a.g.ptr[row * a.g.ld + (int64_t)h * a.vdim + e]);
  }
}

bool tensor_cores(const LatentArgs& a) {
  return !a.exact && (a.kv_type == E_BF16 || a.kv_type == E_F16) && a.rank % 8 == 0 && a.rank <= 512;
}

// The slice count depends only on shapes and capacity, so a captured graph stays valid as positions grow.
int slices(const LatentArgs& a, int64_t rows) {
  const int per_cta = tensor_cores(a) ? LT_H : LA_H;
  const int64_t groups = rows * ((a.heads + per_cta - 1) / per_cta);
  return (int)std::max<int64_t>(1, std::min<int64_t>({LV_SLICES, a.cap / LA_BLOCK, (tensor_cores(a) ? 148 : 296) / groups}));
}

template <int KV, int NT>
int split_tc(const LatentArgs& a, const StepRows& s, const float* qa, float* part, int ns, cudaStream_t st) {
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(latent_split_tc_kernel<KV, NT>), LtSmem<NT>::BYTES)) return 1;
  DYN_CUDA(launch_pdl(latent_split_tc_kernel<KV, NT>, dim3((unsigned)ns, (unsigned)((a.heads + LT_H - 1) / LT_H), (unsigned)s.rows),
                      dim3(256), LtSmem<NT>::BYTES, st, a, s, qa, part));
  return 0;
}

template <int KV, int RL>
int split_simt(const LatentArgs& a, const StepRows& s, const float* qa, float* part, int ns, cudaStream_t st) {
  DYN_CUDA(launch_pdl(latent_split_kernel<KV, RL>, dim3((unsigned)ns, (unsigned)((a.heads + LA_H - 1) / LA_H), (unsigned)s.rows),
                      dim3(256), 0, st, a, s, qa, part));
  return 0;
}

template <int KV>
int run_absorbed(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  const int64_t rows = s.rows;
  float* qa = a.scratch;
  float* part = qa + (rows * a.heads * a.rank + 3) / 4 * 4;
  const int ns = slices(a, rows);
  DYN_CHECK(a.rank <= 1024 && a.dim <= 8192, "latent attention: rank %d or head dim %d is too large", a.rank, a.dim);
  DYN_CHECK(rows <= 65535 && a.heads < 65535, "latent attention: %lld rows in one step", (long long)rows);
  {
    const bool pair = a.uk.enc == E_BF16 && a.rank % 2 == 0;
    const dim3 grid((unsigned)((a.rank + AB_R - 1) / AB_R), (unsigned)a.heads + 1, (unsigned)rows);
    const size_t smem = (size_t)a.dim * 4;
    if (pair)
      DYN_CUDA(launch_pdl(latent_enter_kernel<KV, true>, grid, dim3(256), smem, st, a, s, qa));
    else
      DYN_CUDA(launch_pdl(latent_enter_kernel<KV, false>, grid, dim3(256), smem, st, a, s, qa));
  }
  if (KV != E_F32 && tensor_cores(a)) {
    constexpr int TC = KV == E_F32 ? E_BF16 : KV;  // f32 caches never come here
    if (a.rank <= 64 ? split_tc<TC, 1>(a, s, qa, part, ns, st) : a.rank <= 128 ? split_tc<TC, 2>(a, s, qa, part, ns, st)
        : a.rank <= 256 ? split_tc<TC, 4>(a, s, qa, part, ns, st) : split_tc<TC, 8>(a, s, qa, part, ns, st))
      return 1;
  } else if (a.rank <= 128 ? split_simt<KV, 4>(a, s, qa, part, ns, st) : a.rank <= 256 ? split_simt<KV, 8>(a, s, qa, part, ns, st)
             : a.rank <= 512 ? split_simt<KV, 16>(a, s, qa, part, ns, st) : split_simt<KV, 32>(a, s, qa, part, ns, st)) {
    return 1;
  }
  {
    const bool wide = a.uv.enc == E_BF16 && a.rank % 8 == 0 && a.rank <= 512 && (reinterpret_cast<uintptr_t>(a.uv.data) & 15) == 0;
    const int quads = (a.rank + 3) / 4, groups = a.rank % 4 == 0 && quads <= 128 ? 256 / quads : 1;
    const dim3 grid((unsigned)((a.vdim + LV_E - 1) / LV_E), (unsigned)a.heads, (unsigned)rows);
    const size_t smem = (size_t)groups * a.rank * 4;
    if (wide)
      DYN_CUDA(launch_pdl(latent_value_kernel<true>, grid, dim3(256), smem, st, a, s, part, ns));
    else
      DYN_CUDA(launch_pdl(latent_value_kernel<false>, grid, dim3(256), smem, st, a, s, part, ns));
  }
  count_launch(3);
  DYN_CUDA(cudaGetLastError());
  return 0;
}

// ---- expanded keys and values ---------------------------------------------------------------------
constexpr int EX_D = 128;  // head width of the prefill attention
constexpr int EX_SPLITS = 4;  // K-split sums of the up-projection kept for the expansion to add

// y rows [k heads | v heads] of tokens t0.. -> K, V planes [head][cap][128] bf16, zero padded. With splits > 1
// the rows still lie as that many K-split sums `zstride` floats apart.
__global__ void __launch_bounds__(256)
latent_expand_kernel(const float* __restrict__ k, int64_t ldk, const float* __restrict__ v, int64_t ldv, int splits, int64_t zstride,
                     int heads, int dim, int vdim,
                     int64_t t0, int64_t tokens, int64_t cap, __nv_bfloat162* __restrict__ kx, __nv_bfloat162* __restrict__ vx) {
  const int64_t total = tokens * heads * (EX_D / 2);
  for (int64_t it = blockIdx.x * 256ll + threadIdx.x; it < total; it += (int64_t)gridDim.x * 256) {
    const int c = (int)(it % (EX_D / 2)) * 2;
    const int64_t th = it / (EX_D / 2), h = th % heads, t = th / heads;
    const float* kr = k + t * ldk + h * dim;
    const float* vr = v + t * ldv + h * vdim;
    const int64_t at = ((h * cap + t0 + t) * EX_D + c) / 2;
    float k0 = 0.f, k1 = 0.f, v0 = 0.f, v1 = 0.f;
    for (int z = 0; z < splits; z++, kr += zstride, vr += zstride) {
      if (c < dim) k0 += kr[c];
      if (c + 1 < dim) k1 += kr[c + 1];
      if (c < vdim) v0 += vr[c];
      if (c + 1 < vdim) v1 += vr[c + 1];
    }
    kx[at] = __floats2bfloat162_rn(k0, k1);
    vx[at] = __floats2bfloat162_rn(v0, v1);
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

// Normalised latents of a portion into the cache: one block per row.
template <int KV>
__global__ void __launch_bounds__(128) latent_store_kernel(LatentArgs a, StepRows s) {
  __shared__ float red[4];
  const int tid = threadIdx.x;
  const int64_t r = blockIdx.x;
  const float* d = a.d.ptr + r * a.d.ld;
  float ss = 0.f;
  for (int i = tid; i < a.rank; i += 128) ss = fmaf(d[i], d[i], ss);
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  const float inv = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)a.rank + a.eps);
  typename Lat<KV>::T* dst = reinterpret_cast<typename Lat<KV>::T*>(a.cache) + (slot_of(s, r) * a.cap + pos_of(s, r)) * a.rank;
  for (int i = tid; i < a.rank; i += 128) dst[i] = Lat<KV>::enc(d[i] * inv * aux_load(a.norm.ptr, a.norm.type, i));
}

unsigned ew_grid(int64_t total) { return (unsigned)std::max<int64_t>(1, std::min<int64_t>((total + 255) / 256, 148 * 16)); }

int run_expanded(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  const int64_t rows = s.rows, H = a.heads, end = s.base + rows;
  const int64_t kd = H * a.dim, vd = H * a.vdim;
  __nv_bfloat16* kx = reinterpret_cast<__nv_bfloat16*>(a.scratch);
  __nv_bfloat16* vx = kx + H * a.cap * EX_D;
  float* y = reinterpret_cast<float*>(vx + H * a.cap * EX_D);  // [EX_SPLITS][max_rows, kd + vd]
  float* qp = y + EX_SPLITS * a.max_rows * (kd + vd);          // [rows, H * 128]
  float* ctx = qp + a.max_rows * H * EX_D;
  const __nv_bfloat16* lat = reinterpret_cast<const __nv_bfloat16*>(a.cache) + s.slot * a.cap * a.rank;
  for (int64_t t0 = 0; t0 < end; t0 += a.max_rows) {
    const int64_t n = std::min(a.max_rows, end - t0);
    const float *k = y, *v = y + kd;
    int64_t ldk = kd + vd, ldv = kd + vd;
    int splits = 1;
    if (a.ukv.data && n > 16 && dqgemm_tc_takes(a.ukv, n)) {
      TgIo io;
      io.partial = y, io.partial_bytes = (size_t)EX_SPLITS * a.max_rows * (kd + vd) * 4;
      bool handled = false;
      if (launch_dqgemm_tc(a.ukv, lat + t0 * a.rank, E_BF16, n, y, nullptr, st, &handled, &io)) return 1;
      DYN_CHECK(handled, "dequant GEMM refused a product it had accepted");
      splits = std::max(1, io.splits);
    } else if (a.ukv.data) {
      if (launch_linear(a.ukv, lat + t0 * a.rank, E_BF16, n, y, nullptr, st)) return 1;
    } else {
      v = y + n * kd, ldk = kd, ldv = vd;
      if (launch_linear(a.uk, lat + t0 * a.rank, E_BF16, n, y, nullptr, st) ||
          launch_linear(a.uv, lat + t0 * a.rank, E_BF16, n, y + n * kd, nullptr, st))
        return 1;
    }
    latent_expand_kernel<<<ew_grid(n * H * (EX_D / 2)), 256, 0, st>>>(k, ldk, v, ldv, splits, n * (kd + vd), a.heads, a.dim, a.vdim, t0, n, a.cap,
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
    need = std::max(need, (size_t)r * a.heads * (a.rank + (size_t)slices(a, r) * (a.rank + 4)) + 4);
  if (expands(a) && rows >= EXPAND_MIN_ROWS)
    need = std::max(need, (size_t)a.heads * a.cap * EX_D +
                              (size_t)a.max_rows * a.heads * (EX_SPLITS * (a.dim + a.vdim) + 2 * EX_D) + 64);
  return need;
}

int launch_latent_attention(const LatentArgs& a, const StepRows& s, cudaStream_t st) {
  if (s.rows == 0) return 0;
  if (s.base >= 0 && s.rows >= EXPAND_MIN_ROWS && expands(a)) {
    latent_store_kernel<E_BF16><<<(unsigned)s.rows, 128, 0, st>>>(a, s);
    count_launch();
    return run_expanded(a, s, st);
  }
  switch (a.kv_type) {
    case E_F32: return run_absorbed<E_F32>(a, s, st);
    case E_F16: return run_absorbed<E_F16>(a, s, st);
    case E_BF16: return run_absorbed<E_BF16>(a, s, st);
    default: DYN_CHECK(false, "kv_type %d unsupported", a.kv_type);
  }
  return 0;
}

}  // namespace dyn
