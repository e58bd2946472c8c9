// Gated linear recurrence behind a short causal convolution: two input branches x (recurrent) and y
// (gate), block-diagonal recurrence and input gates, a diagonal f32 state per channel.
//
// The convolution's inputs live in a ring of `taps` rows per slot, position p in row p mod taps, so a
// decode step writes its own row while other CTAs still read the rows before it. Positions before the
// sequence start count as zeros and are never read.
//
// Decode rows: one launch per layer. A CTA takes 16 outputs of one gate block: it forms the block's
// convolution outputs (a few multiplies, repeated by the block's CTAs), then a warp per output reads
// the two gate rows and updates the state.
// Portions: convolution -> gates (a tiled block-diagonal product whose epilogue leaves a_t and the
// increment b_t) -> scan. The scan handles 512 tokens x 16 channels per CTA and pass: a thread composes
// the maps S -> A S + B of its 8 tokens, the 64 segment maps are chained through shared memory, and
// each thread replays its tokens from its start state.
#include <algorithm>

#include "mixers.cuh"

namespace dyn {
namespace {

__device__ __forceinline__ float gelu_tanh_of(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// gate sums -> (a, sqrt(1 - a^2) i u); 1 - a^2 from the logarithm, without cancellation near a = 1
__device__ __forceinline__ void recurrence_terms(float rz, float iz, float u, float c, float lam, float* a, float* b) {
  const float la = -c * sigmoid_of(rz) * softplus_of(lam);
  *a = expf(la);
  *b = sqrtf(-expm1f(2.0f * la)) * sigmoid_of(iz) * u;
}

// ---- decode rows -----------------------------------------------------------------------------
constexpr int RG_OUT = 16, RG_PER_WARP = RG_OUT / 8;

__device__ __forceinline__ float dot8(const uint4& w, const float* u) {
  const uint32_t x[4] = {w.x, w.y, w.z, w.w};
  float s = 0.f;
#pragma unroll
  for (int e = 0; e < 4; e++)
    s = fmaf(__uint_as_float(x[e] << 16), u[2 * e], s), s = fmaf(__uint_as_float(x[e] & 0xffff0000u), u[2 * e + 1], s);
  return s;
}

// WIDE: bf16 gate rows of whole 16-byte pieces; a warp's first piece per lane of its four gate rows is fetched
// before the kernel waits for the products.
template <bool WIDE>
__global__ void __launch_bounds__(256) rglru_step_kernel(RglruArgs a, const int64_t* row_pos, const int64_t* row_seq,
                                                         int64_t pos0, int64_t seq0, int64_t row0) {
  extern __shared__ __align__(16) float u_s[];  // [width / blocks]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n = a.width / a.blocks, slices = (n + RG_OUT - 1) / RG_OUT;
  const int blk = blockIdx.x / slices, slice = blockIdx.x % slices;
  const int64_t r = row0 + blockIdx.y;
  const int pieces = n / 8;
  pdl_trigger();
  uint4 wr[RG_PER_WARP], wi[RG_PER_WARP];
  if (WIDE) {
#pragma unroll
    for (int i = 0; i < RG_PER_WARP; i++) {
      const int o = slice * RG_OUT + warp + 8 * i;
      const int64_t at = (int64_t)blk * n + o;
      if (o < n && lane < pieces) {
        wr[i] = reinterpret_cast<const uint4*>(a.ra.ptr + at * n * 2)[lane];
        wi[i] = reinterpret_cast<const uint4*>(a.ri.ptr + at * n * 2)[lane];
      }
    }
  }
  pdl_wait();
  const int64_t pos = row_pos ? row_pos[r] : pos0, seq = row_seq ? row_seq[r] : seq0;
  float* ring = a.ring + seq * (int64_t)a.taps * a.width;
  const float* x = a.x.ptr + r * a.x.ld;
  for (int c = tid; c < n; c += 256) {
    const int64_t ch = (int64_t)blk * n + c;
    const float xin = x[ch] + vec_at(a.bx, ch);
    float u = vec_at(a.conv, ch * a.taps + a.taps - 1) * xin;
#pragma unroll 4
    for (int j = 1; j < a.taps; j++)
      if (pos >= j) u = fmaf(vec_at(a.conv, ch * a.taps + a.taps - 1 - j), ring[((pos - j) % a.taps) * a.width + ch], u);
    u_s[c] = u + vec_at(a.bc, ch);
    if (slice == 0) ring[(pos % a.taps) * a.width + ch] = xin;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < RG_PER_WARP; i++) {
    const int o = slice * RG_OUT + warp + 8 * i;
    if (o >= n) break;
    const int64_t ch = (int64_t)blk * n + o;
    float rz = 0.f, iz = 0.f;
    if (WIDE) {
      if (lane < pieces) rz = dot8(wr[i], u_s + 8 * lane), iz = dot8(wi[i], u_s + 8 * lane);
      for (int p = lane + 32; p < pieces; p += 32) {
        rz += dot8(reinterpret_cast<const uint4*>(a.ra.ptr + ch * n * 2)[p], u_s + 8 * p);
        iz += dot8(reinterpret_cast<const uint4*>(a.ri.ptr + ch * n * 2)[p], u_s + 8 * p);
      }
    } else {
      for (int k = lane; k < n; k += 32) {
        rz = fmaf(vec_at(a.ra, ch * n + k), u_s[k], rz);
        iz = fmaf(vec_at(a.ri, ch * n + k), u_s[k], iz);
      }
    }
    rz = warp_sum(rz), iz = warp_sum(iz);
    if (lane == 0) {
      float av, bv;
      recurrence_terms(rz + vec_at(a.bra, ch), iz + vec_at(a.bri, ch), u_s[o], a.c, vec_at(a.lam, ch), &av, &bv);
      float* S = a.state + seq * a.width + ch;
      const float s = pos > 0 ? fmaf(av, *S, bv) : bv;
      *S = s;
      a.out[r * a.width + ch] = s * gelu_tanh_of(a.y.ptr[r * a.y.ld + ch] + vec_at(a.by, ch));
    }
  }
}

bool wide_rows(const RglruArgs& a) {
  const int n = a.width / a.blocks;
  auto ok = [&](const Vec& v) { return v.type == E_BF16 && (reinterpret_cast<uintptr_t>(v.ptr) & 15) == 0; };
  return n % 8 == 0 && ok(a.ra) && ok(a.ri);
}

int step_rows(const RglruArgs& a, const int64_t* pos, const int64_t* seq, int64_t pos0, int64_t seq0, int64_t row0,
              int64_t rows, cudaStream_t st) {
  const int n = a.width / a.blocks, slices = (n + RG_OUT - 1) / RG_OUT;
  const size_t smem = (size_t)n * 4;
  DYN_CHECK(smem <= 48 * 1024, "rglru: a gate block of %d channels is too large", n);
  for (int64_t r0 = 0; r0 < rows; r0 += 65535) {
    const dim3 grid((unsigned)(a.blocks * slices), (unsigned)std::min<int64_t>(65535, rows - r0));
    if (wide_rows(a))
      DYN_CUDA(launch_pdl(rglru_step_kernel<true>, grid, dim3(256), smem, st, a, pos, seq, pos0, seq0, row0 + r0));
    else
      DYN_CUDA(launch_pdl(rglru_step_kernel<false>, grid, dim3(256), smem, st, a, pos, seq, pos0, seq0, row0 + r0));
    count_launch();
  }
  DYN_CUDA(cudaGetLastError());
  return 0;
}

// ---- portions ---------------------------------------------------------------------------------
// u[t][ch]; inputs from before the portion come from the ring. A thread takes one channel and CV_T tokens; with
// TAPS > 0 the window of inputs stays in registers.
constexpr int CV_T = 16;
template <int TAPS>
__global__ void __launch_bounds__(128) rglru_conv_kernel(RglruArgs a, int64_t rows, int64_t base, int64_t slot, float* __restrict__ u) {
  const int ch = blockIdx.x * 128 + threadIdx.x;
  if (ch >= a.width) return;
  const float* ring = a.ring + slot * (int64_t)a.taps * a.width;
  const float bx = vec_at(a.bx, ch), bc = vec_at(a.bc, ch);
  const int64_t t0 = (int64_t)blockIdx.y * CV_T;
  auto input = [&](int64_t t) {  // of token base + t, t possibly before the portion
    if (t >= 0) return t < rows ? a.x.ptr[t * a.x.ld + ch] + bx : 0.f;
    return base + t >= 0 ? ring[((base + t) % a.taps) * a.width + ch] : 0.f;
  };
  if constexpr (TAPS > 0) {
    float w[TAPS], in[CV_T + TAPS - 1];
#pragma unroll
    for (int j = 0; j < TAPS; j++) w[j] = vec_at(a.conv, (int64_t)ch * TAPS + j);
#pragma unroll
    for (int j = 0; j < CV_T + TAPS - 1; j++) in[j] = input(t0 + j - (TAPS - 1));
#pragma unroll
    for (int i = 0; i < CV_T; i++) {
      float acc = 0.f;
#pragma unroll
      for (int j = TAPS - 1; j >= 0; j--) acc = fmaf(w[j], in[i + j], acc);
      if (t0 + i < rows) u[(t0 + i) * a.width + ch] = acc + bc;
    }
  } else {
    for (int i = 0; i < CV_T && t0 + i < rows; i++) {
      float acc = 0.f;
      for (int j = 0; j < a.taps; j++)
        acc = fmaf(vec_at(a.conv, (int64_t)ch * a.taps + a.taps - 1 - j), input(t0 + i - j), acc);
      u[(t0 + i) * a.width + ch] = acc + bc;
    }
  }
}

// Gates on the tensor cores for bf16 weights: 64 tokens x 64 outputs of one block per CTA, both products. The f32
// inputs enter as three bf16 terms (hi + mid + lo hold all 24 bits), the weights as stored, so every product
// is exact and the sums are f32: these are gates of a recurrence, not 16-bit activations. Warp w takes 16 tokens
// (w mod 4) of one of the two matrices (w / 4).
constexpr int GT_T = 64, GT_K = 64, GT_P = GT_K + 8;
constexpr int GT_SMEM = (3 * GT_T + 2 * GT_T) * GT_P * 2;
__global__ void __launch_bounds__(256)
rglru_gates_tc_kernel(RglruArgs a, int64_t rows, const float* __restrict__ u, float* __restrict__ av, float* __restrict__ bv) {
  extern __shared__ __align__(16) uint8_t gt_smem[];
  __nv_bfloat16(*us)[GT_T][GT_P] = reinterpret_cast<__nv_bfloat16(*)[GT_T][GT_P]>(gt_smem);              // [term][token][k]
  __nv_bfloat16(*ws)[GT_T][GT_P] = reinterpret_cast<__nv_bfloat16(*)[GT_T][GT_P]>(gt_smem + 3 * GT_T * GT_P * 2);  // [matrix][output][k]
  float(*zs)[GT_T + 4] = reinterpret_cast<float(*)[GT_T + 4]>(gt_smem);                                  // [matrix * 64 + token][output], afterwards
  static_assert(2 * GT_T * (GT_T + 4) * 4 <= GT_SMEM, "gate sums fit the operand tiles");
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int n = a.width / a.blocks, tiles = (n + GT_T - 1) / GT_T;
  const int blk = blockIdx.x / tiles, o0 = (blockIdx.x % tiles) * GT_T;
  const int64_t t0 = (int64_t)blockIdx.y * GT_T;
  const int mt = warp & 3, mat = warp >> 2;
  float acc[8][4] = {};
  constexpr int UQ = GT_T * GT_K / 4 / 256, WQ = 2 * GT_T * GT_K / 8 / 256;
  float4 uq[UQ];
  uint4 wq[WQ];
  auto fetch = [&](int k0) {  // the next slice is under way while the current one is used
#pragma unroll
    for (int j = 0; j < UQ; j++) {
      const int i = tid + 256 * j, tok = i / (GT_K / 4), k = (i % (GT_K / 4)) * 4;  // n is a multiple of 8: whole quads
      uq[j] = t0 + tok < rows && k0 + k < n ? *reinterpret_cast<const float4*>(u + (t0 + tok) * a.width + blk * n + k0 + k)
                                            : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < WQ; j++) {
      const int i = tid + 256 * j, m = i / (GT_T * GT_K / 8), o = (i / (GT_K / 8)) % GT_T, k = (i % (GT_K / 8)) * 8;
      wq[j] = o0 + o < n && k0 + k < n
                  ? *reinterpret_cast<const uint4*>((m ? a.ri.ptr : a.ra.ptr) + (((int64_t)blk * n + o0 + o) * n + k0 + k) * 2)
                  : make_uint4(0, 0, 0, 0);
    }
  };
  fetch(0);
  for (int k0 = 0; k0 < n; k0 += GT_K) {
#pragma unroll
    for (int j = 0; j < UQ; j++) {
      const int i = tid + 256 * j, tok = i / (GT_K / 4), k = (i % (GT_K / 4)) * 4;
      const float x[4] = {uq[j].x, uq[j].y, uq[j].z, uq[j].w};
      uint32_t t3[3][2];
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const __nv_bfloat16 h = __float2bfloat16_rn(x[e]);
        const float r1 = x[e] - __bfloat162float(h);
        const __nv_bfloat16 m = __float2bfloat16_rn(r1);
        const uint32_t b[3] = {__bfloat16_as_ushort(h), __bfloat16_as_ushort(m),
                               __bfloat16_as_ushort(__float2bfloat16_rn(r1 - __bfloat162float(m)))};
#pragma unroll
        for (int s = 0; s < 3; s++) t3[s][e / 2] = e % 2 ? t3[s][e / 2] | (b[s] << 16) : b[s];
      }
#pragma unroll
      for (int s = 0; s < 3; s++) *reinterpret_cast<uint2*>(&us[s][tok][k]) = make_uint2(t3[s][0], t3[s][1]);
    }
#pragma unroll
    for (int j = 0; j < WQ; j++) {
      const int i = tid + 256 * j, m = i / (GT_T * GT_K / 8), o = (i / (GT_K / 8)) % GT_T, k = (i % (GT_K / 8)) * 8;
      *reinterpret_cast<uint4*>(&ws[m][o][k]) = wq[j];
    }
    if (k0 + GT_K < n) fetch(k0 + GT_K);
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < GT_K / 16; kk++) {
      uint32_t af[3][4];
#pragma unroll
      for (int s = 0; s < 3; s++) {
        const __nv_bfloat16 *p0 = &us[s][16 * mt + g][16 * kk + 2 * t], *p1 = &us[s][16 * mt + g + 8][16 * kk + 2 * t];
        af[s][0] = *reinterpret_cast<const uint32_t*>(p0), af[s][1] = *reinterpret_cast<const uint32_t*>(p1);
        af[s][2] = *reinterpret_cast<const uint32_t*>(p0 + 8), af[s][3] = *reinterpret_cast<const uint32_t*>(p1 + 8);
      }
#pragma unroll
      for (int nt = 0; nt < 8; nt++) {
        const __nv_bfloat16* p = &ws[mat][8 * nt + g][16 * kk + 2 * t];
        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(p), b1 = *reinterpret_cast<const uint32_t*>(p + 8);
#pragma unroll
        for (int s = 2; s >= 0; s--)  // small terms first
          asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
              : "+f"(acc[nt][0]), "+f"(acc[nt][1]), "+f"(acc[nt][2]), "+f"(acc[nt][3])
              : "r"(af[s][0]), "r"(af[s][1]), "r"(af[s][2]), "r"(af[s][3]), "r"(b0), "r"(b1));
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int nt = 0; nt < 8; nt++)
#pragma unroll
    for (int e = 0; e < 4; e++) zs[mat * GT_T + 16 * mt + g + 8 * (e >> 1)][8 * nt + 2 * t + (e & 1)] = acc[nt][e];
  __syncthreads();
  const int o = tid % GT_T;
  if (o0 + o >= n) return;
  const int64_t ch = (int64_t)blk * n + o0 + o;
  const float br = vec_at(a.bra, ch), bi = vec_at(a.bri, ch), lam = vec_at(a.lam, ch);
#pragma unroll 4
  for (int tok = tid / GT_T; tok < GT_T && t0 + tok < rows; tok += 256 / GT_T) {
    const int64_t at = (t0 + tok) * a.width + ch;
    recurrence_terms(zs[tok][o] + br, zs[GT_T + tok][o] + bi, u[at], a.c, lam, &av[at], &bv[at]);
  }
}

// Gates of 128 tokens x 64 outputs of one block, f32: both products share the u tile.
constexpr int GG_M = 128, GG_N = 64, GG_K = 16;
__global__ void __launch_bounds__(256)
rglru_gates_kernel(RglruArgs a, int64_t rows, const float* __restrict__ u, float* __restrict__ av, float* __restrict__ bv) {
  __shared__ __align__(16) float us[GG_K][GG_M + 4], rs[GG_K][GG_N + 4], is[GG_K][GG_N + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int n = a.width / a.blocks, tiles = (n + GG_N - 1) / GG_N;
  const int blk = blockIdx.x / tiles, o0 = (blockIdx.x % tiles) * GG_N;
  const int64_t t0 = (int64_t)blockIdx.y * GG_M;
  float ar[8][4] = {}, ai[8][4] = {};
  for (int k0 = 0; k0 < n; k0 += GG_K) {
#pragma unroll
    for (int j = 0; j < GG_M * GG_K / 256; j++) {
      const int i = tid + 256 * j, t = i / GG_K, k = i % GG_K;
      us[k][t] = t0 + t < rows && k0 + k < n ? u[(t0 + t) * a.width + blk * n + k0 + k] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < GG_N * GG_K / 256; j++) {
      const int i = tid + 256 * j, o = i / GG_K, k = i % GG_K;
      const bool live = o0 + o < n && k0 + k < n;
      const int64_t at = ((int64_t)blk * n + o0 + o) * n + k0 + k;
      rs[k][o] = live ? vec_at(a.ra, at) : 0.f;
      is[k][o] = live ? vec_at(a.ri, at) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GG_K; k++) {
      const float4 x0 = *reinterpret_cast<const float4*>(&us[k][4 * ty]), x1 = *reinterpret_cast<const float4*>(&us[k][64 + 4 * ty]);
      const float4 r4 = *reinterpret_cast<const float4*>(&rs[k][4 * tx]), i4 = *reinterpret_cast<const float4*>(&is[k][4 * tx]);
      const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
      const float rv[4] = {r4.x, r4.y, r4.z, r4.w}, iv[4] = {i4.x, i4.y, i4.z, i4.w};
#pragma unroll
      for (int i = 0; i < 8; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) ar[i][j] = fmaf(xv[i], rv[j], ar[i][j]), ai[i][j] = fmaf(xv[i], iv[j], ai[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int o = o0 + 4 * tx + j;
    if (o >= n) continue;
    const int64_t ch = (int64_t)blk * n + o;
    const float br = vec_at(a.bra, ch), bi = vec_at(a.bri, ch), lam = vec_at(a.lam, ch);
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int64_t t = t0 + (i < 4 ? 4 * ty + i : 60 + 4 * ty + i);
      if (t >= rows) continue;
      recurrence_terms(ar[i][j] + br, ai[i][j] + bi, u[t * a.width + ch], a.c, lam, &av[t * a.width + ch], &bv[t * a.width + ch]);
    }
  }
}

constexpr int SC_CH = 16, SC_SEG = 64, SC_LEN = 8, SC_PASS = SC_SEG * SC_LEN;
__global__ void __launch_bounds__(1024)
rglru_scan_kernel(RglruArgs a, int64_t rows, int64_t base, int64_t slot, const float* __restrict__ av, const float* __restrict__ bv) {
  __shared__ float sA[SC_SEG][SC_CH], sB[SC_SEG][SC_CH];
  const int lane = threadIdx.x % SC_CH, seg = threadIdx.x / SC_CH;
  const int ch = blockIdx.x * SC_CH + lane;
  const bool live = ch < a.width;
  float S0 = live && base > 0 ? a.state[slot * a.width + ch] : 0.f;  // state before the pass
  const float by = live ? vec_at(a.by, ch) : 0.f;
  for (int64_t p0 = 0; p0 < rows; p0 += SC_PASS) {
    const int64_t t0 = p0 + seg * SC_LEN;
    float x[SC_LEN], y[SC_LEN], gate[SC_LEN];
#pragma unroll
    for (int i = 0; i < SC_LEN; i++) {
      const bool in = live && t0 + i < rows;
      x[i] = in ? av[(t0 + i) * a.width + ch] : 1.f;
      y[i] = in ? bv[(t0 + i) * a.width + ch] : 0.f;
      gate[i] = in ? a.y.ptr[(t0 + i) * a.y.ld + ch] : 0.f;
    }
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < SC_LEN; i++) B = fmaf(x[i], B, y[i]), A *= x[i];
    sA[seg][lane] = A, sB[seg][lane] = B;
    __syncthreads();
    float S = S0;
#pragma unroll 8
    for (int w = 0; w < SC_SEG; w++) {
      const float n = fmaf(sA[w][lane], S0, sB[w][lane]);
      if (w < seg) S = n;
      S0 = n;
    }
#pragma unroll
    for (int i = 0; i < SC_LEN; i++) {
      S = fmaf(x[i], S, y[i]);
      if (live && t0 + i < rows)
        a.out[(t0 + i) * a.width + ch] = S * gelu_tanh_of(gate[i] + by);
    }
    __syncthreads();
  }
  if (!live) return;
  if (seg == 0) a.state[slot * a.width + ch] = S0;
  // the portion's last inputs go to the ring for the tokens that follow
  if (seg < a.taps && seg < rows) {
    const float bx = vec_at(a.bx, ch);
    float* ring = a.ring + slot * (int64_t)a.taps * a.width;
    for (int64_t b = seg; b < a.taps && b < rows; b += SC_SEG) {
      const int64_t t = rows - 1 - b;
      ring[((base + t) % a.taps) * a.width + ch] = a.x.ptr[t * a.x.ld + ch] + bx;
    }
  }
}

}  // namespace

size_t rglru_scratch_floats(const RglruArgs& a, int64_t rows) { return (size_t)3 * rows * a.width; }

int launch_rglru(const RglruArgs& a, const StepRows& r, cudaStream_t st) {
  if (r.rows == 0) return 0;
  if (r.base < 0) return step_rows(a, r.pos, r.seq, 0, 0, 0, r.rows, st);
  if (r.rows == 1) return step_rows(a, nullptr, nullptr, r.base, r.slot, 0, 1, st);
  DYN_CHECK(r.rows <= 65535, "rglru: portion of %lld tokens", (long long)r.rows);
  float* u = a.scratch;
  float *av = u + r.rows * a.width, *bv = av + r.rows * a.width;
  const dim3 cgrid((unsigned)((a.width + 127) / 128), (unsigned)((r.rows + CV_T - 1) / CV_T));
  if (a.taps == 4)
    rglru_conv_kernel<4><<<cgrid, 128, 0, st>>>(a, r.rows, r.base, r.slot, u);
  else
    rglru_conv_kernel<0><<<cgrid, 128, 0, st>>>(a, r.rows, r.base, r.slot, u);
  const int n = a.width / a.blocks;
  if (!a.exact && wide_rows(a)) {
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(rglru_gates_tc_kernel), GT_SMEM)) return 1;
    rglru_gates_tc_kernel<<<dim3((unsigned)(a.blocks * ((n + GT_T - 1) / GT_T)), (unsigned)((r.rows + GT_T - 1) / GT_T)), 256, GT_SMEM, st>>>(
        a, r.rows, u, av, bv);
  } else
    rglru_gates_kernel<<<dim3((unsigned)(a.blocks * ((n + GG_N - 1) / GG_N)), (unsigned)((r.rows + GG_M - 1) / GG_M)), 256, 0, st>>>(
      a, r.rows, u, av, bv);
  rglru_scan_kernel<<<(unsigned)((a.width + SC_CH - 1) / SC_CH), SC_CH * SC_SEG, 0, st>>>(a, r.rows, r.base, r.slot, av, bv);
  count_launch(3);
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace dyn
