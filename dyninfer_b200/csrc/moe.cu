// Mixture of experts: each row's router logits choose `top` of the experts by sigmoid score; a chosen expert
// runs on the row times its score, an optional shared expert on the row itself; outputs are added to the residual.
// An expert is down(min(gate, limit) * sigmoid(1.702 min(gate, limit)) * (clamp(up, +-limit) + 1)).
//
// A few rows: two launches stream the chosen experts' weights (moe_up_kernel, moe_down_kernel); every CTA picks
// its experts from the logits itself. Scaling the input of gate and up scales their sums, so the score multiplies those.
// More rows: (row, choice) pairs are sorted by expert (moe_plan_kernel; a fixed order, so results do not depend on
// timing), then grouped products run on the tensor cores: f16 matrices by tile copies (gemm_grouped.cu; a session turns bf16
// experts into f16 when their range allows it), others through the grouped form of the dequant GEMM, and in f32 for f32
// sessions and shapes the GEMMs do not take; moe_combine_kernel adds each row's outputs in the order of its choices.
#include <algorithm>

#include "mixers.cuh"

namespace dyn {
namespace {

constexpr int MO_THREADS = 256, MO_WARPS = 8;
constexpr int MO_MAX_EXPERTS = 1024;

__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit), u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_of(1.702f * g) * (u + 1.0f);
}

// The `count` experts with the largest logits, best first (ties: the smaller index), by one warp; take(i, expert, logit).
template <class Take>
__device__ __forceinline__ void choose(const float* z, int experts, int count, Take take) {
  const int lane = threadIdx.x & 31;
  unsigned taken = 0;  // of this lane's experts lane, lane + 32, ...
  for (int i = 0; i < count; i++) {
    float best = -INFINITY;
    int at = 0x7fffffff;
    for (int j = 0; lane + 32 * j < experts; j++) {
      const float v = z[lane + 32 * j];
      if (!(taken >> j & 1) && (v > best || at == 0x7fffffff)) best = v, at = lane + 32 * j;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (oa != 0x7fffffff && (at == 0x7fffffff || ov > best || (ov == best && oa < at))) best = ov, at = oa;
    }
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    take(i, at, best);
  }
}

template <bool BF16>
__device__ __forceinline__ float dot8(const uint4& w, const float4& x, const float4& y) {
  const uint32_t u[4] = {w.x, w.y, w.z, w.w};
  const float v[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 4; i++) {
    float a, b;
    if (BF16) a = __uint_as_float(u[i] << 16), b = __uint_as_float(u[i] & 0xffff0000u);
    else a = f16_bits_to_f32(u[i] & 0xffffu), b = f16_bits_to_f32(u[i] >> 16);
    s = fmaf(a, v[2 * i], s), s = fmaf(b, v[2 * i + 1], s);
  }
  return s;
}
// vectors in shared memory as two planes of four, so that a lane's two reads of a piece of eight are conflict-free
__device__ __forceinline__ float& plane_at(float* xs, int k, int K8) { return xs[((((k >> 2) & 1) * K8 + (k >> 3)) << 2) + (k & 3)]; }

constexpr int MU_OUT = 2;  // outputs per warp
// act[row][slot][f] for f < ff of that slot's expert (slot `top`: the shared one). Normalises its row of x.
template <bool BF16>
__global__ void __launch_bounds__(MO_THREADS) moe_up_kernel(MoeArgs a, const float* __restrict__ x, const void* norm_w, int norm_type,
                                                            float eps, const float* __restrict__ z, float* __restrict__ act) {
  extern __shared__ __align__(16) float mu_x[];  // [2][K / 8] float4
  __shared__ float red[MO_WARPS], s_scale;
  __shared__ int s_expert;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slots = a.top + (a.shared_ff ? 1 : 0), slot = blockIdx.y % slots, wide = max(a.ff, a.shared_ff);
  const int64_t r = blockIdx.y / slots;
  const int K = (int)a.width, K8 = K / 8, ff = slot < a.top ? a.ff : a.shared_ff;
  const int f0 = (blockIdx.x * MO_WARPS + warp) * MU_OUT;
  pdl_trigger();
  if (blockIdx.x * MO_WARPS * MU_OUT >= ff) return;
  pdl_wait();
  float ss = 0.f;
  for (int i = tid; i < K; i += MO_THREADS) {
    const float v = x[r * K + i];
    plane_at(mu_x, i, K8) = v;
    ss = fmaf(v, v, ss);
  }
  if (slot < a.top && warp == 0)
    choose(z + r * a.experts, a.experts, slot + 1, [&](int i, int e, float l) {
      if (i == slot && lane == 0) s_expert = e, s_scale = sigmoid_of(l);
    });
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = warp_sum(lane < MO_WARPS ? red[lane] : 0.f);
  const float inv = 1.0f / sqrtf(ss / (float)K + eps);
  for (int i = tid; i < K; i += MO_THREADS)  // the thread's own elements
    plane_at(mu_x, i, K8) = __fmul_rn(__fmul_rn(plane_at(mu_x, i, K8), inv), aux_load(reinterpret_cast<const uint8_t*>(norm_w), norm_type, i));
  __syncthreads();
  const float4* xs = reinterpret_cast<const float4*>(mu_x);
  const uint8_t *gw = slot < a.top ? a.table[3 * s_expert] : a.shared_gate.data, *uw = slot < a.top ? a.table[3 * s_expert + 1] : a.shared_up.data;
  const float scale = slot < a.top ? s_scale : 1.0f, limit = slot < a.top ? a.limit : a.shared_limit;
  float sum[2 * MU_OUT] = {};
  const uint4* rows[2 * MU_OUT];
#pragma unroll
  for (int o = 0; o < MU_OUT; o++) {
    const int64_t f = min(f0 + o, ff - 1);
    rows[2 * o] = reinterpret_cast<const uint4*>(gw + f * K * 2), rows[2 * o + 1] = reinterpret_cast<const uint4*>(uw + f * K * 2);
  }
  constexpr int U = 4;
  for (int p0 = lane; p0 < K8; p0 += 32 * U) {
    uint4 w[2 * MU_OUT][U];
#pragma unroll
    for (int u = 0; u < U; u++)
#pragma unroll
      for (int o = 0; o < 2 * MU_OUT; o++)
        if (p0 + 32 * u < K8) w[o][u] = __ldcs(rows[o] + p0 + 32 * u);
#pragma unroll
    for (int u = 0; u < U; u++) {
      if (p0 + 32 * u >= K8) break;
      const float4 xa = xs[p0 + 32 * u], xb = xs[K8 + p0 + 32 * u];
#pragma unroll
      for (int o = 0; o < 2 * MU_OUT; o++) sum[o] += dot8<BF16>(w[o][u], xa, xb);
    }
  }
#pragma unroll
  for (int o = 0; o < MU_OUT; o++) {
    const float g = warp_sum(sum[2 * o]) * scale, u = warp_sum(sum[2 * o + 1]) * scale;
    if (lane == 0 && f0 + o < ff) act[(r * slots + slot) * wide + f0 + o] = clamped_glu(g, u, limit);
  }
}

constexpr int MD_THREADS = 1024, MD_WARPS = MD_THREADS / 32, MD_DEPTH = 8, MD_SPAN = 32 * MD_DEPTH;
// hidden[row][n] += sum over the slots of down[n] . act. A CTA owns a block of outputs; their rows, all slots one after the
// other, are cut into spans of MD_SPAN pieces of eight, dealt to the warps.
template <bool BF16>
__global__ void __launch_bounds__(MD_THREADS, 1) moe_down_kernel(MoeArgs a, const float* __restrict__ z, const float* __restrict__ act, float* hidden) {
  extern __shared__ __align__(16) float md_x[];  // planes over all slots' activations, one after the other; then sums
  __shared__ const uint8_t* s_base[64];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slots = a.top + (a.shared_ff ? 1 : 0), wide = max(a.ff, a.shared_ff), total = a.top * a.ff + a.shared_ff, T8 = total / 8;
  const int64_t r = blockIdx.y, W = a.width;
  const int64_t out0 = W * blockIdx.x / gridDim.x;
  const int own = (int)(W * (blockIdx.x + 1) / gridDim.x - out0), parts = (T8 + MD_SPAN - 1) / MD_SPAN;
  pdl_trigger();
  pdl_wait();
  if (warp == 0) {
    choose(z + r * a.experts, a.experts, a.top, [&](int i, int e, float) {
      if (lane == 0) s_base[i] = a.table[3 * e + 2];
    });
    if (lane == 0 && a.shared_ff) s_base[a.top] = a.shared_down.data;
  }
  for (int i = tid; i < total; i += MD_THREADS) {
    const int slot = min(i / a.ff, a.top), f = i - slot * a.ff;
    plane_at(md_x, i, T8) = act[(r * slots + slot) * wide + f];
  }
  __syncthreads();
  const float4* xs = reinterpret_cast<const float4*>(md_x);
  float* sums = md_x + total;  // [own][parts]
  const unsigned ff8 = a.ff / 8;
  for (int unit = warp; unit < own * parts; unit += MD_WARPS) {
    const int o = unit / parts, p0 = (unit - o * parts) * MD_SPAN + lane;
    uint4 w[MD_DEPTH];
#pragma unroll
    for (int u = 0; u < MD_DEPTH; u++) {
      const int p = p0 + 32 * u;
      if (p < T8) {
        const int slot = min((int)((unsigned)p / ff8), a.top), k = p - slot * (int)ff8;
        w[u] = __ldcs(reinterpret_cast<const uint4*>(s_base[slot] + (out0 + o) * (slot < a.top ? a.ff : a.shared_ff) * 2) + k);
      }
    }
    float sum = 0.f;
#pragma unroll
    for (int u = 0; u < MD_DEPTH; u++) {
      const int p = p0 + 32 * u;
      if (p < T8) sum += dot8<BF16>(w[u], xs[p], xs[T8 + p]);
    }
    sum = warp_sum(sum);
    if (lane == 0) sums[unit] = sum;
  }
  __syncthreads();
  for (int o = tid; o < own; o += MD_THREADS) {
    float v = 0.f;
    for (int p = 0; p < parts; p++) v += sums[o * parts + p];
    hidden[r * W + out0 + o] += v;
  }
}

// ---- many rows -----------------------------------------------------------------------------------
// Integer part of the scratch. pair = row * top + choice; sorted by expert, then pair.
struct MoePlan {
  int *ids, *list, *pos;  // [pairs]: expert of a pair; pair at a sorted place; sorted place of a pair
  float* score;           // [pairs]
  int4* tiles;            // [max_tiles]: expert, first sorted place, places (0: none)
  int max_tiles, bn;
};

__global__ void __launch_bounds__(MO_THREADS) moe_choose_kernel(MoeArgs a, const float* __restrict__ z, int64_t rows, MoePlan p) {
  const int lane = threadIdx.x & 31;
  const int64_t r = blockIdx.x * (int64_t)MO_WARPS + (threadIdx.x >> 5);
  if (r >= rows) return;
  choose(z + r * a.experts, a.experts, a.top, [&](int i, int e, float l) {
    if (lane == 0) p.ids[r * a.top + i] = e, p.score[r * a.top + i] = sigmoid_of(l);
  });
}

// CTA = expert: counts of all experts, then this one's places in order of its pairs, and its tiles.
__global__ void __launch_bounds__(MO_THREADS) moe_plan_kernel(MoeArgs a, int pairs, MoePlan p) {
  extern __shared__ int mp_count[];  // [experts]
  __shared__ int warp_n[MO_WARPS], s_start, s_tile, s_tiles;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, e = blockIdx.x;
  for (int i = tid; i < a.experts; i += MO_THREADS) mp_count[i] = 0;
  __syncthreads();
  for (int i = tid; i < pairs; i += MO_THREADS) atomicAdd(&mp_count[p.ids[i]], 1);
  __syncthreads();
  if (warp == 0) {
    int before = 0, tiles = 0, all = 0;
    for (int i = lane; i < a.experts; i += 32) {
      const int t = (mp_count[i] + p.bn - 1) / p.bn;
      all += t;
      if (i < e) before += mp_count[i], tiles += t;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
      before += __shfl_xor_sync(0xffffffffu, before, o), tiles += __shfl_xor_sync(0xffffffffu, tiles, o), all += __shfl_xor_sync(0xffffffffu, all, o);
    if (lane == 0) s_start = before, s_tile = tiles, s_tiles = all;
  }
  __syncthreads();
  const int n = mp_count[e], start = s_start;
  for (int t = tid; t * p.bn < n; t += MO_THREADS) p.tiles[s_tile + t] = make_int4(e, start + t * p.bn, min(p.bn, n - t * p.bn), 0);
  if (e == 0)
    for (int t = s_tiles + tid; t < p.max_tiles; t += MO_THREADS) p.tiles[t] = make_int4(0, 0, 0, 0);
  int at = start;
  for (int i0 = 0; i0 < pairs; i0 += MO_THREADS) {
    const int i = i0 + tid;
    const bool mine = i < pairs && p.ids[i] == e;
    const unsigned b = __ballot_sync(0xffffffffu, mine);
    if (lane == 0) warp_n[warp] = __popc(b);
    __syncthreads();
    int mineat = at + __popc(b & ((1u << lane) - 1)), sum = 0;
#pragma unroll
    for (int w = 0; w < MO_WARPS; w++) {
      if (w < warp) mineat += warp_n[w];
      sum += warp_n[w];
    }
    if (mine) p.list[mineat] = i, p.pos[i] = mineat;
    at += sum;
    __syncthreads();
  }
}

// f32: y[place][n] = sum_k x[row][k] * score * w[expert][n][k]. up: columns [0, ff) are the gate's, [ff, 2 ff) the up's.
constexpr int MG_T = 64, MG_K = 16, MG_P = MG_T + 4;
template <bool UP>
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(MoeArgs a, MoePlan p, const float* __restrict__ x, float* __restrict__ y) {
  __shared__ __align__(16) float xs[MG_K][MG_P], ws[MG_K][MG_P];
  const int4 tile = p.tiles[blockIdx.y];
  if (tile.z == 0) return;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int blocks = (a.ff + MG_T - 1) / MG_T;
  const int64_t K = UP ? a.width : a.ff, N = UP ? a.ff : a.width, ldy = UP ? 2 * a.ff : a.width;
  const int part = UP ? (int)blockIdx.x / blocks : 2;
  const int64_t n0 = (int64_t)(UP ? blockIdx.x % blocks : blockIdx.x) * MG_T;
  const uint8_t* w = a.table[3 * tile.x + part];
  float acc[4][4] = {};
  for (int64_t k0 = 0; k0 < K; k0 += MG_K) {
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int i = tid + 256 * j, r = i / MG_K, k = i % MG_K;
      const bool kin = k0 + k < K;
      float v = 0.f;
      if (kin && r < tile.z) {
        const int place = tile.y + r;
        if (UP) {
          const int pair = p.list[place];
          v = x[(int64_t)(pair / a.top) * K + k0 + k] * p.score[pair];
        } else {
          v = x[(int64_t)place * K + k0 + k];
        }
      }
      xs[k][r] = v;
      ws[k][r] = kin && n0 + r < N ? aux_load(w, a.enc, (n0 + r) * K + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MG_K; k++) {
      const float4 u = *reinterpret_cast<const float4*>(&xs[k][4 * ty]), v = *reinterpret_cast<const float4*>(&ws[k][4 * tx]);
      const float av[4] = {u.x, u.y, u.z, u.w}, bv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    if (4 * ty + i >= tile.z) continue;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int64_t n = n0 + 4 * tx + j;
      if (n < N) y[(int64_t)(tile.y + 4 * ty + i) * ldy + (UP ? part * a.ff : 0) + n] = acc[i][j];
    }
  }
}

__global__ void __launch_bounds__(256) clamped_glu_rows_kernel(const float* __restrict__ gu, int64_t rows, int64_t I, float limit, float* __restrict__ y) {
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < rows * I; i += (int64_t)gridDim.x * 256) {
    const int64_t r = i / I, c = i - r * I;
    y[i] = clamped_glu(gu[r * 2 * I + c], gu[r * 2 * I + I + c], limit);
  }
}
__global__ void __launch_bounds__(256) clamped_glu_kernel(const float* __restrict__ g, const float* __restrict__ u, int64_t n, float limit, float* __restrict__ y) {
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < n; i += (int64_t)gridDim.x * 256) y[i] = clamped_glu(g[i], u[i], limit);
}

// hidden[row] += its choices' outputs, in their order
__global__ void __launch_bounds__(256) moe_combine_kernel(MoeArgs a, MoePlan p, int64_t rows, const float* __restrict__ y, float* hidden) {
  __shared__ int s_pos[64];
  const int64_t r = blockIdx.x, W = a.width;
  if (threadIdx.x < a.top) s_pos[threadIdx.x] = p.pos[r * a.top + threadIdx.x];
  __syncthreads();
  for (int64_t n = blockIdx.y * 256 + threadIdx.x; n < W; n += 256 * gridDim.y) {
    float v = 0.f;
#pragma unroll 4
    for (int i = 0; i < a.top; i++) v += y[(int64_t)s_pos[i] * W + n];
    hidden[r * W + n] += v;
  }
}

// sorted activation operand: the rows' f16 values, the scores in the rows' inverse scales
__global__ void __launch_bounds__(256) moe_gather_kernel(MoeArgs a, MoePlan p, const __half* __restrict__ xh, const float* __restrict__ inv,
                                                         __half* __restrict__ xg, float* __restrict__ inv_g) {
  const int64_t place = blockIdx.x, K8 = a.width / 8;
  const int pair = p.list[place];
  const int64_t r = pair / a.top;
  const uint4* src = reinterpret_cast<const uint4*>(xh + r * a.width);
  uint4* dst = reinterpret_cast<uint4*>(xg + place * a.width);
  for (int64_t i = threadIdx.x; i < K8; i += 256) dst[i] = src[i];
  if (threadIdx.x == 0) inv_g[place] = inv[r] * p.score[pair];
}

size_t up256(size_t n) { return (n + 255) / 256 * 256; }

int tile_rows(const MoeArgs& a, int64_t rows, bool tensor) {
  if (!tensor) return MG_T;
  // one tile per expert up to twice the even share: the tile-copy GEMM's tiles cost what their rows cost, the other's their full width
  const int64_t share = rows * a.top / a.experts + 1, want = a.maps ? 2 * share : share + share / 8;
  return want <= 16 ? 16 : (int)std::min<int64_t>(256, (want + 31) / 32 * 32);
}

bool few_rows(const MoeArgs& a, int64_t rows) {
  auto ok = [](const WRef& w) { return (reinterpret_cast<uintptr_t>(w.data) & 15) == 0; };
  return rows <= 4 && (a.enc == E_BF16 || a.enc == E_F16) && a.width % 8 == 0 && a.ff % 8 == 0 && a.shared_ff % 8 == 0 && a.aligned &&
         a.top < 64 && a.width <= 32 * 1024 && (int64_t)a.top * a.ff + a.shared_ff <= 32 * 1024 &&
         (!a.shared_ff || (a.shared_gate.enc == a.enc && a.shared_up.enc == a.enc && a.shared_down.enc == a.enc && ok(a.shared_gate) &&
                           ok(a.shared_up) && ok(a.shared_down)));
}
bool tensor_shape(const MoeArgs& a) {
  return !a.exact && a.gate_up_table && a.aligned && (a.enc == E_BF16 || a.enc == E_F16) && a.width % 64 == 0 && a.ff % 64 == 0;
}

// Byte layout of the scratch for a step of `rows` rows; z [rows][experts] comes first.
struct MoeBytes {
  size_t plan, gu, act, yo, xr, inv_r, xg, inv_g, total;
  int max_tiles, bn;
};
MoeBytes layout(const MoeArgs& a, int64_t rows) {
  MoeBytes b{};
  const bool tc = tensor_shape(a);
  const size_t pairs = (size_t)rows * a.top;
  b.bn = tile_rows(a, rows, tc);
  b.max_tiles = (int)(pairs / b.bn + std::min<size_t>(pairs, a.experts));
  size_t at = up256((size_t)rows * a.experts * 4);
  auto take = [&](size_t bytes) {
    const size_t here = at;
    at += up256(bytes);
    return here;
  };
  b.plan = take(4 * pairs * 4 + (size_t)b.max_tiles * 16 + 64);
  // a few rows: activations of all slots
  b.gu = take(std::max(pairs * 2 * a.ff * 4, (size_t)std::min<int64_t>(rows, 4) * (a.top + 1) * std::max(a.ff, a.shared_ff) * 4));
  const size_t prows = std::max<size_t>(pairs, b.bn);  // rows of a GEMM operand's buffer
  b.act = take(tc ? prows * a.ff * 2 : pairs * a.ff * 4);
  b.yo = take(pairs * a.width * 4);
  if (tc) {
    b.xr = take((size_t)rows * a.width * 2), b.inv_r = take((size_t)rows * 4);
    b.xg = take(prows * a.width * 2), b.inv_g = take(pairs * 4);
  }
  b.total = at;
  return b;
}

unsigned ew_blocks(int64_t n) { return (unsigned)std::max<int64_t>(1, std::min<int64_t>((n + 255) / 256, 148 * 16)); }

}  // namespace

int launch_clamped_glu_rows(const float* gu, int64_t rows, int64_t I, float limit, float* y, cudaStream_t st) {
  clamped_glu_rows_kernel<<<ew_blocks(rows * I), 256, 0, st>>>(gu, rows, I, limit, y);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}
int launch_clamped_glu(const float* gate, const float* up, int64_t n, float limit, float* y, cudaStream_t st) {
  clamped_glu_kernel<<<ew_blocks(n), 256, 0, st>>>(gate, up, n, limit, y);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

size_t moe_scratch_floats(const MoeArgs& a, int64_t rows) {
  size_t need = layout(a, rows).total;
  for (int64_t r = 1; r < rows; r *= 2) need = std::max(need, layout(a, r).total);
  return need / 4 + 64;
}

bool moe_takes_operand(const MoeArgs& a) { return tensor_shape(a); }
bool moe_streams(const MoeArgs& a, int64_t rows) { return !a.exact && few_rows(a, rows); }

// The whole feed-forward of a few rows: hidden += experts(norm(x)); x may be hidden's buffer only if nothing was added yet.
int launch_moe_few(const MoeArgs& a, const float* x, const void* norm_w, int norm_type, float eps, int64_t rows, const float* z, float* act,
                   cudaStream_t st) {
  const int slots = a.top + (a.shared_ff ? 1 : 0), wide = std::max(a.ff, a.shared_ff);
  const dim3 grid((unsigned)((wide + MO_WARPS * MU_OUT - 1) / (MO_WARPS * MU_OUT)), (unsigned)(rows * slots));
  const size_t smem = (size_t)a.width * 4;
  const bool bf = a.enc == E_BF16;
  const auto kernel = bf ? moe_up_kernel<true> : moe_up_kernel<false>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), 160 * 1024)) return 1;
  DYN_CUDA(launch_pdl(kernel, grid, dim3(MO_THREADS), smem, st, a, x, norm_w, norm_type, eps, z, act));
  count_launch();
  return 0;
}
int launch_moe_few_down(const MoeArgs& a, int64_t rows, const float* z, const float* act, float* hidden, cudaStream_t st) {
  const auto kernel = a.enc == E_BF16 ? moe_down_kernel<true> : moe_down_kernel<false>;
  const int64_t total = (int64_t)a.top * a.ff + a.shared_ff, parts = (total / 8 + MD_SPAN - 1) / MD_SPAN;
  const int64_t blocks = std::min<int64_t>(a.width, std::max(1, sm_count()));
  const size_t smem = (size_t)(total + ((a.width + blocks - 1) / blocks) * parts) * 4;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), 200 * 1024)) return 1;
  DYN_CHECK(smem <= 200 * 1024, "mixture of experts: activations of %lld are too wide", (long long)total);
  const dim3 grid((unsigned)blocks, (unsigned)rows);
  DYN_CUDA(launch_pdl(kernel, grid, dim3(MD_THREADS), smem, st, a, z, act, hidden));
  count_launch();
  return 0;
}
float* moe_few_act(const MoeArgs& a, int64_t rows) {
  return reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(a.scratch) + layout(a, rows).gu);
}

// The chosen experts of many rows: everything up to the outputs [pairs][width] in the scratch.
int launch_moe_experts(const MoeArgs& a, const float* xn, const __half* xh, const float* xinv, int64_t rows, const float* z, cudaStream_t st) {
  const MoeBytes b = layout(a, rows);
  uint8_t* base = reinterpret_cast<uint8_t*>(a.scratch);
  const int64_t pairs = rows * a.top;
  DYN_CHECK(pairs < (1 << 28), "mixture of experts: %lld choices in one step", (long long)pairs);
  MoePlan p;
  p.ids = reinterpret_cast<int*>(base + b.plan), p.list = p.ids + pairs, p.pos = p.list + pairs;
  p.score = reinterpret_cast<float*>(p.pos + pairs);
  p.tiles = reinterpret_cast<int4*>(reinterpret_cast<uint8_t*>(p.ids) + (4 * (size_t)pairs * 4 + 15) / 16 * 16);
  p.max_tiles = b.max_tiles, p.bn = b.bn;
  moe_choose_kernel<<<(unsigned)((rows + MO_WARPS - 1) / MO_WARPS), MO_THREADS, 0, st>>>(a, z, rows, p);
  moe_plan_kernel<<<(unsigned)a.experts, MO_THREADS, (size_t)a.experts * 4, st>>>(a, (int)pairs, p);
  count_launch(2);
  float *gu = reinterpret_cast<float*>(base + b.gu), *yo = reinterpret_cast<float*>(base + b.yo);
  DYN_CHECK(b.max_tiles <= 65535, "mixture of experts: %d tiles in one launch", b.max_tiles);
  if (tensor_shape(a)) {
    __half *xg = reinterpret_cast<__half*>(base + b.xg), *xa = reinterpret_cast<__half*>(base + b.act);
    float* inv_g = reinterpret_cast<float*>(base + b.inv_g);
    if (!xh) {
      __half* xr = reinterpret_cast<__half*>(base + b.xr);
      float* ir = reinterpret_cast<float*>(base + b.inv_r);
      if (launch_activation_prepare(xn, rows, a.width, xr, ir, st)) return 1;
      xh = xr, xinv = ir;
    }
    moe_gather_kernel<<<(unsigned)pairs, 256, 0, st>>>(a, p, xh, xinv, xg, inv_g);
    count_launch();
    if (a.maps) {
      // z sigmoid(1.702 z) > -0.17, so gated values are at most max(limit, 0.17) (limit + 1): scaled to at most 2^13
      int e = 0;
      frexpf(std::max(a.limit, 0.17f) * (a.limit + 1.0f), &e);
      GroupedGemm up;
      up.maps = a.maps, up.tiles = p.tiles, up.max_tiles = p.max_tiles, up.bn = p.bn, up.xh = xg, up.inv_s = inv_g;
      up.M = pairs, up.N = a.ff, up.K = a.width, up.yh = xa, up.limit = a.limit, up.out_scale = ldexpf(1.0f, 13 - e);
      GroupedGemm down = up;
      down.xh = xa, down.N = a.width, down.K = a.ff, down.yh = nullptr, down.y = yo, down.inv_s = nullptr, down.in_scale = ldexpf(1.0f, e - 13);
      return launch_grouped_gemm(up, st) || launch_grouped_gemm(down, st);
    }
    TgGroups g;
    g.tiles = p.tiles, g.max_tiles = p.max_tiles, g.bn = p.bn;
    WRef w;
    w.enc = a.enc, w.rows = 2 * a.ff, w.cols = a.width;
    g.bases = a.gate_up_table;
    if (launch_dqgemm_tc_grouped(w, g, xg, inv_g, pairs, gu, st) ||
        launch_clamped_glu_prepare(gu, pairs, a.ff, a.limit, xa, inv_g, st))
      return 1;
    w.rows = a.width, w.cols = a.ff;
    g.bases = a.down_table;
    if (launch_dqgemm_tc_grouped(w, g, xa, inv_g, pairs, yo, st)) return 1;
  } else {
    float* act = reinterpret_cast<float*>(base + b.act);
    DYN_CHECK(xn, "mixture of experts: f32 rows are missing");
    const unsigned fb = (unsigned)((a.ff + MG_T - 1) / MG_T);
    moe_gemm_f32_kernel<true><<<dim3(2 * fb, (unsigned)p.max_tiles), 256, 0, st>>>(a, p, xn, gu);
    count_launch();
    if (launch_clamped_glu_rows(gu, pairs, a.ff, a.limit, act, st)) return 1;
    moe_gemm_f32_kernel<false><<<dim3((unsigned)((a.width + MG_T - 1) / MG_T), (unsigned)p.max_tiles), 256, 0, st>>>(a, p, act, yo);
    count_launch();
  }
  DYN_CUDA(cudaGetLastError());
  return 0;
}

int launch_moe_combine(const MoeArgs& a, int64_t rows, float* hidden, cudaStream_t st) {
  const MoeBytes b = layout(a, rows);
  uint8_t* base = reinterpret_cast<uint8_t*>(a.scratch);
  const int64_t pairs = rows * a.top;
  MoePlan p{};
  p.pos = reinterpret_cast<int*>(base + b.plan) + 2 * pairs;
  moe_combine_kernel<<<dim3((unsigned)rows, (unsigned)std::min<int64_t>(4, (a.width + 255) / 256)), 256, 0, st>>>(
      a, p, rows, reinterpret_cast<const float*>(base + b.yo), hidden);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

int moe_check(const MoeArgs& a) {
  DYN_CHECK(a.experts >= 1 && a.experts <= MO_MAX_EXPERTS && a.top >= 1 && a.top <= std::min(a.experts, 64) && a.ff >= 1,
            "mixture of %d experts of width %d, %d per token", a.experts, a.ff, a.top);
  return 0;
}

}  // namespace dyn
