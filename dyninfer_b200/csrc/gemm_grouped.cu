// Grouped GEMM of f16 matrices (the experts of a mixture): activation rows sorted by matrix, one CTA per
// (256 weight rows, tile of up to 256 activation rows of one matrix), y^T = W x^T with f32 accumulation.
//
//   * one thread fetches weight and activation chunks of 64 k with 2-D TMA tile copies (hardware 128-byte swizzle) into a ring
//     of stages: two tiles of 128 weight rows and one of activation rows;
//   * one thread of another warp issues tcgen05.mma (kind::f16, M = 128) for both weight tiles: each activation byte
//     that crosses from L2 serves 256 weight rows. Copies and MMAs cover the tile's own rows only (in steps of a copy box
//     and of sixteen): the shared-memory port, which carries every operand byte in and out, is what bounds a chunk;
//   * eight warps read the two accumulators back (tcgen05.ld, lane = weight row).
// GLU form: the two weight tiles are the same 128 rows of gate and up, and the epilogue leaves
// min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, +-limit) + 1) as the next product's f16 operand: such values are
// bounded by the limit, so one power-of-two scale serves all rows.
// Stages hand over through mbarriers; every wait is bounded and reports through the error word, and copies under way
// have landed and the tensor memory is released before the CTA exits.
#include <algorithm>

#include "common.cuh"
#include "tensor_map.cuh"
#include "umma.cuh"

namespace dyn {
namespace {

constexpr int GG_BM = 128, GG_BK = 64, GG_THREADS = 256, GG_MAX_STAGES = 8;
constexpr int GG_A_BYTES = GG_BM * GG_BK * 2;
constexpr int GG_SMEM = 224 * 1024;
constexpr long long GG_SPINS = 1LL << 24;

struct GgArgs {
  const CUtensorMap* maps;  // device, [matrices][3]: gate, up, down
  const int4* tiles;        // matrix, first row, rows
  const float* inv_s;       // scale of every activation row's sums (nullptr: in_scale for all)
  int bn, box, col, nstage;  // most activation rows per tile; rows of a copy box; column of the second accumulator
  int64_t N, K;             // outputs per row (GLU: of the gated ones)
  float* y;
  __half* yh;
  float limit, in_scale, out_scale;
  int* error;
};

__device__ __forceinline__ void tmem_ld16(uint32_t (&v)[16], uint32_t addr) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n\t"
      "tcgen05.wait::ld.sync.aligned;"  // in one statement: no use of the values can move before the wait
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]),
        "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(addr)
      : "memory");
}

template <bool GLU>
__global__ void __launch_bounds__(GG_THREADS, 1) grouped_gemm_kernel(const GgArgs a, const __grid_constant__ CUtensorMap xmap) {
  extern __shared__ __align__(1024) uint8_t gg_smem[];
  __shared__ uint64_t full_bar[GG_MAX_STAGES], empty_bar[GG_MAX_STAGES], accum_bar;
  __shared__ uint32_t tmem_base_s;
  __shared__ int s_abort;
  __shared__ float s_inv[256];
  const int4 tile = a.tiles[blockIdx.y];
  if (tile.z == 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int64_t n0 = (int64_t)blockIdx.x * (GLU ? GG_BM : 2 * GG_BM);
  const int nk = (int)(a.K / GG_BK), nstage = a.nstage, m0 = tile.y, live = tile.z;
  const uint32_t stage_bytes = 2 * GG_A_BYTES + (uint32_t)a.bn * (GG_BK * 2);
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gg_smem) + 1023) & ~uintptr_t(1023));
  if (tid == 0) {
    s_abort = 0;
    for (int i = 0; i < GG_MAX_STAGES; i++) mbar_init(full_bar + i, 1), mbar_init(empty_bar + i, 1);
    mbar_init(&accum_bar, 1);
    mbar_fence_init();
  }
  if (warp == 1) {  // the MMA warp owns the tensor memory
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"((uint32_t)(2 * a.col))
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  for (int j = tid; j < a.bn; j += GG_THREADS) s_inv[j] = j >= live ? 0.f : a.inv_s ? a.inv_s[m0 + j] : a.in_scale;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_d = tmem_base_s;
  const int boxes = (live + a.box - 1) / a.box;
  if (warp == 0 && lane == 0) {
    const CUtensorMap* first = a.maps + 3 * (int64_t)tile.x + (GLU ? 0 : 2);
    const CUtensorMap* second = first + (GLU ? 1 : 0);
    const int row1 = (int)n0 + (GLU ? 0 : GG_BM);
    int issued = 0;
    for (int kc = 0; kc < nk; kc++) {
      const int slot = kc % nstage;
      if (kc >= nstage && !mbar_wait_bounded(empty_bar + slot, (unsigned)(kc / nstage - 1) & 1u, GG_SPINS, &s_abort)) {
        if (!s_abort) s_abort = 1;
        break;
      }
      uint8_t* dst = smem + (size_t)slot * stage_bytes;
      mbar_expect_tx(full_bar + slot, 2 * GG_A_BYTES + (unsigned)(boxes * a.box) * (GG_BK * 2));
      // maps of 32-bit words: 32 of them per chunk of 64 k
      tma_load_2d(dst, first, kc * (GG_BK / 2), (int)n0, full_bar + slot);
      tma_load_2d(dst + GG_A_BYTES, second, kc * (GG_BK / 2), row1, full_bar + slot);
      for (int i = 0; i < boxes; i++)
        tma_load_2d(dst + 2 * GG_A_BYTES + i * a.box * (GG_BK * 2), &xmap, kc * (GG_BK / 2), m0 + i * a.box, full_bar + slot);
      issued++;
    }
    if (s_abort) {  // the copies under way land before the CTA leaves
      int never = 0;
      for (int kc = max(0, issued - nstage); kc < issued; kc++)
        mbar_wait_bounded(full_bar + kc % nstage, (unsigned)(kc / nstage) & 1u, GG_SPINS, &never);
    }
  } else if (warp == 1 && lane == 0) {
    const uint32_t idesc = umma_idesc((live + 15) / 16 * 16), smem0 = smem_u32(smem);
    uint32_t accumulate = 0u;
    for (int kc = 0; kc < nk; kc++) {
      const int slot = kc % nstage;
      if (!mbar_wait_bounded(full_bar + slot, (unsigned)(kc / nstage) & 1u, GG_SPINS, &s_abort)) {
        if (!s_abort) s_abort = 2;
        break;
      }
      tc_fence_after();
      const uint32_t at = smem0 + (uint32_t)slot * stage_bytes;
      const uint64_t a0 = umma_desc(at), a1 = umma_desc(at + GG_A_BYTES), b = umma_desc(at + 2 * GG_A_BYTES);
#pragma unroll
      for (int k4 = 0; k4 < GG_BK / 16; k4++) {  // 16 k further along a swizzled row: +32 bytes, +2 in the descriptor
        umma_f16(tmem_d, a0 + 2 * k4, b + 2 * k4, idesc, accumulate);
        umma_f16(tmem_d + (uint32_t)a.col, a1 + 2 * k4, b + 2 * k4, idesc, accumulate);
        accumulate = 1u;
      }
      umma_commit(empty_bar + slot);
    }
    umma_commit(&accum_bar);  // also reached after a failed wait
  }
  __syncwarp();
  const bool ok = mbar_wait_bounded(&accum_bar, 0, GG_SPINS, &s_abort);
  if (!ok && !s_abort) s_abort = 3;
  tc_fence_after();
  if (ok && !s_abort) {
    const int quarter = warp & 3, half = warp >> 2;
    const uint32_t tbase = tmem_d + ((uint32_t)(quarter * 32) << 16);
    if constexpr (GLU) {
      // the warps of a quarter take the blocks of sixteen activation rows in turn
      const int64_t n = n0 + quarter * 32 + lane;
      for (int j0 = half * 16; j0 < live; j0 += 32) {
        uint32_t g[16], u[16];
        tmem_ld16(g, tbase + (uint32_t)j0);
        tmem_ld16(u, tbase + (uint32_t)(a.col + j0));
        __half* p = a.yh + (int64_t)(m0 + j0) * a.N + n;
#pragma unroll
        for (int j = 0; j < 16; j++) {
          const float s = s_inv[j0 + j];
          const float gv = fminf(__uint_as_float(g[j]) * s, a.limit), uv = fminf(fmaxf(__uint_as_float(u[j]) * s, -a.limit), a.limit);
          const float y = gv * (1.0f / (1.0f + expf(-1.702f * gv))) * (uv + 1.0f);
          if (n < a.N && j0 + j < live) p[(int64_t)j * a.N] = __float2half_rn(y * a.out_scale);
        }
      }
    } else {
      const int64_t n = n0 + half * GG_BM + quarter * 32 + lane;
      for (int j0 = 0; j0 < live; j0 += 16) {
        uint32_t v[16];
        tmem_ld16(v, tbase + (uint32_t)(half * a.col + j0));
        float* p = a.y + (int64_t)(m0 + j0) * a.N + n;
#pragma unroll
        for (int j = 0; j < 16; j++)
          if (n < a.N && j0 + j < live) p[(int64_t)j * a.N] = __uint_as_float(v[j]) * s_inv[j0 + j];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_d), "r"((uint32_t)(2 * a.col)) : "memory");
  if (tid == 0 && s_abort) report_wait_expired(a.error, DEV_ERR_GEMM_PIPE);
}

// bf16 matrices of a table -> f16 in place, or the largest magnitude of all of them.
__global__ void __launch_bounds__(256) plain16_range_kernel(const uint8_t* const* table, int64_t count, int* largest) {
  const uint16_t* w = reinterpret_cast<const uint16_t*>(table[blockIdx.y]);
  float m = 0.f;
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < count; i += (int64_t)gridDim.x * 256) {
    const float v = fabsf(bf16_bits_to_f32(w[i]));
    m = v < 3.0e38f ? fmaxf(m, v) : 3.0e38f;
  }
  m = warp_max(m);
  if ((threadIdx.x & 31) == 0) atomicMax(largest, __float_as_int(m));  // magnitudes order like their bits
}
__global__ void __launch_bounds__(256) plain16_to_f16_kernel(const uint8_t* const* table, int64_t count) {
  uint16_t* w = const_cast<uint16_t*>(reinterpret_cast<const uint16_t*>(table[blockIdx.y]));
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < count; i += (int64_t)gridDim.x * 256)
    w[i] = __half_as_ushort(__float2half_rn(bf16_bits_to_f32(w[i])));
}

}  // namespace

int bf16_table_range(const uint8_t* const* table, int matrices, int64_t count, int* largest_dev, cudaStream_t s) {
  plain16_range_kernel<<<dim3(64, (unsigned)matrices), 256, 0, s>>>(table, count, largest_dev);
  DYN_CUDA(cudaGetLastError());
  return 0;
}
int bf16_table_to_f16(const uint8_t* const* table, int matrices, int64_t count, cudaStream_t s) {
  plain16_to_f16_kernel<<<dim3(64, (unsigned)matrices), 256, 0, s>>>(table, count);
  DYN_CUDA(cudaGetLastError());
  return 0;
}

bool grouped_gemm_takes(int64_t rows, int64_t K) { return rows >= 1 && K >= GG_BK && K % GG_BK == 0; }

// Map of one f16 matrix [rows, K] for grouped_gemm_kernel.
int make_grouped_weight_map(const uint8_t* w, int64_t rows, int64_t K, void* map) {
  return make_row_box_map(w, (size_t)K * 2, rows, GG_BK / 2, GG_BM, reinterpret_cast<CUtensorMap*>(map), true);
}

int launch_grouped_gemm(const GroupedGemm& g, cudaStream_t s) {
  DYN_CHECK(grouped_gemm_takes(g.N, g.K), "grouped GEMM: %lld outputs of %lld", (long long)g.N, (long long)g.K);
  DYN_CHECK((g.bn == 16 || (g.bn >= 32 && g.bn <= 256 && g.bn % 32 == 0)) && g.max_tiles >= 1 && g.max_tiles <= 65535, "grouped GEMM: %d tiles of %d rows",
            g.max_tiles, g.bn);
  GgArgs a;
  a.maps = reinterpret_cast<const CUtensorMap*>(g.maps), a.tiles = g.tiles, a.inv_s = g.inv_s, a.bn = g.bn;
  a.box = std::min(32, g.bn);
  a.col = 32;
  while (a.col < g.bn) a.col *= 2;
  const int stage = 2 * GG_A_BYTES + g.bn * GG_BK * 2;
  a.nstage = std::min(GG_MAX_STAGES, (GG_SMEM - 1024) / stage);
  a.N = g.N, a.K = g.K, a.y = g.y, a.yh = g.yh, a.limit = g.limit, a.in_scale = g.in_scale, a.out_scale = g.out_scale;
  a.error = device_error_word();
  if (!a.error) return 1;
  CUtensorMap xmap;
  if (make_row_box_map(reinterpret_cast<const uint8_t*>(g.xh), (size_t)g.K * 2, std::max<int64_t>(g.M, g.bn), GG_BK / 2, a.box, &xmap, true)) return 1;
  const size_t smem = (size_t)a.nstage * stage + 1024;
  const int per = g.yh ? GG_BM : 2 * GG_BM;
  const dim3 grid((unsigned)((g.N + per - 1) / per), (unsigned)g.max_tiles);
  const auto kernel = g.yh ? grouped_gemm_kernel<true> : grouped_gemm_kernel<false>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), GG_SMEM)) return 1;
  kernel<<<grid, GG_THREADS, smem, s>>>(a, xmap);
  count_launch();
  DYN_CUDA(cudaGetLastError());
  return 0;
}

}  // namespace dyn
