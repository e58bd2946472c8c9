// Internal session declarations shared by session.cu (ABI, upload, GQA decoder) and session_mixers.cu
// (decoders whose layers carry recurrent or latent-attention mixers).
#pragma once

#include <algorithm>
#include <map>
#include <string>
#include <utility>
#include <vector>

#include "common.cuh"
#include "decode_mega.cuh"
#include "mixers.cuh"

namespace dyn {
struct NormW {
  const void* ptr = nullptr;
  int type = E_F32;
  uint64_t bytes = 0;
};

struct LayerW {
  NormW attn_norm, ffn_norm, q_norm, k_norm;
  WRef q, k, v, o, gate, up, down;
  // rows of consecutive matrices seen as one (data == nullptr: not laid back to back)
  WRef qkv;     // [q; k] or [q; k; v]
  int qkv_parts = 0;
  WRef gate_up; // [gate; up]
};

// One layer of a decoder whose layers are listed one by one: which mixer, its sizes, its feed-forward.
enum MixerKind { MIX_RETENTION = 0, MIX_RGLRU = 1, MIX_LATENT = 2, MIX_SOFTMAX = 3, MIX_DELTA = 4 };
struct MixerCfg {
  MixerKind kind = MIX_RETENTION;
  int tensors = 0;  // the layer whose parameters this one runs with (itself, or one it shares them with)
  bool parallel = false;  // mixer and feed-forward read the same residual row; otherwise one after the other
  int ff = 0;       // width of the gated feed-forward, 0: none
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot_dims = 0;
  double rot_base = 0;
  std::vector<double> decay;
  int width = 0, blocks = 0, taps = 0;
  int rank = 0;
  float scale = 0.f, softcap = 0.f;
  bool bias = false;  // products of the mixer have biases
  // a mixture of experts instead of the feed-forward (experts > 0), with a shared one (shared_ff > 0)
  int experts = 0, top = 0, expert_ff = 0, shared_ff = 0;
  float expert_limit = 0.f, shared_limit = 0.f;
  bool feeds_forward() const { return ff > 0 || experts > 0; }
  int gated_width() const { return experts ? shared_ff : ff; }  // width of the matrices gate, up and down
  // cached elements per token and slot
  size_t cached() const {
    return kind == MIX_LATENT ? (size_t)rank : kind == MIX_SOFTMAX ? (size_t)kv_heads * (dim + vdim) : 0;
  }
  bool same_sizes(const MixerCfg& o) const {
    return heads == o.heads && kv_heads == o.kv_heads && dim == o.dim && vdim == o.vdim && rot_dims == o.rot_dims && width == o.width &&
           blocks == o.blocks && taps == o.taps && rank == o.rank && bias == o.bias && ff == o.ff && experts == o.experts &&
           expert_ff == o.expert_ff && shared_ff == o.shared_ff;
  }
};

struct MixerLayer {
  MixerCfg c;
  NormW norm1, norm2;
  std::vector<WRef> in;       // input products; matrices laid back to back are one
  int part_in[6] = {}, parts = 0;
  int64_t part_col[6] = {};   // part p = columns from part_col[p] of product part_in[p]
  WRef o, gate, up, gate_up, down;
  NormW by, bx, conv, bc, ra, bra, ri, bri, lam, lat_norm;
  WRef uk, uv, ukv;
  NormW qb, kb, vb, ob;       // softmax attention
  NormW conv_q, conv_k, conv_v, a_log, dt, head_norm;  // delta rule
  WRef router;
  MoeArgs moe;                // experts' tables and shapes; scratch is the session's
  double* freq = nullptr;     // device tables of the owning layer
  float* decay = nullptr;
  size_t state_off = 0, state_floats = 0;  // per slot: floats in the state pool (regions [slot][...])
  size_t ring_off = 0, ring_floats = 0;
};

struct ModelCfg {
  bool exact = false;            // every product in f32 (descriptor "compute": "f32")
  std::vector<MixerCfg> mixers;  // non-empty: one entry per layer
  int layers = 0, hidden = 0, inter = 0, heads = 0, kv_heads = 0, head_dim = 0, vocab = 0;
  float eps = 1e-6f, theta = 10000.f;
  // what the stored norm weights count from (0: plain weights), and the factor of the logits
  float norm_offset = 0.f, logit_scale = 1.f;
  bool qk_norm = true, rope = true;
  int batch = 1;
  int kv2_type = E_BF16;  // element type used when the KV cache is configured with 2 bytes
  bool persistent = true;  // single-token steps run as the persistent decode kernel
  // tensor parallelism: heads / kv_heads / inter above are this rank's share; the lm_head holds
  // lm_rows = vocab / tp_world consecutive rows starting at tp_rank * lm_rows
  int tp_rank = 0, tp_world = 1, lm_rows = 0;
};

}  // namespace dyn

using namespace dyn;

struct dyninfer_cuda_session_t {
  int device = 0;
  cudaStream_t stream = nullptr;
  cudaEvent_t tm0 = nullptr, tm1 = nullptr;  // dyninfer_cuda_session_timer
  ModelCfg cfg;
  FreqTable freq;
  // parameters
  uint8_t* arena = nullptr;
  uint64_t arena_bytes = 0;
  uint64_t weight_bytes = 0;         // sum of uploaded range lengths
  uint64_t decode_weight_bytes = 0;  // linears + lm_head + norm vectors
  WRef embed, lm_head;
  NormW out_norm;
  std::vector<LayerW> layers;
  // KV pool
  bool kv_configured = false;
  size_t page_size = 0, chunk_size = 0, kv_elem = 0, pages = 0;
  int kv_type = E_F32;
  uint8_t* kcache = nullptr;  // [layer][seq][nkv][cap][d]
  uint8_t* vcache = nullptr;
  size_t kv_bytes_each = 0;
  // decoders with mixers: latent planes [layer][slot][cap][rank] instead of K and V, recurrent state in f32
  // ([layer][slot][...], position 0 starts from an empty state), the position every slot has reached
  // (-1: the last step of the slot failed, it must start over)
  std::vector<MixerLayer> mix;
  uint8_t* lcache = nullptr;
  size_t lcache_bytes = 0;
  float* state = nullptr;
  size_t state_floats = 0;
  float* mix_scratch = nullptr;
  size_t mix_scratch_floats = 0;
  float* tables = nullptr;       // decays, angles per position, norm weights counted from an offset
  const uint8_t** expert_tables = nullptr;  // addresses of the experts' matrices
  uint8_t* expert_maps = nullptr;           // their tensor maps
  std::vector<int64_t> slot_pos;
  // logits of several rows of a portion
  float* want_logits = nullptr;  // [want_cap, vocab]
  float* want_logits_host = nullptr;
  int64_t* want_index_dev = nullptr;
  int64_t want_cap = 0;
  // scratch
  int64_t max_rows = 0;
  float *hidden = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *ctx = nullptr,
        *act = nullptr, *up = nullptr, *logits = nullptr;
  // many-row steps: the dequant GEMM's activation operand written by the norm / SwiGLU kernels, and the
  // K-split sums of o / down waiting for the residual + norm kernel
  __half* xh = nullptr;
  float *xinv = nullptr, *gpart = nullptr;
  __half* xh2 = nullptr;  // a second operand, for layers whose branches read one residual row
  float* xinv2 = nullptr;
  int64_t xh_rows = 0, xh_cols = 0;
  size_t gpart_bytes = 0;
  float *qkv1 = nullptr, *gu1 = nullptr;  // rows of [q | k | v] and of [gate | up] for the fused products
  int64_t *tokens_dev = nullptr, *row_pos_dev = nullptr, *row_seq_dev = nullptr,
          *out_token_dev = nullptr, *hist_dev = nullptr, *hist_count_dev = nullptr;
  size_t hist_cap = 0;
  void* argmax_scratch = nullptr;
  float* batch_logits = nullptr;      // [batch, vocab], allocated by the first batched step
  int64_t* batch_tokens_dev = nullptr; // [batch]
  float* batch_logits_host = nullptr;  // pinned, allocated when logits are first requested
  // pinned host staging
  float* logits_host = nullptr;
  int64_t* stage_host = nullptr;  // [0]=token [1]=pos [2]=seq [3]=out token, then chunk arrays
  // persistent decode kernel
  bool mega = false;
  int mega_grid = 0, mega_nslot = 0, mega_xs = 0, mega_max_split = 1;
  size_t mega_smem = 0;
  MegaLayer* mega_layers = nullptr;
  int64_t* io_dev = nullptr;  // [0] token [1] position [2] slot [3] produced token [4] error word
  unsigned long long* prof_dev = nullptr;
  unsigned long long* trace_dev = nullptr;  // [grid][layers + 1][16] event stamps (DYNINFER_CUDA_TRACE=1)
  uint8_t* prog_dev = nullptr;  // [grid] program blobs
  MegaProgLayout mega_lay;
  float* ll_dev = nullptr;  // hand-off vectors of (value, epoch) pairs, one allocation
  size_t ll_off[7] = {};    // float offsets: hidden0, hidden1, qkv, ctx, part, act, amax
  unsigned mega_epoch = 0;  // epochs used so far (each launch takes layers + 2)
  // graphs
  cudaGraphExec_t decode_graph = nullptr;  // H2D token/pos + forward + D2H token
  cudaGraphExec_t loop_graph = nullptr;    // forward + device-side advance
  std::map<int64_t, std::pair<cudaGraphExec_t, uint64_t>> batch_graphs;  // rows -> batched step (graph, nodes)
  uint64_t graph_nodes = 0, loop_nodes = 0;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  // tensor parallelism (tp_world > 1): communicator, partial-sum scratch, per-rank logits
  void* tp_comm = nullptr;
  float* tp_part = nullptr;    // [max_rows, hidden] partial o_proj / down products of ranks > 0
  float* tp_logits = nullptr;  // [max(1, batch), lm_rows] this rank's slice of the logits
  float* tp_gather = nullptr;  // [tp_world, batch, lm_rows] gathered slices of a batched step
  bool tp_warm = false;        // the collectives have run once outside a capture
  TpPeer peer;                 // peer-memory exchange (used instead of the all-reduce once attached)
  // scratch of the single-row products (K-slice partial sums), owned here so that a captured step
  // has no allocation nodes between its kernels
  void* scratch = nullptr;
  size_t scratch_bytes = 0;
  // statistics
  dyninfer_cuda_allocator_statistics_t stats{};
  uint64_t launches = 0;
};

namespace dyn {

typedef ::dyninfer_cuda_session_t Session;

inline int dev_alloc(Session* s, void** out, size_t bytes) {
  DYN_CUDA(cudaMalloc(out, bytes ? bytes : 16));
  s->stats.device_bytes_allocated += bytes;
  uint64_t live = s->stats.device_bytes_allocated - s->stats.device_bytes_freed;
  s->stats.device_bytes_peak = std::max(s->stats.device_bytes_peak, live);
  return 0;
}
inline void dev_free(Session* s, void* p, size_t bytes) {
  if (!p) return;
  cudaFree(p);
  s->stats.device_bytes_freed += bytes;
}
inline int host_alloc(Session* s, void** out, size_t bytes) {
  DYN_CUDA(cudaMallocHost(out, bytes ? bytes : 16));
  s->stats.host_bytes_allocated += bytes;
  uint64_t live = s->stats.host_bytes_allocated - s->stats.host_bytes_freed;
  s->stats.host_bytes_peak = std::max(s->stats.host_bytes_peak, live);
  return 0;
}

// session_mixers.cu
struct Json;
struct ParamTable;  // lookup of uploaded parameters, session.cu
int parse_mixers(const Json& desc, ModelCfg* cfg);
// Names whose matrices are worth placing back to back (one product), per layer that owns tensors.
std::vector<std::vector<std::string>> mixer_place_runs(const ModelCfg& cfg);
int bind_mixers(Session* s, const ParamTable& t, uint64_t* decode_bytes);
int configure_mixers(Session* s, int64_t rows);
int ensure_mixer_pages(Session* s, size_t page_count);
int reset_mixers(Session* s);
size_t mixer_cache_elements(const ModelCfg& cfg);  // cached elements per token and slot, all layers
int enqueue_mixer_layers(Session* s, int64_t rows, int64_t chunk_start, int64_t chunk_slot);
// A step of rows starting at `start` in `slot`: recurrent state cannot be rewound.
int mixer_check_position(Session* s, int64_t slot, int64_t start);

// session.cu
struct ParamTable {
  virtual int linear(const std::string& name, int64_t rows, int64_t cols, WRef* out) const = 0;
  virtual int plain(const std::string& name, const std::vector<int64_t>& shape, NormW* out) const = 0;
  virtual ~ParamTable() = default;
};
// The derived weights scale * (offset + w) of a norm, in f32 at `dst` (device); *w then refers to them.
int derive_norm(Session* s, NormW* w, int64_t n, float offset, float scale, float* dst);
bool follows_in_arena(const WRef& a, const WRef& b);
int session_linear(Session* s, const WRef& w, const void* x, int x_type, int64_t m, float* y, const float* residual);

}  // namespace dyn
