// Decoders whose layers are listed one by one, each with a mixer of its own kind (retention, gated
// linear recurrence, latent attention, softmax attention, gated delta rule) and optionally a gated
// feed-forward or a mixture of experts, after the mixer or beside it: descriptor entries, binding of
// parameters, caches and states, and the layers of a step.
//
// A layer may run with another layer's parameters; its cache and state are always its own. The steps,
// graphs, batching and ABI around the layers are the session's (session.cu).
#include <math.h>
#include <string.h>

#include "json_min.h"
#include "session.cuh"

namespace dyn {

int parse_mixers(const Json& desc, ModelCfg* cfg) {
  const Json* list = desc.get("mixers");
  if (!list) return 0;
  DYN_CHECK(list->kind == Json::Arr && (int)list->arr.size() == cfg->layers && cfg->layers > 0,
            "descriptor `mixers` must list all %d layers", cfg->layers);
  for (int l = 0; l < cfg->layers; l++) {
    const Json& j = list->arr[l];
    MixerCfg m;
    const std::string kind = j.string("type", "");
    auto num = [&](const char* k) { return (int)j.number(k, 0); };
    m.tensors = (int)j.number("tensors", l);
    m.ff = num("ff");
    m.heads = num("heads"), m.dim = num("dim"), m.vdim = num("vdim");
    m.kv_heads = num("kv_heads"), m.parallel = num("parallel") != 0;
    m.rot_dims = num("rot_dims"), m.rot_base = j.number("rot_base", 0);
    DYN_CHECK(m.tensors >= 0 && m.tensors < cfg->layers && m.ff >= 0, "layer %d: bad `tensors` or `ff`", l);
    DYN_CHECK(m.rot_dims >= 0 && m.rot_dims <= m.dim && m.rot_dims % 2 == 0 && (m.rot_dims == 0 || m.rot_base > 0),
              "layer %d: rotation of %d dims in heads of %d", l, m.rot_dims, m.dim);
    m.experts = num("experts"), m.top = num("top"), m.expert_ff = num("expert_ff"), m.shared_ff = num("shared_ff");
    m.expert_limit = (float)j.number("expert_limit", 0), m.shared_limit = (float)j.number("shared_limit", 0);
    DYN_CHECK(m.experts >= 0 && m.shared_ff >= 0 && (m.experts == 0 || m.ff == 0), "layer %d: dense and expert feed-forwards", l);
    const bool grouped = m.heads > 0 && m.kv_heads > 0 && m.heads % m.kv_heads == 0 && m.dim > 0 && m.vdim > 0;
    if (kind == "retention") {
      m.kind = MIX_RETENTION;
      const Json* d = j.get("decay");
      DYN_CHECK(d && d->kind == Json::Arr && (int)d->arr.size() == m.heads, "layer %d: one decay per head", l);
      for (auto& v : d->arr) m.decay.push_back(v.num);
      DYN_CHECK(m.heads > 0 && m.dim > 0 && m.vdim > 0, "layer %d: retention sizes", l);
    } else if (kind == "rglru") {
      m.kind = MIX_RGLRU;
      m.width = num("width"), m.blocks = num("blocks"), m.taps = num("taps");
      DYN_CHECK(m.width > 0 && m.blocks > 0 && m.taps > 0 && m.width % m.blocks == 0,
                "layer %d: recurrence of width %d, %d gate blocks, %d taps", l, m.width, m.blocks, m.taps);
    } else if (kind == "latent_attention") {
      m.kind = MIX_LATENT;
      m.rank = num("rank"), m.scale = (float)j.number("scale", 0);
      DYN_CHECK(m.heads > 0 && m.dim > 0 && m.vdim > 0 && m.rank > 0 && m.rank <= 1024, "layer %d: latent attention sizes", l);
    } else if (kind == "softmax_attention") {
      m.kind = MIX_SOFTMAX;
      m.scale = (float)j.number("scale", 0), m.softcap = (float)j.number("softcap", 0), m.bias = num("bias") != 0;
      DYN_CHECK(grouped && m.softcap >= 0, "layer %d: softmax attention sizes", l);
    } else if (kind == "gated_delta") {
      m.kind = MIX_DELTA;
      m.taps = num("taps");
      DYN_CHECK(grouped && m.taps > 0, "layer %d: delta rule sizes", l);
    } else {
      DYN_CHECK(false, "E_KERNEL_COVERAGE: layer %d has a mixer without a cuda kernel: `%s`", l, kind.c_str());
    }
    cfg->mixers.push_back(m);
  }
  for (int l = 0; l < cfg->layers; l++)
    DYN_CHECK(cfg->mixers[cfg->mixers[l].tensors].kind == cfg->mixers[l].kind &&
                  cfg->mixers[cfg->mixers[l].tensors].tensors == cfg->mixers[l].tensors,
              "layer %d runs with the parameters of layer %d, which has other ones", l, cfg->mixers[l].tensors);
  return 0;
}

static std::string layer_name(int l) { return "blk." + std::to_string(l) + "."; }

static std::vector<std::string> input_names(const MixerCfg& m, int l) {
  const std::string b = layer_name(l);
  switch (m.kind) {
    case MIX_RETENTION: return {b + "attn_q.weight", b + "attn_k.weight", b + "attn_v.weight", b + "attn_gate.weight"};
    case MIX_RGLRU: return {b + "rec_y.weight", b + "rec_x.weight"};
    case MIX_SOFTMAX: return {b + "attn_q.weight", b + "attn_k.weight", b + "attn_v.weight"};
    case MIX_DELTA:
      return {b + "attn_q.weight", b + "attn_k.weight", b + "attn_v.weight", b + "attn_gate.weight", b + "delta_beta.weight",
              b + "delta_decay.weight"};
    default: return {b + "attn_q.weight", b + "attn_kv_down.weight", b + "attn_gate.weight"};
  }
}

std::vector<std::vector<std::string>> mixer_place_runs(const ModelCfg& cfg) {
  std::vector<std::vector<std::string>> runs;
  for (int l = 0; l < cfg.layers; l++) {
    const MixerCfg& m = cfg.mixers[l];
    if (m.tensors != l) continue;
    const std::string b = layer_name(l);
    runs.push_back(input_names(m, l));
    if (m.kind == MIX_LATENT) runs.push_back({b + "attn_k_up.weight", b + "attn_v_up.weight"});
    if (m.gated_width()) runs.push_back({b + "ffn_gate.weight", b + "ffn_up.weight"});
    for (int e = 0; e < m.experts; e++) {
      const std::string x = b + "expert_" + std::to_string(e);
      runs.push_back({x + "_gate.weight", x + "_up.weight"});
    }
  }
  return runs;
}

// The experts of layer l: shapes, and device tables of their matrices' addresses from `table` on.
static int bind_experts(const ModelCfg& c, int l, const ParamTable& t, MixerLayer* L, std::vector<const uint8_t*>* host, const uint8_t** table) {
  const MixerCfg& m = c.mixers[l];
  const std::string b = layer_name(l);
  MoeArgs& a = L->moe;
  if (t.linear(b + "ffn_router.weight", m.experts, c.hidden, &L->router)) return 1;
  a.experts = m.experts, a.top = m.top, a.ff = m.expert_ff, a.shared_ff = m.shared_ff;
  a.limit = m.expert_limit, a.shared_limit = m.shared_limit, a.width = c.hidden, a.exact = c.exact;
  a.shared_gate = L->gate, a.shared_up = L->up, a.shared_down = L->down;
  if (moe_check(a)) return 1;
  a.aligned = true;
  bool joined = true;
  const size_t at = host->size();
  std::vector<const uint8_t*> gate_up, down;
  for (int e = 0; e < m.experts; e++) {
    const std::string x = b + "expert_" + std::to_string(e);
    WRef w[3];
    if (t.linear(x + "_gate.weight", m.expert_ff, c.hidden, &w[0]) || t.linear(x + "_up.weight", m.expert_ff, c.hidden, &w[1]) ||
        t.linear(x + "_down.weight", c.hidden, m.expert_ff, &w[2]))
      return 1;
    if (e == 0) a.enc = w[0].enc;
    for (const WRef& r : w) {
      DYN_CHECK(r.enc == a.enc && (r.enc == E_F32 || r.enc == E_F16 || r.enc == E_BF16), "layer %d: experts must share a plain type", l);
      a.aligned = a.aligned && (reinterpret_cast<uintptr_t>(r.data) & 15) == 0;
      host->push_back(r.data);
    }
    joined = joined && follows_in_arena(w[0], w[1]);
    gate_up.push_back(w[0].data), down.push_back(w[2].data);
  }
  a.table = table + at;
  a.gate_up_table = joined ? table + host->size() : nullptr;
  host->insert(host->end(), gate_up.begin(), gate_up.end());
  a.down_table = table + host->size();
  host->insert(host->end(), down.begin(), down.end());
  return 0;
}

// Experts the tile-copy GEMM takes: bf16 matrices become f16 in place when all of them, and the shared expert's, keep their
// bits there (largest magnitude between 2^-8 and 2^15: nothing overflows, and what f16 drops below 2^-25 is less than 2^-17 of
// it), then tensor maps of every matrix. That GEMM's gated values share one scale, set by the limit: wide limits stay out.
static int prepare_experts(Session* s, MixerLayer* L, const std::vector<const uint8_t*>& host, size_t at, uint8_t* maps) {
  MoeArgs& a = L->moe;
  const int64_t count = (int64_t)a.ff * a.width, shared = (int64_t)a.shared_ff * a.width;
  const int matrices = 3 * a.experts;
  if (a.limit > 64.f) return 0;
  if (a.exact || !a.aligned || !grouped_gemm_takes(a.ff, a.width) || !grouped_gemm_takes(a.width, a.ff)) return 0;
  if (a.enc == E_BF16) {
    WRef* own[4] = {&L->gate, &L->up, &L->down, &L->gate_up};
    for (int i = 0; a.shared_ff && i < 3; i++)
      if (own[i]->enc != E_BF16) return 0;
    int* largest = nullptr;
    const uint8_t** extra = nullptr;
    const uint8_t* shared_host[3] = {L->gate.data, L->up.data, L->down.data};
    if (dev_alloc(s, (void**)&largest, 256)) return 1;
    extra = reinterpret_cast<const uint8_t**>(largest + 2);
    DYN_CUDA(cudaMemset(largest, 0, 8));
    DYN_CUDA(cudaMemcpy(extra, shared_host, sizeof(shared_host), cudaMemcpyHostToDevice));
    int bits[2] = {0, 0};
    if (bf16_table_range(a.table, matrices, count, largest, s->stream) ||
        (a.shared_ff && bf16_table_range(extra, 3, shared, largest + 1, s->stream)))
      return 1;
    DYN_CUDA(cudaStreamSynchronize(s->stream));
    DYN_CUDA(cudaMemcpy(bits, largest, sizeof(bits), cudaMemcpyDeviceToHost));
    auto fits = [](int b) {
      float v;
      memcpy(&v, &b, 4);
      return v >= 0x1p-8f && v <= 0x1p15f;
    };
    const bool ok = fits(bits[0]) && (!a.shared_ff || fits(bits[1]));
    if (ok && (bf16_table_to_f16(a.table, matrices, count, s->stream) || (a.shared_ff && bf16_table_to_f16(extra, 3, shared, s->stream)))) return 1;
    DYN_CUDA(cudaStreamSynchronize(s->stream));
    dev_free(s, largest, 256);
    if (!ok) return 0;
    a.enc = E_F16;
    for (WRef* w : own)
      if (w->data) w->enc = E_F16;
    a.shared_gate = L->gate, a.shared_up = L->up, a.shared_down = L->down;
  }
  if (a.enc != E_F16) return 0;
  std::vector<uint8_t> blob((size_t)matrices * GROUPED_MAP_BYTES + 64);
  uint8_t* p = blob.data() + (64 - reinterpret_cast<uintptr_t>(blob.data()) % 64) % 64;  // maps are made on 64-byte boundaries
  for (int i = 0; i < matrices; i++)
    if (make_grouped_weight_map(host[at + i], i % 3 == 2 ? a.width : a.ff, i % 3 == 2 ? a.ff : a.width, p + (size_t)i * GROUPED_MAP_BYTES))
      return 1;
  DYN_CUDA(cudaMemcpy(maps, p, (size_t)matrices * GROUPED_MAP_BYTES, cudaMemcpyHostToDevice));
  a.maps = maps;
  return 0;
}

int bind_mixers(Session* s, const ParamTable& t, uint64_t* decode_bytes) {
  const ModelCfg& c = s->cfg;
  const int64_t H = c.hidden;
  s->mix.resize(c.layers);
  size_t floats = 0;
  std::vector<size_t> decay_at(c.layers), freq_at(c.layers), norm_at(c.layers);
  size_t pointers = 0;
  for (int l = 0; l < c.layers; l++) {
    const MixerCfg& m = c.mixers[l];
    if (m.tensors != l) continue;
    if (m.rot_dims) freq_at[l] = floats, floats += m.rot_dims;  // doubles first, on even offsets
    if (m.kind == MIX_RETENTION) decay_at[l] = floats, floats += (m.heads + 1) / 2 * 2;
    if (c.norm_offset != 0.f) norm_at[l] = floats, floats += (2 * H + 1) / 2 * 2;
    pointers += (size_t)m.experts * 5;
  }
  const bool scaled = c.norm_offset != 0.f || c.logit_scale != 1.f;
  const size_t out_norm_at = floats;
  if (scaled) floats += H;
  if (dev_alloc(s, (void**)&s->tables, floats * 4)) return 1;
  if (pointers && dev_alloc(s, (void**)&s->expert_tables, pointers * sizeof(void*))) return 1;
  std::vector<const uint8_t*> addresses;
  // the output norm also carries the logits' factor: head (s x) = s head x
  if (scaled && derive_norm(s, &s->out_norm, H, c.norm_offset, c.logit_scale, s->tables + out_norm_at)) return 1;
  for (int l = 0; l < c.layers; l++) {
    MixerLayer& L = s->mix[l];
    const MixerCfg& m = c.mixers[l];
    L.c = m;
    if (m.tensors != l) continue;
    const std::string b = layer_name(l);
    std::vector<int64_t> in_rows;
    int64_t out_cols = 0;
    if (m.rot_dims) {
      std::vector<double> f(m.rot_dims / 2);
      for (size_t i = 0; i < f.size(); i++) f[i] = pow(m.rot_base, -2.0 * (double)i / m.rot_dims);
      L.freq = reinterpret_cast<double*>(s->tables + freq_at[l]);
      DYN_CUDA(cudaMemcpy(L.freq, f.data(), f.size() * 8, cudaMemcpyHostToDevice));
    }
    if (m.kind == MIX_RETENTION) {
      const int64_t qd = (int64_t)m.heads * m.dim, vd = (int64_t)m.heads * m.vdim;
      in_rows = {qd, qd, vd, vd}, out_cols = vd;
      std::vector<float> d(m.decay.begin(), m.decay.end());
      L.decay = s->tables + decay_at[l];
      DYN_CUDA(cudaMemcpy(L.decay, d.data(), d.size() * 4, cudaMemcpyHostToDevice));
    } else if (m.kind == MIX_RGLRU) {
      in_rows = {m.width, m.width}, out_cols = m.width;
      const int64_t n = m.width / m.blocks;
      if (t.plain(b + "rec_y.bias", {m.width}, &L.by) || t.plain(b + "rec_x.bias", {m.width}, &L.bx) ||
          t.plain(b + "rec_conv.weight", {m.width, m.taps}, &L.conv) || t.plain(b + "rec_conv.bias", {m.width}, &L.bc) ||
          t.plain(b + "rec_a_gate.weight", {m.blocks, n, n}, &L.ra) || t.plain(b + "rec_a_gate.bias", {m.blocks, n}, &L.bra) ||
          t.plain(b + "rec_i_gate.weight", {m.blocks, n, n}, &L.ri) || t.plain(b + "rec_i_gate.bias", {m.blocks, n}, &L.bri) ||
          t.plain(b + "rec_lambda", {m.width}, &L.lam))
        return 1;
    } else if (m.kind == MIX_SOFTMAX) {
      const int64_t qd = (int64_t)m.heads * m.dim, kd = (int64_t)m.kv_heads * m.dim, vd = (int64_t)m.kv_heads * m.vdim;
      in_rows = {qd, kd, vd}, out_cols = (int64_t)m.heads * m.vdim;
      if (m.bias && (t.plain(b + "attn_q.bias", {qd}, &L.qb) || t.plain(b + "attn_k.bias", {kd}, &L.kb) ||
                     t.plain(b + "attn_v.bias", {vd}, &L.vb) || t.plain(b + "attn_output.bias", {H}, &L.ob)))
        return 1;
    } else if (m.kind == MIX_DELTA) {
      const int64_t kd = (int64_t)m.kv_heads * m.dim, vd = (int64_t)m.heads * m.vdim;
      in_rows = {kd, kd, vd, vd, m.heads, m.heads}, out_cols = vd;
      if (t.plain(b + "conv_q.weight", {kd, m.taps}, &L.conv_q) || t.plain(b + "conv_k.weight", {kd, m.taps}, &L.conv_k) ||
          t.plain(b + "conv_v.weight", {vd, m.taps}, &L.conv_v) || t.plain(b + "delta_a_log", {m.heads}, &L.a_log) ||
          t.plain(b + "delta_dt.bias", {m.heads}, &L.dt) || t.plain(b + "head_norm.weight", {m.vdim}, &L.head_norm))
        return 1;
    } else {
      const int64_t qd = (int64_t)m.heads * m.dim, vd = (int64_t)m.heads * m.vdim;
      in_rows = {qd, m.rank, vd}, out_cols = vd;
      if (t.plain(b + "attn_kv_norm.weight", {m.rank}, &L.lat_norm) ||
          t.linear(b + "attn_k_up.weight", qd, m.rank, &L.uk) || t.linear(b + "attn_v_up.weight", vd, m.rank, &L.uv))
        return 1;
      for (const WRef* w : {&L.uk, &L.uv})
        DYN_CHECK(w->enc == E_F32 || w->enc == E_F16 || w->enc == E_BF16, "layer %d: latent up-projections must be a plain type", l);
      if (follows_in_arena(L.uk, L.uv)) L.ukv = L.uk, L.ukv.rows += L.uv.rows;
    }
    const auto names = input_names(m, l);
    L.parts = (int)names.size();
    WRef prev;
    for (int p = 0; p < L.parts; p++) {
      WRef w;
      if (t.linear(names[p], in_rows[p], H, &w)) return 1;
      if (p && follows_in_arena(prev, w)) {
        L.part_col[p] = L.in.back().rows;
        L.in.back().rows += w.rows;
      } else {
        L.part_col[p] = 0;
        L.in.push_back(w);
      }
      L.part_in[p] = (int)L.in.size() - 1;
      prev = w;
    }
    if (t.plain(b + "attn_norm.weight", {H}, &L.norm1) ||
        t.linear(b + (m.kind == MIX_RGLRU ? "rec_output.weight" : "attn_output.weight"), H, out_cols, &L.o))
      return 1;
    if (m.feeds_forward() && t.plain(b + "ffn_norm.weight", {H}, &L.norm2)) return 1;
    if (const int ff = m.gated_width()) {
      if (t.linear(b + "ffn_gate.weight", ff, H, &L.gate) || t.linear(b + "ffn_up.weight", ff, H, &L.up) ||
          t.linear(b + "ffn_down.weight", H, ff, &L.down))
        return 1;
      if (follows_in_arena(L.gate, L.up)) L.gate_up = L.gate, L.gate_up.rows += L.up.rows;
    }
    if (m.experts && bind_experts(c, l, t, &L, &addresses, s->expert_tables)) return 1;
    if (c.norm_offset != 0.f) {
      if (derive_norm(s, &L.norm1, H, c.norm_offset, 1.f, s->tables + norm_at[l])) return 1;
      if (L.norm2.ptr && derive_norm(s, &L.norm2, H, c.norm_offset, 1.f, s->tables + norm_at[l] + H)) return 1;
    }
  }
  if (!addresses.empty()) {
    DYN_CUDA(cudaMemcpy(s->expert_tables, addresses.data(), addresses.size() * sizeof(void*), cudaMemcpyHostToDevice));
    if (dev_alloc(s, (void**)&s->expert_maps, addresses.size() * GROUPED_MAP_BYTES)) return 1;
    for (int l = 0; l < c.layers; l++) {
      MixerLayer& L = s->mix[l];
      if (c.mixers[l].tensors != l || !L.moe.experts) continue;
      const size_t at = L.moe.table - s->expert_tables;
      if (prepare_experts(s, &L, addresses, at, s->expert_maps + at * GROUPED_MAP_BYTES)) return 1;
    }
  }
  // layers that run with another layer's parameters; state regions
  size_t off = 0;
  for (int l = 0; l < c.layers; l++) {
    const MixerCfg& m = c.mixers[l];
    if (m.tensors != l) {
      s->mix[l] = s->mix[m.tensors];
      s->mix[l].c = m;
      DYN_CHECK(c.mixers[m.tensors].same_sizes(m),
                "layer %d runs with the parameters of layer %d but has other sizes", l, m.tensors);
    }
    MixerLayer& L = s->mix[l];
    L.state_floats = m.kind == MIX_RETENTION || m.kind == MIX_DELTA ? (size_t)m.heads * m.dim * m.vdim
                     : m.kind == MIX_RGLRU                          ? (size_t)m.width
                                                                    : 0;
    L.ring_floats = m.kind == MIX_RGLRU   ? (size_t)m.taps * m.width
                    : m.kind == MIX_DELTA ? (size_t)m.taps * (2 * m.kv_heads * m.dim + m.heads * m.vdim)
                                          : 0;
    auto region = [&](size_t per_slot) {
      const size_t at = off;
      off += ((size_t)c.batch * per_slot + 63) / 64 * 64;
      return at;
    };
    L.state_off = region(L.state_floats);
    L.ring_off = region(L.ring_floats);
    for (const WRef& w : L.in) *decode_bytes += w.total_bytes();
    for (const WRef* w : {&L.o, &L.gate, &L.up, &L.down, &L.uk, &L.uv, &L.router})
      if (w->data) *decode_bytes += w->total_bytes();
    for (const NormW* w : {&L.norm1, &L.norm2, &L.by, &L.bx, &L.conv, &L.bc, &L.ra, &L.bra, &L.ri, &L.bri, &L.lam, &L.lat_norm, &L.qb,
                           &L.kb, &L.vb, &L.ob, &L.conv_q, &L.conv_k, &L.conv_v, &L.a_log, &L.dt, &L.head_norm})
      *decode_bytes += w->bytes;
    if (m.experts) *decode_bytes += 3ull * m.top * m.expert_ff * H * enc_row_bytes(L.moe.enc, 1);  // one row's experts
  }
  s->state_floats = off;
  s->slot_pos.assign((size_t)c.batch, 0);
  return 0;
}

size_t mixer_cache_elements(const ModelCfg& cfg) {
  size_t n = 0;
  for (const MixerCfg& m : cfg.mixers) n += m.cached();
  return n;
}

static Vec vec(const NormW& w) {
  Vec v;
  v.ptr = reinterpret_cast<const uint8_t*>(w.ptr), v.type = w.type;
  return v;
}

static int64_t input_width(const MixerLayer& L) {
  int64_t n = 0;
  for (const WRef& w : L.in) n += w.rows;
  return n;
}

// Where part p of the layer's input products lies when the products of `rows` rows are written to `buf`
// one after the other.
static Rows part_rows(const MixerLayer& L, float* buf, int64_t rows, int p) {
  for (int i = 0; i < L.part_in[p]; i++) buf += rows * L.in[i].rows;
  Rows r;
  r.ptr = buf + L.part_col[p], r.ld = L.in[L.part_in[p]].rows;
  return r;
}

static uint8_t* cache_plane(Session* s, int layer, int64_t cap) {
  size_t elems = 0;
  for (int l = 0; l < layer; l++) elems += (size_t)s->cfg.batch * cap * s->mix[l].c.cached();
  return s->lcache + elems * s->kv_elem;
}

static RetentionArgs retention_args(Session* s, const MixerLayer& L, int64_t rows) {
  RetentionArgs a;
  a.q = part_rows(L, s->qkv1, rows, 0), a.k = part_rows(L, s->qkv1, rows, 1);
  a.v = part_rows(L, s->qkv1, rows, 2), a.g = part_rows(L, s->qkv1, rows, 3);
  a.heads = L.c.heads, a.dim = L.c.dim, a.vdim = L.c.vdim, a.rot_dims = L.c.rot_dims;
  a.freq = L.freq, a.decay = L.decay;
  a.state = s->state + L.state_off, a.out = s->ctx, a.scratch = s->mix_scratch, a.eps = s->cfg.eps, a.exact = s->cfg.exact;
  return a;
}

static RglruArgs rglru_args(Session* s, const MixerLayer& L, int64_t rows) {
  RglruArgs a;
  a.y = part_rows(L, s->qkv1, rows, 0), a.x = part_rows(L, s->qkv1, rows, 1);
  a.width = L.c.width, a.blocks = L.c.blocks, a.taps = L.c.taps;
  a.by = vec(L.by), a.bx = vec(L.bx), a.conv = vec(L.conv), a.bc = vec(L.bc), a.ra = vec(L.ra), a.bra = vec(L.bra);
  a.ri = vec(L.ri), a.bri = vec(L.bri), a.lam = vec(L.lam);
  a.state = s->state + L.state_off, a.ring = s->state + L.ring_off;
  a.out = s->ctx, a.scratch = s->mix_scratch, a.exact = s->cfg.exact;
  return a;
}

static LatentArgs latent_args(Session* s, const MixerLayer& L, int layer, int64_t rows, int64_t cap) {
  LatentArgs a;
  a.q = part_rows(L, s->qkv1, rows, 0), a.d = part_rows(L, s->qkv1, rows, 1), a.g = part_rows(L, s->qkv1, rows, 2);
  a.heads = L.c.heads, a.dim = L.c.dim, a.vdim = L.c.vdim, a.rank = L.c.rank;
  a.scale = L.c.scale, a.eps = s->cfg.eps, a.norm = vec(L.lat_norm);
  a.uk = L.uk, a.uv = L.uv, a.ukv = L.ukv;
  a.cache = cache_plane(s, layer, cap), a.kv_type = s->kv_type, a.cap = cap;
  a.out = s->ctx, a.scratch = s->mix_scratch, a.exact = s->cfg.exact, a.max_rows = s->max_rows;
  return a;
}

static SoftmaxArgs softmax_args(Session* s, const MixerLayer& L, int layer, int64_t rows, int64_t cap) {
  SoftmaxArgs a;
  a.q = part_rows(L, s->qkv1, rows, 0), a.k = part_rows(L, s->qkv1, rows, 1), a.v = part_rows(L, s->qkv1, rows, 2);
  a.heads = L.c.heads, a.kv_heads = L.c.kv_heads, a.dim = L.c.dim, a.vdim = L.c.vdim, a.rot_dims = L.c.rot_dims;
  a.freq = L.freq, a.scale = L.c.scale, a.softcap = L.c.softcap, a.qb = vec(L.qb), a.kb = vec(L.kb), a.vb = vec(L.vb);
  uint8_t* keys = cache_plane(s, layer, cap);
  a.kcache = keys, a.vcache = keys + (size_t)s->cfg.batch * cap * L.c.kv_heads * L.c.dim * s->kv_elem;
  a.kv_type = s->kv_type, a.cap = cap, a.out = s->ctx, a.scratch = s->mix_scratch, a.exact = s->cfg.exact;
  return a;
}

static DeltaArgs delta_args(Session* s, const MixerLayer& L, int64_t rows) {
  DeltaArgs a;
  Rows* parts[6] = {&a.q, &a.k, &a.v, &a.g, &a.b, &a.a};
  for (int p = 0; p < 6; p++) *parts[p] = part_rows(L, s->qkv1, rows, p);
  a.heads = L.c.heads, a.kv_heads = L.c.kv_heads, a.dim = L.c.dim, a.vdim = L.c.vdim, a.taps = L.c.taps;
  a.conv_q = vec(L.conv_q), a.conv_k = vec(L.conv_k), a.conv_v = vec(L.conv_v);
  a.a_log = vec(L.a_log), a.dt = vec(L.dt), a.norm = vec(L.head_norm);
  a.state = s->state + L.state_off, a.ring = s->state + L.ring_off;
  a.out = s->ctx, a.scratch = s->mix_scratch, a.eps = s->cfg.eps, a.exact = s->cfg.exact;
  return a;
}

static MoeArgs moe_args(Session* s, const MixerLayer& L) {
  MoeArgs a = L.moe;
  a.limit = L.c.expert_limit, a.shared_limit = L.c.shared_limit, a.top = L.c.top;
  a.scratch = s->mix_scratch;
  return a;
}

static int grow_mix_scratch(Session* s, int64_t rows, int64_t cap) {
  size_t need = 0;
  for (int l = 0; l < s->cfg.layers; l++) {
    const MixerLayer& L = s->mix[l];
    if (L.c.kind == MIX_RETENTION) need = std::max(need, retention_scratch_floats(retention_args(s, L, rows), rows));
    else if (L.c.kind == MIX_RGLRU) need = std::max(need, rglru_scratch_floats(rglru_args(s, L, rows), rows));
    else if (L.c.kind == MIX_SOFTMAX) need = std::max(need, softmax_scratch_floats(softmax_args(s, L, l, rows, cap), rows));
    else if (L.c.kind == MIX_DELTA) need = std::max(need, delta_scratch_floats(delta_args(s, L, rows), rows));
    else need = std::max(need, latent_scratch_floats(latent_args(s, L, l, rows, cap), rows));
    if (L.c.experts) need = std::max(need, moe_scratch_floats(moe_args(s, L), rows));
  }
  if (need <= s->mix_scratch_floats) return 0;
  dev_free(s, s->mix_scratch, s->mix_scratch_floats * 4);
  s->mix_scratch = nullptr, s->mix_scratch_floats = 0;
  if (dev_alloc(s, (void**)&s->mix_scratch, need * 4)) return 1;
  s->mix_scratch_floats = need;
  return 0;
}

// Activation scratch and the recurrent state, at the first configuration.
int configure_mixers(Session* s, int64_t rows) {
  const ModelCfg& c = s->cfg;
  int64_t proj = 0, ctx = 0, ff = 0;
  bool beside = false;
  for (const MixerLayer& L : s->mix) {
    proj = std::max(proj, input_width(L));
    ctx = std::max(ctx, L.o.cols);
    ff = std::max<int64_t>(ff, L.c.gated_width());
    beside = beside || (L.c.parallel && L.c.feeds_forward());
  }
  const int64_t wide = std::max({(int64_t)c.hidden, ctx, ff}), alloc = rows + rows / 2 + 64;
  if (dev_alloc(s, (void**)&s->hidden, (size_t)rows * c.hidden * 4) ||
      dev_alloc(s, (void**)&s->xn, (size_t)rows * c.hidden * 4) ||
      dev_alloc(s, (void**)&s->ctx, (size_t)rows * ctx * 4) ||
      dev_alloc(s, (void**)&s->act, (size_t)rows * std::max<int64_t>(1, ff) * 4) ||
      (!c.exact && rows >= 64 &&
       (dev_alloc(s, (void**)&s->xh, (size_t)alloc * wide * 2) || dev_alloc(s, (void**)&s->xinv, (size_t)alloc * 4) ||
        dev_alloc(s, (void**)&s->gpart, (size_t)8 * rows * c.hidden * 4))) ||
      (!c.exact && rows >= 64 && beside &&
       (dev_alloc(s, (void**)&s->xh2, (size_t)alloc * c.hidden * 2) || dev_alloc(s, (void**)&s->xinv2, (size_t)alloc * 4))) ||
      dev_alloc(s, (void**)&s->qkv1, (size_t)rows * proj * 4) ||
      dev_alloc(s, (void**)&s->gu1, (size_t)rows * 2 * std::max<int64_t>(1, ff) * 4) ||
      dev_alloc(s, (void**)&s->tokens_dev, (size_t)rows * 8) || dev_alloc(s, (void**)&s->row_pos_dev, (size_t)rows * 8) ||
      dev_alloc(s, (void**)&s->row_seq_dev, (size_t)rows * 8) ||
      host_alloc(s, (void**)&s->stage_host, (size_t)(8 + 3 * rows) * 8) ||
      dev_alloc(s, (void**)&s->state, s->state_floats * 4))
    return 1;
  if (s->xh) s->xh_rows = alloc, s->xh_cols = wide, s->gpart_bytes = (size_t)8 * rows * c.hidden * 4;
  s->max_rows = rows;
  DYN_CUDA(cudaMemset(s->state, 0, s->state_floats * 4));
  return 0;
}

int ensure_mixer_pages(Session* s, size_t page_count) {
  const ModelCfg& c = s->cfg;
  const int64_t cap = (int64_t)(page_count * s->page_size), old = (int64_t)(s->pages * s->page_size);
  const size_t bytes = mixer_cache_elements(c) * c.batch * (size_t)cap * s->kv_elem;
  uint8_t* fresh = nullptr;
  if (bytes) {
    if (dev_alloc(s, (void**)&fresh, bytes)) return 1;
    DYN_CUDA(cudaMemsetAsync(fresh, 0, bytes, s->stream));
    if (s->pages) {  // keep what is cached: every layer's slots are planes of their own
      size_t from = 0, to = 0;
      for (const MixerLayer& L : s->mix) {
        auto move = [&](size_t planes, size_t width) -> int {
          const size_t src = (size_t)old * width * s->kv_elem, dst = (size_t)cap * width * s->kv_elem;
          DYN_CUDA(cudaMemcpy2DAsync(fresh + to, dst, s->lcache + from, src, src, planes, cudaMemcpyDeviceToDevice, s->stream));
          from += src * planes, to += dst * planes;
          return 0;
        };
        if (L.c.kind == MIX_LATENT && move(c.batch, L.c.rank)) return 1;
        if (L.c.kind == MIX_SOFTMAX && (move((size_t)c.batch * L.c.kv_heads, L.c.dim) || move((size_t)c.batch * L.c.kv_heads, L.c.vdim)))
          return 1;
      }
    }
    DYN_CUDA(cudaStreamSynchronize(s->stream));
    dev_free(s, s->lcache, s->lcache_bytes);
    s->lcache = fresh, s->lcache_bytes = bytes;
  }
  return grow_mix_scratch(s, s->max_rows, cap);
}

int reset_mixers(Session* s) {
  if (s->lcache) DYN_CUDA(cudaMemsetAsync(s->lcache, 0, s->lcache_bytes, s->stream));
  if (s->state_floats) DYN_CUDA(cudaMemsetAsync(s->state, 0, s->state_floats * 4, s->stream));
  DYN_CUDA(cudaStreamSynchronize(s->stream));
  std::fill(s->slot_pos.begin(), s->slot_pos.end(), 0);
  return 0;
}

int mixer_check_position(Session* s, int64_t slot, int64_t start) {
  if (s->cfg.mixers.empty() || start == 0) return 0;
  const int64_t at = s->slot_pos[(size_t)slot];
  DYN_CHECK(at >= 0, "slot %lld: its last step failed, the sequence must start over at position 0", (long long)slot);
  DYN_CHECK(start == at, "slot %lld is at position %lld: recurrent state cannot continue at %lld", (long long)slot,
            (long long)at, (long long)start);
  return 0;
}

int enqueue_mixer_layers(Session* s, int64_t rows, int64_t chunk_start, int64_t chunk_slot) {
  const ModelCfg& c = s->cfg;
  cudaStream_t st = s->stream;
  const int64_t H = c.hidden, cap = (int64_t)(s->pages * s->page_size);
  StepRows step;
  step.rows = rows, step.pos = s->row_pos_dev, step.seq = s->row_seq_dev;
  step.base = chunk_start, step.slot = chunk_slot;
  // Many rows whose products all go to the dequant GEMM: the norm kernels write its operand themselves and
  // the K-split sums of the output and down projections are added inside the norm that follows.
  bool fuse = !c.exact && rows >= 64 && s->xh && H <= 8192;
  for (const MixerLayer& L : s->mix) {
    auto takes = [&](const WRef& w) {
      return !w.data || (dqgemm_tc_takes(w, rows) && dqgemm_tc_padded_rows(w, rows) <= s->xh_rows);
    };
    for (const WRef& w : L.in) fuse = fuse && takes(w);
    for (const WRef* w : {&L.o, &L.gate, &L.up, &L.down, &L.router}) fuse = fuse && takes(*w);
    // experts that only the f32 products take read the normalised rows in f32
    if (L.c.experts) fuse = fuse && moe_takes_operand(moe_args(s, L));
  }
  // A few rows of 16-bit weights: the streaming GEMV normalises its input and gates its output itself.
  bool stream = rows <= 4;
  for (const MixerLayer& L : s->mix) {
    for (const WRef& w : L.in) stream = stream && gemv_plain_takes(w, rows);
    if (L.c.ff) stream = stream && L.gate_up.data && gemv_plain_takes(L.gate_up, rows);
    if (L.c.experts) stream = stream && gemv_plain_takes(L.router, rows) && moe_streams(moe_args(s, L), rows);
  }
  GemvForm form;
  auto streamed = [&](const WRef& w, const float* x, float* y) -> int {
    bool handled = false;
    if (launch_gemv_plain(w, x, E_F32, (int)rows, y, nullptr, st, &handled, form)) return 1;
    DYN_CHECK(handled, "streaming GEMV refused a product it had accepted");
    return 0;
  };
  int pending = 0;  // K-split sums in gpart that `hidden` still lacks
  const __half* operand = nullptr;  // what from_norm multiplies in the fused form, and its scales
  const float* operand_inv = nullptr;
  auto norm = [&](const NormW& w, const NormPair& pair = NormPair()) -> int {
    operand = s->xh, operand_inv = s->xinv;
    if (stream) {
      form.norm_w = w.ptr, form.norm_type = w.type, form.eps = c.eps;
      return 0;
    }
    if (!fuse) return launch_rms_norm(s->hidden, w.ptr, w.type, rows, H, c.eps, s->xn, st);
    const int splits = pending;
    pending = 0;
    return splits > 1 ? launch_norm_prepare(nullptr, s->gpart, splits, s->hidden, s->hidden, w.ptr, w.type, rows, H, c.eps,
                                            s->xh, s->xinv, st, pair)
                      : launch_norm_prepare(s->hidden, nullptr, 0, nullptr, pair.bias ? s->hidden : nullptr, w.ptr, w.type, rows, H,
                                            c.eps, s->xh, s->xinv, st, pair);
  };
  // x == nullptr: the prepared operand
  auto gemm = [&](const WRef& w, const float* x, const __half* xh, const float* xinv, float* y, const float* residual, bool defer) -> int {
    TgIo io;
    if (!x) io.xh = xh, io.inv_s = xinv, io.rows_alloc = s->xh_rows;
    if (defer) io.partial = s->gpart, io.partial_bytes = s->gpart_bytes;
    bool handled = false;
    if (launch_dqgemm_tc(w, x, E_F32, rows, y, residual, st, &handled, &io)) return 1;
    DYN_CHECK(handled, "dequant GEMM refused a product it had accepted");
    if (defer) pending = io.splits;
    return 0;
  };
  // a product of the normalised rows
  auto from_norm = [&](const WRef& w, float* y) -> int {
    if (stream) return streamed(w, s->hidden, y);
    return fuse ? gemm(w, nullptr, operand, operand_inv, y, nullptr, false) : session_linear(s, w, s->xn, E_F32, rows, y, nullptr);
  };
  // hidden += W x; `last`: no norm of this function follows to add deferred sums
  auto to_hidden = [&](const WRef& w, const float* x, bool prepared, bool last) -> int {
    return fuse ? gemm(w, prepared ? nullptr : x, s->xh, s->xinv, s->hidden, s->hidden, !last)
                : session_linear(s, w, x, E_F32, rows, s->hidden, s->hidden);
  };
  for (int l = 0; l < c.layers; l++) {
    const MixerLayer& L = s->mix[l];
    const bool final_layer = l + 1 == c.layers;
    const bool forward = L.c.feeds_forward();
    const bool beside = L.c.parallel && forward;  // the feed-forward reads the residual as the mixer does
    // many rows: both norms, and the output bias into the residual, in one launch; the mixer's output may then follow at once
    const bool paired = beside && fuse && s->xh2;
    NormPair pair;
    if (paired) pair.w = L.norm2.ptr, pair.type = L.norm2.type, pair.xh = s->xh2, pair.inv_s = s->xinv2, pair.bias = L.ob.ptr, pair.bias_type = L.ob.type;
    if (norm(L.norm1, pair)) return 1;
    float* y = s->qkv1;
    for (const WRef& w : L.in) {
      if (from_norm(w, y)) return 1;
      y += rows * w.rows;
    }
    bool mixed_operand = false;  // the mixer's output is the operand in xh (the input products are done with it)
    int rc;
    switch (L.c.kind) {
      case MIX_RETENTION: rc = launch_retention(retention_args(s, L, rows), step, st); break;
      case MIX_RGLRU: rc = launch_rglru(rglru_args(s, L, rows), step, st); break;
      case MIX_SOFTMAX: rc = launch_softmax_attention(softmax_args(s, L, l, rows, cap), step, st); break;
      case MIX_DELTA: {
        DeltaArgs a = delta_args(s, L, rows);
        mixed_operand = fuse && step.base >= 0 && delta_writes_operand(a) && (!beside || paired);
        if (mixed_operand) a.xh = s->xh, a.xinv = s->xinv;
        rc = launch_delta(a, step, st);
        break;
      }
      default: rc = launch_latent_attention(latent_args(s, L, l, rows, cap), step, st);
    }
    if (rc) return 1;
    // the mixer's output into the residual
    auto add_mixer = [&](bool last) -> int {
      if (!L.ob.ptr || paired) return to_hidden(L.o, s->ctx, mixed_operand, last);
      if (stream && gemv_plain_takes(L.o, rows)) {
        GemvForm f;
        f.bias = L.ob.ptr, f.bias_type = L.ob.type;
        bool handled = false;
        return launch_gemv_plain(L.o, s->ctx, E_F32, (int)rows, s->hidden, s->hidden, st, &handled, f);
      }
      return to_hidden(L.o, s->ctx, false, last) || launch_add_bias(s->hidden, L.ob.ptr, L.ob.type, rows, H, st);
    };
    if ((!beside || paired) && add_mixer(paired || (final_layer && !forward))) return 1;
    if (!forward) continue;
    if (paired) operand = s->xh2, operand_inv = s->xinv2;
    else if (norm(L.norm2)) return 1;
    // products of the experts up to their outputs; the router's logits lie at the start of the scratch
    const MoeArgs moe = L.c.experts ? moe_args(s, L) : MoeArgs();
    float* const z = s->mix_scratch;
    if (L.c.experts) {
      if (from_norm(L.router, z)) return 1;
      if (stream) {
        float* const act = moe_few_act(moe, rows);
        if (launch_moe_few(moe, s->hidden, L.norm2.ptr, L.norm2.type, c.eps, rows, z, act, st) || (beside && !paired && add_mixer(true)) ||
            launch_moe_few_down(moe, rows, z, act, s->hidden, st))
          return 1;
        continue;
      }
      if (launch_moe_experts(moe, fuse ? nullptr : s->xn, fuse ? operand : nullptr, operand_inv, rows, z, st)) return 1;
    }
    const int64_t ff = L.c.gated_width();
    bool prepared = false;
    if (ff && stream) {
      form.pairs = 1;
      if (from_norm(L.gate_up, s->act)) return 1;
      form.pairs = 0;
    } else if (ff && L.gate_up.data) {
      if (from_norm(L.gate_up, s->gu1)) return 1;
      prepared = fuse;
      const float limit = L.c.shared_limit;
      if (L.c.experts ? (fuse ? launch_clamped_glu_prepare(s->gu1, rows, ff, limit, s->xh, s->xinv, st)
                              : launch_clamped_glu_rows(s->gu1, rows, ff, limit, s->act, st))
                      : (fuse ? launch_silu_prepare(s->gu1, rows, ff, s->xh, s->xinv, st)
                              : launch_silu_mul_rows(s->gu1, rows, ff, s->act, st)))
        return 1;
    } else if (ff) {
      float* up = s->gu1 + rows * ff;
      if (from_norm(L.gate, s->gu1) || from_norm(L.up, up) ||
          (L.c.experts ? launch_clamped_glu(s->gu1, up, rows * ff, L.c.shared_limit, s->act, st)
                       : launch_silu_mul(s->gu1, up, rows * ff, s->act, st)))
        return 1;
    }
    if (beside && !paired && add_mixer(true)) return 1;
    if (ff && to_hidden(L.down, s->act, prepared, final_layer)) return 1;
    if (L.c.experts && launch_moe_combine(moe, rows, s->hidden, st)) return 1;
  }
  return 0;
}

}  // namespace dyn
