// Token mixers other than GQA attention: kernels' arguments and launchers. Every mixer reads the
// output of its layer's input products (f32, possibly column ranges of one fused product, hence the
// separate row strides) and writes the rows that feed its output projection.
//
// A step is either a set of independent rows, each the next token of its own slot (decode), or a
// portion: consecutive tokens of one slot. Positions are absolute; a row at position 0 starts from
// an empty state whatever the slot held before, so a slot is reused without clearing it.
#pragma once

#include "common.cuh"

namespace dyn {

// Rows of one projection: element (r, c) at ptr[r * ld + c].
struct Rows {
  float* ptr = nullptr;
  int64_t ld = 0;
};
// A vector or small table in its checkpoint type.
struct Vec {
  const uint8_t* ptr = nullptr;
  int type = E_BF16;
};
// Which tokens a launch covers.
struct StepRows {
  int64_t rows = 0;
  const int64_t* pos = nullptr;  // device, absolute position of each row
  const int64_t* seq = nullptr;  // device, slot of each row
  int64_t base = -1, slot = 0;   // base >= 0: a portion of slot `slot` starting at position `base`
};

// The angle of a position, reduced in double precision: p * f is far from 0 for long contexts.
__device__ __forceinline__ void sincos_position(int64_t pos, double freq, float* sv, float* cv) {
  const double turns = (double)pos * freq * 0.15915494309189535;  // 1 / 2 pi
  const double frac = turns - rint(turns);
  sincospif((float)(2.0 * frac), sv, cv);
}

__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_of(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float vec_at(const Vec& v, int64_t i) { return aux_load(v.ptr, v.type, i); }

// ---- retention: fixed-decay linear attention (retention.cu) ----
//   S_t = decay_h S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t,  out = o_t / rms(o_t) * silu(g_t)
// q and k rotated (rotate-half on the first rot_dims of a head), k scaled by dim^-1/2 afterwards.
struct RetentionArgs {
  Rows q, k, v, g;
  int heads = 0, dim = 0, vdim = 0, rot_dims = 0;
  const double* freq = nullptr;   // [rot_dims / 2] angles per position
  const float* decay = nullptr;   // [heads]
  float* state = nullptr;         // [slot][heads][dim][vdim]
  float* out = nullptr;           // [rows, heads * vdim]
  float* scratch = nullptr;       // retention_scratch_floats
  float eps = 0.f;
  bool exact = false;             // f32 products only
};
size_t retention_scratch_floats(const RetentionArgs& a, int64_t rows);
int launch_retention(const RetentionArgs& a, const StepRows& r, cudaStream_t st);

// ---- gated linear recurrence behind a short convolution (rglru.cu) ----
//   u = conv(x + bx) + bc;  r, i = sigmoid(block-diagonal products of u);  log a = -c r softplus(lam)
//   S_t = a S_{t-1} + sqrt(1 - a^2) i u,  out = S_t * gelu_tanh(y + by)
struct RglruArgs {
  Rows y, x;
  int width = 0, blocks = 0, taps = 0;
  float c = 8.0f;
  Vec by, bx, conv, bc, ra, bra, ri, bri, lam;
  float* state = nullptr;   // [slot][width]
  float* ring = nullptr;    // [slot][taps][width]: convolution input of position p in row p mod taps
  float* out = nullptr;     // [rows, width]
  float* scratch = nullptr; // rglru_scratch_floats
  bool exact = false;       // f32 products only
};
size_t rglru_scratch_floats(const RglruArgs& a, int64_t rows);
int launch_rglru(const RglruArgs& a, const StepRows& r, cudaStream_t st);

// ---- attention over cached latents, without positions (latent_attention.cu) ----
//   c_t = rms_norm(d_t) * w (cached);  score = scale (q . W_uk c);  out = softmax W_uv c * sigmoid(g)
struct LatentArgs {
  Rows q, d, g;
  int heads = 0, dim = 0, vdim = 0, rank = 0;
  float scale = 0.f, eps = 0.f;
  Vec norm;
  WRef uk, uv, ukv;               // ukv: [uk; uv] as one matrix when they lie back to back
  void* cache = nullptr;          // [slot][cap][rank]
  int kv_type = E_F32;
  int64_t cap = 0;
  float* out = nullptr;           // [rows, heads * vdim]
  float* scratch = nullptr;       // latent_scratch_floats
  bool exact = false;
  int64_t max_rows = 0;           // rows the expansion of the cache is done in
};
size_t latent_scratch_floats(const LatentArgs& a, int64_t rows);
int launch_latent_attention(const LatentArgs& a, const StepRows& r, cudaStream_t st);

// ---- softmax attention over cached keys and values (softmax_attention.cu) ----
//   score = softcap tanh(scale (q . k) / softcap), causal; q and k rotated (rotate-half on the first rot_dims of a
//   head); query head h reads kv head h / (heads / kv_heads); values may have another width than keys
struct SoftmaxArgs {
  Rows q, k, v;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot_dims = 0;
  const double* freq = nullptr;   // [rot_dims / 2] angles per position
  float scale = 0.f, softcap = 0.f;  // softcap 0: scores as they are
  Vec qb, kb, vb;                 // added to the products (ptr nullptr: none)
  void *kcache = nullptr, *vcache = nullptr;  // [slot][kv head][cap][dim] and [..][vdim]
  int kv_type = E_F32;
  int64_t cap = 0;
  float* out = nullptr;           // [rows, heads * vdim]
  float* scratch = nullptr;       // softmax_scratch_floats
  bool exact = false;
};
size_t softmax_scratch_floats(const SoftmaxArgs& a, int64_t rows);
int launch_softmax_attention(const SoftmaxArgs& a, const StepRows& r, cudaStream_t st);

// ---- gated delta rule behind short convolutions (delta.cu) ----
//   q, k, v = silu(conv(.)); q, k to unit length per head, q times dim^-1/2; decay g = exp(-exp(A) softplus(a + dt)),
//   beta = sigmoid(b);  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   out = o / rms(o) * norm * silu(gate); value head h reads q/k head h / (heads / kv_heads)
struct DeltaArgs {
  Rows q, k, v, g, b, a;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0;
  Vec conv_q, conv_k, conv_v;     // [channels, taps], last column on the current token
  Vec a_log, dt, norm;
  float* state = nullptr;         // [slot][heads][dim][vdim]
  float* ring = nullptr;          // [slot][taps][q | k | v channels]: convolution input of position p in row p mod taps
  float* out = nullptr;           // [rows, heads * vdim]
  float* scratch = nullptr;       // delta_scratch_floats
  __half* xh = nullptr;           // portions of several rows: the output as the dequant GEMM's operand instead of f32
  float* xinv = nullptr;
  float eps = 0.f, unit_eps = 1e-6f;
  bool exact = false;             // f32 products only
};
bool delta_writes_operand(const DeltaArgs& a);
size_t delta_scratch_floats(const DeltaArgs& a, int64_t rows);
int launch_delta(const DeltaArgs& a, const StepRows& r, cudaStream_t st);

// ---- mixture of experts (moe.cu) ----
//   the `top` experts with the largest sigmoid(router . h); sum of expert(score * h) + shared(h), with
//   expert(h) = down(min(gate h, limit) sigmoid(1.702 min(gate h, limit)) (clamp(up h, +-limit) + 1))
struct MoeArgs {
  int experts = 0, top = 0, ff = 0, shared_ff = 0;  // shared_ff 0: no shared expert
  float limit = 0.f, shared_limit = 0.f;
  int64_t width = 0;
  int enc = E_BF16;                         // type of all experts' matrices
  bool aligned = false;                     // they start on 16-byte boundaries
  const uint8_t* const* table = nullptr;    // device, [experts][gate, up, down]
  // device, [experts]: [gate; up] as one matrix each (nullptr: not laid back to back), down
  const uint8_t* const *gate_up_table = nullptr, *const* down_table = nullptr;
  const void* maps = nullptr;               // device, tensor maps of f16 matrices [experts][gate, up, down] (nullptr: none)
  WRef shared_gate, shared_up, shared_down;
  float* scratch = nullptr;                 // moe_scratch_floats; the router logits [rows, experts] come first
  bool exact = false;
};
int moe_check(const MoeArgs& a);
size_t moe_scratch_floats(const MoeArgs& a, int64_t rows);
// A few rows: launch_moe_few forms act (moe_few_act) from norm(x) and the router logits z, shared expert included;
// launch_moe_few_down adds the outputs to hidden.
bool moe_streams(const MoeArgs& a, int64_t rows);
float* moe_few_act(const MoeArgs& a, int64_t rows);
int launch_moe_few(const MoeArgs& a, const float* x, const void* norm_w, int norm_type, float eps, int64_t rows, const float* z, float* act,
                   cudaStream_t st);
int launch_moe_few_down(const MoeArgs& a, int64_t rows, const float* z, const float* act, float* hidden, cudaStream_t st);
// Many rows: the chosen experts' outputs into the scratch (rows as xn in f32, or as the GEMM's operand xh, xinv), then
// into hidden. The shared expert is the caller's.
// Whether the experts read the operand (otherwise xn).
bool moe_takes_operand(const MoeArgs& a);
int launch_moe_experts(const MoeArgs& a, const float* xn, const __half* xh, const float* xinv, int64_t rows, const float* z, cudaStream_t st);
int launch_moe_combine(const MoeArgs& a, int64_t rows, float* hidden, cudaStream_t st);
// y = clamped_glu(gate, up): rows of [gate | up], or two matrices
int launch_clamped_glu_rows(const float* gate_up, int64_t rows, int64_t inter, float limit, float* y, cudaStream_t st);
int launch_clamped_glu(const float* gate, const float* up, int64_t n, float limit, float* y, cudaStream_t st);

// y[m, n] = sum_k x[m, k] w[n, k] (+ residual) with f32 products and accumulation for plain weights of
// any shape (gemm_f32.cu).
int launch_gemm_f32(const WRef& w, const void* x, int x_type, int64_t m, float* y, const float* residual,
                    cudaStream_t s);
// The same for every encoding: the kernels that multiply in f32 only, whatever the row count.
int launch_linear_exact(const WRef& w, const void* x, int x_type, int64_t m, float* y, const float* residual,
                        cudaStream_t s);
// RMSNorm of the rows of x that `index` lists: y[j] = norm(x[index[j]]).
int launch_rms_norm_indexed(const float* x, const int64_t* index, const void* w, int w_type, int64_t rows,
                            int64_t width, float eps, float* y, cudaStream_t s);

}  // namespace dyn
