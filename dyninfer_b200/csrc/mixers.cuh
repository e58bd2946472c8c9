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
