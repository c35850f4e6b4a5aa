// Retention: linear attention with a fixed decay per head.  Per head, with R_t the rotation of position t,
//   S_t = decay S_{t-1} + (R_t k_t / sqrt(dim)) v_t^T,   o_t = S_t^T R_t q_t,   y_t = o_t / rms(o_t) * silu(g_t)
// over a float32 state S [dim, vdim] that a sequence carries from token to token.  Not in the reference (all of its attention
// is softmax attention, src/NN.jl:343-387).
// Lightning attention is the same recurrence without rotation and key scale, silu on q, k and v, and one norm over all heads' outputs
// together: with `ssq` set the kernels leave y_t = o_t w gate and the heads' sums of o_t^2; whoever multiplies y by the output
// projection applies the norm's scale, one number per token.
#pragma once
#include "common.cuh"

namespace lmb {

// Tokens start[b] .. start[b] + len[b] - 1 of the packed rows are positions pos0[b] .. of sequence b.
struct RetentionView {
  int B = 0;
  const int* start = nullptr;
  const int* len = nullptr;
  const int* pos0 = nullptr;
  int total = 0;                      // packed rows (bounds of the tensor maps)
  int H = 0, dim = 0, vdim = 0;
  int rot_dims = 0;                   // features of q and k still to be rotated, in neighbouring pairs (2i, 2i + 1); 0: rotated already
  const float* inv_freq = nullptr;    // [rot_dims / 2]
  const float* decay = nullptr;       // [H][decay_pitch]: powers 0 .. decay_pitch - 1
  int decay_pitch = 0;
  float eps = 0.f;
  float k_scale = 1.f;
  float* state = nullptr;             // [B][H][dim][round_up(vdim, 4)]
  // rows [T, pitch] of the projections: head a of q at column a * dim and so on;
  // raw_gate: what is still to be applied to g (1: silu, 2: sigmoid); raw_act: q, k and v still lack their silu (token by token only)
  const void *q = nullptr, *k = nullptr, *v = nullptr, *g = nullptr;
  int q_pitch = 0, k_pitch = 0, v_pitch = 0, g_pitch = 0;
  int in_f32 = 1, raw_gate = 1, raw_act = 0;
  const float* out_w = nullptr;       // [H * vdim] (with ssq)
  float* ssq = nullptr;               // token t, head a: ssq[t * ssq_t + a * ssq_h]
  int ssq_t = 0, ssq_h = 0;
  void* out = nullptr;                // model dtype: [T, ldo] row-major, or GEMV activations of padding bp
  int ldo = 0, bp = 0;
};

int32_t retention_configure();
// token after token: decoding, short portions, float32, any sizes
int32_t retention_steps(Ctx* ctx, int dtype, const RetentionView& v, cudaStream_t st);
// chunks of 64 tokens on the tensor cores: bf16 rows, rotated, gated (raw_gate 0), row-major output
bool retention_chunks_ok(const RetentionView& v);
int32_t retention_chunks(Ctx* ctx, const RetentionView& v, cudaStream_t st);
// the same in chunks of 128 tokens with tcgen05 (csrc/retention_tc.cu)
bool retention_tc_ok(const RetentionView& v);
int32_t retention_tc(Ctx* ctx, const RetentionView& v, cudaStream_t st);
int32_t retention_tc_configure();
// angle tables of T tokens: tab[t * n + i] = (cos, sin) of pos[t] * inv_freq[i]
int32_t angle_table(Ctx* ctx, float2* tab, const float* inv_freq, int n, const int* pos, int T, cudaStream_t st);

}  // namespace lmb
