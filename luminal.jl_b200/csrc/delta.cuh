// Gated delta rule with one decay per key channel.  Per head, over a float32 state S [dim, vdim] that a sequence carries along:
//   S <- diag(g_t) S;   S <- S + k_t (beta_t (v_t - S^T k_t))^T;   o_t = S^T q_t;   y_t = o_t / rms(o_t) * w * gate_t
// with q, k, v after a causal convolution over time and silu, q and k unit vectors (q also divided by sqrt(dim)),
// g = exp(-exp(A) softplus(decay + bias)) and beta a sigmoid.  Query / key heads may serve several value heads.
// Not in the reference (all of its attention is softmax attention, src/NN.jl:343-387).
#pragma once
#include "common.cuh"

namespace lmb {

// Tokens start[b] .. start[b] + len[b] - 1 of the packed rows are positions pos0[b] .. of sequence b.
struct DeltaView {
  int B = 0;
  const int *start = nullptr, *len = nullptr, *pos0 = nullptr;
  int total = 0;                                   // packed rows
  const int *seq = nullptr, *pos = nullptr;        // of every packed row (delta_conv)
  int H = 0, G = 0, dim = 0, vdim = 0, taps = 0;   // value heads, query / key heads (head h uses h / (H / G))
  float eps = 0.f;
  float* state = nullptr;                          // [B][H][dim][round_up(vdim, 4)]
  float* ring = nullptr;                           // [B][taps][channels]: raw input of position p in slot p % taps; channels q | k | v
  const float* conv = nullptr;                     // [taps][channels], tap 0 meets the current token
  const float *a_log = nullptr, *dt_bias = nullptr, *norm = nullptr;       // [H], [H * dim], [vdim]
  // rows of the projections, head a of q at column a * dim and so on
  const void *q = nullptr, *k = nullptr, *v = nullptr;
  int q_pitch = 0, k_pitch = 0, v_pitch = 0;
  const float* b = nullptr;                        // [.., H] before the sigmoid
  int b_pitch = 0;
  // raw: q, k, v are float32 inputs of the convolution, `decay` is before bias and softplus, `gate` float32 before its sigmoid; one token per
  // sequence.  Otherwise: q, k, v in the model dtype after silu, scales rq, rk [.., G] (1 / |q| / sqrt(dim), 1 / |k|), `decay` the logarithm of g,
  // `gate` in the model dtype after its sigmoid.
  int raw = 0;
  const float *rq = nullptr, *rk = nullptr;
  const float* decay = nullptr;                    // [.., H * dim]
  int decay_pitch = 0;
  const void* gate = nullptr;                      // [.., H * vdim]
  int gate_pitch = 0;
  void* out = nullptr;                             // model dtype: [T, ldo] row-major, or GEMV activations of padding bp
  int ldo = 0, bp = 0;
};

int32_t delta_configure();
// convolution, silu and head lengths of packed rows: out [T, channels] in the model dtype, rq and rk [T, G]; then the ring
int32_t delta_conv(Ctx* ctx, int dtype, const DeltaView& v, void* out, float* rq, float* rk, cudaStream_t st);
// token after token: decoding, short portions, float32
int32_t delta_steps(Ctx* ctx, int dtype, const DeltaView& v, cudaStream_t st);
// chunks of 64 tokens on the tensor cores (csrc/delta_chunk.cu): bf16 prepared rows, heads up to 128 wide
bool delta_chunks_ok(const DeltaView& v);
int32_t delta_chunks(Ctx* ctx, const DeltaView& v, cudaStream_t st);
int32_t delta_chunk_configure();
// the same with tcgen05 (csrc/delta_tc.cu), for heads wider than 64
bool delta_tc_ok(const DeltaView& v);
int32_t delta_tc(Ctx* ctx, const DeltaView& v, cudaStream_t st);
int32_t delta_tc_configure();

}  // namespace lmb
