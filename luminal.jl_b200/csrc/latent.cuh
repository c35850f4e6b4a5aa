// Latent attention: every token caches one latent row c [kv_rank] and one rotated key part [rot_dim] that all heads share;
// head a's keys and values are Wuk_a c and Wuv_a c.  Two ways to attend:
//   absorbed  q'_a = Wuk_a^T q_a is compared with the latents themselves and the weighted latents go through Wuv_a after the
//             softmax: the cache is read once for all heads.  One new token per sequence, short portions, float32.
//   expanded  the context's keys and values are multiplied out by one GEMM and attended by the tensor-core flash kernel
//             (csrc/flash_tc.cu): long portions.
// Nothing like it in the reference, whose attention caches keys and values per head (src/NN.jl:343-387).
#pragma once
#include "common.cuh"

namespace lmb {

// T tokens: token t is position pos[t] of sequence seq[t]
struct LatentView {
  int T = 0;
  const int* seq = nullptr;
  const int* pos = nullptr;
  int H = 0, dim = 0, vdim = 0, q_rank = 0, kv_rank = 0, rot_dim = 0, rot_dims = 0, rot_interleaved = 1;
  int q_rotated = 0;                // latent_absorb: the queries' positional parts are rotated already
  int rot = 0, ld = 0;              // cache row: latent from 0, rotated part from `rot`, `ld` elements (the gaps are zero)
  int64_t seq_stride = 0;           // cache elements per sequence
  const float* inv_freq = nullptr;  // [rot_dims / 2]
  float scale = 1.f, eps = 0.f;
};

int32_t latent_configure();

// proj [T, pitch] float32 holds the projections of one layer: the query latent from column q0 and, if cache != NULL, latent and
// key part from column kv0.  xq <- RMSNorm(query latent) in the model dtype, row-major [T, ldxq] or, bp > 0, a GEMV activation
// buffer of that padding; the normed latent and the rotated key part go to the cache rows of the tokens and, if packed != NULL,
// also to row t of packed [T, ld].
int32_t latent_prep(Ctx* ctx, int dtype, const LatentView& v, const float* proj, int pitch, int q0, int kv0, const float* q_norm,
                    const float* kv_norm, void* xq, int ldxq, int bp, void* cache, void* packed, cudaStream_t st);
// q [T, H * (dim + rot_dim)] (float32 if q_f32, else the model dtype) -> qa [T, H, ld] in the model dtype, ordered like a cache
// row: the absorbed part and the rotated part
// (w_ukt: W_uk with every head transposed, [H, kv_rank, dim])
int32_t latent_absorb(Ctx* ctx, int dtype, const LatentView& v, const void* q, int q_f32, const void* w_ukt, void* qa, cudaStream_t st);
// softmax over positions 0 .. pos[t] of the token's sequence: the weighted latents, as partial results per share of the keys (nsplit >= 1)
// or whole (nsplit 0, the CUDA-core kernel); part holds plan.part_floats
struct LatentAttnPlan { int nsplit = 0; int64_t part_floats = 0; };
LatentAttnPlan latent_attn_plan(const Ctx* ctx, int dtype, const LatentView& v, int T, int ctx_len);
int32_t latent_attend(Ctx* ctx, int dtype, const LatentView& v, const void* qa, const void* cache, const LatentAttnPlan& plan, float* part, cudaStream_t st);
// out[t, a * vdim + i] = sigmoid(gate[t, a]) (Wuv_a olat[t, a])_i in the model dtype, row-major [T, ldo] or GEMV activations (bp > 0)
int32_t latent_expand(Ctx* ctx, int dtype, const LatentView& v, const float* part, const LatentAttnPlan& plan, const void* w_uv, const float* gate,
                      int gate_pitch, void* out, int ldo, int bp, cudaStream_t st);
// rotates the positional part of q [T, H * (dim + rot_dim)] in place (bf16; where the projection's epilogue could not)
int32_t latent_rotate_q(Ctx* ctx, const LatentView& v, void* q, cudaStream_t st);

}  // namespace lmb
