// Grouped-query attention over the last `window` positions with rotated, root-mean-square-normed queries and keys and bounded
// scores.  Keys and values are cached row-major per head, as they enter the products: keys after rotation and norm.
//   q, k <- rms over the head of the rotated rows;  s = cap tanh(scale q . k / cap);  softmax over the visible keys
// The reference's attention has none of these (src/NN.jl:343-387); long portions run the flash kernel (csrc/flash_tc.cu).
#pragma once
#include "common.cuh"

namespace lmb {

// T tokens: token t is position pos[t] of sequence seq[t]
struct WindowView {
  int T = 0;
  const int* seq = nullptr;
  const int* pos = nullptr;
  int H = 0, G = 0, dim = 0, vdim = 0;      // query heads, key / value heads (query head h reads h / (H / G))
  int k_ld = 0, v_ld = 0, cap = 0;          // cache rows [sequence][G][cap][ld], zero behind the width
  void *keys = nullptr, *values = nullptr;
  int rot_dims = 0, rot_interleaved = 1;
  const float* inv_freq = nullptr;          // [rot_dims / 2]
  const float2* angles = nullptr;           // [T][rot_dims / 2] (cos, sin), or NULL: computed
  float rot_scale = 1.f;                    // factor of cosine and sine
  float scale = 1.f, score_cap = 0.f, eps = 0.f;
  int window = 0;                           // 0: all earlier positions
};

// rows of the projections: head a of q at column a * dim and so on; k == NULL: another layer's keys and values are read
struct WindowRows {
  const void *q = nullptr, *k = nullptr, *v = nullptr;
  int q_pitch = 0, k_pitch = 0, v_pitch = 0;
  int in_f32 = 0;
};

int32_t window_configure();
// q_out [T, H * dim] in the model dtype <- rotated, normed queries (may be the input rows); keys and values to the tokens' cache rows
int32_t window_prep(Ctx* ctx, int dtype, const WindowView& v, const WindowRows& in, void* q_out, cudaStream_t st);

struct WindowPlan { int nsplit = 0; int64_t part_floats = 0; int n_counters = 0; };      // nsplit 0: the CUDA-core kernel
// T tokens that look at no more than ctx_len positions
WindowPlan window_plan(const Ctx* ctx, int dtype, const WindowView& v, int T, int ctx_len);
// out[t, a * vdim + i]: row-major [T, ldo] or GEMV activations of padding bp.  in.in_f32 with a tensor-core plan: the kernel does
// window_prep's work itself (one token per sequence); otherwise in.q are prepared queries.  counters: zero between launches
int32_t window_attend(Ctx* ctx, int dtype, const WindowView& v, const WindowRows& in, const WindowPlan& plan, float* part, unsigned* counters, void* out,
                      int ldo, int bp, cudaStream_t st);

}  // namespace lmb
