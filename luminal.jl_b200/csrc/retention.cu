// Kernels of retention (see retention.cuh).
#include "pdl.cuh"
#include "retention.cuh"

namespace lmb {
namespace {

constexpr int kStepThreads = 128;

// One CTA per (head, sequence).  Thread (c, w): four value columns 4 c .., rows w, w + W, ... of the state, where W = threads / column
// groups; a thread owns its elements of the state for all tokens, so only q, k, v and the partial outputs go through shared memory.
template <typename IT, typename OT>
__global__ void __launch_bounds__(kStepThreads) retention_step_kernel(const RetentionView v) {
  extern __shared__ float sm[];
  __shared__ float red[kStepThreads / 32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int D = v.dim, V = v.vdim, V4 = (V + 3) >> 2;         // state rows are V4 float4s
  const int cols = min(V4, kStepThreads), W = kStepThreads / cols;
  float* qs = sm;                      // [D]
  float* ks = qs + ((D + 3) & ~3);     // [D]
  float* vs = ks + ((D + 3) & ~3);     // [4 V4]
  float* os = vs + 4 * V4;             // [W][4 V4]
  pdl_launch_dependents();
  pdl_wait();
  const int n = v.len[b], t0 = v.start[b], p0 = v.pos0[b];
  if (n <= 0) return;
  const float decay = v.decay[h * v.decay_pitch + 1];
  const float kscale = 1.0f / sqrtf((float)D);
  float4* S = reinterpret_cast<float4*>(v.state) + ((int64_t)b * v.H + h) * D * V4;
  const int c0 = tid % cols, w = tid / cols;
  for (int i = 0; i < n; ++i) {
    const int64_t t = t0 + i;
    const IT* q = reinterpret_cast<const IT*>(v.q) + t * v.q_pitch + h * D;
    const IT* k = reinterpret_cast<const IT*>(v.k) + t * v.k_pitch + h * D;
    const IT* vv = reinterpret_cast<const IT*>(v.v) + t * v.v_pitch + h * V;
    for (int d = tid; d < D; d += kStepThreads) {
      float qv = to_f32(q[d]), kv = to_f32(k[d]);
      if (d < v.rot_dims) {
        const int half = v.rot_dims >> 1;
        const int idx = v.rot_interleaved ? d >> 1 : (d < half ? d : d - half);
        const bool second = v.rot_interleaved ? (d & 1) : d >= half;
        const int other = v.rot_interleaved ? (d ^ 1) : (second ? d - half : d + half);
        float s, c;
        sincosf((float)(p0 + i) * v.inv_freq[idx], &s, &c);
        if (!second) s = -s;
        qv = qv * c + to_f32(q[other]) * s;
        kv = kv * c + to_f32(k[other]) * s;
      }
      qs[d] = qv;
      ks[d] = kv * kscale;
    }
    for (int d = tid; d < 4 * V4; d += kStepThreads) vs[d] = d < V ? to_f32(vv[d]) : 0.f;
    __syncthreads();
    if (w < W) {
      for (int c = c0; c < V4; c += cols) {
        const float4 vc = *reinterpret_cast<const float4*>(vs + 4 * c);
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int d = w; d < D; d += W) {
          float4 s = S[(int64_t)d * V4 + c];
          const float kd = ks[d], qd = qs[d];
          s.x = fmaf(kd, vc.x, decay * s.x); s.y = fmaf(kd, vc.y, decay * s.y);
          s.z = fmaf(kd, vc.z, decay * s.z); s.w = fmaf(kd, vc.w, decay * s.w);
          S[(int64_t)d * V4 + c] = s;
          o.x = fmaf(qd, s.x, o.x); o.y = fmaf(qd, s.y, o.y); o.z = fmaf(qd, s.z, o.z); o.w = fmaf(qd, s.w, o.w);
        }
        *reinterpret_cast<float4*>(os + w * 4 * V4 + 4 * c) = o;
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < V; d += kStepThreads) {
      float o = 0.f;
      for (int j = 0; j < W; ++j) o += os[j * 4 * V4 + d];
      vs[d] = o;                       // this token's v is used up
      ss += o * o;
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int j = 0; j < kStepThreads / 32; ++j) tot += red[j];
    const float inv = 1.0f / sqrtf(tot / (float)V + v.eps);
    const IT* g = reinterpret_cast<const IT*>(v.g) + t * v.g_pitch + h * V;
    OT* out = reinterpret_cast<OT*>(v.out);
    for (int d = tid; d < V; d += kStepThreads) {
      float gv = to_f32(g[d]);
      if (v.raw_gate) gv = gv / (1.0f + expf(-gv));
      const int col = h * V + d;
      out[v.bp > 0 ? Layout<OT>::x_offset((int)t, col, v.bp) : t * v.ldo + col] = from_f32<OT>(vs[d] * inv * gv);
    }
    __syncthreads();                   // vs, red and os are rewritten by the next token
  }
}

size_t step_smem(const RetentionView& v) {
  const int V4 = (v.vdim + 3) >> 2, cols = V4 < kStepThreads ? V4 : kStepThreads, W = kStepThreads / cols;
  return (size_t)(2 * ((v.dim + 3) & ~3) + 4 * V4 + W * 4 * V4) * 4;
}

}  // namespace

int32_t retention_configure() { return LMB200_OK; }

int32_t retention_steps(Ctx* ctx, int dtype, const RetentionView& v, cudaStream_t st) {
  const size_t smem = step_smem(v);
  LMB_REQUIRE(smem <= 48 * 1024, "retention: heads of %d x %d", v.dim, v.vdim);
  const dim3 grid((unsigned)v.H, (unsigned)v.B);
  if (dtype != LMB200_BF16) {
    LMB_REQUIRE(v.in_f32, "retention: float32 models have float32 projections");
    LMB_CUDA(launch_k(retention_step_kernel<float, float>, grid, dim3(kStepThreads), smem, st, v));
  } else if (v.in_f32) {
    LMB_CUDA(launch_k(retention_step_kernel<float, __nv_bfloat16>, grid, dim3(kStepThreads), smem, st, v));
  } else {
    LMB_CUDA(launch_k(retention_step_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(kStepThreads), smem, st, v));
  }
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
