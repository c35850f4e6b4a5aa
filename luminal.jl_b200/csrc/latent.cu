// Kernels of latent attention (see latent.cuh).
#include <math_constants.h>

#include "latent.cuh"
#include "pdl.cuh"

namespace lmb {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kTok = 8;                 // tokens per CTA of the per-head products: one read of a head's matrix serves all of them

__device__ __forceinline__ float block_sum(float v, float* red, int threads) {      // red: [threads / 32]
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < threads / 32; ++i) t += red[i];
  return t;
}

// feature i of a rotated vector u[0 .. dims): pair (lo, hi) of i, the pair's index and which of the two i is
__device__ __forceinline__ void rot_pair(int i, int dims, int interleaved, int* lo, int* hi, int* idx, bool* second) {
  if (interleaved) { *idx = i >> 1; *second = i & 1; *lo = i & ~1; *hi = i | 1; }
  else { const int half = dims >> 1; *second = i >= half; *idx = *second ? i - half : i; *lo = *idx; *hi = *idx + half; }
}
template <typename F>
__device__ __forceinline__ float rotated(F u, int i, int dims, int interleaved, int pos, const float* inv_freq) {
  if (i >= dims) return u(i);
  int lo, hi, idx;
  bool second;
  rot_pair(i, dims, interleaved, &lo, &hi, &idx, &second);
  float s, c;
  sincosf((float)pos * inv_freq[idx], &s, &c);
  return second ? u(hi) * c + u(lo) * s : u(lo) * c - u(hi) * s;
}

template <typename WT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentView v, const float* __restrict__ proj, int pitch, int q0, int kv0,
                                                          const float* __restrict__ q_norm, const float* __restrict__ kv_norm,
                                                          WT* __restrict__ xq, int ldxq, int bp, WT* __restrict__ cache) {
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const float* q = proj + (int64_t)t * pitch + q0;
  float ss = 0.f;
  for (int i = tid; i < v.q_rank; i += 256) ss += q[i] * q[i];
  const float inv = 1.0f / sqrtf(block_sum(ss, red, 256) / (float)v.q_rank + v.eps);
  for (int i = tid; i < v.q_rank; i += 256)
    xq[bp > 0 ? Layout<WT>::x_offset(t, i, bp) : (int64_t)t * ldxq + i] = from_f32<WT>(q[i] * inv * q_norm[i]);
  if (!cache) return;
  const float* kv = proj + (int64_t)t * pitch + kv0;
  ss = 0.f;
  for (int i = tid; i < v.kv_rank; i += 256) ss += kv[i] * kv[i];
  const float kinv = 1.0f / sqrtf(block_sum(ss, red, 256) / (float)v.kv_rank + v.eps);
  const int pos = v.pos[t];
  WT* row = cache + v.seq[t] * v.seq_stride + (int64_t)pos * v.ld;
  for (int i = tid; i < v.kv_rank; i += 256) row[i] = from_f32<WT>(kv[i] * kinv * kv_norm[i]);
  const float* kr = kv + v.kv_rank;
  for (int i = tid; i < v.rot_dim; i += 256)
    row[v.rot + i] = from_f32<WT>(rotated([&](int j) { return kr[j]; }, i, v.rot_dims, v.rot_interleaved, pos, v.inv_freq));
}

// one CTA: head blockIdx.x, tokens kTok * blockIdx.y ..
template <typename WT, typename QT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LatentView v, const QT* __restrict__ q, const WT* __restrict__ w_uk,
                                                            WT* __restrict__ qa) {
  extern __shared__ float qs[];                        // [dim][kTok]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t0 = blockIdx.y * kTok, n = min(kTok, v.T - t0), tid = threadIdx.x;
  const int qd = v.dim + v.rot_dim;
  const int64_t pitch = (int64_t)v.H * qd;
  for (int i = tid; i < v.dim * kTok; i += 256) {
    const int t = i / v.dim, d = i - t * v.dim;
    qs[d * kTok + t] = t < n ? to_f32(q[(t0 + t) * pitch + h * qd + d]) : 0.f;
  }
  for (int i = tid; i < v.rot_dim * n; i += 256) {
    const int t = i / v.rot_dim, d = i - t * v.rot_dim;
    const QT* qr = q + (t0 + t) * pitch + h * qd + v.dim;
    qa[((int64_t)(t0 + t) * v.H + h) * v.ld + v.rot + d] =
        from_f32<WT>(rotated([&](int j) { return to_f32(qr[j]); }, d, v.rot_dims, v.rot_interleaved, v.pos[t0 + t], v.inv_freq));
  }
  __syncthreads();
  for (int r = 2 * tid; r < v.kv_rank; r += 512) {     // two latent columns per thread
    const bool two = r + 1 < v.kv_rank;
    const WT* w = w_uk + (int64_t)h * v.dim * v.kv_rank + r;
    float a0[kTok], a1[kTok];
#pragma unroll
    for (int t = 0; t < kTok; ++t) a0[t] = a1[t] = 0.f;
#pragma unroll 4
    for (int d = 0; d < v.dim; ++d) {
      const float w0 = to_f32(w[(int64_t)d * v.kv_rank]), w1 = two ? to_f32(w[(int64_t)d * v.kv_rank + 1]) : 0.f;
      const float4 x0 = *reinterpret_cast<const float4*>(qs + d * kTok), x1 = *reinterpret_cast<const float4*>(qs + d * kTok + 4);
      const float x[kTok] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
      for (int t = 0; t < kTok; ++t) { a0[t] = fmaf(x[t], w0, a0[t]); a1[t] = fmaf(x[t], w1, a1[t]); }
    }
#pragma unroll
    for (int t = 0; t < kTok; ++t) {
      if (t >= n) continue;
      WT* o = qa + ((int64_t)(t0 + t) * v.H + h) * v.ld + r;
      o[0] = from_f32<WT>(a0[t]);
      if (two) o[1] = from_f32<WT>(a1[t]);
    }
  }
}

// One CTA per (head, token): online softmax over tiles of kSimple keys, any sizes and dtype, CUDA cores.
constexpr int kSimple = 128;
template <typename WT>
__global__ void __launch_bounds__(kSimple) latent_attend_simple_kernel(const LatentView v, const WT* __restrict__ qa, const WT* __restrict__ cache,
                                                                       float* __restrict__ olat) {
  extern __shared__ float sm[];                        // q [ld] | o [kv_rank] | p [kSimple]
  __shared__ float red[kSimple / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  float* qs = sm;
  float* os = sm + v.ld;
  float* ps = os + v.kv_rank;
  const WT* q = qa + ((int64_t)t * v.H + h) * v.ld;
  for (int i = tid; i < v.ld; i += kSimple) qs[i] = to_f32(q[i]);
  for (int i = tid; i < v.kv_rank; i += kSimple) os[i] = 0.f;
  const int n = v.pos[t] + 1;
  const WT* base = cache + v.seq[t] * v.seq_stride;
  float m = -CUDART_INF_F, l = 0.f;
  __syncthreads();
  for (int k0 = 0; k0 < n; k0 += kSimple) {
    const int key = k0 + tid;
    float s = -CUDART_INF_F;
    if (key < n) {
      const WT* row = base + (int64_t)key * v.ld;
      float acc = 0.f;
      for (int i = 0; i < v.kv_rank; ++i) acc = fmaf(qs[i], to_f32(row[i]), acc);
      for (int i = v.rot; i < v.rot + v.rot_dim; ++i) acc = fmaf(qs[i], to_f32(row[i]), acc);
      s = acc * v.scale;
    }
    float mx = s;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
    float mn = m;
    for (int i = 0; i < kSimple / 32; ++i) mn = fmaxf(mn, red[i]);
    const float p = exp2f((s - mn) * kLog2e), alpha = exp2f((m - mn) * kLog2e);
    ps[tid] = p;
    m = mn;
    l = l * alpha + block_sum(p, red, kSimple);        // its barriers also publish ps
    const int cnt = min(kSimple, n - k0);
    for (int r = tid; r < v.kv_rank; r += kSimple) {
      float acc = os[r] * alpha;
      for (int i = 0; i < cnt; ++i) acc = fmaf(ps[i], to_f32(base[(int64_t)(k0 + i) * v.ld + r]), acc);
      os[r] = acc;
    }
    __syncthreads();
  }
  const float inv = 1.0f / l;
  for (int r = tid; r < v.kv_rank; r += kSimple) olat[((int64_t)t * v.H + h) * v.kv_rank + r] = os[r] * inv;
}

// one CTA: head blockIdx.x, tokens kTok * blockIdx.y ..; one warp per value feature, lanes over the latent
template <typename WT>
__global__ void __launch_bounds__(256) latent_expand_kernel(const LatentView v, const float* __restrict__ olat, const WT* __restrict__ w_uv,
                                                            const float* __restrict__ gate, int gate_pitch, WT* __restrict__ out, int ldo,
                                                            int bp) {
  extern __shared__ float xs[];                        // [kTok][kv_rank]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t0 = blockIdx.y * kTok, n = min(kTok, v.T - t0), tid = threadIdx.x, lane = tid & 31;
  const int R = v.kv_rank;
  for (int i = tid; i < kTok * R; i += 256) {
    const int t = i / R;
    xs[i] = t < n ? olat[((int64_t)(t0 + t) * v.H + h) * R + (i - t * R)] : 0.f;
  }
  __syncthreads();
  for (int d = tid >> 5; d < v.vdim; d += 8) {
    const WT* w = w_uv + ((int64_t)h * v.vdim + d) * R;
    float a[kTok];
#pragma unroll
    for (int t = 0; t < kTok; ++t) a[t] = 0.f;
    for (int r = lane; r < R; r += 32) {
      const float wv = to_f32(w[r]);
#pragma unroll
      for (int t = 0; t < kTok; ++t) a[t] = fmaf(xs[t * R + r], wv, a[t]);
    }
#pragma unroll
    for (int t = 0; t < kTok; ++t)
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) a[t] += __shfl_xor_sync(0xffffffffu, a[t], off);
    float mine = 0.f;
#pragma unroll
    for (int t = 0; t < kTok; ++t) mine = lane == t ? a[t] : mine;
    if (lane < n) {
      const int t = t0 + lane, col = h * v.vdim + d;
      const float g = 1.0f / (1.0f + expf(-gate[(int64_t)t * gate_pitch + h]));
      out[bp > 0 ? Layout<WT>::x_offset(t, col, bp) : (int64_t)t * ldo + col] = from_f32<WT>(mine * g);
    }
  }
}

}  // namespace

int32_t latent_configure() { return LMB200_OK; }

int32_t latent_prep(Ctx* ctx, int dtype, const LatentView& v, const float* proj, int pitch, int q0, int kv0, const float* q_norm,
                    const float* kv_norm, void* xq, int ldxq, int bp, void* cache, cudaStream_t st) {
  if (dtype == LMB200_BF16)
    LMB_CUDA(launch_k(latent_prep_kernel<__nv_bfloat16>, dim3(v.T), dim3(256), 0, st, v, proj, pitch, q0, kv0, q_norm, kv_norm,
                      (__nv_bfloat16*)xq, ldxq, bp, (__nv_bfloat16*)cache));
  else
    LMB_CUDA(launch_k(latent_prep_kernel<float>, dim3(v.T), dim3(256), 0, st, v, proj, pitch, q0, kv0, q_norm, kv_norm, (float*)xq, ldxq, bp,
                      (float*)cache));
  ctx->launches++;
  return LMB200_OK;
}

int32_t latent_absorb(Ctx* ctx, int dtype, const LatentView& v, const void* q, int q_f32, const void* w_uk, void* qa, cudaStream_t st) {
  const dim3 grid((unsigned)v.H, (unsigned)ceil_div(v.T, kTok));
  const size_t smem = (size_t)v.dim * kTok * 4;
  LMB_REQUIRE(smem <= 48 * 1024 && grid.y <= 65535, "latent attention: head width %d, %d tokens", v.dim, v.T);
  if (dtype != LMB200_BF16)
    LMB_CUDA(launch_k(latent_absorb_kernel<float, float>, grid, dim3(256), smem, st, v, (const float*)q, (const float*)w_uk, (float*)qa));
  else if (q_f32)
    LMB_CUDA(launch_k(latent_absorb_kernel<__nv_bfloat16, float>, grid, dim3(256), smem, st, v, (const float*)q, (const __nv_bfloat16*)w_uk,
                      (__nv_bfloat16*)qa));
  else
    LMB_CUDA(launch_k(latent_absorb_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), smem, st, v, (const __nv_bfloat16*)q,
                      (const __nv_bfloat16*)w_uk, (__nv_bfloat16*)qa));
  ctx->launches++;
  return LMB200_OK;
}

LatentAttnPlan latent_attn_plan(const Ctx* ctx, int dtype, int T, int H, int kv_rank, int ctx_len) {
  (void)ctx; (void)dtype; (void)T; (void)H; (void)kv_rank; (void)ctx_len;
  return LatentAttnPlan();
}

int32_t latent_attend(Ctx* ctx, int dtype, const LatentView& v, const void* qa, const void* cache, const LatentAttnPlan& plan, float* part,
                      unsigned* counters, float* olat, cudaStream_t st) {
  (void)plan; (void)part; (void)counters;
  const size_t smem = (size_t)(v.ld + v.kv_rank + kSimple) * 4;
  LMB_REQUIRE(smem <= 48 * 1024, "latent attention: latent width %d", v.kv_rank);
  LMB_REQUIRE(v.T <= 65535, "latent attention: %d tokens in one absorbed launch", v.T);
  const dim3 grid((unsigned)v.H, (unsigned)v.T);
  if (dtype == LMB200_BF16)
    LMB_CUDA(launch_k(latent_attend_simple_kernel<__nv_bfloat16>, grid, dim3(kSimple), smem, st, v, (const __nv_bfloat16*)qa,
                      (const __nv_bfloat16*)cache, olat));
  else
    LMB_CUDA(launch_k(latent_attend_simple_kernel<float>, grid, dim3(kSimple), smem, st, v, (const float*)qa, (const float*)cache, olat));
  ctx->launches++;
  return LMB200_OK;
}

int32_t latent_expand(Ctx* ctx, int dtype, const LatentView& v, const float* olat, const void* w_uv, const float* gate, int gate_pitch,
                      void* out, int ldo, int bp, cudaStream_t st) {
  const dim3 grid((unsigned)v.H, (unsigned)ceil_div(v.T, kTok));
  const size_t smem = (size_t)kTok * v.kv_rank * 4;
  LMB_REQUIRE(smem <= 48 * 1024 && grid.y <= 65535, "latent attention: latent width %d, %d tokens", v.kv_rank, v.T);
  if (dtype == LMB200_BF16)
    LMB_CUDA(launch_k(latent_expand_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, v, olat, (const __nv_bfloat16*)w_uv, gate, gate_pitch,
                      (__nv_bfloat16*)out, ldo, bp));
  else
    LMB_CUDA(launch_k(latent_expand_kernel<float>, grid, dim3(256), smem, st, v, olat, (const float*)w_uv, gate, gate_pitch, (float*)out, ldo, bp));
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
