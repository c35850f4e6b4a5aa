// Kernels of latent attention (see latent.cuh).
#include <math_constants.h>

#include <algorithm>

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
                                                          WT* __restrict__ xq, int ldxq, int bp, WT* __restrict__ cache,
                                                          WT* __restrict__ packed) {
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
  WT* row2 = packed ? packed + (int64_t)t * v.ld : nullptr;
  for (int i = tid; i < v.kv_rank; i += 256) {
    const WT c = from_f32<WT>(kv[i] * kinv * kv_norm[i]);
    row[i] = c;
    if (row2) row2[i] = c;
  }
  const float* kr = kv + v.kv_rank;
  for (int i = tid; i < v.rot_dim; i += 256) {
    const WT c = from_f32<WT>(rotated([&](int j) { return kr[j]; }, i, v.rot_dims, v.rot_interleaved, pos, v.inv_freq));
    row[v.rot + i] = c;
    if (row2) row2[v.rot + i] = c;
  }
}

// the positional part of every head's query, in place: one CTA per token, a thread per (head, pair)
__global__ void __launch_bounds__(128) latent_rotate_q_kernel(const LatentView v, __nv_bfloat16* __restrict__ q) {
  extern __shared__ float2 cs[];                       // [rot_dims / 2] cosine, sine
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, half = v.rot_dims >> 1, qd = v.dim + v.rot_dim;
  for (int i = threadIdx.x; i < half; i += 128) {
    float s, c;
    sincosf((float)v.pos[t] * v.inv_freq[i], &s, &c);
    cs[i] = make_float2(c, s);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < v.H * half; i += 128) {
    const int h = i / half, p = i - h * half;
    __nv_bfloat16* r = q + ((int64_t)t * v.H + h) * qd + v.dim;
    const int lo = v.rot_interleaved ? 2 * p : p, hi = v.rot_interleaved ? 2 * p + 1 : p + half;
    const float a = __bfloat162float(r[lo]), b = __bfloat162float(r[hi]);
    r[lo] = __float2bfloat16_rn(a * cs[p].x - b * cs[p].y);
    r[hi] = __float2bfloat16_rn(b * cs[p].x + a * cs[p].y);
  }
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
        from_f32<WT>(rotated([&](int j) { return to_f32(qr[j]); }, d, v.q_rotated ? 0 : v.rot_dims, v.rot_interleaved, v.pos[t0 + t], v.inv_freq));
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

// ---------------------------------------------------------------------------------------------
// bf16 absorbed attention, split over the keys.  One CTA = 8 warps: the 16 MT heads of one group of one token against `keys_per_cta`
// keys in tiles of 64.  The latent rows of a tile arrive once (cp.async, two stages, row pitch an odd number of 16-byte chunks) and serve
// as keys (S = Q' C^T, 16 keys x 16 heads per warp) and as values (O += P C, every warp a slice of the latent's columns); the scores and
// the running softmax stay float32.  Splits are merged by the last CTA of a (token, head group) to finish, in split order.
// ---------------------------------------------------------------------------------------------
constexpr int kLatThreads = 256, kLatKeys = 64, kLatStages = 2;
constexpr int kScorePitch = kLatKeys + 4, kProbPitch = kLatKeys + 8;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LatTile {                        // shared-memory shape of a row: latent padded to R16, rotated part padded to P16
  int R16, P16, pitch;                  // pitch in elements
};
__host__ __device__ inline LatTile lat_tile(int kv_rank, int rot_dim) {
  LatTile t;
  t.R16 = (kv_rank + 15) & ~15;
  t.P16 = (rot_dim + 15) & ~15;
  t.pitch = t.R16 + t.P16 + 8;
  return t;
}
size_t lat_smem(int MT, int kv_rank, int rot_dim) {
  const LatTile t = lat_tile(kv_rank, rot_dim);
  return (size_t)(kLatStages * kLatKeys + MT * 16) * t.pitch * 2 + (size_t)2 * 16 * kScorePitch * 4 + (size_t)MT * 16 * kProbPitch * 2 +
         (size_t)MT * 16 * 3 * 4;
}

__device__ __forceinline__ int lat_keys_per_cta(int n, int nsplit) { return (((n + nsplit - 1) / nsplit + kLatKeys - 1) / kLatKeys) * kLatKeys; }

template <int NT, int MT>
__global__ void __launch_bounds__(kLatThreads, 1) latent_attend_tc_kernel(const LatentView v, const __nv_bfloat16* __restrict__ qa,
                                                                          const __nv_bfloat16* __restrict__ cache, int nsplit, float* __restrict__ part,
                                                                          unsigned* __restrict__ counters, float* __restrict__ olat) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ int is_last;
  const LatTile L = lat_tile(v.kv_rank, v.rot_dim);
  constexpr int M = MT * 16;
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(sm_raw);                    // [stage][key][pitch]
  __nv_bfloat16* sQ = sK + kLatStages * kLatKeys * L.pitch;                        // [M][pitch]
  float* sS = reinterpret_cast<float*>(sQ + M * L.pitch);                          // [2][16][kScorePitch]: head tiles (MT 2) or halves of the features (MT 1)
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(sS + 2 * 16 * kScorePitch); // [M][kProbPitch]
  float* sA = reinterpret_cast<float*>(sP + M * kProbPitch);                       // [M] rescale, [M] max, [M] sum
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int groups = (v.H + M - 1) / M;
  const int t = blockIdx.x / groups, hg = blockIdx.x - t * groups;
  pdl_launch_dependents();
  pdl_wait();
  const int n = v.pos[t] + 1;
  const int kpc = lat_keys_per_cta(n, nsplit);
  const int k_begin = blockIdx.y * kpc, k_end = min(n, k_begin + kpc);
  if (k_begin >= n) return;
  const int tiles = (k_end - k_begin + kLatKeys - 1) / kLatKeys;
  const __nv_bfloat16* base = cache + v.seq[t] * v.seq_stride;
  const int chunks = v.ld >> 3, c_chunks = v.rot >> 3;

  auto load_tile = [&](int j) {
    __nv_bfloat16* dst = sK + (j & 1) * kLatKeys * L.pitch;
    const int key0 = k_begin + j * kLatKeys;
    for (int i = tid; i < kLatKeys * chunks; i += kLatThreads) {
      const int key = i / chunks, c = i - key * chunks;
      const int col = c < c_chunks ? c * 8 : L.R16 + (c - c_chunks) * 8;
      const bool ok = key0 + key < k_end;
      const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst + key * L.pitch + col);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(base + (int64_t)(ok ? key0 + key : k_begin) * v.ld + c * 8),
                   "r"(ok ? 16 : 0)
                   : "memory");
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  // the padding between and behind the parts is never written by a copy: zero it once
  for (int i = tid; i < (kLatStages * kLatKeys + M) * L.pitch / 8; i += kLatThreads) reinterpret_cast<uint4*>(sm_raw)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  load_tile(0);
  if (tiles > 1) load_tile(1);
  for (int i = tid; i < M * chunks; i += kLatThreads) {
    const int h = i / chunks, c = i - h * chunks;
    const int col = c < c_chunks ? c * 8 : L.R16 + (c - c_chunks) * 8;
    if (hg * M + h < v.H)
      *reinterpret_cast<uint4*>(sQ + h * L.pitch + col) = *reinterpret_cast<const uint4*>(qa + ((int64_t)t * v.H + hg * M + h) * v.ld + c * 8);
  }

  const int KS = (L.R16 + L.P16) >> 4;                 // 16-feature steps of the scores
  const int half = warp & 1, kg = warp >> 1;           // MT 2: head tile; MT 1: which half of the steps
  const int ks0 = MT == 2 ? 0 : (half ? (KS + 1) / 2 : 0), ks1 = MT == 2 ? KS : (half ? KS : (KS + 1) / 2);
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
  constexpr int TPR = kLatThreads / M, KPT = kLatKeys / TPR;        // softmax: threads per head, keys per thread
  const int srow = tid / TPR, spart = tid % TPR;
  const float cs = v.scale * kLog2e;
  float m_run = -CUDART_INF_F, l_run = 0.f;
  const uint32_t qaddr = (uint32_t)__cvta_generic_to_shared(sQ + ((MT == 2 ? half * 16 : 0) + (lane & 15)) * L.pitch + (lane >> 4) * 8);
  const int col0 = warp * NT * 8;                      // this warp's slice of the latent's columns

  for (int j = 0; j < tiles; ++j) {
    if (j + 1 < tiles) asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    else asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    const __nv_bfloat16* K = sK + (j & 1) * kLatKeys * L.pitch;
    {
      float s0[2][4], s1[2][4];                        // even and odd steps, two 8-key tiles
#pragma unroll
      for (int i = 0; i < 4; ++i) s0[0][i] = s0[1][i] = s1[0][i] = s1[1][i] = 0.f;
      const uint32_t kaddr = (uint32_t)__cvta_generic_to_shared(K + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * L.pitch + ((lane >> 3) & 1) * 8);
      int ks = ks0;
#pragma unroll 2
      for (; ks + 1 < ks1; ks += 2) {
        uint32_t a[4], b[4], a2[4], b2[4];
        ldsm4(a, qaddr + ks * 32);
        ldsm4(b, kaddr + ks * 32);
        ldsm4(a2, qaddr + ks * 32 + 32);
        ldsm4(b2, kaddr + ks * 32 + 32);
        mma16816(s0[0], a, b[0], b[1]);
        mma16816(s0[1], a, b[2], b[3]);
        mma16816(s1[0], a2, b2[0], b2[1]);
        mma16816(s1[1], a2, b2[2], b2[3]);
      }
      if (ks < ks1) {
        uint32_t a[4], b[4];
        ldsm4(a, qaddr + ks * 32);
        ldsm4(b, kaddr + ks * 32);
        mma16816(s0[0], a, b[0], b[1]);
        mma16816(s0[1], a, b[2], b[3]);
      }
      float* o = sS + half * 16 * kScorePitch + (lane >> 2) * kScorePitch + kg * 16 + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        *reinterpret_cast<float2*>(o + i * 8) = make_float2(s0[i][0] + s1[i][0], s0[i][1] + s1[i][1]);
        *reinterpret_cast<float2*>(o + 8 * kScorePitch + i * 8) = make_float2(s0[i][2] + s1[i][2], s0[i][3] + s1[i][3]);
      }
    }
    __syncthreads();
    {
      float s[KPT];
      float mx = -CUDART_INF_F;
      const int key0 = k_begin + j * kLatKeys + spart * KPT;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        float x = sS[srow * kScorePitch + spart * KPT + i];
        if (MT == 1) x += sS[16 * kScorePitch + srow * kScorePitch + spart * KPT + i];
        s[i] = key0 + i < k_end ? x * cs : -CUDART_INF_F;
        mx = fmaxf(mx, s[i]);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float mn = fmaxf(m_run, mx);               // finite: every tile holds at least one key
      const float alpha = exp2f(m_run - mn);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float p0 = exp2f(s[i] - mn), p1 = exp2f(s[i + 1] - mn);
        sum += p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(sP + srow * kProbPitch + spart * KPT + i) = __floats2bfloat162_rn(p0, p1);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l_run = l_run * alpha + sum;
      m_run = mn;
      if (spart == 0) sA[srow] = alpha;
    }
    __syncthreads();
    if (col0 < L.R16) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = sA[m * 16 + (lane >> 2)], a1 = sA[m * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i) { acc[m][i][0] *= a0; acc[m][i][1] *= a0; acc[m][i][2] *= a1; acc[m][i][3] *= a1; }
      }
#pragma unroll
      for (int ks = 0; ks < kLatKeys / 16; ++ks) {
        uint32_t p[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          ldsm4(p[m], (uint32_t)__cvta_generic_to_shared(sP + (m * 16 + (lane & 15)) * kProbPitch + ks * 16 + (lane >> 4) * 8));
        const uint32_t vaddr = (uint32_t)__cvta_generic_to_shared(K + (ks * 16 + (lane & 15)) * L.pitch + col0 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
          if (col0 + i * 8 >= L.R16) break;
          uint32_t b[4];
          ldsm4_trans(b, vaddr + i * 16);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma16816(acc[m][i], p[m], b[0], b[1]);
            mma16816(acc[m][i + 1], p[m], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                                   // the stage is free
    if (j + 2 < tiles) load_tile(j + 2);
  }
  if (spart == 0) { sA[M + srow] = m_run; sA[2 * M + srow] = l_run; }
  __syncthreads();
  const int R = v.kv_rank;
  const int nvalid = (n + kpc - 1) / kpc;
  auto each = [&](auto f) {                            // f(head row, column, value) of this thread's accumulators
    if (col0 >= L.R16) return;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int row = m * 16 + (lane >> 2) + (e >> 1) * 8, col = col0 + i * 8 + (lane & 3) * 2 + (e & 1);
          if (col < R && hg * M + row < v.H) f(row, col, acc[m][i][e]);
        }
  };
  if (nvalid == 1) {
    each([&](int row, int col, float x) { olat[((int64_t)t * v.H + hg * M + row) * R + col] = x / sA[2 * M + row]; });
    return;
  }
  const int64_t slot_floats = (int64_t)M * (R + 2);
  float* mine = part + ((int64_t)blockIdx.x * nsplit + blockIdx.y) * slot_floats;
  each([&](int row, int col, float x) { mine[(int64_t)row * R + col] = x; });
  if (tid < M) { mine[(int64_t)M * R + tid] = sA[M + tid]; mine[(int64_t)M * R + M + tid] = sA[2 * M + tid]; }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const unsigned prev = atomicAdd(&counters[blockIdx.x], 1u);
    is_last = prev == (unsigned)nvalid - 1u;
    if (is_last) counters[blockIdx.x] = 0u;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  const float* p0 = part + (int64_t)blockIdx.x * nsplit * slot_floats;
  float* wgt = sS;                                     // [M]: 1 / denominator, then the weights split by split
  if (tid < M) {
    float mx = -CUDART_INF_F, den = 0.f;
    for (int i = 0; i < nvalid; ++i) mx = fmaxf(mx, __ldcg(p0 + i * slot_floats + (int64_t)M * R + tid));
    for (int i = 0; i < nvalid; ++i)
      den += exp2f(__ldcg(p0 + i * slot_floats + (int64_t)M * R + tid) - mx) * __ldcg(p0 + i * slot_floats + (int64_t)M * R + M + tid);
    wgt[tid] = mx;
    wgt[M + tid] = 1.0f / den;
  }
  __syncthreads();
  for (int i = tid; i < M * R; i += kLatThreads) {
    const int row = i / R, col = i - row * R;
    if (hg * M + row >= v.H) continue;
    const float mx = wgt[row], inv = wgt[M + row];
    float x = 0.f;
#pragma unroll 4
    for (int k = 0; k < nvalid; ++k) x += exp2f(__ldcg(p0 + k * slot_floats + (int64_t)M * R + row) - mx) * __ldcg(p0 + k * slot_floats + i);
    olat[((int64_t)t * v.H + hg * M + row) * R + col] = x * inv;
  }
}

bool lat_tc_ok(int kv_rank, int rot_dim) { return kv_rank <= 512 && lat_smem(2, kv_rank, rot_dim) <= 220 * 1024; }
int lat_mt(int H) { return H > 16 ? 2 : 1; }
int lat_nt(int kv_rank) { return kv_rank <= 128 ? 2 : (kv_rank <= 256 ? 4 : 8); }

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

int32_t latent_configure() {
#define LMB_CFG(NT)                                                                                                                  \
  LMB_CUDA(cudaFuncSetAttribute(latent_attend_tc_kernel<NT, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));           \
  LMB_CUDA(cudaFuncSetAttribute(latent_attend_tc_kernel<NT, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024))
  LMB_CFG(2);
  LMB_CFG(4);
  LMB_CFG(8);
#undef LMB_CFG
  return LMB200_OK;
}

int32_t latent_prep(Ctx* ctx, int dtype, const LatentView& v, const float* proj, int pitch, int q0, int kv0, const float* q_norm,
                    const float* kv_norm, void* xq, int ldxq, int bp, void* cache, void* packed, cudaStream_t st) {
  if (dtype == LMB200_BF16)
    LMB_CUDA(launch_k(latent_prep_kernel<__nv_bfloat16>, dim3(v.T), dim3(256), 0, st, v, proj, pitch, q0, kv0, q_norm, kv_norm,
                      (__nv_bfloat16*)xq, ldxq, bp, (__nv_bfloat16*)cache, (__nv_bfloat16*)packed));
  else
    LMB_CUDA(launch_k(latent_prep_kernel<float>, dim3(v.T), dim3(256), 0, st, v, proj, pitch, q0, kv0, q_norm, kv_norm, (float*)xq, ldxq, bp,
                      (float*)cache, (float*)packed));
  ctx->launches++;
  return LMB200_OK;
}

int32_t latent_rotate_q(Ctx* ctx, const LatentView& v, void* q, cudaStream_t st) {
  if (v.rot_dims == 0) return LMB200_OK;
  LMB_CUDA(launch_k(latent_rotate_q_kernel, dim3((unsigned)v.T), dim3(128), (size_t)(v.rot_dims / 2) * 8, st, v, (__nv_bfloat16*)q));
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

// The split whose CTAs fill whole waves of the SMs: cost = waves x (keys per CTA + a fixed share for the queries, the merge and the
// first tile's latency).  Every sequence divides its own context by the same split count.
LatentAttnPlan latent_attn_plan(const Ctx* ctx, int dtype, int T, int H, int kv_rank, int rot_dim, int ctx_len) {
  LatentAttnPlan p;
  if (dtype != LMB200_BF16 || !lat_tc_ok(kv_rank, rot_dim)) return p;
  const int M = 16 * lat_mt(H);
  const int64_t pairs = (int64_t)T * ceil_div(H, M), resident = ctx->sm_count;
  const int64_t max_split = std::min<int64_t>(64, ceil_div(ctx_len, 2 * kLatKeys));
  int64_t best = 1, best_cost = -1;
  for (int64_t ns = 1; ns <= std::max<int64_t>(1, max_split); ++ns) {
    const int64_t keys = round_up(ceil_div(ctx_len, ns), kLatKeys);
    const int64_t cost = ceil_div(pairs * ns, resident) * (keys + 192);
    if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = ns; }
  }
  p.nsplit = (int)best;
  if (best > 1) {
    p.part_floats = pairs * best * M * (kv_rank + 2);
    p.counters = pairs;
  }
  return p;
}

int32_t latent_attend(Ctx* ctx, int dtype, const LatentView& v, const void* qa, const void* cache, const LatentAttnPlan& plan, float* part,
                      unsigned* counters, float* olat, cudaStream_t st) {
  if (dtype == LMB200_BF16 && plan.nsplit >= 1 && lat_tc_ok(v.kv_rank, v.rot_dim)) {
    const int MT = lat_mt(v.H), NT = lat_nt(v.kv_rank);
    const dim3 grid((unsigned)(v.T * ceil_div(v.H, 16 * MT)), (unsigned)plan.nsplit);
    const size_t smem = lat_smem(MT, v.kv_rank, v.rot_dim);
    auto go = [&](auto kern) {
      return launch_k(kern, grid, dim3(kLatThreads), smem, st, v, (const __nv_bfloat16*)qa, (const __nv_bfloat16*)cache, plan.nsplit, part, counters, olat);
    };
    if (MT == 1) LMB_CUDA(NT == 2 ? go(latent_attend_tc_kernel<2, 1>) : NT == 4 ? go(latent_attend_tc_kernel<4, 1>) : go(latent_attend_tc_kernel<8, 1>));
    else LMB_CUDA(NT == 2 ? go(latent_attend_tc_kernel<2, 2>) : NT == 4 ? go(latent_attend_tc_kernel<4, 2>) : go(latent_attend_tc_kernel<8, 2>));
    ctx->launches++;
    return LMB200_OK;
  }
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
