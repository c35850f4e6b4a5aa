// Kernels of latent attention (see latent.cuh).
#include <math_constants.h>

#include <algorithm>

#include "latent.cuh"
#include "pdl.cuh"
#include "tc.cuh"

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
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LatentView v, const QT* __restrict__ q, const WT* __restrict__ w_ukt,
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
    const WT* w = w_ukt + ((int64_t)h * v.kv_rank + r) * v.dim;
    float a0[kTok], a1[kTok];
#pragma unroll
    for (int t = 0; t < kTok; ++t) a0[t] = a1[t] = 0.f;
#pragma unroll 4
    for (int d = 0; d < v.dim; ++d) {
      const float w0 = to_f32(w[d]), w1 = two ? to_f32(w[v.dim + d]) : 0.f;
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
// bf16 absorbed attention, split over the keys.  One CTA holds the 16 MT heads of one group of one token; its 16 warps are two teams of
// 8 that take the 32-key tiles of the CTA's share in turn, so that one team's products run during the other's softmax.  A tile's
// latent rows arrive by bulk copies (one per row, two stages per team; the row pitch is an odd number of 16-byte chunks) and serve as keys
// (S = Q' C^T: all heads x 16 keys x a quarter of the features per warp) and as values (O += P C: every warp a slice of the latent's columns).  Scores
// and the running softmax stay float32.  A CTA leaves (O, max, sum) of its keys; latent_expand merges the splits.
// ---------------------------------------------------------------------------------------------
constexpr int kTeams = 2, kTeamThreads = 256, kLatThreads = kTeams * kTeamThreads, kLatKeys = 32, kLatStages = 2;
constexpr int kScorePitch = kLatKeys + 4, kProbPitch = kLatKeys + 8, kParts = 4;      // kParts: the features of a score are summed in four parts

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  mma16816(c, a[0], a[1], a[2], a[3], b0, b1);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

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
  return (size_t)(kTeams * kLatStages * kLatKeys + MT * 16) * t.pitch * 2 +
         (size_t)kTeams * MT * 16 * (kParts * kScorePitch * 4 + kProbPitch * 2 + 4);
}
// keys per split: every sequence divides its own context by the same split count, in whole tiles of every team
__host__ __device__ inline int lat_keys_per_cta(int n, int nsplit) {
  constexpr int unit = kTeams * kLatKeys;
  return (((n + nsplit - 1) / nsplit + unit - 1) / unit) * unit;
}
// partial results of (token, head group, split): O [16 MT][kv_rank], then max and sum per head (log2 units)
__host__ __device__ inline int64_t lat_slot(int M, int kv_rank) { return (int64_t)M * (kv_rank + 2); }

template <int NT, int MT>
__global__ void __launch_bounds__(kLatThreads, 1) latent_attend_tc_kernel(const LatentView v, const __nv_bfloat16* __restrict__ qa,
                                                                          const __nv_bfloat16* __restrict__ cache, int nsplit,
                                                                          float* __restrict__ part, int* err) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ __align__(8) uint64_t full[kTeams][kLatStages];
  const LatTile L = lat_tile(v.kv_rank, v.rot_dim);
  constexpr int M = MT * 16;
  const int tid = threadIdx.x, lane = tid & 31, team = tid / kTeamThreads, tt = tid - team * kTeamThreads, warp = tt >> 5;
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(sm_raw) + team * kLatStages * kLatKeys * L.pitch;        // [stage][key][pitch]
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sm_raw) + kTeams * kLatStages * kLatKeys * L.pitch;      // [M][pitch]
  float* scores = reinterpret_cast<float*>(sQ + M * L.pitch);
  float* sS = scores + team * kParts * M * kScorePitch;                                                         // [part][M][kScorePitch]
  __nv_bfloat16* probs = reinterpret_cast<__nv_bfloat16*>(scores + kTeams * kParts * M * kScorePitch);
  __nv_bfloat16* sP = probs + team * M * kProbPitch;                                                            // [M][kProbPitch]
  float* sA = reinterpret_cast<float*>(probs + kTeams * M * kProbPitch) + team * M;                             // [M] rescale
  const int groups = (v.H + M - 1) / M;
  const int t = blockIdx.x / groups, hg = blockIdx.x - t * groups;
  auto team_sync = [&]() { asm volatile("bar.sync %0, %1;\n" ::"r"(1 + team), "n"(kTeamThreads) : "memory"); };
  if (tid == 0) {
    for (int i = 0; i < kTeams; ++i)
      for (int s = 0; s < kLatStages; ++s) tc::mbar_init(&full[i][s], 1);
    tc::mbar_init_fence();
  }
  // the padding between and behind the parts, and rows past the context, are never written by a copy: zero everything once
  for (int i = tid; i < (kTeams * kLatStages * kLatKeys + M) * L.pitch / 8; i += kLatThreads) reinterpret_cast<uint4*>(sm_raw)[i] = make_uint4(0, 0, 0, 0);
  tc::fence_async_smem();
  pdl_launch_dependents();
  pdl_wait();
  const int n = v.pos[t] + 1;
  const int kpc = lat_keys_per_cta(n, nsplit);
  const int k_begin = blockIdx.y * kpc, k_end = min(n, k_begin + kpc);
  if (k_begin >= n) return;
  __syncthreads();
  const int all_tiles = (k_end - k_begin + kLatKeys - 1) / kLatKeys;
  const int tiles = (all_tiles - team + kTeams - 1) / kTeams;         // this team's: team, team + 2, ...
  const __nv_bfloat16* base = cache + v.seq[t] * v.seq_stride;
  const bool one_piece = v.rot == L.R16;
  // every warp of the team issues the copies of four rows (one warp for all of them would hold the others up at the next barrier)
  auto load_tile = [&](int j) {
    constexpr int kRows = kLatKeys / (kTeamThreads / 32);
    const int key0 = k_begin + (j * kTeams + team) * kLatKeys, valid = min(kLatKeys, k_end - key0), row = warp * kRows + lane;
    uint64_t* bar = &full[team][j % kLatStages];
    if (tt == 0) tc::mbar_expect_tx(bar, (uint32_t)(valid * v.ld * 2));
    if (lane < kRows && row < valid) {
      __nv_bfloat16* dst = sK + ((j % kLatStages) * kLatKeys + row) * L.pitch;
      const __nv_bfloat16* src = base + (int64_t)(key0 + row) * v.ld;
      if (one_piece) tc::bulk_g2s(dst, src, (uint32_t)(v.ld * 2), bar);
      else {
        tc::bulk_g2s(dst, src, (uint32_t)(v.rot * 2), bar);
        if (v.ld > v.rot) tc::bulk_g2s(dst + L.R16, src + v.rot, (uint32_t)((v.ld - v.rot) * 2), bar);
      }
    }
  };
  for (int j = 0; j < min(tiles, kLatStages); ++j) load_tile(j);
  const int chunks = v.ld >> 3, c_chunks = v.rot >> 3;
  for (int h = tid >> 5; h < M; h += kLatThreads / 32)
    if (hg * M + h < v.H)
      for (int c = lane; c < chunks; c += 32)
        *reinterpret_cast<uint4*>(sQ + h * L.pitch + (c < c_chunks ? c * 8 : L.R16 + (c - c_chunks) * 8)) =
            *reinterpret_cast<const uint4*>(qa + ((int64_t)t * v.H + hg * M + h) * v.ld + c * 8);
  __syncthreads();

  // scores: warp = (16-key group, quarter of the feature steps), all heads
  const int KS = (L.R16 + L.P16) >> 4;
  const int kg = warp & 1, part_i = warp >> 1;
  const int ks0 = part_i * KS / kParts, ks1 = (part_i + 1) * KS / kParts;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
  constexpr int TPR = kTeamThreads / M, KPT = kLatKeys / TPR;       // softmax: threads per head, keys per thread
  const int srow = tt / TPR, spart = tt % TPR;
  const float cs = v.scale * kLog2e;
  float m_run = -CUDART_INF_F, l_run = 0.f;
  const uint32_t qaddr = smem_addr(sQ + (lane & 15) * L.pitch + (lane >> 4) * 8), qnext = (uint32_t)(16 * L.pitch * 2);
  const int col0 = warp * NT * 8;                      // this warp's slice of the latent's columns
  bool dead = false;

  for (int j = 0; j < tiles; ++j) {
    tc::mbar_wait(&full[team][j % kLatStages], (j / kLatStages) & 1, dead, err);
    const __nv_bfloat16* K = sK + (j % kLatStages) * kLatKeys * L.pitch;
    const int key0 = k_begin + (j * kTeams + team) * kLatKeys;
    {
      float sc[MT][2][4];                              // two 8-key tiles per head tile
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i) sc[m][0][i] = sc[m][1][i] = 0.f;
      const uint32_t kaddr = smem_addr(K + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * L.pitch + ((lane >> 3) & 1) * 8);
#pragma unroll 5
      for (int ks = ks0; ks < ks1; ++ks) {
        uint32_t a[MT][4], b[4];
        ldsm4(b, kaddr + ks * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(a[m], qaddr + m * qnext + ks * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma16816(sc[m][0], a[m], b[0], b[1]);
          mma16816(sc[m][1], a[m], b[2], b[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float* o = sS + (part_i * M + m * 16 + (lane >> 2)) * kScorePitch + kg * 16 + (lane & 3) * 2;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          *reinterpret_cast<float2*>(o + i * 8) = make_float2(sc[m][i][0], sc[m][i][1]);
          *reinterpret_cast<float2*>(o + 8 * kScorePitch + i * 8) = make_float2(sc[m][i][2], sc[m][i][3]);
        }
      }
    }
    team_sync();                                       // the scores are there; everyone is past the previous tile
    {
      float s[KPT];
      float mx = -CUDART_INF_F;
      const float* sp = sS + srow * kScorePitch + spart * KPT;
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float2 a = *reinterpret_cast<const float2*>(sp + i), b = *reinterpret_cast<const float2*>(sp + M * kScorePitch + i);
        const float2 c = *reinterpret_cast<const float2*>(sp + 2 * M * kScorePitch + i), d = *reinterpret_cast<const float2*>(sp + 3 * M * kScorePitch + i);
        s[i] = ((a.x + b.x) + (c.x + d.x)) * cs;
        s[i + 1] = ((a.y + b.y) + (c.y + d.y)) * cs;
      }
      if (key0 + kLatKeys > k_end) {
#pragma unroll
        for (int i = 0; i < KPT; ++i)
          if (key0 + spart * KPT + i >= k_end) s[i] = -CUDART_INF_F;
      }
#pragma unroll
      for (int i = 0; i < KPT; ++i) mx = fmaxf(mx, s[i]);
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float mn = fmaxf(m_run, mx);               // finite: every tile holds at least one key
      const float alpha = ex2(m_run - mn);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float p0 = ex2(s[i] - mn), p1 = ex2(s[i + 1] - mn);
        sum += p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(sP + srow * kProbPitch + spart * KPT + i) = __floats2bfloat162_rn(p0, p1);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l_run = l_run * alpha + sum;
      m_run = mn;
      if (spart == 0) sA[srow] = alpha;
    }
    if (j >= 1 && j + 1 < tiles) load_tile(j + 1);        // into the stage of tile j - 1
    team_sync();
    if (col0 < L.R16) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = sA[m * 16 + (lane >> 2)], a1 = sA[m * 16 + (lane >> 2) + 8];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int i = 0; i < NT; ++i) { acc[m][i][0] *= a0; acc[m][i][1] *= a0; acc[m][i][2] *= a1; acc[m][i][3] *= a1; }
        }
      }
#pragma unroll
      for (int ks = 0; ks < kLatKeys / 16; ++ks) {
        uint32_t p[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(p[m], smem_addr(sP + (m * 16 + (lane & 15)) * kProbPitch + ks * 16 + (lane >> 4) * 8));
        const uint32_t vaddr = smem_addr(K + (ks * 16 + (lane & 15)) * L.pitch + col0 + (lane >> 4) * 8);
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
  }
  // The second team hands its accumulators over through shared memory (a thread's counterpart owns the same elements), and the
  // first leaves the merged result of the CTA's keys.
  const int R = v.kv_rank;
  float* stat = reinterpret_cast<float*>(probs);       // [team][max, sum][M]
  float* hand = reinterpret_cast<float*>(sm_raw);      // [MT * NT * 4][kTeamThreads], over the key stages (and, for narrow latents, the scores)
  __syncthreads();
  if (spart == 0) { stat[(2 * team) * M + srow] = m_run; stat[(2 * team + 1) * M + srow] = l_run; }
  if (team == 1) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) hand[((m * NT + i) * 4 + e) * kTeamThreads + tt] = acc[m][i][e];
  }
  __syncthreads();
  if (team == 1) return;
  float* mine = part + ((int64_t)blockIdx.x * nsplit + blockIdx.y) * lat_slot(M, R);
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e2 = 0; e2 < 2; ++e2) {
      const int row = m * 16 + (lane >> 2) + e2 * 8;
      const float m0 = stat[row], m1 = stat[2 * M + row], mx = fmaxf(m0, m1);          // the first team has had a tile: m0 is finite
      const float w0 = ex2(m0 - mx), w1 = ex2(m1 - mx);
      if (warp == 0 && (lane & 3) == 0) { mine[(int64_t)M * R + row] = mx; mine[(int64_t)M * R + M + row] = stat[M + row] * w0 + stat[3 * M + row] * w1; }
      if (col0 >= L.R16) continue;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int col = col0 + i * 8 + (lane & 3) * 2;
        const float* o = hand + ((m * NT + i) * 4 + e2 * 2) * kTeamThreads + tt;
        const float x = acc[m][i][2 * e2] * w0 + o[0] * w1, y = acc[m][i][2 * e2 + 1] * w0 + o[kTeamThreads] * w1;
        if (col < R) *reinterpret_cast<float2*>(mine + (int64_t)row * R + col) = make_float2(x, y);       // R is even
      }
    }
}

// ---------------------------------------------------------------------------------------------
// Products of one head's matrix W [N, K] (row-major, 16-byte rows) with up to 16 tokens: 8 warps share the N / 8 column tiles of the CTA's
// slice.  Within 32 features lane tq takes the eight from 8 tq on for both operands, so every fragment is one 16-byte load.
// ---------------------------------------------------------------------------------------------
constexpr int kHeadTok = 16;

// sA: [kHeadTok][pitch] bf16, zero behind K (pitch covers K rounded up to 32); f(token row, column n, value)
template <typename F>
__device__ __forceinline__ void head_product(const __nv_bfloat16* __restrict__ W, int N, int K, int n_begin, int n_end, const __nv_bfloat16* sA, int pitch, F f) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tq = lane & 3;
  for (int n0 = n_begin + warp * 16; n0 < n_end; n0 += 8 * 16) {          // two column tiles at a time
    float c[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const __nv_bfloat16* w0 = W + (int64_t)min(n0 + g, N - 1) * K;
    const __nv_bfloat16* w1 = W + (int64_t)min(n0 + 8 + g, N - 1) * K;
#pragma unroll 4
    for (int k = 8 * tq; k - 8 * tq < K; k += 32) {
      const bool in = k < K;
      const uint4 z = make_uint4(0, 0, 0, 0);
      const uint4 b0 = in ? __ldg(reinterpret_cast<const uint4*>(w0 + k)) : z, b1 = in ? __ldg(reinterpret_cast<const uint4*>(w1 + k)) : z;
      const uint4 a0 = *reinterpret_cast<const uint4*>(sA + g * pitch + k), a1 = *reinterpret_cast<const uint4*>(sA + (g + 8) * pitch + k);
      mma16816(c[0], a0.x, a1.x, a0.y, a1.y, b0.x, b0.y);
      mma16816(c[1], a0.x, a1.x, a0.y, a1.y, b1.x, b1.y);
      mma16816(c[0], a0.z, a1.z, a0.w, a1.w, b0.z, b0.w);
      mma16816(c[1], a0.z, a1.z, a0.w, a1.w, b1.z, b1.w);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = n0 + 8 * i + 2 * tq + (e & 1);
        if (n < n_end) f(g + 8 * (e >> 1), n, c[i][e]);
      }
  }
}
__host__ __device__ inline int head_pitch(int K) { return ((K + 31) & ~31) + 8; }

// queries against the latents: head blockIdx.x, tokens 16 * blockIdx.y .., latent columns of slice blockIdx.z; W_uk as [H, kv_rank, dim]
template <typename QT>
__global__ void __launch_bounds__(256) latent_absorb_tc_kernel(const LatentView v, const QT* __restrict__ q, const __nv_bfloat16* __restrict__ w_ukt,
                                                               __nv_bfloat16* __restrict__ qa) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* sA = reinterpret_cast<__nv_bfloat16*>(sm_raw);
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t0 = blockIdx.y * kHeadTok, n = min(kHeadTok, v.T - t0), tid = threadIdx.x;
  const int qd = v.dim + v.rot_dim, pitch = head_pitch(v.dim);
  const int64_t qp = (int64_t)v.H * qd;
  for (int t = tid >> 5; t < kHeadTok; t += 8)
    for (int d = tid & 31; d < pitch; d += 32)
      sA[t * pitch + d] = __float2bfloat16_rn(t < n && d < v.dim ? to_f32(q[(t0 + t) * qp + h * qd + d]) : 0.f);
  if (blockIdx.z == 0)
    for (int i = tid; i < v.rot_dim * n; i += 256) {
      const int t = i / v.rot_dim, d = i - t * v.rot_dim;
      const QT* qr = q + (t0 + t) * qp + h * qd + v.dim;
      qa[((int64_t)(t0 + t) * v.H + h) * v.ld + v.rot + d] = __float2bfloat16_rn(
          rotated([&](int j) { return to_f32(qr[j]); }, d, v.q_rotated ? 0 : v.rot_dims, v.rot_interleaved, v.pos[t0 + t], v.inv_freq));
    }
  __syncthreads();
  const int R = v.kv_rank, per = (((R + gridDim.z - 1) / gridDim.z) + 15) & ~15, r0 = blockIdx.z * per;
  head_product(w_ukt + (int64_t)h * R * v.dim, R, v.dim, r0, min(R, r0 + per), sA, pitch, [&](int t, int r, float x) {
    if (t < n) qa[((int64_t)(t0 + t) * v.H + h) * v.ld + r] = __float2bfloat16_rn(x);
  });
}

// merges the partial results of a head's keys, multiplies the weighted latents out to values and gates them: head blockIdx.x, tokens
// tok * blockIdx.y .. (tok <= kHeadTok; few tokens per CTA spread the merging over the SMs), value columns of slice blockIdx.z
__global__ void __launch_bounds__(256) latent_expand_tc_kernel(const LatentView v, const float* __restrict__ part, int nsplit, int M,
                                                               const __nv_bfloat16* __restrict__ w_uv, const float* __restrict__ gate, int gate_pitch,
                                                               __nv_bfloat16* __restrict__ out, int ldo, int bp, int tok) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* sA = reinterpret_cast<__nv_bfloat16*>(sm_raw);
  __shared__ float s_gate[kHeadTok];
  const int R = v.kv_rank, pitch = head_pitch(R);
  float* s_w = reinterpret_cast<float*>(sA + kHeadTok * pitch);                // [kHeadTok][nsplit] weights of the partial results
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t0 = blockIdx.y * tok, n = min(tok, v.T - t0), tid = threadIdx.x, lane = tid & 31;
  const int groups = (v.H + M - 1) / M, hg = h / M, row = h - hg * M, np = nsplit;
  const int64_t slot = lat_slot(M, R);
  for (int t = tid >> 5; t < n; t += 8) {
    const float* p = part + ((int64_t)(t0 + t) * groups + hg) * np * slot + (int64_t)M * R + row;
    const int ctx = v.pos[t0 + t] + 1, kpc = lat_keys_per_cta(ctx, nsplit);
    float mx = -CUDART_INF_F;
    for (int i = lane; i < np; i += 32) {
      const float m = i * kpc < ctx ? __ldcg(p + i * slot) : -CUDART_INF_F;
      s_w[t * np + i] = m;
      mx = fmaxf(mx, m);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    float den = 0.f;
    for (int i = lane; i < np; i += 32) {
      const float m = s_w[t * np + i];
      const float w = m == -CUDART_INF_F ? 0.f : exp2f(m - mx);
      s_w[t * np + i] = w;
      if (w > 0.f) den += w * __ldcg(p + i * slot + M);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) den += __shfl_xor_sync(0xffffffffu, den, off);
    if (lane == 0) s_gate[t] = 1.0f / (den * (1.0f + expf(-gate[(int64_t)(t0 + t) * gate_pitch + h])));       // gate / denominator
  }
  __syncthreads();
  // four latent columns per thread; the loads do not depend on the weights (a share nobody wrote holds stale numbers, weight 0)
  const int q4 = pitch >> 2;
  for (int i = tid; i < kHeadTok * q4; i += 256) {
    const int t = i / q4, r = (i - t * q4) * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < n && r < R) {
      const float* p = part + ((int64_t)(t0 + t) * groups + hg) * np * slot + (int64_t)row * R + r;
#pragma unroll 8
      for (int k = 0; k < np; ++k) {
        const float4 y = __ldcg(reinterpret_cast<const float4*>(p + k * slot));
        const float w = s_w[t * np + k];
        if (w > 0.f) { x.x += w * y.x; x.y += w * y.y; x.z += w * y.z; x.w += w * y.w; }
      }
      const float s = s_gate[t];
      x.x *= s; x.y *= s; x.z *= s; x.w *= s;
    }
    __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(sA + t * pitch + r);
    o[0] = __floats2bfloat162_rn(x.x, x.y);
    o[1] = __floats2bfloat162_rn(x.z, x.w);
  }
  __syncthreads();
  const int V = v.vdim, per = (((V + gridDim.z - 1) / gridDim.z) + 15) & ~15, n0 = blockIdx.z * per;
  head_product(w_uv + (int64_t)h * V * R, V, R, n0, min(V, n0 + per), sA, pitch, [&](int t, int d, float x) {
    if (t < n) out[bp > 0 ? Layout<__nv_bfloat16>::x_offset(t0 + t, h * V + d, bp) : (int64_t)(t0 + t) * ldo + h * V + d] = __float2bfloat16_rn(x);
  });
}

// column slices that give every SM a CTA, each at least 64 columns
unsigned head_slices(const Ctx* ctx, int64_t ctas, int N) {
  int64_t z = ctas >= ctx->sm_count ? 1 : ceil_div(ctx->sm_count, ctas);
  return (unsigned)std::max<int64_t>(1, std::min<int64_t>(z, N / 64));
}

constexpr size_t kLatMaxSmem = 226 * 1024;
bool lat_tc_ok(const LatentView& v) {
  return v.kv_rank <= 512 && v.kv_rank % 8 == 0 && v.dim % 8 == 0 && lat_smem(2, v.kv_rank, v.rot_dim) <= kLatMaxSmem;
}
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
  LMB_CUDA(cudaFuncSetAttribute(latent_attend_tc_kernel<NT, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatMaxSmem));           \
  LMB_CUDA(cudaFuncSetAttribute(latent_attend_tc_kernel<NT, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatMaxSmem))
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

int32_t latent_absorb(Ctx* ctx, int dtype, const LatentView& v, const void* q, int q_f32, const void* w_ukt, void* qa, cudaStream_t st) {
  if (dtype == LMB200_BF16 && lat_tc_ok(v)) {
    const int64_t tg = ceil_div(v.T, kHeadTok);
    const dim3 grid((unsigned)v.H, (unsigned)tg, head_slices(ctx, v.H * tg, v.kv_rank));
    const size_t smem = (size_t)kHeadTok * head_pitch(v.dim) * 2;
    if (q_f32) LMB_CUDA(launch_k(latent_absorb_tc_kernel<float>, grid, dim3(256), smem, st, v, (const float*)q, (const __nv_bfloat16*)w_ukt, (__nv_bfloat16*)qa));
    else LMB_CUDA(launch_k(latent_absorb_tc_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, v, (const __nv_bfloat16*)q, (const __nv_bfloat16*)w_ukt, (__nv_bfloat16*)qa));
    ctx->launches++;
    return LMB200_OK;
  }
  const dim3 grid((unsigned)v.H, (unsigned)ceil_div(v.T, kTok));
  const size_t smem = (size_t)v.dim * kTok * 4;
  LMB_REQUIRE(smem <= 48 * 1024 && grid.y <= 65535, "latent attention: head width %d, %d tokens", v.dim, v.T);
  if (dtype != LMB200_BF16)
    LMB_CUDA(launch_k(latent_absorb_kernel<float, float>, grid, dim3(256), smem, st, v, (const float*)q, (const float*)w_ukt, (float*)qa));
  else if (q_f32)
    LMB_CUDA(launch_k(latent_absorb_kernel<__nv_bfloat16, float>, grid, dim3(256), smem, st, v, (const float*)q, (const __nv_bfloat16*)w_ukt,
                      (__nv_bfloat16*)qa));
  else
    LMB_CUDA(launch_k(latent_absorb_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), smem, st, v, (const __nv_bfloat16*)q,
                      (const __nv_bfloat16*)w_ukt, (__nv_bfloat16*)qa));
  ctx->launches++;
  return LMB200_OK;
}

// The split whose CTAs fill whole waves of the SMs: cost = waves x (keys per CTA + a fixed share for the queries, the merge and the
// first tile's latency).  Every sequence divides its own context by the same split count.
LatentAttnPlan latent_attn_plan(const Ctx* ctx, int dtype, const LatentView& v, int T, int ctx_len) {
  LatentAttnPlan p;
  p.part_floats = (int64_t)T * v.H * v.kv_rank;                  // the CUDA-core kernel's output
  if (dtype != LMB200_BF16 || !lat_tc_ok(v)) return p;
  const int M = 16 * lat_mt(v.H);
  const int64_t pairs = (int64_t)T * ceil_div(v.H, M), resident = ctx->sm_count;
  const int64_t max_split = std::max<int64_t>(1, std::min<int64_t>(64, ceil_div(ctx_len, 4 * kLatKeys)));
  int64_t best = 1, best_cost = -1;
  for (int64_t ns = 1; ns <= max_split; ++ns) {
    const int64_t cost = ceil_div(pairs * ns, resident) * (lat_keys_per_cta(ctx_len, (int)ns) + 192);
    if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = ns; }
  }
  p.nsplit = (int)best;
  p.part_floats = pairs * best * lat_slot(M, v.kv_rank);
  return p;
}

int32_t latent_attend(Ctx* ctx, int dtype, const LatentView& v, const void* qa, const void* cache, const LatentAttnPlan& plan, float* part, cudaStream_t st) {
  if (plan.nsplit >= 1) {
    LMB_REQUIRE(dtype == LMB200_BF16 && lat_tc_ok(v), "latent attention: the plan is not this layer's");
    const int MT = lat_mt(v.H), NT = lat_nt(v.kv_rank);
    const dim3 grid((unsigned)(v.T * ceil_div(v.H, 16 * MT)), (unsigned)plan.nsplit);
    const size_t smem = lat_smem(MT, v.kv_rank, v.rot_dim);
    auto go = [&](auto kern) {
      return launch_k(kern, grid, dim3(kLatThreads), smem, st, v, (const __nv_bfloat16*)qa, (const __nv_bfloat16*)cache, plan.nsplit, part, ctx->dev_err);
    };
    if (MT == 1) LMB_CUDA(NT == 2 ? go(latent_attend_tc_kernel<2, 1>) : NT == 4 ? go(latent_attend_tc_kernel<4, 1>) : go(latent_attend_tc_kernel<8, 1>));
    else LMB_CUDA(NT == 2 ? go(latent_attend_tc_kernel<2, 2>) : NT == 4 ? go(latent_attend_tc_kernel<4, 2>) : go(latent_attend_tc_kernel<8, 2>));
    ctx->launches++;
    return LMB200_OK;
  }
  float* olat = part;
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

int32_t latent_expand(Ctx* ctx, int dtype, const LatentView& v, const float* part, const LatentAttnPlan& plan, const void* w_uv, const float* gate,
                      int gate_pitch, void* out, int ldo, int bp, cudaStream_t st) {
  if (plan.nsplit >= 1) {
    int tok = kHeadTok;
    while (tok > 2 && v.H * ceil_div(v.T, tok) < ctx->sm_count) tok >>= 1;
    const int64_t tg = ceil_div(v.T, tok);
    const dim3 grid((unsigned)v.H, (unsigned)tg, head_slices(ctx, v.H * tg, v.vdim));
    const size_t smem = (size_t)kHeadTok * head_pitch(v.kv_rank) * 2 + (size_t)kHeadTok * plan.nsplit * 4;
    LMB_CUDA(launch_k(latent_expand_tc_kernel, grid, dim3(256), smem, st, v, part, plan.nsplit, 16 * lat_mt(v.H), (const __nv_bfloat16*)w_uv, gate,
                      gate_pitch, (__nv_bfloat16*)out, ldo, bp, tok));
    ctx->launches++;
    return LMB200_OK;
  }
  const float* olat = part;
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
