// Retention over long portions on the fifth-generation tensor cores: chunks of 128 tokens, tcgen05.mma with the scores, both
// outputs and the state in tensor memory.
//
// A CTA (or a pair of them for value widths above 128, 128 value columns each) owns one head of one sequence and walks its
// chunks; row i, key j of a chunk with n valid tokens, decay g, scale = 1 / sqrt(dim):
//   A = Q K^T                                   M 128 x N 128 x K dim          -> columns P
//   P = A * scale g^(i - j) for j <= i          registers; back to P's columns as bf16 pairs hi | lo (x = hi + lo to about 2^-17)
//   I = Q S                                     S of the previous chunk from shared memory, hi and lo      -> columns I
//   O = P V                                     P from tensor memory, hi and lo                            -> columns O
//   S = g^n S + (scale g^(n - 1 - j) K)^T V     weighted keys hi and lo; S (float32) accumulates in tensor memory
//   y_i = (O_i + g^(i + 1) I_i) / rms * gate
// so q, k, v enter as bf16 and everything the decays touch keeps float32's leading 16 bits.
// Warps: 0-7 scores and outputs (two threads per row), 8-15 state and weighted keys (two threads per row), 16 issues the MMAs, 17
// the TMA loads (K in two buffers, Q and V in one each: they are free again half a chunk before they are needed).
// The weighted keys' hi part overwrites K in place: the layout is the swizzled tile K came in, the weight is one number per row.
#include <cuda.h>

#include "pdl.cuh"
#include "retention.cuh"
#include "tc.cuh"

namespace lmb {
namespace {

constexpr int kT = 128;                                  // tokens per chunk, rows of every tile
constexpr int kSub = kT * 128;                           // bytes of a sub-tile [128 rows][64 columns], 128-byte swizzle
constexpr int kTile = 2 * kSub;                          // 128 x 128 bf16
constexpr int kThreads = 18 * 32;
constexpr uint32_t kColP = 0, kColO = 128, kColI = 256, kColS = 384;
constexpr int offQ = 0, offK = kTile, offKl = 3 * kTile, offV = 4 * kTile, offSh = 5 * kTile, offSl = 6 * kTile, offEnd = 7 * kTile;
struct Tail {                                            // behind the tiles
  uint64_t q_full, q_empty, k_full[2], k_empty[2], v_full, v_empty, s_full, p_ready, kt_ready, st_ready, o_full, o_empty, m4_done, x_full;
  uint32_t tmem;
  float pw[kT + 4];                                      // decay^0 .. decay^128
  float ssq[2][kT];                                      // sums of squares of the two column halves
  float peer[2][kT];                                     // the other CTA's rows, by chunk parity
};
constexpr size_t kSmem = (size_t)offEnd + sizeof(Tail);
static_assert(kSmem <= 227 * 1024, "shared memory");

__device__ __forceinline__ uint64_t desc(uint32_t saddr, uint32_t lbo, uint32_t sbo) {       // 128-byte swizzle
  return (uint64_t)((saddr & 0x3FFFF) >> 4) | ((uint64_t)(lbo >> 4) << 16) | ((uint64_t)(sbo >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// K-major operand (rows of 128 bytes), features 16 ks ..
__device__ __forceinline__ uint64_t desc_k(uint32_t tile, int ks) { return desc(tile + (ks >> 2) * kSub + (ks & 3) * 32, 16, 1024); }
// operand whose rows are the contraction index, rows 16 ks ..
__device__ __forceinline__ uint64_t desc_mn(uint32_t tile, int ks) { return desc(tile + ks * 2048, kSub, 1024); }
__device__ __forceinline__ void mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {        // A from tensor memory
  asm volatile(
      "{\n.reg .pred p;\nsetp.ne.b32 p, %4, 0;\ntcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}\n" ::"r"(d), "r"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void tma_3d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(tc::smem_u32(dst)),
      "l"(reinterpret_cast<uint64_t>(map)), "r"(c0), "r"(c1), "r"(c2), "r"(tc::smem_u32(bar))
      : "memory");
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack2bf(uint32_t u) {
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&u);
  return make_float2(__low2float(h), __high2float(h));
}
// wait for signals of the other CTA of the pair (acquire at cluster scope), bounded like tc::mbar_wait
__device__ __forceinline__ void mbar_wait_cluster(uint64_t* bar, uint32_t parity, bool& dead, int* err) {
  if (dead) return;
  const long long t0 = clock64();
  for (;;) {
    uint32_t ok;
    asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\nselp.u32 %0, 1, 0, p;\n}\n"
                 : "=r"(ok) : "r"(tc::smem_u32(bar)), "r"(parity) : "memory");
    if (ok) return;
    if (clock64() - t0 > tc::kWaitLimit) { dead = true; if (err) atomicExch(err, 1); return; }
  }
}

__global__ void __launch_bounds__(kThreads, 1) retention_tc_kernel(const RetentionView v, const __grid_constant__ CUtensorMap qmap,
                                                                   const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap,
                                                                   int* err) {
  using namespace tc;
  extern __shared__ __align__(1024) unsigned char smem[];
  Tail& tl = *reinterpret_cast<Tail*>(smem + offEnd);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pair = gridDim.x, slice = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  if (tid == 0) {
    if (smem_u32(smem) & 1023) atomicExch(err, 1);       // the swizzle needs 1024-byte tiles
    mbar_init(&tl.q_full, 1); mbar_init(&tl.q_empty, 1); mbar_init(&tl.v_full, 1); mbar_init(&tl.v_empty, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&tl.k_full[i], 1); mbar_init(&tl.k_empty[i], 1); }
    mbar_init(&tl.s_full, 1); mbar_init(&tl.o_full, 1); mbar_init(&tl.m4_done, 1);
    mbar_init(&tl.p_ready, 8); mbar_init(&tl.kt_ready, 8); mbar_init(&tl.st_ready, 8); mbar_init(&tl.o_empty, 8);
    mbar_init(&tl.x_full, kT);
    mbar_init_fence();
  }
  for (int i = tid; i <= kT; i += kThreads) tl.pw[i] = v.decay[(int64_t)h * v.decay_pitch + i];      // constants of the model
  if (warp == 16) tmem_alloc(&tl.tmem, 512);
  fence_before();
  __syncthreads();
  if (pair > 1) {                                        // both CTAs' barriers exist before anyone arrives on them
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
  }
  fence_after();
  const uint32_t tmem = tl.tmem;
  pdl_launch_dependents();
  pdl_wait();
  bool dead = false;
  const int n_all = v.len[b], t_first = v.start[b];
  const int chunks = (n_all + kT - 1) / kT;              // 0: nothing to do (uniform over the pair)
  const int D = v.dim, V = v.vdim, ld = (V + 3) & ~3, c0 = slice * 128;
  const float* pw = tl.pw;
  const float scale = v.k_scale;
  const uint32_t lane_base = (uint32_t)(32 * (warp & 3)) << 16;

  if (warp == 17) {
    if (lane == 0) {
      for (int c = 0; c < chunks; ++c) {
        const int t0 = t_first + c * kT, kb = c & 1;
        mbar_wait(&tl.k_empty[kb], ((c >> 1) & 1) ^ 1, dead, err);
        mbar_expect_tx(&tl.k_full[kb], kTile);
        for (int s = 0; s < 2; ++s) tma_3d(smem + offK + kb * kTile + s * kSub, &kmap, s * 64, h, t0, &tl.k_full[kb]);
        mbar_wait(&tl.q_empty, (c & 1) ^ 1, dead, err);
        mbar_expect_tx(&tl.q_full, kTile);
        for (int s = 0; s < 2; ++s) tma_3d(smem + offQ + s * kSub, &qmap, s * 64, h, t0, &tl.q_full);
        mbar_wait(&tl.v_empty, (c & 1) ^ 1, dead, err);
        mbar_expect_tx(&tl.v_full, kTile);
        for (int s = 0; s < 2; ++s) tma_3d(smem + offV + s * kSub, &vmap, c0 + s * 64, h, t0, &tl.v_full);
      }
    }
    __syncwarp();
  } else if (warp == 16) {
    constexpr uint32_t kKK = idesc_bf16(128, 128, false, false), kKM = idesc_bf16(128, 128, false, true), kMM = idesc_bf16(128, 128, true, true);
    const uint32_t base = smem_u32(smem);
    const int ds = (D + 15) >> 4;                        // 16-feature steps (the tiles are zero behind dim)
    auto scores = [&](int c) {
      mbar_wait(&tl.q_full, c & 1, dead, err);
      mbar_wait(&tl.k_full[c & 1], (c >> 1) & 1, dead, err);
      fence_after();
      if (lane == 0) {
        for (int ks = 0; ks < ds; ++ks) mma_f16(tmem + kColP, desc_k(base + offQ, ks), desc_k(base + offK + (c & 1) * kTile, ks), kKK, ks ? 1u : 0u);
        commit(&tl.s_full);
      }
      __syncwarp();
    };
    if (chunks > 0) scores(0);
    for (int c = 0; c < chunks; ++c) {
      if (c) mbar_wait(&tl.o_empty, (c - 1) & 1, dead, err);
      mbar_wait(&tl.st_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
        for (int ks = 0; ks < ds; ++ks) mma_f16(tmem + kColI, desc_k(base + offQ, ks), desc_mn(base + offSh, ks), kKM, ks ? 1u : 0u);
        for (int ks = 0; ks < ds; ++ks) mma_f16(tmem + kColI, desc_k(base + offQ, ks), desc_mn(base + offSl, ks), kKM, 1u);
        commit(&tl.q_empty);
      }
      __syncwarp();
      mbar_wait(&tl.v_full, c & 1, dead, err);
      mbar_wait(&tl.p_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
        for (int ks = 0; ks < 8; ++ks) mma_ts(tmem + kColO, tmem + kColP + ks * 8, desc_mn(base + offV, ks), kKM, ks ? 1u : 0u);
        for (int ks = 0; ks < 8; ++ks) mma_ts(tmem + kColO, tmem + kColP + 64 + ks * 8, desc_mn(base + offV, ks), kKM, 1u);
        commit(&tl.o_full);
      }
      __syncwarp();
      mbar_wait(&tl.kt_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
        for (int ks = 0; ks < 8; ++ks) mma_f16(tmem + kColS, desc_mn(base + offK + (c & 1) * kTile, ks), desc_mn(base + offV, ks), kMM, 1u);
        for (int ks = 0; ks < 8; ++ks) mma_f16(tmem + kColS, desc_mn(base + offKl, ks), desc_mn(base + offV, ks), kMM, 1u);
        commit(&tl.m4_done);
        commit(&tl.v_empty);
        commit(&tl.k_empty[c & 1]);
      }
      __syncwarp();
      if (c + 1 < chunks) scores(c + 1);
    }
  } else if (warp >= 8) {
    // ------------------------------ state and weighted keys ------------------------------
    const int half = (warp - 8) >> 2, row = 32 * (warp & 3) + lane;            // state row (feature) / token
    float* state = v.state + (((int64_t)b * v.H + h) * D + row) * ld + c0 + half * 64;
    const int cols = min(64, ld - c0 - half * 64);                             // valid state columns of this thread (a multiple of 4, or <= 0)
    auto put = [&](int col, const float (&x)[16]) {                            // 16 columns from `col` (of the half) to shared memory, hi and lo
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split2(x[8 * q + 2 * e], x[8 * q + 2 * e + 1], hi[e], lo[e]);
        const int at = half * kSub + row * 128 + ((((col >> 3) + q) ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(smem + offSh + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(smem + offSl + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    };
    for (int c = 0; c < chunks; ++c) {
      const int n = min(kT, n_all - c * kT);
      const float wn = pw[n];
      if (c) { mbar_wait(&tl.m4_done, (c - 1) & 1, dead, err); fence_after(); }
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        float x[16];
        if (c == 0) {
#pragma unroll
          for (int i = 0; i < 16; i += 4) {
            const float4 y = row < D && ch * 16 + i < cols ? *reinterpret_cast<const float4*>(state + ch * 16 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[i] = y.x; x[i + 1] = y.y; x[i + 2] = y.z; x[i + 3] = y.w;
          }
        } else {
          tmem_ld16(x, tmem + lane_base + kColS + half * 64 + ch * 16);
        }
        put(ch * 16, x);
        uint32_t u[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(x[i] * wn);
        tmem_st16_nowait(tmem + lane_base + kColS + half * 64 + ch * 16, u);
      }
      tmem_st_wait();
      fence_before();
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.st_ready);
      mbar_wait(&tl.k_full[c & 1], (c >> 1) & 1, dead, err);
      mbar_wait(&tl.s_full, c & 1, dead, err);           // K has been multiplied with Q: its tile may become the weighted keys
      const float kw = row < n ? scale * pw[n - 1 - row] : 0.f;
      unsigned char* kt = smem + offK + (c & 1) * kTile + half * kSub + row * 128;
      unsigned char* kl = smem + offKl + half * kSub + row * 128;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int at = ((i + row) & 7) << 4;             // the order does not matter, the rotation keeps the lanes on different banks
        uint4 x = *reinterpret_cast<const uint4*>(kt + at), lo;
        uint32_t* xi = reinterpret_cast<uint32_t*>(&x);
        uint32_t* li = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 y = unpack2bf(xi[e]);
          split2(y.x * kw, y.y * kw, xi[e], li[e]);
        }
        *reinterpret_cast<uint4*>(kt + at) = x;
        *reinterpret_cast<uint4*>(kl + at) = lo;
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.kt_ready);
    }
    if (chunks > 0) {
      mbar_wait(&tl.m4_done, (chunks - 1) & 1, dead, err);
      fence_after();
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        float x[16];
        tmem_ld16(x, tmem + lane_base + kColS + half * 64 + ch * 16);
        if (row < D) {
#pragma unroll
          for (int i = 0; i < 16; i += 4)
            if (ch * 16 + i < cols) *reinterpret_cast<float4*>(state + ch * 16 + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
        }
      }
    }
  } else {
    // ------------------------------ scores and outputs ------------------------------
    const int half = warp >> 2, row = 32 * (warp & 3) + lane, pair_bar = 1 + (warp & 3);
    const float wi = pw[row + 1], g1 = pw[1];
    for (int c = 0; c < chunks; ++c) {
      const int n = min(kT, n_all - c * kT);
      const int64_t t = t_first + (int64_t)c * kT + row;
      const int col = h * V + c0 + half * 64, left = V - c0 - half * 64;       // valid columns: a multiple of 8, or <= 0
      const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(v.g) + t * v.g_pitch + col;
      if (row < n && left > 0) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(gate));
      mbar_wait(&tl.s_full, c & 1, dead, err);
      fence_after();
      uint32_t hi[32], lo[32];
      const bool any = half * 64 <= 32 * (warp & 3) + 31;                      // some key of this half is not in the rows' future
      if (any) {
#pragma unroll
        for (int ch = 0; ch < 4; ++ch) {
          float s[16];
          tmem_ld16(s, tmem + lane_base + kColP + half * 64 + ch * 16);
          // weights from the nearest key of the sixteen outwards: one table entry, then one factor per key
          const int d = row - (half * 64 + ch * 16 + 15);                      // distance to the last key
          float w = scale * pw[max(d, 0)];
#pragma unroll
          for (int i = 15; i >= 0; --i) {
            const bool seen = d + 15 - i >= 0;
            s[i] = seen ? s[i] * w : 0.f;
            if (seen) w *= g1;
          }
#pragma unroll
          for (int i = 0; i < 16; i += 2) split2(s[i], s[i + 1], hi[ch * 8 + i / 2], lo[ch * 8 + i / 2]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) hi[i] = lo[i] = 0u;
      }
      asm volatile("bar.sync %0, 64;\n" ::"r"(pair_bar) : "memory");           // the other half of the row has read its scores too
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        uint32_t a[16], l[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) { a[i] = hi[16 * q + i]; l[i] = lo[16 * q + i]; }
        tmem_st16_nowait(tmem + lane_base + kColP + half * 32 + q * 16, a);
        tmem_st16_nowait(tmem + lane_base + kColP + 64 + half * 32 + q * 16, l);
      }
      tmem_st_wait();
      fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.p_ready);

      mbar_wait(&tl.o_full, c & 1, dead, err);
      fence_after();
      float o[64];
      float ss = 0.f;
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        float x[16], y[16];
        tmem_ld16(x, tmem + lane_base + kColO + half * 64 + ch * 16);
        tmem_ld16(y, tmem + lane_base + kColI + half * 64 + ch * 16);
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float z = fmaf(wi, y[i], x[i]);
          o[ch * 16 + i] = z;
          ss = fmaf(z, z, ss);
        }
      }
      fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.o_empty);
      tl.ssq[half][row] = ss;
      asm volatile("bar.sync %0, 64;\n" ::"r"(pair_bar) : "memory");
      ss += tl.ssq[half ^ 1][row];
      if (pair > 1) {
        if (half == 0) {
          uint32_t at, bar;
          asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(at) : "r"(smem_u32(&tl.peer[c & 1][row])), "r"((uint32_t)(slice ^ 1)));
          asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(bar) : "r"(smem_u32(&tl.x_full)), "r"((uint32_t)(slice ^ 1)));
          asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(at), "f"(ss) : "memory");
          asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];\n" ::"r"(bar) : "memory");
        }
        mbar_wait_cluster(&tl.x_full, c & 1, dead, err);
        ss += tl.peer[c & 1][row];
      }
      const float inv = v.ssq ? 1.0f : 1.0f / sqrtf(ss / (float)V + v.eps);
      if (row < n) {
        if (v.ssq && half == 0 && slice == 0) v.ssq[t * v.ssq_t + h * v.ssq_h] = ss;
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(v.out) + t * v.ldo + col;
#pragma unroll
        for (int q0 = 0; q0 < 8; q0 += 4) {                                    // four gate vectors in flight
          uint4 gu[4];
#pragma unroll
          for (int q = 0; q < 4; ++q)
            gu[q] = (q0 + q) * 8 < left ? __ldg(reinterpret_cast<const uint4*>(gate + (q0 + q) * 8)) : make_uint4(0, 0, 0, 0);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            uint32_t* gi = reinterpret_cast<uint32_t*>(&gu[q]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float2 g = unpack2bf(gi[e]);
              const int i = (q0 + q) * 8 + 2 * e;
              if (v.out_w && i < left) { const float2 w = __ldg(reinterpret_cast<const float2*>(v.out_w + col + i)); g.x *= w.x; g.y *= w.y; }
              const __nv_bfloat162 r = __floats2bfloat162_rn(o[i] * inv * g.x, o[i + 1] * inv * g.y);
              gi[e] = *reinterpret_cast<const uint32_t*>(&r);
            }
            if ((q0 + q) * 8 < left) *reinterpret_cast<uint4*>(out + (q0 + q) * 8) = gu[q];
          }
        }
      }
    }
  }
  fence_before();
  __syncthreads();
  if (warp == 16) {
    fence_after();
    tmem_dealloc(tmem, 512);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                  const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess && qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(ptr);
    else
      cudaGetLastError();
  }
  return fn;
}
// [T tokens][H heads][width] inside rows of `pitch` elements; a box is 128 tokens x 64 features of one head
int32_t head_map(CUtensorMap* map, const void* base, int width, int H, int T, int pitch) {
  EncodeTiledFn enc = encode_fn();
  if (!enc) return fail(LMB200_ECUDA, "retention: cuTensorMapEncodeTiled is not available");
  const cuuint64_t dims[3] = {(cuuint64_t)width, (cuuint64_t)H, (cuuint64_t)T};
  const cuuint64_t strides[2] = {(cuuint64_t)width * 2, (cuuint64_t)pitch * 2};
  const cuuint32_t box[3] = {64, 1, (cuuint32_t)kT};
  const cuuint32_t estr[3] = {1, 1, 1};
  const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(LMB200_ECUDA, "retention: cuTensorMapEncodeTiled failed (%d)", (int)r);
  return LMB200_OK;
}

}  // namespace

int32_t retention_tc_configure() {
  LMB_CUDA(cudaFuncSetAttribute(retention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmem));
  return LMB200_OK;
}

// heads no wider than a tile; narrow heads (64 x 64 and below) are better off in the 64-token chunks of csrc/retention.cu
bool retention_tc_ok(const RetentionView& v) {
  return retention_chunks_ok(v) && v.dim <= 128 && v.vdim <= 256 && (v.dim > 64 || v.vdim > 64) && v.g_pitch % 8 == 0 && v.ldo % 8 == 0 &&
         v.decay_pitch > kT && v.total > 0;
}

int32_t retention_tc(Ctx* ctx, const RetentionView& v, cudaStream_t st) {
  LMB_REQUIRE(retention_tc_ok(v), "retention: heads of %d x %d have no 128-token kernel", v.dim, v.vdim);
  CUtensorMap qmap, kmap, vmap;
  LMB_TRY(head_map(&qmap, v.q, v.dim, v.H, v.total, v.q_pitch));
  LMB_TRY(head_map(&kmap, v.k, v.dim, v.H, v.total, v.k_pitch));
  LMB_TRY(head_map(&vmap, v.v, v.vdim, v.H, v.total, v.v_pitch));
  const unsigned slices = (unsigned)ceil_div(v.vdim, 128);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, (unsigned)v.H, (unsigned)v.B);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = kSmem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  LMB_CUDA(cudaLaunchKernelEx(&cfg, retention_tc_kernel, v, qmap, kmap, vmap, ctx->dev_err));
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
