// Channel-wise gated delta rule over long portions on the fifth-generation tensor cores: the algorithm of csrc/delta_chunk.cu (chunks of
// 64 tokens; kt, qt, kb, A, B as defined there) with its products on tcgen05.mma and the state in tensor memory.
//
// One CTA per (value head, sequence).  Everything is transposed: the 128 lanes of tensor memory are value columns.  Per chunk
//   [Y | O]^T = S^T [kt | qt]^T        S^T from tensor memory as bf16 pairs hi | lo, kt and qt hi and lo in shared memory
//   X = beta (V - Y),  U^T = X^T T^T   T = (I + A)^-1, 64 x 64
//   O^T += U^T B^T,   S^T = S^T diag(e^{G_end}) + U^T kb
// every product as hi hi + lo hi + hi lo (x = hi + lo to about 2^-17), accumulated in float32.
//   [A | B] = [kt | qt] (k e^{-G})^T   mild chunks, from shared memory; other chunks with mma.sync, block by block
// Mild: no channel decays by more than 2^-160 in the chunk.  There G counts from the middle, G - G_end / 2, so that e^G and e^-G stay within
// 2^80, and the operand of the first product is S e^{G_end / 2}.  (A and B above their diagonals may overflow; those elements are dropped.)
// Tensor memory columns: [Y then U | O] 128, S 128, [S hi | S lo, later X hi | X lo] 128, [U hi | U lo] 64, [A, B] 64 (lanes: tokens).
// Warps: 0-7 own the value columns (two threads per column): they turn S, X and U into operands and write the outputs; 8-15 prepare the
// next chunk (decay sums, kt, qt, kb, A and B, T in float32) while the others work on this one; 16 issues the other MMAs, 17
// and 18 the TMA loads.  All waits are bounded.
#include <cuda.h>

#include "delta.cuh"
#include "mma_sync.cuh"
#include "pdl.cuh"
#include "tc.cuh"

namespace lmb {
namespace {

constexpr int kC = 64, kW = 128;                        // tokens per chunk; head width, padded with zeros
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kDiagMax = 80.0f, kDecayMin = -150.0f;  // as in csrc/delta_chunk.cu
constexpr int kThreads = 19 * 32;
constexpr uint32_t cYO = 0, cS = 128, cSh = 256, cSl = 320, cXh = 256, cXl = 288, cUh = 384, cUl = 416, cBlk = 448;
constexpr int kPv = kW, kPg = kW, kPt = 72;             // row pitches: raw rows, decay sums, float32 A and T
// shared memory; tiles in the 128-byte swizzle
constexpr int kSub = 128 * 128, kSub64 = 64 * 128;      // sub-tiles [128 rows][64 columns], [64 rows][64 columns]
constexpr int oKQh = 0, oKQl = oKQh + 2 * kSub;         // rows 0-63 kt, 64-127 qt
constexpr int oKbh = oKQl + 2 * kSub, oKbl = oKbh + 2 * kSub64;
constexpr int oTh = oKbl + 2 * kSub64, oTl = oTh + kSub64, oBh = oTl + kSub64, oBl = oBh + kSub64;
constexpr int oK = oBl + kSub64, oQ = oK + 2 * kSub64;  // raw rows; mild chunks then k e^{-G} as a tile, hi over K, lo over Q
constexpr int oV = oQ + 2 * kSub64;                     // v, later the outputs on their way out
constexpr int oG = oV + 2 * kSub64;                     // log decays, their sums; later A and T in float32
constexpr int oEnd = oG + 2 * kC * kPt * 4;
static_assert(kC * kPg * 4 <= 2 * kC * kPt * 4 && kC * kPv * 2 <= 2 * kSub64, "what lies over something else fits");
struct Tail {
  uint64_t raw_full, raw_empty, g_full, g_empty, v_full, v_empty, kq_ready, blk_done, tb_ready, kb_ready, s_ready, x_ready, u_ready, yo_done, u_done, o_done, s_done;
  uint32_t tmem;
  alignas(16) float R[5][kW];                           // decay sums before blocks 1 .. 3 of 16 tokens, and of the whole chunk
  alignas(16) float E[2][kW];                           // e^{G_end}, by chunk parity
  alignas(16) float M[2][kW];                           // e^{G_end / 2}, or 1 in other than mild chunks
  float row[2][3][kC];                                  // beta, 1 / |k|, 1 / |q| / sqrt(dim), by chunk parity
  float sum[4][kC];                                     // sums of squares of the outputs per 32 value columns
};
constexpr size_t kSmem = (size_t)oEnd + sizeof(Tail);
static_assert(kSmem <= 227 * 1024 && oEnd % 16 == 0, "shared memory");

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint64_t desc(uint32_t saddr, uint32_t lbo, uint32_t sbo) {       // 128-byte swizzle
  return (uint64_t)((saddr & 0x3FFFF) >> 4) | ((uint64_t)(lbo >> 4) << 16) | ((uint64_t)(sbo >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {        // A from tensor memory
  asm volatile(
      "{\n.reg .pred p;\nsetp.ne.b32 p, %4, 0;\ntcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}\n" ::"r"(d), "r"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
// byte of (row, column) in a swizzled tile of sub-tiles `sub` bytes apart
__device__ __forceinline__ int swz(int row, int col, int sub) { return (col >> 6) * sub + row * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4) + (col & 7) * 2; }
__device__ __forceinline__ void tma_3d(void* dst, const CUtensorMap* map, int c1, int c2, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(tc::smem_u32(dst)),
      "l"(reinterpret_cast<uint64_t>(map)), "r"(0), "r"(c1), "r"(c2), "r"(tc::smem_u32(bar))
      : "memory");
}
// one 16 x 8 tile of A B over 16 ks .. contraction steps, A and B row-major float32 of pitch kPt, operands as bf16 pairs hi + lo
__device__ __forceinline__ void mm_tile(float (&c)[4], const float* A, const float* B, int k0, int k1, int g, int tq) {
  c[0] = c[1] = c[2] = c[3] = 0.f;
  for (int k = k0; k < k1; k += 16) {
    uint32_t ah[4], al[4], bh[2], bl[2];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 x = *reinterpret_cast<const float2*>(A + (g + 8 * (e & 1)) * kPt + k + 2 * tq + 8 * (e >> 1));
      split2(x.x, x.y, ah[e], al[e]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float* x = B + (k + 2 * tq + 8 * e) * kPt + g;
      split2(x[0], x[kPt], bh[e], bl[e]);
    }
    mma16816(c, ah, bh[0], bh[1]);
    mma16816(c, al, bh[0], bh[1]);
    mma16816(c, ah, bl[0], bl[1]);
  }
}
__device__ __forceinline__ void prep_sync() { asm volatile("bar.sync 3, 256;\n" ::: "memory"); }

__global__ void __launch_bounds__(kThreads, 1) delta_tc_kernel(const DeltaView v, const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap qmap,
                                                                const __grid_constant__ CUtensorMap vmap, const __grid_constant__ CUtensorMap gmap, int* err) {
  using namespace tc;
  typedef __nv_bfloat16 bf;
  extern __shared__ __align__(1024) unsigned char smem[];
  Tail& tl = *reinterpret_cast<Tail*>(smem + oEnd);
  bf *sK = (bf*)(smem + oK), *sQ = (bf*)(smem + oQ), *sV = (bf*)(smem + oV);
  float* sG = (float*)(smem + oG);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, b = blockIdx.y, D = v.dim, V = v.vdim, ld = (V + 3) & ~3, a = h / (v.H / v.G);
  if (tid == 0) {
    if (smem_u32(smem) & 1023) atomicExch(err, 1);       // the swizzle needs 1024-byte tiles
    mbar_init(&tl.raw_full, 2); mbar_init(&tl.g_full, 1); mbar_init(&tl.v_full, 1); mbar_init(&tl.blk_done, 1); mbar_init(&tl.yo_done, 1); mbar_init(&tl.u_done, 1); mbar_init(&tl.o_done, 1); mbar_init(&tl.s_done, 1);
    mbar_init(&tl.raw_empty, 8); mbar_init(&tl.g_empty, 8); mbar_init(&tl.v_empty, 8); mbar_init(&tl.kb_ready, 8); mbar_init(&tl.kq_ready, 8); mbar_init(&tl.tb_ready, 8);
    mbar_init(&tl.s_ready, 8); mbar_init(&tl.x_ready, 8); mbar_init(&tl.u_ready, 8);
    mbar_init_fence();
  }
  // what lies behind the widths and above the triangles stays zero
  for (int i = tid; i < (oG - oTh) / 16; i += kThreads) reinterpret_cast<uint4*>(smem + oTh)[i] = make_uint4(0, 0, 0, 0);
  fence_async_smem();
  if (warp == 16) tmem_alloc(&tl.tmem, 512);
  fence_before();
  __syncthreads();
  fence_after();
  const uint32_t tmem = tl.tmem;
  pdl_launch_dependents();
  pdl_wait();
  bool dead = false;
  const int n_all = v.len[b], t_first = v.start[b];
  const int chunks = (n_all + kC - 1) / kC;              // 0: nothing to do

  if (warp >= 17) {
    // ------------------------------ rows of log g, k and q; of v.  What a box takes in behind the portion counts as zero (beta, decay) ------------------------------
    for (int c = 0; c < chunks; ++c) {
      const int t0 = t_first + c * kC;
      if (warp == 17) {
        mbar_wait(&tl.g_empty, (c & 1) ^ 1, dead, err);
        if (lane == 0) {
          mbar_expect_tx(&tl.g_full, kC * kW * 4);
          tma_3d(sG, &gmap, h, t0, &tl.g_full);
        }
        mbar_wait(&tl.raw_empty, (c & 1) ^ 1, dead, err);
        if (lane == 0) {
          mbar_expect_tx(&tl.raw_full, 2 * kC * kW * 2);
          tma_3d(sK, &kmap, a, t0, &tl.raw_full);
          tma_3d(sQ, &qmap, a, t0, &tl.raw_full);
        }
        float (*row)[kC] = tl.row[c & 1];                // the tokens' scalars go with them
#pragma unroll
        for (int r = lane; r < kC; r += 32) {
          const bool ok = c * kC + r < n_all;
          const int64_t t = (int64_t)t0 + (ok ? r : 0);
          const float x = v.b[t * v.b_pitch + h], y = v.rk[t * v.G + a], z = v.rq[t * v.G + a];
          row[0][r] = ok ? 1.0f / (1.0f + expf(-x)) : 0.f;
          row[1][r] = ok ? y : 0.f;
          row[2][r] = ok ? z : 0.f;
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&tl.raw_full);
      } else {
        mbar_wait(&tl.v_empty, (c & 1) ^ 1, dead, err);
        if (lane == 0) {
          mbar_expect_tx(&tl.v_full, kC * kW * 2);
          tma_3d(sV, &vmap, h, t0, &tl.v_full);
        }
      }
    }
    __syncwarp();
  } else if (warp == 16) {
    // ------------------------------ MMA issue ------------------------------
    constexpr uint32_t kN128 = idesc_bf16(128, 128, false, false), kN64 = idesc_bf16(128, 64, false, false), kN128m = idesc_bf16(128, 128, false, true);
    const uint32_t base = smem_u32(smem);
    for (int c = 0; c < chunks; ++c) {
      mbar_wait(&tl.kq_ready, c & 1, dead, err);
      mbar_wait(&tl.s_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
#pragma unroll
        for (int p = 0; p < 3; ++p)                      // hi hi, lo hi, hi lo
          for (int ks = 0; ks < 8; ++ks)
            mma_ts(tmem + cYO, tmem + (p == 1 ? cSl : cSh) + ks * 8, desc(base + (p == 2 ? oKQl : oKQh) + (ks >> 2) * kSub + (ks & 3) * 32, 16, 1024), kN128, p | ks ? 1u : 0u);
        commit(&tl.yo_done);
      }
      __syncwarp();
      mbar_wait(&tl.tb_ready, c & 1, dead, err);
      mbar_wait(&tl.x_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
#pragma unroll
        for (int p = 0; p < 3; ++p)
          for (int ks = 0; ks < 4; ++ks)
            mma_ts(tmem + cYO, tmem + (p == 1 ? cXl : cXh) + ks * 8, desc(base + (p == 2 ? oTl : oTh) + ks * 32, 16, 1024), kN64, p | ks ? 1u : 0u);
        commit(&tl.u_done);
      }
      __syncwarp();
      mbar_wait(&tl.u_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
#pragma unroll
        for (int p = 0; p < 3; ++p)
          for (int ks = 0; ks < 4; ++ks)
            mma_ts(tmem + cYO + 64, tmem + (p == 1 ? cUl : cUh) + ks * 8, desc(base + (p == 2 ? oBl : oBh) + ks * 32, 16, 1024), kN64, 1u);
        commit(&tl.o_done);
      }
      __syncwarp();
      mbar_wait(&tl.kb_ready, c & 1, dead, err);
      fence_after();
      if (lane == 0) {
#pragma unroll
        for (int p = 0; p < 3; ++p)
          for (int ks = 0; ks < 4; ++ks)
            mma_ts(tmem + cS, tmem + (p == 1 ? cUl : cUh) + ks * 8, desc(base + (p == 2 ? oKbl : oKbh) + ks * 2048, kSub64, 1024), kN128m, 1u);
        commit(&tl.s_done);
      }
      __syncwarp();
    }
  } else if (warp >= 8) {
    // ------------------------------ preparation of a chunk ------------------------------
    const int pt = tid - 256, pw = warp - 8, g = lane >> 2, tq = lane & 3;
    const int ch = pt >> 1, hf = pt & 1;                 // decay sums: channel, half of the chunk
    const int quad = warp & 3, side = pw >> 2;           // A and B: 32 rows of [A | B], half of their columns
    int n_mild = 0;                                      // phases of blk_done
    for (int c = 0; c < chunks; ++c) {
      const int n = min(kC, n_all - c * kC);
      const float *beta = tl.row[c & 1][0], *rk = tl.row[c & 1][1], *rq = tl.row[c & 1][2];
      float* E = tl.E[c & 1];
      // ---- decay sums (log2 units): in sG from the start of each block of 16 tokens, in R before the block
      mbar_wait(&tl.g_full, c & 1, dead, err);
      float tot[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        float gl[16], s = 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) gl[r] = ch < D && hf * 32 + q * 16 + r < n ? sG[(hf * 32 + q * 16 + r) * kPg + ch] : 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          s += fmaxf(gl[r] * kLog2e, kDecayMin);
          sG[(hf * 32 + q * 16 + r) * kPg + ch] = s;
        }
        tot[q] = s;
      }
      const float mine = tot[0] + tot[1], other = __shfl_xor_sync(0xffffffffu, mine, 1), before = hf ? other : 0.f;
      if (hf) tl.R[2][ch] = before;
      tl.R[hf ? 3 : 1][ch] = before + tot[0];
      const float all = hf ? other + mine : mine + other;
      if (!hf) {
        tl.R[4][ch] = all;
        E[ch] = ex2(all);
      }
      int mild;
      {                                                  // over the preparing warps
        int p = all >= -2 * kDiagMax;
        asm volatile("{\n.reg .pred p, q;\nsetp.ne.s32 p, %1, 0;\nbarrier.red.and.pred q, 3, 256, p;\nselp.s32 %0, 1, 0, q;\n}\n" : "=r"(mild) : "r"(p) : "memory");
      }
      if (!hf) tl.M[c & 1][ch] = mild ? ex2(0.5f * all) : 1.f;
      // ---- kt, qt, and k e^{-G} over the raw rows
      mbar_wait(&tl.raw_full, c & 1, dead, err);
      if (c) mbar_wait(&tl.yo_done, (c - 1) & 1, dead, err);
      {
        uint2 mh[8], ml[8];
        float4 mid = make_float4(0.f, 0.f, 0.f, 0.f);
        if (mild) {
          mid = *reinterpret_cast<const float4*>(&tl.R[4][(pt & 31) * 4]);
          mid.x *= 0.5f; mid.y *= 0.5f; mid.z *= 0.5f; mid.w *= 0.5f;
        }
#pragma unroll
        for (int it = 0; it < 8; ++it) {
          const int r = (pt >> 5) + 8 * it, d = (pt & 31) * 4, at = r * kW + d;
          const float4 L = *reinterpret_cast<const float4*>(sG + r * kPg + d);
          const float4 Rv = it < 2 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(&tl.R[it >> 1][d]);
          uint2 ku = *reinterpret_cast<const uint2*>(sK + at), qu = *reinterpret_cast<const uint2*>(sQ + at);
          if (d >= D) {                                  // behind the width: whatever lay over the raw rows before
            ku = qu = make_uint2(0u, 0u);
            if (!mild) *reinterpret_cast<uint2*>(sK + at) = *reinterpret_cast<uint2*>(sQ + at) = ku;
          }
          const float2 k0 = unpack_bf16(ku.x), k1 = unpack_bf16(ku.y), q0 = unpack_bf16(qu.x), q1 = unpack_bf16(qu.y);
          const float kr = rk[r], qr = rq[r];
          const float G[4] = {Rv.x + L.x - mid.x, Rv.y + L.y - mid.y, Rv.z + L.z - mid.z, Rv.w + L.w - mid.w};
          const float k[4] = {k0.x * kr, k0.y * kr, k1.x * kr, k1.y * kr}, q[4] = {q0.x * qr, q0.y * qr, q1.x * qr, q1.y * qr};
          float e[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) e[j] = ex2(G[j]);
          const int to = swz(r, d, kSub);
          uint2 hi, lo;
          split2(k[0] * e[0], k[1] * e[1], hi.x, lo.x);
          split2(k[2] * e[2], k[3] * e[3], hi.y, lo.y);
          *reinterpret_cast<uint2*>(smem + oKQh + to) = hi;
          *reinterpret_cast<uint2*>(smem + oKQl + to) = lo;
          split2(q[0] * e[0], q[1] * e[1], hi.x, lo.x);
          split2(q[2] * e[2], q[3] * e[3], hi.y, lo.y);
          *reinterpret_cast<uint2*>(smem + oKQh + to + 64 * 128) = hi;
          *reinterpret_cast<uint2*>(smem + oKQl + to + 64 * 128) = lo;
          if (mild) {
            split2(k[0] * ex2(-G[0]), k[1] * ex2(-G[1]), mh[it].x, ml[it].x);
            split2(k[2] * ex2(-G[2]), k[3] * ex2(-G[3]), mh[it].y, ml[it].y);
          }
        }
        if (mild) {
          prep_sync();                                   // every raw row has been read
#pragma unroll
          for (int it = 0; it < 8; ++it) {
            const int to = swz((pt >> 5) + 8 * it, (pt & 31) * 4, kSub64);
            *reinterpret_cast<uint2*>(smem + oK + to) = mh[it];
            *reinterpret_cast<uint2*>(smem + oQ + to) = ml[it];
          }
        }
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.kq_ready);
      prep_sync();
      if (mild && pt == 0) {
        constexpr uint32_t kN64 = idesc_bf16(128, 64, false, false);
        const uint32_t base = smem_u32(smem);
        fence_after();
#pragma unroll
        for (int p = 0; p < 3; ++p)
          for (int ks = 0; ks < 8; ++ks)
            mma_f16(tmem + cBlk, desc(base + (p == 1 ? oKQl : oKQh) + (ks >> 2) * kSub + (ks & 3) * 32, 16, 1024),
                    desc(base + (p == 2 ? oQ : oK) + (ks >> 2) * kSub64 + (ks & 3) * 32, 16, 1024), kN64, p | ks ? 1u : 0u);
        commit(&tl.blk_done);
      }
      __syncwarp();
      // ---- A and B of other than mild chunks: 16 x 16 blocks in registers, first one per warp (0-3 on the diagonal), then the A or the B
      // part of two more
      auto block_of = [](int task, int* rt, int* st) {
        const int off = task - 4;
        *rt = task < 4 ? task : off == 0 ? 1 : off < 3 ? 2 : 3;
        *st = task < 4 ? task : off == 0 ? 0 : off < 3 ? off - 1 : off - 3;
      };
      auto block = [&](int rt, int st, bool do_a, bool do_b, float (&ca)[2][4], float (&cb)[2][4]) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) ca[j][e] = cb[j][e] = 0.f;
        if (16 * rt >= n) return;
        const bool diag = rt == st;
        {
          bool direct = false;
          if (diag) {
            float m = 0.f;
            for (int d = lane; d < kW; d += 32) m = fmaxf(m, -sG[(rt * 16 + 15) * kPg + d]);
            direct = __any_sync(0xffffffffu, !(m <= kDiagMax));
          }
          if (!direct) {
#pragma unroll 1
            for (int kk = 0; kk < 8; ++kk) {
              uint32_t xh[4], xl[4], bh[4], bl[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) {              // B operand: column tile e >> 1, channels 2 tq + 8 (e & 1)
                const int r = st * 16 + g + 8 * (e >> 1), d = kk * 16 + 2 * tq + 8 * (e & 1);
                const float2 G = *reinterpret_cast<const float2*>(sG + r * kPg + d), Rt = rt ? *reinterpret_cast<const float2*>(&tl.R[rt][d]) : make_float2(0.f, 0.f);
                const float2 Rs = st ? *reinterpret_cast<const float2*>(&tl.R[st][d]) : make_float2(0.f, 0.f);
                const float2 k = unpack_bf16(*reinterpret_cast<const uint32_t*>(sK + r * kW + d));
                split2(k.x * ex2(Rt.x - Rs.x - G.x), k.y * ex2(Rt.y - Rs.y - G.y), bh[e], bl[e]);
              }
#pragma unroll
              for (int part = 0; part < 2; ++part) {
                if (part == 0 ? !do_a : !do_b) continue;
                const bf* src = part == 0 ? sK : sQ;
                float (&cc)[2][4] = part == 0 ? ca : cb;
#pragma unroll
                for (int e = 0; e < 4; ++e) {            // A operand: rows g + 8 (e & 1), channels 2 tq + 8 (e >> 1)
                  const int r = rt * 16 + g + 8 * (e & 1), d = kk * 16 + 2 * tq + 8 * (e >> 1);
                  const float2 G = *reinterpret_cast<const float2*>(sG + r * kPg + d), x = unpack_bf16(*reinterpret_cast<const uint32_t*>(src + r * kW + d));
                  split2(x.x * ex2(G.x), x.y * ex2(G.y), xh[e], xl[e]);
                }
                mma16816(cc[0], xh, bh[0], bh[1]); mma16816(cc[1], xh, bh[2], bh[3]);
                mma16816(cc[0], xl, bh[0], bh[1]); mma16816(cc[1], xl, bh[2], bh[3]);
                mma16816(cc[0], xh, bl[0], bl[1]); mma16816(cc[1], xh, bl[2], bl[3]);
              }
            }
          } else {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const int r = rt * 16 + g + 8 * (e >> 1), s = rt * 16 + 8 * j + 2 * tq + (e & 1);
                if (s > r) continue;
                float x = 0.f, y = 0.f;
                for (int d = 0; d < D; ++d) {
                  const float w = __bfloat162float(sK[s * kW + d]) * ex2(sG[r * kPg + d] - sG[s * kPg + d]);
                  x = fmaf(__bfloat162float(sK[r * kW + d]), w, x);
                  y = fmaf(__bfloat162float(sQ[r * kW + d]), w, y);
                }
                ca[j][e] = x;
                cb[j][e] = y;
              }
          }
        }
        // scales and the triangle
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int tl_ = g + 8 * (e >> 1), sl = 8 * j + 2 * tq + (e & 1), t = rt * 16 + tl_, s = st * 16 + sl;
            ca[j][e] *= beta[t] * rk[t] * rk[s];
            cb[j][e] *= rq[t] * rk[s];
            if (diag && sl >= tl_) ca[j][e] = 0.f;
            if (diag && sl > tl_) cb[j][e] = 0.f;
          }
      };
      auto write_kb = [&]() {
#pragma unroll 4
        for (int it = 0; it < 8; ++it) {
          const int r = (pt >> 5) + 8 * it, d = (pt & 31) * 4, to = swz(r, d, kSub64);
          float2 k0, k1;
          float f[4];
          if (mild) {
            const float4 X = *reinterpret_cast<const float4*>(&tl.M[c & 1][d]);
            const uint2 ku = *reinterpret_cast<const uint2*>(smem + oK + to), lu = *reinterpret_cast<const uint2*>(smem + oQ + to);
            const float2 l0 = unpack_bf16(lu.x), l1 = unpack_bf16(lu.y);
            k0 = unpack_bf16(ku.x); k1 = unpack_bf16(ku.y);
            k0.x += l0.x; k0.y += l0.y; k1.x += l1.x; k1.y += l1.y;
            f[0] = X.x; f[1] = X.y; f[2] = X.z; f[3] = X.w;
          } else {
            const uint2 ku = *reinterpret_cast<const uint2*>(sK + r * kW + d);
            const float4 L = *reinterpret_cast<const float4*>(sG + r * kPg + d), all4 = *reinterpret_cast<const float4*>(&tl.R[4][d]);
            const float4 Rv = it < 2 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(&tl.R[it >> 1][d]);
            const float kr = rk[r];
            k0 = unpack_bf16(ku.x); k1 = unpack_bf16(ku.y);
            f[0] = kr * ex2(all4.x - Rv.x - L.x); f[1] = kr * ex2(all4.y - Rv.y - L.y); f[2] = kr * ex2(all4.z - Rv.z - L.z); f[3] = kr * ex2(all4.w - Rv.w - L.w);
          }
          uint2 hi, lo;
          split2(k0.x * f[0], k0.y * f[1], hi.x, lo.x);
          split2(k1.x * f[2], k1.y * f[3], hi.y, lo.y);
          *reinterpret_cast<uint2*>(smem + oKbh + to) = hi;
          *reinterpret_cast<uint2*>(smem + oKbl + to) = lo;
        }
      };
      // ---- A in float32 over the decay sums, B as an operand
      float *sA = sG, *sT = sG + kC * kPt;
      if (mild) {
        if (c) mbar_wait(&tl.s_done, (c - 1) & 1, dead, err);   // all products of the chunk before: kb, T and B are free
        write_kb();                                      // while A and B are multiplied
        mbar_wait(&tl.blk_done, n_mild++ & 1, dead, err);
        fence_after();
        float x[32];
        tmem_ld32(x, tmem + ((uint32_t)(32 * quad) << 16) + cBlk + side * 32);
        fence_before();
        const int t = 32 * (quad & 1) + lane, s0 = side * 32;
        if (quad < 2) {
          const float bt = beta[t];
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const auto z = [&](int j) { return s0 + i + j < t ? x[i + j] * bt : 0.f; };
            *reinterpret_cast<float4*>(sA + t * kPt + s0 + i) = make_float4(z(0), z(1), z(2), z(3));
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 hi, lo;
            const auto z = [&](int j) { return s0 + i + j <= t ? x[i + j] : 0.f; };
            split2(z(0), z(1), hi.x, lo.x); split2(z(2), z(3), hi.y, lo.y); split2(z(4), z(5), hi.z, lo.z); split2(z(6), z(7), hi.w, lo.w);
            const int to = swz(t, s0 + i, 0);
            *reinterpret_cast<uint4*>(smem + oBh + to) = hi;
            *reinterpret_cast<uint4*>(smem + oBl + to) = lo;
          }
        }
      } else {
        float a1[2][4], b1[2][4], a2[2][4], b2[2][4];
        int rt1, st1, rt2 = 0, st2 = 0;
        block_of(pw, &rt1, &st1);
        block(rt1, st1, true, true, a1, b1);
        if (pw < 4) {
          block_of(8 + (pw >> 1), &rt2, &st2);
          block(rt2, st2, (pw & 1) == 0, pw & 1, a2, b2);
        }
        if (c) mbar_wait(&tl.s_done, (c - 1) & 1, dead, err);
        write_kb();
        auto put_b = [&](int rt, int st, const float (&cb)[2][4]) {
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e2 = 0; e2 < 2; ++e2) {
              uint32_t hi, lo;
              split2(cb[j][2 * e2], cb[j][2 * e2 + 1], hi, lo);
              const int to = swz(rt * 16 + g + 8 * e2, st * 16 + 8 * j + 2 * tq, 0);
              *reinterpret_cast<uint32_t*>(smem + oBh + to) = hi;
              *reinterpret_cast<uint32_t*>(smem + oBl + to) = lo;
            }
        };
        put_b(rt1, st1, b1);
        if (pw < 4 && (pw & 1)) put_b(rt2, st2, b2);
        prep_sync();                                     // decay sums and raw rows have been read
        auto put_a = [&](int rt, int st, const float (&ca)[2][4]) {
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e2 = 0; e2 < 2; ++e2)
              *reinterpret_cast<float2*>(sA + (rt * 16 + g + 8 * e2) * kPt + st * 16 + 8 * j + 2 * tq) = make_float2(ca[j][2 * e2], ca[j][2 * e2 + 1]);
        };
        put_a(rt1, st1, a1);
        if (pw < 4 && (pw & 1) == 0) put_a(rt2, st2, a2);
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) { mbar_arrive(&tl.kb_ready); mbar_arrive(&tl.raw_empty); }
      prep_sync();
      // ---- T = (I + A)^-1: 16 x 16 diagonal blocks, then twice [[P, 0], [R, Q]]^-1 = [[P', 0], [-Q' R P', Q']]
      if (pw < 4) {
        const float* M = sA + (pw * 16) * kPt + pw * 16;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float y = i == (lane & 15) ? 1.f : 0.f;
#pragma unroll
          for (int k = 0; k < i; ++k) y = fmaf(-M[i * kPt + k], x[k], y);
          x[i] = y;
        }
        if (lane < 16) {
#pragma unroll
          for (int i = 0; i < 16; ++i) sT[(pw * 16 + i) * kPt + pw * 16 + lane] = x[i];
        }
      }
      prep_sync();
      auto put_tile = [&](float* to, const float (&x)[4], float sign) {
        *reinterpret_cast<float2*>(to + g * kPt + 2 * tq) = make_float2(sign * x[0], sign * x[1]);
        *reinterpret_cast<float2*>(to + (g + 8) * kPt + 2 * tq) = make_float2(sign * x[2], sign * x[3]);
      };
      {                                                  // R P' of the two 32-blocks, into the empty blocks above the diagonal; then -Q' of it
        float x[4];
        const int blk = (pw >> 1) & 1, n0 = (pw & 1) * 8;
        float *D0 = sT + blk * 32 * kPt + blk * 32, *D1 = D0 + 16 * kPt + 16, *up = D0 + 16, *low = D0 + 16 * kPt;
        if (pw < 4) {
          mm_tile(x, sA + (blk * 32 + 16) * kPt + blk * 32, D0 + n0, 0, 16, g, tq);
          put_tile(up + n0, x, 1.f);
          __syncwarp();                                  // a warp reads only the columns it wrote
          mm_tile(x, D1, up + n0, 0, 16, g, tq);
          put_tile(low + n0, x, -1.f);
        }
      }
      prep_sync();
      {                                                  // the same for the halves; P' and Q' are zero above their diagonal blocks (scratch lies there)
        float x[4];
        const int m0 = (pw >> 2) * 16, n0 = (pw & 3) * 8;
        mm_tile(x, sA + (32 + m0) * kPt, sT + n0, n0 & 16, 32, g, tq);
        put_tile(sT + m0 * kPt + 32 + n0, x, 1.f);
        prep_sync();
        mm_tile(x, sT + (32 + m0) * kPt + 32, sT + 32 + n0, 0, m0 + 16, g, tq);
        put_tile(sT + (32 + m0) * kPt + n0, x, -1.f);
      }
      prep_sync();
      {                                                  // sixteen elements of a row, zero above the triangle
        const int r = pt >> 2, c0 = (pt & 3) * 16;
        const bool in = c0 <= r;
#pragma unroll
        for (int i = 0; i < 16; i += 8) {
          const float* x = sT + r * kPt + c0 + i;
          uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
          if (in) {
            const float4 x0 = *reinterpret_cast<const float4*>(x), x1 = *reinterpret_cast<const float4*>(x + 4);
            split2(x0.x, x0.y, hi.x, lo.x); split2(x0.z, x0.w, hi.y, lo.y); split2(x1.x, x1.y, hi.z, lo.z); split2(x1.z, x1.w, hi.w, lo.w);
          }
          const int to = swz(r, c0 + i, 0);
          *reinterpret_cast<uint4*>(smem + oTh + to) = hi;
          *reinterpret_cast<uint4*>(smem + oTl + to) = lo;
        }
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) { mbar_arrive(&tl.tb_ready); mbar_arrive(&tl.g_empty); }
    }
  } else {
    // ------------------------------ value columns ------------------------------
    const int half = warp >> 2, quad = warp & 3, col = 32 * quad + lane;
    const uint32_t lanes = tmem + ((uint32_t)(32 * quad) << 16);
    float* state = v.state + ((int64_t)b * v.H + h) * D * ld + col;
    const float wn = col < V ? __ldg(v.norm + col) : 0.f;
    for (int c = 0; c < chunks; ++c) {
      const int n = min(kC, n_all - c * kC);
      const int64_t t0 = t_first + (int64_t)c * kC + half * 32;
      const float *beta = tl.row[c & 1][0] + half * 32, *E = tl.E[c & 1], *M = tl.M[c & 1];
      // ---- S as an operand, and decayed
      mbar_wait(&tl.kq_ready, c & 1, dead, err);
      if (c) { mbar_wait(&tl.s_done, (c - 1) & 1, dead, err); fence_after(); }
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float x[16];
        const int d0 = half * 64 + q * 16;
        if (c == 0) {
#pragma unroll
          for (int i = 0; i < 16; ++i) x[i] = d0 + i < D && col < V ? state[(int64_t)(d0 + i) * ld] : 0.f;
        } else {
          tmem_ld16(x, lanes + cS + d0);
        }
        uint32_t hi[8], lo[8], u[16];
#pragma unroll
        for (int i = 0; i < 16; i += 2) split2(x[i] * M[d0 + i], x[i + 1] * M[d0 + i + 1], hi[i / 2], lo[i / 2]);
#pragma unroll
        for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(x[i] * E[d0 + i]);
        tmem_st16_nowait(lanes + cS + d0, u);
        asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};\n" ::"r"(lanes + cSh + d0 / 2), "r"(hi[0]), "r"(hi[1]), "r"(hi[2]), "r"(hi[3]),
                     "r"(hi[4]), "r"(hi[5]), "r"(hi[6]), "r"(hi[7]) : "memory");
        asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};\n" ::"r"(lanes + cSl + d0 / 2), "r"(lo[0]), "r"(lo[1]), "r"(lo[2]), "r"(lo[3]),
                     "r"(lo[4]), "r"(lo[5]), "r"(lo[6]), "r"(lo[7]) : "memory");
      }
      tmem_st_wait();
      fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.s_ready);
      // ---- X
      mbar_wait(&tl.v_full, c & 1, dead, err);
      float x[32];
      uint32_t hi[16], lo[16];
      {
        bf vv[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) vv[i] = col < V ? sV[(half * 32 + i) * kPv + col] : __float2bfloat16_rn(0.f);
        mbar_wait(&tl.yo_done, c & 1, dead, err);
        fence_after();
        tmem_ld32(x, lanes + cYO + half * 32);
#pragma unroll
        for (int i = 0; i < 32; i += 2)
          split2(beta[i] * (__bfloat162float(vv[i]) - x[i]), beta[i + 1] * (__bfloat162float(vv[i + 1]) - x[i + 1]), hi[i / 2], lo[i / 2]);
      }
      tmem_st16_nowait(lanes + cXh + half * 16, hi);
      tmem_st16_nowait(lanes + cXl + half * 16, lo);
      tmem_st_wait();
      fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.x_ready);
      // the gates of the output pieces this thread will store: pass p, rows of half a chunk's quarter, eight value columns
      const int hr = tid & 127, piece = (hr & 15) * 8;   // 128 threads: 8 rows x 16 pieces at a time
      uint4 gates[4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const int r = p * 8 + (hr >> 4);
        gates[p] = half * 32 + r < n && piece < V ? __ldg(reinterpret_cast<const uint4*>(reinterpret_cast<const bf*>(v.gate) + (t0 + r) * v.gate_pitch + h * V + piece))
                                                  : make_uint4(0, 0, 0, 0);
      }
      mbar_wait(&tl.u_done, c & 1, dead, err);
      fence_after();
      tmem_ld32(x, lanes + cYO + half * 32);
#pragma unroll
      for (int i = 0; i < 32; i += 2) split2(x[i], x[i + 1], hi[i / 2], lo[i / 2]);
      tmem_st16_nowait(lanes + cUh + half * 16, hi);
      tmem_st16_nowait(lanes + cUl + half * 16, lo);
      tmem_st_wait();
      fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.u_ready);
      // ---- outputs: lane i ends with token i's sum of squares over the warp's 32 value columns
      mbar_wait(&tl.o_done, c & 1, dead, err);
      fence_after();
      tmem_ld32(x, lanes + cYO + 64 + half * 32);
      float ss[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) ss[i] = x[i] * x[i];
#pragma unroll
      for (int w = 16; w > 0; w >>= 1) {
        const bool up = (lane & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) {
          const float send = up ? ss[i] : ss[i + w], keep = up ? ss[i + w] : ss[i];
          ss[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
        }
      }
      tl.sum[quad][half * 32 + lane] = ss[0];
      asm volatile("bar.sync %0, 128;\n" ::"r"(1 + half) : "memory");
      const float all = tl.sum[0][half * 32 + lane] + tl.sum[1][half * 32 + lane] + tl.sum[2][half * 32 + lane] + tl.sum[3][half * 32 + lane];
      const float inv = 1.0f / sqrtf(all / (float)V + v.eps);
      // turned through the place of v, sixteen tokens at a time: [16][128] float32 per half, then whole pieces of token rows
      float* stage = reinterpret_cast<float*>(smem + oV) + half * 16 * kW;
#pragma unroll
      for (int p = 0; p < 2; ++p) {
#pragma unroll
        for (int i = 0; i < 16; ++i) stage[i * kW + col] = x[p * 16 + i] * __shfl_sync(0xffffffffu, inv, p * 16 + i) * wn;
        asm volatile("bar.sync %0, 128;\n" ::"r"(1 + half) : "memory");
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int rl = q * 8 + (hr >> 4), r = p * 16 + rl;
          const float4 y0 = *reinterpret_cast<const float4*>(stage + rl * kW + piece), y1 = *reinterpret_cast<const float4*>(stage + rl * kW + piece + 4);
          uint4 gu = gates[p * 2 + q];
          const float y[8] = {y0.x, y0.y, y0.z, y0.w, y1.x, y1.y, y1.z, y1.w};
          uint32_t* gi = reinterpret_cast<uint32_t*>(&gu);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 gt = unpack_bf16(gi[e]);
            const __nv_bfloat162 o = __floats2bfloat162_rn(y[2 * e] * gt.x, y[2 * e + 1] * gt.y);
            gi[e] = *reinterpret_cast<const uint32_t*>(&o);
          }
          if (half * 32 + r < n && piece < V) *reinterpret_cast<uint4*>(reinterpret_cast<bf*>(v.out) + (t0 + r) * v.ldo + h * V + piece) = gu;
        }
        asm volatile("bar.sync %0, 128;\n" ::"r"(1 + half) : "memory");
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tl.v_empty);
    }
    if (chunks > 0) {
      mbar_wait(&tl.s_done, (chunks - 1) & 1, dead, err);
      fence_after();
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float x[16];
        const int d0 = half * 64 + q * 16;
        tmem_ld16(x, lanes + cS + d0);
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (d0 + i < D && col < V) state[(int64_t)(d0 + i) * ld] = x[i];
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
// [T tokens][heads][width] inside rows of `pitch` elements; a box is 64 tokens x 128 features of one head, rows dense, zeros behind the width
int32_t rows_map(CUtensorMap* map, const void* base, bool f32, int width, int heads, int T, int pitch) {
  static EncodeTiledFn enc = nullptr;
  if (!enc) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) != cudaSuccess || qres != cudaDriverEntryPointSuccess) {
      cudaGetLastError();
      return fail(LMB200_ECUDA, "delta rule: cuTensorMapEncodeTiled is not available");
    }
    enc = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  const int e = f32 ? 4 : 2;
  const cuuint64_t dims[3] = {(cuuint64_t)width, (cuuint64_t)heads, (cuuint64_t)T};
  const cuuint64_t strides[2] = {(cuuint64_t)width * e, (cuuint64_t)pitch * e};
  const cuuint32_t box[3] = {(cuuint32_t)kW, 1, (cuuint32_t)kC};
  const cuuint32_t estr[3] = {1, 1, 1};
  const CUresult r = enc(map, f32 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT32 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(LMB200_ECUDA, "delta rule: cuTensorMapEncodeTiled failed (%d)", (int)r);
  return LMB200_OK;
}

}  // namespace

int32_t delta_tc_configure() {
  LMB_CUDA(cudaFuncSetAttribute(delta_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmem));
  return LMB200_OK;
}

// heads no wider than a tile; narrow ones (64 x 64 and below) are better off in csrc/delta_chunk.cu
bool delta_tc_ok(const DeltaView& v) { return delta_chunks_ok(v) && (v.dim > 64 || v.vdim > 64); }

int32_t delta_tc(Ctx* ctx, const DeltaView& v, cudaStream_t st) {
  LMB_REQUIRE(delta_tc_ok(v), "delta rule: heads of %d x %d have no kernel on tcgen05", v.dim, v.vdim);
  CUtensorMap kmap, qmap, vmap, gmap;
  LMB_TRY(rows_map(&kmap, v.k, false, v.dim, v.G, v.total, v.k_pitch));
  LMB_TRY(rows_map(&qmap, v.q, false, v.dim, v.G, v.total, v.q_pitch));
  LMB_TRY(rows_map(&vmap, v.v, false, v.vdim, v.H, v.total, v.v_pitch));
  LMB_TRY(rows_map(&gmap, v.decay, true, v.dim, v.H, v.total, v.decay_pitch));
  LMB_CUDA(launch_k(delta_tc_kernel, dim3((unsigned)v.H, (unsigned)v.B), dim3(kThreads), kSmem, st, v, kmap, qmap, vmap, gmap, ctx->dev_err));
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
