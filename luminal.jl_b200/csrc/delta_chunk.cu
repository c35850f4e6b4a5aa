// Channel-wise gated delta rule over long portions, in chunks of 64 tokens on the tensor cores (see delta.cuh).
//
// One CTA per (value head, sequence); log decays are summed up along the chunk, G_t = sum of log g up to and with t.  With
//   kt_t = k_t e^{G_t},  qt_t = q_t e^{G_t},  kb_s = k_s e^{G_end - G_s}
//   A_ts = beta_t sum_d k_t k_s e^{G_t - G_s} (s < t),   B_ts = sum_d q_t k_s e^{G_t - G_s} (s <= t)
// the recurrence is
//   (I + A) U = beta (V - kt S),   O = qt S + B U,   S <- diag(e^{G_end}) S + kb^T U
// A and B for any decays: where a whole chunk decays by no more than 2^-kDiagMax, they are products of kt, qt and k_s e^{-G_s}.  Else the
// rows t of a 16-token block are taken relative to the block's start R, e^{G_t - R} e^{R - G_s}, and no exponent is positive for s in an
// earlier block; inside the block the second factor grows, again no further than 2^kDiagMax, or its 16 x 16 sums are taken term by term.  (I + A) is solved block by block with the inverses of its 16 x 16 diagonal blocks.
// Everything the decays or the state touch enters the products as bf16 pairs hi + lo (x to about 2^-17) in three products.
// All products are taken transposed (M = 16 value columns): a warp owns 16 value columns, its part of the state stays in its
// accumulator registers over the whole portion and is an A operand without a move, and so is U; warps meet only to share
// kt, qt, kb, A and B.
#include "delta.cuh"
#include "mma_sync.cuh"
#include "pdl.cuh"
#include "tc.cuh"

namespace lmb {
namespace {

constexpr int kC = 64, kB = kC / 16;
constexpr int kBlk = 16 * 24;                       // elements of a 16 x 16 block of A, B or an inverse (rows of 48 bytes: no bank conflicts)
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kDiagMax = 80.0f;                   // log2 units: e^{R - G_s} up to 2^80
constexpr float kDecayMin = -150.0f;                // a factor below any float32

template <int DK, int DV>
struct Smem {
  static constexpr int kWarps = DV / 16, kThreads = 32 * kWarps;
  static constexpr int pk = DK + 8, pv = DV + 8, pg = DK + 4, po = DV + 4;
  static constexpr int kRow = kC * pk * 2;          // bytes of one [64][pk] bf16 matrix
  static constexpr int oKt = 0, oQt = oKt + 2 * kRow, oKb = oQt + 2 * kRow;          // hi then lo each
  static constexpr int oA = oKb + 2 * kRow;                                          // 6 blocks below the diagonal, hi then lo
  static constexpr int oB = oA + 2 * 6 * kBlk * 2;                                   // 10 blocks
  static constexpr int oT = oB + 2 * 10 * kBlk * 2;                                  // 4 inverses
  static constexpr int oK = oT + 2 * 4 * kBlk * 2, oQ = oK + kRow, oG = oQ + kRow;   // raw rows; G float32
  static constexpr int oV = oG + kC * pg * 4;
  static constexpr int oD = oV + kC * pv * 2;                                        // 4 diagonal blocks float32 [16][17]
  static constexpr int oR = oD + 4 * 16 * 17 * 4;                                    // [5][DK]: e^{G_end}, G before blocks 1 .. 3, G_end
  static constexpr int oRow = oR + 5 * DK * 4;                                       // beta, rk, rq: 2 x [3][64]
  static constexpr int total = oRow + 2 * 3 * kC * 4;
  static_assert(kC * po * 4 <= 4 * kRow, "the staged outputs fit over kt and qt");
  static_assert(total <= 227 * 1024, "shared memory");
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

// acc (16 x 16 as two n8 tiles) += or -= (ah + al) (bh + bl)^T without the product of the two low parts
__device__ __forceinline__ void mma3(float (&c0)[4], float (&c1)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4],
                                     const uint32_t (&bl)[4]) {
  mma16816(c0, ah, bh[0], bh[1]);
  mma16816(c1, ah, bh[2], bh[3]);
  mma16816(c0, al, bh[0], bh[1]);
  mma16816(c1, al, bh[2], bh[3]);
  mma16816(c0, ah, bl[0], bl[1]);
  mma16816(c1, ah, bl[2], bl[3]);
}
// two n8 accumulator tiles (16 x 16) as an A operand
__device__ __forceinline__ void frag_of(const float (&c0)[4], const float (&c1)[4], uint32_t (&h)[4], uint32_t (&l)[4]) {
  split2(c0[0], c0[1], h[0], l[0]);
  split2(c0[2], c0[3], h[1], l[1]);
  split2(c1[0], c1[1], h[2], l[2]);
  split2(c1[2], c1[3], h[3], l[3]);
}

template <int DK, int DV>
__global__ void __launch_bounds__(Smem<DK, DV>::kThreads, 1) delta_chunk_kernel(const DeltaView v) {
  typedef Smem<DK, DV> SM;
  typedef __nv_bfloat16 bf;
  constexpr int NW = SM::kWarps, NT = SM::kThreads, pk = SM::pk, pv = SM::pv, pg = SM::pg, ND = DK / 16;
  extern __shared__ __align__(128) unsigned char sm[];
  bf *sKt = (bf*)(sm + SM::oKt), *sQt = (bf*)(sm + SM::oQt), *sKb = (bf*)(sm + SM::oKb);
  bf *sA = (bf*)(sm + SM::oA), *sB = (bf*)(sm + SM::oB), *sT = (bf*)(sm + SM::oT);
  bf *sK = (bf*)(sm + SM::oK), *sQ = (bf*)(sm + SM::oQ), *sV = (bf*)(sm + SM::oV);
  float *sG = (float*)(sm + SM::oG), *sD = (float*)(sm + SM::oD), *sR = (float*)(sm + SM::oR), *sRow = (float*)(sm + SM::oRow);
  float* sO = (float*)(sm + SM::oKt);
  constexpr int kLoT = kC * pk, kLoA = 6 * kBlk, kLoB = 10 * kBlk, kLoI = 4 * kBlk;          // distance of the low parts (elements)
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int h = blockIdx.x, b = blockIdx.y, D = v.dim, V = v.vdim, ld = (V + 3) & ~3, a = h / (v.H / v.G);
  pdl_launch_dependents();
  pdl_wait();
  const int n_all = v.len[b], t_first = v.start[b];
  if (n_all <= 0) return;
  const int chunks = (n_all + kC - 1) / kC;

  // a thread copies 16-byte pieces of one column range, rows r0, r0 + step, ...
  float row_b = 0.f, row_k = 0.f, row_q = 0.f;                 // of token tid, on their way to sRow
  auto load_kqg = [&](int c) {
    const int64_t t0 = t_first + (int64_t)c * kC;
    const int n = min(kC, n_all - c * kC);
    {
      constexpr int step = NT / (DK / 8);
      const int r0 = tid / (DK / 8), d = (tid - r0 * (DK / 8)) * 8;
      const bool in = d < D;
      const bf* k = reinterpret_cast<const bf*>(v.k) + t0 * v.k_pitch + a * D + (in ? d : 0);
      const bf* q = reinterpret_cast<const bf*>(v.q) + t0 * v.q_pitch + a * D + (in ? d : 0);
#pragma unroll
      for (int r = r0; r < kC; r += step) {
        const bool ok = in && r < n;
        tc::cp_async16(smem_addr(sK + r * pk + d), k + (ok ? r * v.k_pitch : 0), ok ? 16u : 0u);
        tc::cp_async16(smem_addr(sQ + r * pk + d), q + (ok ? r * v.q_pitch : 0), ok ? 16u : 0u);
      }
    }
    {
      constexpr int step = NT / (DK / 4);
      const int r0 = tid / (DK / 4), d = (tid - r0 * (DK / 4)) * 4;
      const bool in = d < D;
      const float* x = v.decay + t0 * v.decay_pitch + h * D + (in ? d : 0);
#pragma unroll
      for (int r = r0; r < kC; r += step) {
        const bool ok = in && r < n;
        tc::cp_async16(smem_addr(sG + r * pg + d), x + (ok ? r * v.decay_pitch : 0), ok ? 16u : 0u);
      }
    }
    if (tid < kC) {
      const bool ok = tid < n;
      row_b = ok ? v.b[(t0 + tid) * v.b_pitch + h] : 0.f;
      row_k = ok ? v.rk[(t0 + tid) * v.G + a] : 0.f;
      row_q = ok ? v.rq[(t0 + tid) * v.G + a] : 0.f;
    }
  };
  auto store_rows = [&](int c) {
    if (tid >= kC) return;
    float* row = sRow + (c & 1) * 3 * kC;
    row[tid] = c * kC + tid < n_all ? 1.0f / (1.0f + expf(-row_b)) : 0.f;
    row[kC + tid] = row_k;
    row[2 * kC + tid] = row_q;
  };
  auto load_v = [&](int c) {
    const int64_t t0 = t_first + (int64_t)c * kC;
    const int n = min(kC, n_all - c * kC);
    constexpr int step = NT / (DV / 8);
    const int r0 = tid / (DV / 8), d = (tid - r0 * (DV / 8)) * 8;
    const bool in = d < V;
    const bf* x = reinterpret_cast<const bf*>(v.v) + t0 * v.v_pitch + h * V + (in ? d : 0);
#pragma unroll
    for (int r = r0; r < kC; r += step) {
      const bool ok = in && r < n;
      tc::cp_async16(smem_addr(sV + r * pv + d), x + (ok ? r * v.v_pitch : 0), ok ? 16u : 0u);
    }
  };
  load_kqg(0);
  store_rows(0);
  load_v(0);
  tc::cp_async_commit();

  // the state, transposed: value column warp * 16 + g (+ 8), key channels 8 j + 2 tq, + 1
  float S[DK / 8][4];
  float* state = v.state + ((int64_t)b * v.H + h) * D * ld;
  const int vc = warp * 16 + g;
#pragma unroll
  for (int j = 0; j < DK / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 8 * j + 2 * tq + (e & 1), c = vc + 8 * (e >> 1);
      S[j][e] = d < D && c < V ? state[(int64_t)d * ld + c] : 0.f;
    }

  for (int c = 0; c < chunks; ++c) {
    const int n = min(kC, n_all - c * kC);
    const float *beta = sRow + (c & 1) * 3 * kC, *rk = beta + kC, *rq = rk + kC;
    tc::cp_async_wait<0>();
    __syncthreads();
    // ---- running sums of the log decays (log2 units): in sG from the block's start on (a large decay costs only its own block
    // precision), R[b] = the sum before block b > 0, R[4] = G_end, R[0] = e^{G_end}
    int mild = 1;
    for (int d = tid; d < DK; d += NT) {
      float R = 0.f;
#pragma unroll
      for (int blk = 0; blk < kB; ++blk) {
        if (blk) sR[blk * DK + d] = R;
        float s = 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          s += fmaxf(sG[(blk * 16 + r) * pg + d] * kLog2e, kDecayMin);
          sG[(blk * 16 + r) * pg + d] = s;
        }
        R += s;
      }
      sR[kB * DK + d] = R;
      sR[d] = ex2(R);
      mild = mild && R >= -kDiagMax;
    }
    mild = __syncthreads_and(mild);
    // ---- kt, qt, kb; mild chunks: k e^{-G} over the raw rows (hi over K, lo over Q)
#pragma unroll 2
    for (int i = tid; i < kC * (DK / 4); i += NT) {
      const int r = i / (DK / 4), d = (i - r * (DK / 4)) * 4, at = r * pk + d;
      const float4 L = *reinterpret_cast<const float4*>(sG + r * pg + d), E = *reinterpret_cast<const float4*>(sR + kB * DK + d);
      const float4 Rv = r < 16 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sR + (r >> 4) * DK + d);
      const uint2 ku = *reinterpret_cast<const uint2*>(sK + at), qu = *reinterpret_cast<const uint2*>(sQ + at);
      const float2 k0 = unpack_bf16(ku.x), k1 = unpack_bf16(ku.y), q0 = unpack_bf16(qu.x), q1 = unpack_bf16(qu.y);
      const float kr = rk[r], qr = rq[r];
      const float G[4] = {Rv.x + L.x, Rv.y + L.y, Rv.z + L.z, Rv.w + L.w};
      const float Eb[4] = {E.x - Rv.x - L.x, E.y - Rv.y - L.y, E.z - Rv.z - L.z, E.w - Rv.w - L.w};
      const float k[4] = {k0.x * kr, k0.y * kr, k1.x * kr, k1.y * kr}, q[4] = {q0.x * qr, q0.y * qr, q1.x * qr, q1.y * qr};
      float e[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) e[j] = ex2(G[j]);
      auto put = [&](bf* m, float x0, float x1, float x2, float x3) {
        uint2 hi, lo;
        split2(x0, x1, hi.x, lo.x);
        split2(x2, x3, hi.y, lo.y);
        *reinterpret_cast<uint2*>(m + at) = hi;
        return lo;
      };
      *reinterpret_cast<uint2*>(sKt + kLoT + at) = put(sKt, k[0] * e[0], k[1] * e[1], k[2] * e[2], k[3] * e[3]);
      *reinterpret_cast<uint2*>(sQt + kLoT + at) = put(sQt, q[0] * e[0], q[1] * e[1], q[2] * e[2], q[3] * e[3]);
      if (mild) {
        const float4 X = *reinterpret_cast<const float4*>(sR + d);                              // e^{G_end}
        const float m[4] = {k[0] * ex2(-G[0]), k[1] * ex2(-G[1]), k[2] * ex2(-G[2]), k[3] * ex2(-G[3])};
        *reinterpret_cast<uint2*>(sKb + kLoT + at) = put(sKb, m[0] * X.x, m[1] * X.y, m[2] * X.z, m[3] * X.w);
        *reinterpret_cast<uint2*>(sQ + at) = put(sK, m[0], m[1], m[2], m[3]);
      } else {
        *reinterpret_cast<uint2*>(sKb + kLoT + at) = put(sKb, k[0] * ex2(Eb[0]), k[1] * ex2(Eb[1]), k[2] * ex2(Eb[2]), k[3] * ex2(Eb[3]));
      }
    }
    if (mild) __syncthreads();
    // ---- blocks (rt, st), st <= rt, of A and B: M = 16 rows t, N = 16 rows s
    // tasks 0 - 3: the diagonal ones, which also are inverted; then the A and the B part of the six others
    for (int task = warp; task < 16; task += NW) {
      const int off = (task - 4) >> 1, rt = task < 4 ? task : off == 0 ? 1 : off < 3 ? 2 : 3, st = task < 4 ? task : off == 0 ? 0 : off < 3 ? off - 1 : off - 3;
      const bool do_a = task < 4 || (task & 1) == 0, do_b = task < 4 || (task & 1);
      if (16 * rt >= n) continue;                               // rows behind the portion's end
      const float* R = sR + rt * DK;
      const bool diag = rt == st;
      bool direct = false;
      if (diag && !mild) {
        float m = 0.f;
        for (int d = lane; d < DK; d += 32) m = fmaxf(m, -sG[(rt * 16 + 15) * pg + d]);
        direct = __any_sync(0xffffffffu, !(m <= kDiagMax));
      }
      float ca[2][4], cb[2][4];                                 // k k and q k sums: rows t = g, g + 8; columns s = 8 j + 2 tq, + 1
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) ca[j][e] = cb[j][e] = 0.f;
      if (mild) {
        const uint32_t ao = (uint32_t)((rt * 16 + (lane & 15)) * pk + (lane >> 4) * 8) * 2;
        const uint32_t bo = (uint32_t)((st * 16 + (lane & 7) + ((lane >> 4) << 3)) * pk + ((lane >> 3) & 1) * 8) * 2;
        const uint32_t kt = smem_addr(sKt) + ao, qt = smem_addr(sQt) + ao, k2h = smem_addr(sK) + bo, k2l = smem_addr(sQ) + bo;
        float cx[2][2][4], cy[2][2][4];                         // the three products on accumulators of their own: short chains
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) cx[0][j][e] = cx[1][j][e] = cy[0][j][e] = cy[1][j][e] = 0.f;
        auto three = [&](float (&c0)[2][4], float (&c1)[2][4], float (&c2)[2][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4],
                         const uint32_t (&bl)[4]) {
          mma16816(c0[0], ah, bh[0], bh[1]); mma16816(c0[1], ah, bh[2], bh[3]);
          mma16816(c1[0], al, bh[0], bh[1]); mma16816(c1[1], al, bh[2], bh[3]);
          mma16816(c2[0], ah, bl[0], bl[1]); mma16816(c2[1], ah, bl[2], bl[3]);
        };
#pragma unroll 2
        for (int kk = 0; kk < ND; ++kk) {
          uint32_t ah[4], al[4], bh[4], bl[4];
          ldsm4(bh, k2h + kk * 32);
          ldsm4(bl, k2l + kk * 32);
          if (do_a) {
            ldsm4(ah, kt + kk * 32);
            ldsm4(al, kt + kLoT * 2 + kk * 32);
            three(ca, cx[0], cx[1], ah, al, bh, bl);
          }
          if (do_b) {
            ldsm4(ah, qt + kk * 32);
            ldsm4(al, qt + kLoT * 2 + kk * 32);
            three(cb, cy[0], cy[1], ah, al, bh, bl);
          }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) { ca[j][e] += cx[0][j][e] + cx[1][j][e]; cb[j][e] += cy[0][j][e] + cy[1][j][e]; }
      } else if (!direct) {
#pragma unroll 2
        for (int kk = 0; kk < ND; ++kk) {
          uint32_t kh[4], kl[4], qh[4], ql[4], bh[4], bl[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {                         // A operand: rows g + 8 (e & 1), channels 2 tq + 8 (e >> 1)
            const int r = rt * 16 + g + 8 * (e & 1), d = kk * 16 + 2 * tq + 8 * (e >> 1);
            const float2 G = *reinterpret_cast<const float2*>(sG + r * pg + d);
            const float e0 = ex2(G.x), e1 = ex2(G.y);
            const float2 k = unpack_bf16(*reinterpret_cast<const uint32_t*>(sK + r * pk + d)), q = unpack_bf16(*reinterpret_cast<const uint32_t*>(sQ + r * pk + d));
            if (do_a) split2(k.x * e0, k.y * e1, kh[e], kl[e]);
            if (do_b) split2(q.x * e0, q.y * e1, qh[e], ql[e]);
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) {                         // B operand: column tile e >> 1, channels 2 tq + 8 (e & 1)
            const int r = st * 16 + g + 8 * (e >> 1), d = kk * 16 + 2 * tq + 8 * (e & 1);
            const float2 G = *reinterpret_cast<const float2*>(sG + r * pg + d), Rt = rt ? *reinterpret_cast<const float2*>(R + d) : make_float2(0.f, 0.f);
            const float2 Rs = st ? *reinterpret_cast<const float2*>(sR + st * DK + d) : make_float2(0.f, 0.f);
            const float2 k = unpack_bf16(*reinterpret_cast<const uint32_t*>(sK + r * pk + d));
            split2(k.x * ex2(Rt.x - Rs.x - G.x), k.y * ex2(Rt.y - Rs.y - G.y), bh[e], bl[e]);
          }
          if (do_a) mma3(ca[0], ca[1], kh, kl, bh, bl);
          if (do_b) mma3(cb[0], cb[1], qh, ql, bh, bl);
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
              const float w = __bfloat162float(sK[s * pk + d]) * ex2(sG[r * pg + d] - sG[s * pg + d]);
              x = fmaf(__bfloat162float(sK[r * pk + d]), w, x);
              y = fmaf(__bfloat162float(sQ[r * pk + d]), w, y);
            }
            ca[j][e] = x;
            cb[j][e] = y;
          }
      }
      // scales, the triangle, and into shared memory
      const int blk = rt * (rt + 1) / 2 + st, blk_a = rt * (rt - 1) / 2 + st;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e2 = 0; e2 < 2; ++e2) {
          const int tl = g + 8 * e2, sl = 8 * j + 2 * tq, t = rt * 16 + tl, s = st * 16 + sl;
          const float bt = mild ? beta[t] : beta[t] * rk[t], qt = mild ? 1.f : rq[t], k0 = mild ? 1.f : rk[s], k1 = mild ? 1.f : rk[s + 1];
          float a0 = ca[j][2 * e2] * bt * k0, a1 = ca[j][2 * e2 + 1] * bt * k1;
          float b0 = cb[j][2 * e2] * qt * k0, b1 = cb[j][2 * e2 + 1] * qt * k1;
          if (diag) {
            if (sl >= tl) a0 = 0.f;
            if (sl + 1 >= tl) a1 = 0.f;
            if (sl > tl) b0 = 0.f;
            if (sl + 1 > tl) b1 = 0.f;
            sD[(rt * 16 + tl) * 17 + sl] = a0;
            sD[(rt * 16 + tl) * 17 + sl + 1] = a1;
          }
          uint32_t hi, lo;
          if (do_b) {
            split2(b0, b1, hi, lo);
            *reinterpret_cast<uint32_t*>(sB + blk * kBlk + tl * 24 + sl) = hi;
            *reinterpret_cast<uint32_t*>(sB + kLoB + blk * kBlk + tl * 24 + sl) = lo;
          }
          if (!diag && do_a) {                                          // subtracted where it is used
            split2(-a0, -a1, hi, lo);
            *reinterpret_cast<uint32_t*>(sA + blk_a * kBlk + tl * 24 + sl) = hi;
            *reinterpret_cast<uint32_t*>(sA + kLoA + blk_a * kBlk + tl * 24 + sl) = lo;
          }
        }
      if (diag) {                                               // inverse of the unit lower triangular block, a column per lane
        __syncwarp();
        const float* M = sD + rt * 16 * 17;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float y = i == (lane & 15) ? 1.f : 0.f;
#pragma unroll
          for (int k = 0; k < i; ++k) y = fmaf(-M[i * 17 + k], x[k], y);
          x[i] = y;
        }
        if (lane < 16) {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const bf hi = __float2bfloat16_rn(x[i]);
            sT[rt * kBlk + i * 24 + lane] = hi;
            sT[kLoI + rt * kBlk + i * 24 + lane] = __float2bfloat16_rn(x[i] - __bfloat162float(hi));
          }
        }
      }
    }
    __syncthreads();                                            // raw rows are free, everything below reads what they became
    if (c + 1 < chunks) load_kqg(c + 1);
    tc::cp_async_commit();

    const int nb = (n + 15) >> 4;
    // ---- Y = kt S and O = qt S, transposed
    float Y[2 * kB][4], O[2 * kB][4];
#pragma unroll
    for (int i = 0; i < 2 * kB; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) Y[i][e] = O[i][e] = 0.f;
    {
      // B operands: rows = tokens, columns = channels
      const uint32_t off = (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * pk + ((lane >> 3) & 1) * 8) * 2;
      const uint32_t kt = smem_addr(sKt) + off, qt = smem_addr(sQt) + off;
#pragma unroll
      for (int kk = 0; kk < ND; ++kk) {
        uint32_t sh[4], sl[4];
        frag_of(S[2 * kk], S[2 * kk + 1], sh, sl);
#pragma unroll
        for (int i = 0; i < kB; ++i) {
          if (i >= nb) break;
          uint32_t bh[4], bl[4];
          ldsm4(bh, kt + (uint32_t)(i * 16 * pk + kk * 16) * 2);
          ldsm4(bl, kt + (uint32_t)(kLoT + i * 16 * pk + kk * 16) * 2);
          mma3(Y[2 * i], Y[2 * i + 1], sh, sl, bh, bl);
          ldsm4(bh, qt + (uint32_t)(i * 16 * pk + kk * 16) * 2);
          ldsm4(bl, qt + (uint32_t)(kLoT + i * 16 * pk + kk * 16) * 2);
          mma3(O[2 * i], O[2 * i + 1], sh, sl, bh, bl);
        }
      }
    }
    // ---- U, block by block: U_a = T_a (beta (V - Y) - sum_b A_ab U_b)
    uint32_t uh[kB][4], ul[kB][4];
    const uint32_t boff = (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * 24 + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int i = 0; i < kB; ++i) {
      if (i >= nb) {
#pragma unroll
        for (int e = 0; e < 4; ++e) uh[i][e] = ul[i][e] = 0u;
        continue;
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = i * 16 + 8 * j + 2 * tq + (e & 1);
          Y[2 * i + j][e] = beta[t] * (__bfloat162float(sV[t * pv + vc + 8 * (e >> 1)]) - Y[2 * i + j][e]);
        }
#pragma unroll
      for (int s = 0; s < kB; ++s) {
        if (s >= i) break;
        uint32_t bh[4], bl[4];
        const uint32_t at = smem_addr(sA + (i * (i - 1) / 2 + s) * kBlk) + boff;
        ldsm4(bh, at);
        ldsm4(bl, at + kLoA * 2);
        mma3(Y[2 * i], Y[2 * i + 1], uh[s], ul[s], bh, bl);
      }
      uint32_t xh[4], xl[4], bh[4], bl[4];
      frag_of(Y[2 * i], Y[2 * i + 1], xh, xl);
      const uint32_t at = smem_addr(sT + i * kBlk) + boff;
      ldsm4(bh, at);
      ldsm4(bl, at + kLoI * 2);
      float u0[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f};
      mma3(u0, u1, xh, xl, bh, bl);
      frag_of(u0, u1, uh[i], ul[i]);
    }
    // ---- O += B U
#pragma unroll
    for (int i = 0; i < kB; ++i) {
      if (i >= nb) break;
#pragma unroll
      for (int s = 0; s < kB; ++s) {
        if (s > i) break;
        uint32_t bh[4], bl[4];
        const uint32_t at = smem_addr(sB + (i * (i + 1) / 2 + s) * kBlk) + boff;
        ldsm4(bh, at);
        ldsm4(bl, at + kLoB * 2);
        mma3(O[2 * i], O[2 * i + 1], uh[s], ul[s], bh, bl);
      }
    }
    // ---- S <- e^{G_end} S + kb^T U
#pragma unroll
    for (int j = 0; j < DK / 8; ++j) {
      const float2 E = *reinterpret_cast<const float2*>(sR + 8 * j + 2 * tq);
      S[j][0] *= E.x; S[j][1] *= E.y; S[j][2] *= E.x; S[j][3] *= E.y;
    }
    {
      const uint32_t kb = smem_addr(sKb) + (uint32_t)((lane & 15) * pk + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int s = 0; s < kB; ++s) {
        if (s >= nb) break;
#pragma unroll
        for (int kk = 0; kk < ND; ++kk) {
          uint32_t bh[4], bl[4];
          ldsm4_trans(bh, kb + (uint32_t)(s * 16 * pk + kk * 16) * 2);
          ldsm4_trans(bl, kb + (uint32_t)(kLoT + s * 16 * pk + kk * 16) * 2);
          mma3(S[2 * kk], S[2 * kk + 1], uh[s], ul[s], bh, bl);
        }
      }
    }
    // ---- outputs: through shared memory to whole token rows
    constexpr int kVec = kC * (DV / 8) / NT;                    // 16-byte pieces of the gate and of the output per thread
    uint4 gates[kVec];
#pragma unroll
    for (int j = 0; j < kVec; ++j) {
      const int i = tid + j * NT, r = i / (DV / 8), d = (i - r * (DV / 8)) * 8;
      gates[j] = r < n && d < V ? __ldg(reinterpret_cast<const uint4*>(reinterpret_cast<const bf*>(v.gate) + (t_first + (int64_t)c * kC + r) * v.gate_pitch + h * V + d))
                                : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();                                            // kt and qt have been read by everyone
    if (c + 1 < chunks) load_v(c + 1);
    tc::cp_async_commit();
#pragma unroll
    for (int i = 0; i < 2 * kB; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) sO[(8 * i + 2 * tq + (e & 1)) * SM::po + vc + 8 * (e >> 1)] = O[i][e];
    __syncthreads();
    {
      constexpr int L = DV / 8;                                 // lanes that share a token row
      const int d = (tid % L) * 8;
      float w[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = d < V ? __ldg(v.norm + d + e) : 0.f;
      float o[kVec][8], ss[kVec];
#pragma unroll
      for (int j = 0; j < kVec; ++j) {
        const float* row = sO + (tid / L + j * (NT / L)) * SM::po + d;
        const float4 x = *reinterpret_cast<const float4*>(row), y = *reinterpret_cast<const float4*>(row + 4);
        o[j][0] = x.x; o[j][1] = x.y; o[j][2] = x.z; o[j][3] = x.w; o[j][4] = y.x; o[j][5] = y.y; o[j][6] = y.z; o[j][7] = y.w;
        ss[j] = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss[j] = fmaf(o[j][e], o[j][e], ss[j]);      // zero behind the width
      }
#pragma unroll
      for (int off = L / 2; off > 0; off >>= 1)
#pragma unroll
        for (int j = 0; j < kVec; ++j) ss[j] += __shfl_xor_sync(0xffffffffu, ss[j], off);
#pragma unroll
      for (int j = 0; j < kVec; ++j) {
        const int r = tid / L + j * (NT / L);
        if (r >= n || d >= V) continue;
        const float inv = 1.0f / sqrtf(ss[j] / (float)V + v.eps);
        uint32_t* gi = reinterpret_cast<uint32_t*>(&gates[j]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 gt = unpack_bf16(gi[e]);
          const __nv_bfloat162 y = __floats2bfloat162_rn(o[j][2 * e] * inv * w[2 * e] * gt.x, o[j][2 * e + 1] * inv * w[2 * e + 1] * gt.y);
          gi[e] = *reinterpret_cast<const uint32_t*>(&y);
        }
        *reinterpret_cast<uint4*>(reinterpret_cast<bf*>(v.out) + (t_first + (int64_t)c * kC + r) * v.ldo + h * V + d) = gates[j];
      }
    }
    if (c + 1 < chunks) store_rows(c + 1);
  }
#pragma unroll
  for (int j = 0; j < DK / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 8 * j + 2 * tq + (e & 1), c = vc + 8 * (e >> 1);
      if (d < D && c < V) state[(int64_t)d * ld + c] = S[j][e];
    }
}

template <int DK, int DV>
int32_t launch(const DeltaView& v, cudaStream_t st) {
  LMB_CUDA(launch_k(delta_chunk_kernel<DK, DV>, dim3((unsigned)v.H, (unsigned)v.B), dim3(Smem<DK, DV>::kThreads), (size_t)Smem<DK, DV>::total, st, v));
  return LMB200_OK;
}

}  // namespace

int32_t delta_chunk_configure() {
#define LMB_CFG(DK, DV) LMB_CUDA(cudaFuncSetAttribute(delta_chunk_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, Smem<DK, DV>::total))
  LMB_CFG(64, 64);
  LMB_CFG(64, 128);
  LMB_CFG(128, 64);
  LMB_CFG(128, 128);
#undef LMB_CFG
  return LMB200_OK;
}

bool delta_chunks_ok(const DeltaView& v) {
  const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return !v.raw && v.bp == 0 && v.dim % 8 == 0 && v.vdim % 8 == 0 && v.dim <= 128 && v.vdim <= 128 && v.q_pitch % 8 == 0 && v.k_pitch % 8 == 0 &&
         v.v_pitch % 8 == 0 && v.decay_pitch % 4 == 0 && v.gate_pitch % 8 == 0 && v.ldo % 8 == 0 && aligned(v.q) && aligned(v.k) && aligned(v.v) &&
         aligned(v.decay) && aligned(v.gate) && aligned(v.out) && v.H <= 65535 && v.B <= 65535;
}

int32_t delta_chunks(Ctx* ctx, const DeltaView& v, cudaStream_t st) {
  LMB_REQUIRE(delta_chunks_ok(v), "delta rule: heads of %d x %d have no chunk kernel", v.dim, v.vdim);
  if (v.dim <= 64) LMB_TRY(v.vdim <= 64 ? (launch<64, 64>(v, st)) : (launch<64, 128>(v, st)));
  else LMB_TRY(v.vdim <= 64 ? (launch<128, 64>(v, st)) : (launch<128, 128>(v, st)));
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
