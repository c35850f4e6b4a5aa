// Kernels of retention (see retention.cuh).
#include "activations.cuh"
#include "mma_sync.cuh"
#include "pdl.cuh"
#include "retention.cuh"

namespace lmb {
namespace {

constexpr int kStepMax = 512;           // threads per CTA: 512 where few (head, sequence) pairs leave SMs idle, else 128

// One CTA per (head, sequence).  Thread (c, w): four value columns 4 c .., rows w, w + W, ... of the state, where W = threads / column
// groups; a thread owns its elements of the state for all tokens, so only q, k, v and the partial outputs go through shared memory.
template <typename IT, typename OT>
__global__ void __launch_bounds__(kStepMax) retention_step_kernel(const RetentionView v) {
  extern __shared__ float sm[];
  __shared__ float red[kStepMax / 32];
  const int kStepThreads = blockDim.x;
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
  const float kscale = v.k_scale;
  float4* S = reinterpret_cast<float4*>(v.state) + ((int64_t)b * v.H + h) * D * V4;
  const int c0 = tid % cols, w = tid / cols;
  for (int i = 0; i < n; ++i) {
    const int64_t t = t0 + i;
    const IT* q = reinterpret_cast<const IT*>(v.q) + t * v.q_pitch + h * D;
    const IT* k = reinterpret_cast<const IT*>(v.k) + t * v.k_pitch + h * D;
    const IT* vv = reinterpret_cast<const IT*>(v.v) + t * v.v_pitch + h * V;
    for (int d = tid; d < D; d += kStepThreads) {
      float qv = to_f32(q[d]), kv = to_f32(k[d]);
      if (v.raw_act) { qv = silu_f32(qv); kv = silu_f32(kv); }
      if (d < v.rot_dims) {
        float s, c;
        sincosf((float)(p0 + i) * v.inv_freq[d >> 1], &s, &c);
        if (!(d & 1)) s = -s;
        qv = qv * c + to_f32(q[d ^ 1]) * s;
        kv = kv * c + to_f32(k[d ^ 1]) * s;
      }
      qs[d] = qv;
      ks[d] = kv * kscale;
    }
    for (int d = tid; d < 4 * V4; d += kStepThreads) vs[d] = d >= V ? 0.f : v.raw_act ? silu_f32(to_f32(vv[d])) : to_f32(vv[d]);
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
    for (int j = 0; j < kStepThreads / 32; ++j) tot += red[j];
    const float inv = v.ssq ? 1.0f : 1.0f / sqrtf(tot / (float)V + v.eps);
    if (v.ssq && tid == 0) v.ssq[t * v.ssq_t + h * v.ssq_h] = tot;
    const IT* g = reinterpret_cast<const IT*>(v.g) + t * v.g_pitch + h * V;
    OT* out = reinterpret_cast<OT*>(v.out);
    for (int d = tid; d < V; d += kStepThreads) {
      float gv = to_f32(g[d]);
      if (v.raw_gate) gv = v.raw_gate == 1 ? silu_f32(gv) : sigmoid_f32(gv);
      const int col = h * V + d;
      if (v.out_w) gv *= v.out_w[col];
      out[v.bp > 0 ? Layout<OT>::x_offset((int)t, col, v.bp) : t * v.ldo + col] = from_f32<OT>(vs[d] * inv * gv);
    }
    __syncthreads();                   // vs, red and os are rewritten by the next token
  }
}

size_t step_smem(const RetentionView& v, int threads) {
  const int V4 = (v.vdim + 3) >> 2, cols = V4 < threads ? V4 : threads, W = threads / cols;
  return (size_t)(2 * ((v.dim + 3) & ~3) + 4 * V4 + W * 4 * V4) * 4;
}

// ---------------------------------------------------------------------------------------------
// Chunks of 64 tokens on the tensor cores.  A cluster owns one head of one sequence, each of its CTAs a slice of the value columns; the
// state stays in the accumulator registers over the whole portion.  Per chunk (rows i, keys j of the chunk, n of them valid):
//   O  = diag(decay^(i + 1)) Q S                    state before the chunk
//   O += (Q K^T * scale decay^(i - j), j <= i) V
//   S  = decay^n S + (scale decay^(n - 1 - j) K)^T V
// q, k, v are bf16; everything the decays touch keeps float32's leading 16 bits: S, the weighted scores and the weighted keys enter
// the products as bf16 pairs hi + lo (x = hi + lo to about 2^-17).  Warps: 4 row groups x NG column groups of CG value columns; in the
// state update a row group is a quarter of the state's rows.  The heads' root mean squares are summed over the cluster through distributed shared memory.
// ---------------------------------------------------------------------------------------------
constexpr int kC = 64;

template <int DK, int CG, int NG>
struct ChunkSmem {
  static constexpr int pk = DK + 8, pv = CG * NG + 8;                // row pitches (elements): an odd number of 16-byte chunks
  static constexpr int kQK = kC * pk, kV = kC * pv, kS = DK * pv;
  static constexpr size_t bytes = (size_t)(2 * (2 * kQK + kV) + 2 * kS) * 2 + (size_t)(NG * kC + 2 * 8 * kC + 72) * 4;
};

template <int DK, int CG, int NG>
__global__ void __launch_bounds__(128 * NG, 1) retention_chunk_kernel(const RetentionView v) {
  typedef ChunkSmem<DK, CG, NG> SM;
  constexpr int NT = CG / 8, MT = DK / 64, kThreads = 128 * NG, DVC = CG * NG;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sm_raw);     // [2][kC][pk]
  __nv_bfloat16* sK = sQ + 2 * SM::kQK;
  __nv_bfloat16* sV = sK + 2 * SM::kQK;                             // [2][kC][pv]
  __nv_bfloat16* sSh = sV + 2 * SM::kV;                             // [DK][pv] state, leading and trailing halves
  __nv_bfloat16* sSl = sSh + SM::kS;
  float* s_ssq = reinterpret_cast<float*>(sSl + SM::kS);            // [NG][kC]
  float* s_xch = s_ssq + NG * kC;                                   // [2][8][kC]: every CTA's sums of squares
  float* s_pw = s_xch + 2 * 8 * kC;                                 // decay^0 .. decay^64
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rw = warp & 3, cg = warp >> 2, g = lane >> 2, tq = lane & 3;
  const int slices = gridDim.x, slice = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  pdl_launch_dependents();
  pdl_wait();
  const int n_all = v.len[b], t_first = v.start[b];
  if (n_all <= 0) return;
  const int D = v.dim, V = v.vdim, ld = (V + 3) & ~3;
  const int c0 = slice * DVC;                                       // first value column of this CTA
  const float scale = v.k_scale;
  for (int i = tid; i <= kC; i += kThreads) s_pw[i] = v.decay[h * v.decay_pitch + i];

  auto load = [&](int c) {
    const int64_t t0 = t_first + (int64_t)c * kC;
    const int n = min(kC, n_all - c * kC), buf = c & 1;
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(v.q) + t0 * v.q_pitch + h * D;
    const __nv_bfloat16* k = reinterpret_cast<const __nv_bfloat16*>(v.k) + t0 * v.k_pitch + h * D;
    const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(v.v) + t0 * v.v_pitch + h * V + c0;
    for (int i = tid; i < kC * (DK / 8); i += kThreads) {
      const int r = i / (DK / 8), d = (i - r * (DK / 8)) * 8;
      const bool ok = r < n && d < D;
      const int64_t oq = ok ? (int64_t)r * v.q_pitch + d : 0, ok_ = ok ? (int64_t)r * v.k_pitch + d : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr(sQ + buf * SM::kQK + r * SM::pk + d)), "l"(q + oq), "r"(ok ? 16 : 0) : "memory");
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr(sK + buf * SM::kQK + r * SM::pk + d)), "l"(k + ok_), "r"(ok ? 16 : 0) : "memory");
    }
    for (int i = tid; i < kC * (DVC / 8); i += kThreads) {
      const int r = i / (DVC / 8), d = (i - r * (DVC / 8)) * 8;
      const bool ok = r < n && c0 + d < V;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr(sV + buf * SM::kV + r * SM::pv + d)),
                   "l"(ok ? x + (int64_t)r * v.v_pitch + d : x - c0), "r"(ok ? 16 : 0)
                   : "memory");
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  load(0);

  // the state of this warp: rows rw * DK / 4 + 16 m + g (+ 8), columns cg * CG + 8 nt + 2 tq (+ 1) of the slice
  float S[MT][NT][4];
  float* state = v.state + ((int64_t)b * v.H + h) * D * ld;
  auto state_at = [&](int m, int nt, int e2, bool* ok) -> float* {
    const int d = rw * (DK / 4) + m * 16 + g + e2 * 8, col = c0 + cg * CG + nt * 8 + 2 * tq;
    *ok = d < D && col + 1 < ld;
    return state + (int64_t)d * ld + col;
  };
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e2 = 0; e2 < 2; ++e2) {
        bool ok;
        const float* p = state_at(m, nt, e2, &ok);
        const float2 x = ok ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
        S[m][nt][2 * e2] = x.x;
        S[m][nt][2 * e2 + 1] = x.y;
      }
  auto publish_state = [&]() {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e2 = 0; e2 < 2; ++e2) {
          uint32_t hi, lo;
          split2(S[m][nt][2 * e2], S[m][nt][2 * e2 + 1], hi, lo);
          const int at = (rw * (DK / 4) + m * 16 + g + e2 * 8) * SM::pv + cg * CG + nt * 8 + 2 * tq;
          *reinterpret_cast<uint32_t*>(sSh + at) = hi;
          *reinterpret_cast<uint32_t*>(sSl + at) = lo;
        }
  };
  publish_state();
  if (slices > 1) {                                    // every CTA of the cluster runs before anyone writes into its shared memory
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
  }
  const int chunks = (n_all + kC - 1) / kC;
  const int r0 = rw * 16;
  for (int c = 0; c < chunks; ++c) {
    const int n = min(kC, n_all - c * kC), buf = c & 1;
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    if (c + 1 < chunks) load(c + 1);
    const __nv_bfloat16* Q = sQ + buf * SM::kQK;
    const __nv_bfloat16* K = sK + buf * SM::kQK;
    const __nv_bfloat16* X = sV + buf * SM::kV;
    float O[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;
    {
      float P[8][4];                                    // scores of 16 rows x 64 keys
#pragma unroll
      for (int i = 0; i < 8; ++i) P[i][0] = P[i][1] = P[i][2] = P[i][3] = 0.f;
      const uint32_t qa = smem_addr(Q + (r0 + (lane & 15)) * SM::pk + (lane >> 4) * 8);
      const uint32_t ka = smem_addr(K + ((lane & 7) + ((lane >> 4) << 3)) * SM::pk + ((lane >> 3) & 1) * 8);
      const uint32_t sh = smem_addr(sSh + (lane & 15) * SM::pv + cg * CG + (lane >> 4) * 8), lo_off = (uint32_t)SM::kS * 2;
#pragma unroll 2
      for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t a[4];
        ldsm4(a, qa + ks * 32);
#pragma unroll
        for (int jt = 0; jt < 4; ++jt) {
          if (jt > rw) break;
          uint32_t kb[4];
          ldsm4(kb, ka + jt * 16 * SM::pk * 2 + ks * 32);
          mma16816(P[2 * jt], a, kb[0], kb[1]);
          mma16816(P[2 * jt + 1], a, kb[2], kb[3]);
        }
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t hb[4], lb[4];
          ldsm4_trans(hb, sh + ks * 16 * SM::pv * 2 + nt * 16);
          ldsm4_trans(lb, sh + lo_off + ks * 16 * SM::pv * 2 + nt * 16);
          mma16816(O[nt], a, hb[0], hb[1]);
          mma16816(O[nt + 1], a, hb[2], hb[3]);
          mma16816(O[nt], a, lb[0], lb[1]);
          mma16816(O[nt + 1], a, lb[2], lb[3]);
        }
      }
      const float w0 = s_pw[r0 + g + 1], w1 = s_pw[r0 + g + 9];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { O[nt][0] *= w0; O[nt][1] *= w0; O[nt][2] *= w1; O[nt][3] *= w1; }
#pragma unroll
      for (int jt = 0; jt < 4; ++jt) {
        if (jt > rw) break;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {                   // a-fragment q: rows g + 8 (q & 1), keys 8 (q >> 1) + 2 tq, + 1
          const int i = r0 + g + 8 * (q & 1), j = jt * 16 + 8 * (q >> 1) + 2 * tq;
          const float* p = P[2 * jt + (q >> 1)] + 2 * (q & 1);
          const float x = j <= i ? p[0] * (scale * s_pw[i - j]) : 0.f;
          const float y = j + 1 <= i ? p[1] * (scale * s_pw[i - j - 1]) : 0.f;
          split2(x, y, ph[q], pl[q]);
        }
        const uint32_t va = smem_addr(X + (jt * 16 + (lane & 15)) * SM::pv + cg * CG + (lane >> 4) * 8);
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t vb[4];
          ldsm4_trans(vb, va + nt * 16);
          mma16816(O[nt], ph, vb[0], vb[1]);
          mma16816(O[nt + 1], ph, vb[2], vb[3]);
          mma16816(O[nt], pl, vb[0], vb[1]);
          mma16816(O[nt + 1], pl, vb[2], vb[3]);
        }
      }
    }
    // sums of squares of the rows over this warp's columns
    float q0 = 0.f, q1 = 0.f;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      q0 += O[nt][0] * O[nt][0] + O[nt][1] * O[nt][1];
      q1 += O[nt][2] * O[nt][2] + O[nt][3] * O[nt][3];
    }
    q0 += __shfl_xor_sync(0xffffffffu, q0, 1);
    q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
    q1 += __shfl_xor_sync(0xffffffffu, q1, 1);
    q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
    if (tq == 0) { s_ssq[cg * kC + r0 + g] = q0; s_ssq[cg * kC + r0 + g + 8] = q1; }
    // state update
    const float wn = s_pw[n];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { S[m][nt][0] *= wn; S[m][nt][1] *= wn; S[m][nt][2] *= wn; S[m][nt][3] *= wn; }
#pragma unroll
    for (int kk = 0; kk < kC / 16; ++kk) {
      if (kk * 16 >= n) break;
      float kw[4];                                      // weights of tokens 2 tq, + 1, + 8, + 9 of this step
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = kk * 16 + 2 * tq + (e & 1) + 8 * (e >> 1);
        kw[e] = t < n ? scale * s_pw[n - 1 - t] : 0.f;
      }
      uint32_t vb[NT / 2][4];
#pragma unroll
      for (int i = 0; i < NT / 2; ++i) ldsm4_trans(vb[i], smem_addr(X + (kk * 16 + (lane & 15)) * SM::pv + cg * CG + i * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t a[4], ah[4], al[4];
        ldsm4_trans(a, smem_addr(K + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * SM::pk + rw * (DK / 4) + m * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int q = 0; q < 4; ++q) {                   // fragments 0, 1: tokens 2 tq, + 1; 2, 3: + 8
          const float2 x = unpack_bf16(a[q]);
          split2(x.x * kw[2 * (q >> 1)], x.y * kw[2 * (q >> 1) + 1], ah[q], al[q]);
        }
#pragma unroll
        for (int i = 0; i < NT / 2; ++i) {
          mma16816(S[m][2 * i], ah, vb[i][0], vb[i][1]);
          mma16816(S[m][2 * i + 1], ah, vb[i][2], vb[i][3]);
          mma16816(S[m][2 * i], al, vb[i][0], vb[i][1]);
          mma16816(S[m][2 * i + 1], al, vb[i][2], vb[i][3]);
        }
      }
    }
    __syncthreads();                                    // sums written, everyone is done with the old state in shared memory
    const float* sums = s_ssq;
    int n_sums = NG;
    if (slices > 1) {
      float* mine = s_xch + (c & 1) * 8 * kC + slice * kC;
      for (int i = tid; i < slices * kC; i += kThreads) {
        const int peer = i / kC, row = i - peer * kC;
        float x = 0.f;
#pragma unroll
        for (int k = 0; k < NG; ++k) x += s_ssq[k * kC + row];
        uint32_t remote;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(remote) : "r"(smem_addr(mine + row)), "r"((uint32_t)peer));
        asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(remote), "f"(x) : "memory");
      }
      asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    }
    publish_state();
    if (slices > 1) {
      asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
      sums = s_xch + (c & 1) * 8 * kC;
      n_sums = slices;
    }
    q0 = q1 = 0.f;
    for (int k = 0; k < n_sums; ++k) { q0 += sums[k * kC + r0 + g]; q1 += sums[k * kC + r0 + g + 8]; }
    const float i0 = v.ssq ? 1.0f : 1.0f / sqrtf(q0 / (float)V + v.eps), i1 = v.ssq ? 1.0f : 1.0f / sqrtf(q1 / (float)V + v.eps);
    if (v.ssq && slice == 0 && cg == 0 && tq == 0) {
      const int64_t t = t_first + (int64_t)c * kC + r0 + g;
      if (r0 + g < n) v.ssq[t * v.ssq_t + h * v.ssq_h] = q0;
      if (r0 + g + 8 < n) v.ssq[(t + 8) * v.ssq_t + h * v.ssq_h] = q1;
    }
#pragma unroll
    for (int e2 = 0; e2 < 2; ++e2) {
      const int row = r0 + g + e2 * 8;
      if (row >= n) continue;
      const int64_t t = t_first + (int64_t)c * kC + row;
      const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(v.g) + t * v.g_pitch + h * V;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(v.out) + t * v.ldo + h * V;
      const float inv = e2 ? i1 : i0;
      uint32_t gu[NT];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int col = c0 + cg * CG + nt * 8 + 2 * tq;
        gu[nt] = col < V ? *reinterpret_cast<const uint32_t*>(gate + col) : 0u;
      }
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int col = c0 + cg * CG + nt * 8 + 2 * tq;
        if (col >= V) continue;
        float2 gv = unpack_bf16(gu[nt]);
        if (v.out_w) { gv.x *= v.out_w[h * V + col]; gv.y *= v.out_w[h * V + col + 1]; }
        *reinterpret_cast<__nv_bfloat162*>(out + col) = __floats2bfloat162_rn(O[nt][2 * e2] * inv * gv.x, O[nt][2 * e2 + 1] * inv * gv.y);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e2 = 0; e2 < 2; ++e2) {
        bool ok;
        float* p = state_at(m, nt, e2, &ok);
        if (ok) *reinterpret_cast<float2*>(p) = make_float2(S[m][nt][2 * e2], S[m][nt][2 * e2 + 1]);
      }
}

template <int DK, int CG, int NG>
int32_t launch_chunks(Ctx* ctx, const RetentionView& v, cudaStream_t st) {
  const unsigned slices = (unsigned)ceil_div(v.vdim, CG * NG);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, (unsigned)v.H, (unsigned)v.B);
  cfg.blockDim = dim3(128 * NG);
  cfg.dynamicSmemBytes = ChunkSmem<DK, CG, NG>::bytes;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  LMB_CUDA(cudaLaunchKernelEx(&cfg, retention_chunk_kernel<DK, CG, NG>, v));
  ctx->launches++;
  return LMB200_OK;
}

__global__ void angle_table_kernel(float2* __restrict__ tab, const float* __restrict__ inv_freq, int n, const int* __restrict__ pos, int T) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x;
  if (i >= (int64_t)T * n) return;
  const int t = (int)(i / n);
  float s, c;
  sincosf((float)pos[t] * inv_freq[i - (int64_t)t * n], &s, &c);
  tab[i] = make_float2(c, s);
}

}  // namespace

int32_t retention_configure() {
#define LMB_CFG(DK, CG, NG)                                                                                                  \
  LMB_CUDA(cudaFuncSetAttribute(retention_chunk_kernel<DK, CG, NG>, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                (int)ChunkSmem<DK, CG, NG>::bytes))
  LMB_CFG(64, 64, 1);
  LMB_CFG(64, 64, 2);
  LMB_CFG(128, 64, 1);
  LMB_CFG(128, 64, 2);
  LMB_CFG(256, 32, 2);
#undef LMB_CFG
  return retention_tc_configure();
}

int32_t angle_table(Ctx* ctx, float2* tab, const float* inv_freq, int n, const int* pos, int T, cudaStream_t st) {
  LMB_CUDA(launch_k(angle_table_kernel, dim3((unsigned)ceil_div((int64_t)T * n, 256)), dim3(256), 0, st, tab, inv_freq, n, pos, T));
  ctx->launches++;
  return LMB200_OK;
}

bool retention_chunks_ok(const RetentionView& v) {
  const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return !v.in_f32 && !v.raw_gate && v.rot_dims == 0 && v.bp == 0 && v.dim % 8 == 0 && v.vdim % 8 == 0 && v.dim <= 256 && v.q_pitch % 8 == 0 &&
         v.k_pitch % 8 == 0 && v.v_pitch % 8 == 0 && v.g_pitch % 2 == 0 && v.ldo % 2 == 0 && aligned(v.q) && aligned(v.k) && aligned(v.v) &&
         aligned(v.g) && aligned(v.out) && v.decay_pitch > kC && v.H <= 65535 && v.B <= 65535 &&
         ceil_div(v.vdim, v.dim <= 128 ? 128 : 64) <= 8;
}

int32_t retention_chunks(Ctx* ctx, const RetentionView& v, cudaStream_t st) {
  LMB_REQUIRE(retention_chunks_ok(v), "retention: heads of %d x %d have no chunk kernel", v.dim, v.vdim);
  if (v.dim > 128) return launch_chunks<256, 32, 2>(ctx, v, st);
  // two column groups per CTA share the scores; one each where that would leave SMs without a CTA
  const bool two = v.vdim > 64 && ((int64_t)v.B * v.H * ceil_div(v.vdim, 128) >= ctx->sm_count * 3 / 4 || ceil_div(v.vdim, 64) > 8);
  if (v.dim > 64) return two ? launch_chunks<128, 64, 2>(ctx, v, st) : launch_chunks<128, 64, 1>(ctx, v, st);
  return two ? launch_chunks<64, 64, 2>(ctx, v, st) : launch_chunks<64, 64, 1>(ctx, v, st);
}

int32_t retention_steps(Ctx* ctx, int dtype, const RetentionView& v, cudaStream_t st) {
  const int threads = (int64_t)v.B * v.H < 2 * ctx->sm_count ? kStepMax : 128;
  const size_t smem = step_smem(v, threads);
  LMB_REQUIRE(smem <= 48 * 1024, "retention: heads of %d x %d", v.dim, v.vdim);
  const dim3 grid((unsigned)v.H, (unsigned)v.B);
  if (dtype != LMB200_BF16) {
    LMB_REQUIRE(v.in_f32, "retention: float32 models have float32 projections");
    LMB_CUDA(launch_k(retention_step_kernel<float, float>, grid, dim3(threads), smem, st, v));
  } else if (v.in_f32) {
    LMB_CUDA(launch_k(retention_step_kernel<float, __nv_bfloat16>, grid, dim3(threads), smem, st, v));
  } else {
    LMB_CUDA(launch_k(retention_step_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(threads), smem, st, v));
  }
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
