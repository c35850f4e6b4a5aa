// Kernels of windowed attention (see window_attn.cuh).
#include <math_constants.h>

#include <algorithm>

#include "mma_sync.cuh"
#include "pdl.cuh"
#include "tc.cuh"
#include "window_attn.cuh"

namespace lmb {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

// pair p of a head: features lo and hi; the first rot_dims / 2 pairs rotate
__device__ __forceinline__ void pair_of(const WindowView& v, int p, int* lo, int* hi) {
  const int half = v.rot_dims >> 1;
  if (p >= half || v.rot_interleaved) { *lo = 2 * p; *hi = 2 * p + 1; }
  else { *lo = p; *hi = p + half; }
}
__device__ __forceinline__ float2 turn(const WindowView& v, int t, int pos, int p, float a, float b) {
  float c, s;
  if (v.angles) {
    const float2 cs = __ldg(v.angles + (int64_t)t * (v.rot_dims >> 1) + p);
    c = cs.x; s = cs.y;
  } else {
    // the product's rounding error is turned back to first order: at position 1000 it is 1000 times a float's resolution
    const float f = v.inv_freq[p], x = (float)pos * f, err = fmaf((float)pos, f, -x);
    sincosf(x, &s, &c);
    const float s0 = s;
    s = fmaf(err, c, s);
    c = fmaf(-err, s0, c);
  }
  c *= v.rot_scale; s *= v.rot_scale;
  return make_float2(a * c - b * s, b * c + a * s);
}

// One warp: the rotated and normed head `src` (dim features) through `put(feature, value)`.  Heads wider than 512 read their row twice.
template <typename IT, typename F>
__device__ __forceinline__ void norm_head(const WindowView& v, const IT* src, int t, int pos, int lane, F put) {
  constexpr int kKeep = 8;
  const int pairs = (v.dim + 1) >> 1, half = v.rot_dims >> 1;
  float2 keep[kKeep];
  float ss = 0.f;
  auto load = [&](int p) {
    int lo, hi;
    pair_of(v, p, &lo, &hi);
    float2 x = make_float2(to_f32(src[lo]), hi < v.dim ? to_f32(src[hi]) : 0.f);
    return p < half ? turn(v, t, pos, p, x.x, x.y) : x;
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int p = lane + 32 * i;
    keep[i] = p < pairs ? load(p) : make_float2(0.f, 0.f);
    ss += keep[i].x * keep[i].x + keep[i].y * keep[i].y;
  }
  for (int p = lane + 32 * kKeep; p < pairs; p += 32) { const float2 x = load(p); ss += x.x * x.x + x.y * x.y; }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  const float inv = 1.0f / sqrtf(ss / (float)v.dim + v.eps);
  auto store = [&](int p, float2 x) {
    int lo, hi;
    pair_of(v, p, &lo, &hi);
    put(lo, x.x * inv);
    if (hi < v.dim) put(hi, x.y * inv);
  };
  for (int p = lane + 32 * kKeep; p < pairs; p += 32) {
    const float2 x = load(p);          // in place too: a pair's features belong to one lane
    store(p, x);
  }
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int p = lane + 32 * i;
    if (p < pairs) store(p, keep[i]);
  }
}

// a warp per (token, head): queries, then keys, then values
template <typename IT, typename WT>
__global__ void __launch_bounds__(256) window_prep_kernel(const WindowView v, const WindowRows in, WT* __restrict__ q_out) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = v.H + (in.k ? 2 * v.G : 0);
  const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= (int64_t)v.T * units) return;
  const int t = (int)(id / units), u = (int)(id - (int64_t)t * units);
  const int pos = v.pos[t];
  if (u < v.H) {
    WT* o = q_out + ((int64_t)t * v.H + u) * v.dim;
    norm_head(v, reinterpret_cast<const IT*>(in.q) + (int64_t)t * in.q_pitch + u * v.dim, t, pos, lane, [&](int d, float x) { o[d] = from_f32<WT>(x); });
    return;
  }
  if (pos < 0 || pos >= v.cap) return;
  const int a = (u - v.H) % v.G;
  const int64_t row = ((int64_t)v.seq[t] * v.G + a) * v.cap + pos;
  if (u < v.H + v.G) {
    WT* o = reinterpret_cast<WT*>(v.keys) + row * v.k_ld;
    norm_head(v, reinterpret_cast<const IT*>(in.k) + (int64_t)t * in.k_pitch + a * v.dim, t, pos, lane, [&](int d, float x) { o[d] = from_f32<WT>(x); });
  } else {
    WT* o = reinterpret_cast<WT*>(v.values) + row * v.v_ld;
    const IT* s = reinterpret_cast<const IT*>(in.v) + (int64_t)t * in.v_pitch + a * v.vdim;
    for (int d = lane; d < v.vdim; d += 32) o[d] = from_f32<WT>(to_f32(s[d]));
  }
}

// The same for neighbouring pairs and even widths up to 64 NP: a warp takes kHeads heads of one token, their loads in flight together; the
// token's angles are read once
constexpr int kHeads = 4;
template <typename IT, typename WT, int NP>
__global__ void __launch_bounds__(256) window_prep_rows_kernel(const WindowView v, const WindowRows in, WT* q_out) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = v.H + (in.k ? v.G : 0), groups = (units + kHeads - 1) / kHeads, vgroups = in.k ? (v.G + kHeads - 1) / kHeads : 0;
  const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= (int64_t)v.T * (groups + vgroups)) return;
  const int t = (int)(id / (groups + vgroups)), gr = (int)(id - (int64_t)t * (groups + vgroups));
  const int pos = v.pos[t];
  const bool cached = pos >= 0 && pos < v.cap;
  const int64_t row0 = (int64_t)v.seq[t] * v.G * v.cap + pos;          // key head a: + a * cap
  if (gr >= groups) {
    if (!cached) return;
    for (int a = (gr - groups) * kHeads; a < min(v.G, (gr - groups + 1) * kHeads); ++a) {
      WT* o = reinterpret_cast<WT*>(v.values) + (row0 + (int64_t)a * v.cap) * v.v_ld;
      const IT* s = reinterpret_cast<const IT*>(in.v) + (int64_t)t * in.v_pitch + a * v.vdim;
      for (int d = lane; d < v.vdim; d += 32) o[d] = from_f32<WT>(to_f32(s[d]));
    }
    return;
  }
  float2 x[kHeads][NP];
#pragma unroll
  for (int e = 0; e < kHeads; ++e) {
    const int u = gr * kHeads + e;
    const IT* s = u < v.H ? reinterpret_cast<const IT*>(in.q) + (int64_t)t * in.q_pitch + u * v.dim
                          : reinterpret_cast<const IT*>(in.k) + (int64_t)t * in.k_pitch + (u - v.H) * v.dim;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int d = 2 * (lane + 32 * i);
      x[e][i] = u < units && d < v.dim ? load_pair(s + d) : make_float2(0.f, 0.f);
    }
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int p = lane + 32 * i;
    if (p >= (v.rot_dims >> 1)) continue;
    const float2 cs = turn(v, t, pos, p, 1.f, 0.f);                  // (cosine, sine), scaled
#pragma unroll
    for (int e = 0; e < kHeads; ++e) x[e][i] = make_float2(x[e][i].x * cs.x - x[e][i].y * cs.y, x[e][i].y * cs.x + x[e][i].x * cs.y);
  }
  float ss[kHeads];
#pragma unroll
  for (int e = 0; e < kHeads; ++e) {
    ss[e] = 0.f;
#pragma unroll
    for (int i = 0; i < NP; ++i) ss[e] += x[e][i].x * x[e][i].x + x[e][i].y * x[e][i].y;
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1)
#pragma unroll
    for (int e = 0; e < kHeads; ++e) ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], off);
#pragma unroll
  for (int e = 0; e < kHeads; ++e) {
    const int u = gr * kHeads + e;
    if (u >= units || (u >= v.H && !cached)) continue;
    const float inv = 1.0f / sqrtf(ss[e] / (float)v.dim + v.eps);
    WT* o = u < v.H ? q_out + ((int64_t)t * v.H + u) * v.dim : reinterpret_cast<WT*>(v.keys) + (row0 + (int64_t)(u - v.H) * v.cap) * v.k_ld;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int d = 2 * (lane + 32 * i);
      if (d < v.dim) store_pair(o + d, x[e][i].x * inv, x[e][i].y * inv);
    }
  }
}

__device__ __forceinline__ float bound_score(const WindowView& v, float s) {       // s = q . k
  s *= v.scale;
  return v.score_cap > 0.f ? v.score_cap * tanhf(s / v.score_cap) : s;
}

// CUDA cores, any widths: one CTA per (token, query head), 128 keys at a time
constexpr int kSimple = 128;
template <typename WT>
__global__ void __launch_bounds__(kSimple) window_simple_kernel(const WindowView v, const WT* __restrict__ q, WT* __restrict__ out, int ldo, int bp) {
  extern __shared__ float sm[];              // q [dim] | o [vdim] | p [kSimple]
  __shared__ float red[kSimple / 32];
  float* qs = sm;
  float* os = qs + v.dim;
  float* ps = os + v.vdim;
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  const int pos = v.pos[t], a = h / (v.H / v.G);
  const int lo = v.window > 0 ? max(0, pos - v.window + 1) : 0;
  const WT* K = reinterpret_cast<const WT*>(v.keys) + ((int64_t)v.seq[t] * v.G + a) * v.cap * v.k_ld;
  const WT* V = reinterpret_cast<const WT*>(v.values) + ((int64_t)v.seq[t] * v.G + a) * v.cap * v.v_ld;
  for (int d = tid; d < v.dim; d += kSimple) qs[d] = to_f32(q[((int64_t)t * v.H + h) * v.dim + d]);
  for (int d = tid; d < v.vdim; d += kSimple) os[d] = 0.f;
  __syncthreads();
  auto block_red = [&](float x, bool mx) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float y = __shfl_xor_sync(0xffffffffu, x, off);
      x = mx ? fmaxf(x, y) : x + y;
    }
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = x;
    __syncthreads();
    float r = red[0];
    for (int i = 1; i < kSimple / 32; ++i) r = mx ? fmaxf(r, red[i]) : r + red[i];
    return r;
  };
  float m = -CUDART_INF_F, l = 0.f;
  for (int k0 = lo; k0 <= pos; k0 += kSimple) {
    const int key = k0 + tid, n = min(kSimple, pos + 1 - k0);
    float s = -CUDART_INF_F;
    if (key <= pos) {
      const WT* kr = K + (int64_t)key * v.k_ld;
      s = 0.f;
      for (int d = 0; d < v.dim; ++d) s = fmaf(qs[d], to_f32(kr[d]), s);
      s = bound_score(v, s);
    }
    const float mn = fmaxf(m, block_red(s, true)), alpha = expf(m - mn);
    const float p = key <= pos ? expf(s - mn) : 0.f;
    ps[tid] = p;
    l = l * alpha + block_red(p, false);     // (its barriers also publish ps)
    m = mn;
    for (int d = tid; d < v.vdim; d += kSimple) {
      float o = os[d] * alpha;
      for (int i = 0; i < n; ++i) o = fmaf(ps[i], to_f32(V[(int64_t)(k0 + i) * v.v_ld + d]), o);
      os[d] = o;
    }
    __syncthreads();
  }
  const float inv = 1.0f / l;
  for (int d = tid; d < v.vdim; d += kSimple) {
    const int col = h * v.vdim + d;
    out[bp > 0 ? Layout<WT>::x_offset(t, col, bp) : (int64_t)t * ldo + col] = from_f32<WT>(os[d] * inv);
  }
}

// ---------------------------------------------------------------------------------------------
// Tensor cores (mma.sync), one or a few queries per sequence: bound by reading the cache.  A CTA owns a run of keys of one token and
// up to 8 query heads of one key head; each of its 4 warps streams blocks of 16 keys through its own ring in shared memory:
//   S[key, head]  = K[key, :] . Q[head, :]        M = keys, N = heads
//   O^T[d, head] += V^T[d, key] P[key, head]      M = d, N = heads
// Warps, then CTAs (the last one to finish), are merged with the (max, sum, weighted O) rule.
// ---------------------------------------------------------------------------------------------
constexpr int kThreads = 128, kRing = 3;

__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t a) {
  uint32_t d;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;\n" : "=r"(d) : "r"(a));
  return d;
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// cap tanh(s / cap) through one exponential and one reciprocal, absolute error a few 1e-7 cap
__device__ __forceinline__ float bound_fast(float s, float cap, float two_over_cap) { return cap - 2.0f * __fdividef(cap, 1.0f + __expf(fminf(s * two_over_cap, 80.0f))); }

template <int DK, int DV>
constexpr size_t split_smem() {
  const size_t ring = (size_t)4 * kRing * 16 * ((DK + 8) + (DV + 8)) * 2, merge = (size_t)4 * 8 * DV * 4;
  return 8 * (DK + 8) * 2 + (ring > merge ? ring : merge);
}

template <int DK, int DV, bool PREP>
__global__ void __launch_bounds__(kThreads) window_split_kernel(const WindowView v, const WindowRows in, int nsplit, float* __restrict__ part,
                                                                unsigned* __restrict__ counters, __nv_bfloat16* __restrict__ out, int ldo, int bp) {
  constexpr int PK = DK + 8, PV = DV + 8, NK = DK / 16, NV = DV / 16;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ float sm_m[4][8], sm_l[4][8];
  __shared__ int is_last;
  __shared__ float2 s_cs[PREP ? DK / 2 : 1];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sm_raw);            // [8][PK]
  __nv_bfloat16* ring = sQ + 8 * PK;                                       // [4 warps][kRing][16][PK | PV]
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int gq = v.H / v.G, hb_n = (gq + 7) >> 3;
  const int unit = blockIdx.x, hb = unit % hb_n, ta = unit / hb_n, t = ta / v.G, a = ta - t * v.G;
  const int h0 = a * gq + hb * 8, nh = min(8, gq - hb * 8);
  const int nk = (v.dim + 15) >> 4, nv = (v.vdim + 15) >> 4;
  __nv_bfloat16* stage = ring + warp * kRing * 16 * (PK + PV);
  // columns behind the width never come from memory
  for (int i = tid; i < 8 * PK; i += kThreads) sQ[i] = __float2bfloat16_rn(0.f);
  for (int i = lane; i < kRing * 16; i += 32)
    for (int c = v.k_ld; c < nk * 16; ++c) stage[(i >> 4) * 16 * (PK + PV) + (i & 15) * PK + c] = __float2bfloat16_rn(0.f);
  pdl_wait();
  const int pos = v.pos[t];
  const int lo = v.window > 0 ? max(0, pos - v.window + 1) : 0;
  const int lo16 = lo & ~15, n_keys = pos + 1 - lo16;
  const int kpc = (((n_keys + nsplit - 1) / nsplit + 63) >> 6) << 6;
  const int nvalid = (n_keys + kpc - 1) / kpc;
  const int k_begin = lo16 + blockIdx.y * kpc, k_end = min(pos + 1, k_begin + kpc);
  if (k_begin > pos) return;
  __nv_bfloat16* K = reinterpret_cast<__nv_bfloat16*>(v.keys) + ((int64_t)v.seq[t] * v.G + a) * v.cap * v.k_ld;
  __nv_bfloat16* V = reinterpret_cast<__nv_bfloat16*>(v.values) + ((int64_t)v.seq[t] * v.G + a) * v.cap * v.v_ld;
  __syncthreads();
  const int kpw = kpc >> 2, wb = k_begin + warp * kpw, we = min(k_end, wb + kpw);
  const int blocks = we > wb ? (we - wb + 15) >> 4 : 0;
  const int kc = v.k_ld >> 3, vc = v.v_ld >> 3;
  auto load = [&](int i) {
    __nv_bfloat16* sk = stage + (i % kRing) * 16 * (PK + PV);
    __nv_bfloat16* sv = sk + 16 * PK;
    const int key0 = wb + i * 16;
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      const int r = (lane >> 2) + 8 * rr;
      const __nv_bfloat16* kr = K + (int64_t)(key0 + r) * v.k_ld;
      const __nv_bfloat16* vr = V + (int64_t)(key0 + r) * v.v_ld;
#pragma unroll
      for (int c0 = 0; c0 < DK / 8; c0 += 4)
        if (c0 + tq < kc) tc::cp_async16(tc::smem_u32(sk + r * PK + (c0 + tq) * 8), kr + (c0 + tq) * 8, 16u);
#pragma unroll
      for (int c0 = 0; c0 < DV / 8; c0 += 4)
        if (c0 + tq < vc) tc::cp_async16(tc::smem_u32(sv + r * PV + (c0 + tq) * 8), vr + (c0 + tq) * 8, 16u);
    }
  };
  // the first blocks are on their way while the queries are prepared (not the one that gets the newest key)
  int early = 0;
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) {
    if (i < blocks && (!PREP || wb + i * 16 + 16 <= pos)) { load(i); early = i + 1; }
  }
  if (PREP) {
    const bool newest = in.k && k_end == pos + 1;
    for (int p = tid; p < (v.rot_dims >> 1); p += kThreads) s_cs[p] = turn(v, t, pos, p, 1.f, 0.f);
    if (newest) {
      __nv_bfloat16* o = V + (int64_t)pos * v.v_ld;
      const float* x = reinterpret_cast<const float*>(in.v) + (int64_t)t * in.v_pitch + a * v.vdim;
      for (int d = tid; d < v.vdim; d += kThreads) o[d] = __float2bfloat16_rn(x[d]);
    }
    __syncthreads();
    for (int u = warp; u < nh + (newest ? 1 : 0); u += 4) {
      const float* x = u < nh ? reinterpret_cast<const float*>(in.q) + (int64_t)t * in.q_pitch + (h0 + u) * v.dim
                              : reinterpret_cast<const float*>(in.k) + (int64_t)t * in.k_pitch + a * v.dim;
      __nv_bfloat16* o = u < nh ? sQ + u * PK : K + (int64_t)pos * v.k_ld;
      float2 y[DK / 64];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < DK / 64; ++i) {
        const int p = lane + 32 * i;
        int lo, hi;
        pair_of(v, p, &lo, &hi);
        y[i] = make_float2(lo < v.dim ? x[lo] : 0.f, hi < v.dim ? x[hi] : 0.f);
        if (p < (v.rot_dims >> 1)) {
          const float2 cs = s_cs[p];
          y[i] = make_float2(y[i].x * cs.x - y[i].y * cs.y, y[i].y * cs.x + y[i].x * cs.y);
        }
        ss += y[i].x * y[i].x + y[i].y * y[i].y;
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
      const float inv = 1.0f / sqrtf(ss / (float)v.dim + v.eps);
#pragma unroll
      for (int i = 0; i < DK / 64; ++i) {
        int lo, hi;
        pair_of(v, lane + 32 * i, &lo, &hi);
        if (lo < v.dim) o[lo] = __float2bfloat16_rn(y[i].x * inv);
        if (hi < v.dim) o[hi] = __float2bfloat16_rn(y[i].y * inv);
      }
    }
    __threadfence_block();
  } else {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(in.q) + (int64_t)t * in.q_pitch + (int64_t)h0 * v.dim;
    for (int i = tid; i < nh * v.dim; i += kThreads) sQ[(i / v.dim) * PK + i % v.dim] = q[i];
  }
  __syncthreads();
  uint32_t qf[NK][2];                        // B operand: Q[head g][16 dk + 2 tq, + 1] and + 8
#pragma unroll
  for (int dk = 0; dk < NK; ++dk) {
    qf[dk][0] = *reinterpret_cast<const uint32_t*>(sQ + g * PK + 16 * dk + 2 * tq);
    qf[dk][1] = *reinterpret_cast<const uint32_t*>(sQ + g * PK + 16 * dk + 2 * tq + 8);
  }
  float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.f, l1 = 0.f;
  float o[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const float two_over_cap = v.score_cap > 0.f ? 2.0f / v.score_cap : 0.f;
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) {
    if (i < blocks && i >= early) load(i);
    tc::cp_async_commit();
  }
  for (int i = 0; i < blocks; ++i) {
    if (i + kRing - 1 < blocks) load(i + kRing - 1);
    tc::cp_async_commit();
    tc::cp_async_wait<kRing - 1>();
    __syncwarp();
    const __nv_bfloat16* sk = stage + (i % kRing) * 16 * (PK + PV);
    const __nv_bfloat16* sv = sk + 16 * PK;
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t ka = tc::smem_u32(sk + (lane & 15) * PK + (lane >> 4) * 8);
#pragma unroll
    for (int dk = 0; dk < NK; ++dk) {
      if (dk >= nk) break;
      uint32_t kf[4];
      ldsm4(kf, ka + dk * 32);
      mma16816(s, kf, qf[dk][0], qf[dk][1]);
    }
    const int key0 = wb + i * 16 + g;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = key0 + 8 * (e >> 1);
      s[e] *= v.scale;
      if (v.score_cap > 0.f) s[e] = bound_fast(s[e], v.score_cap, two_over_cap);
      if (key < lo || key > pos) s[e] = -CUDART_INF_F;
    }
    float bm0 = fmaxf(s[0], s[2]), bm1 = fmaxf(s[1], s[3]);
#pragma unroll
    for (int off = 4; off < 32; off <<= 1) {
      bm0 = fmaxf(bm0, __shfl_xor_sync(0xffffffffu, bm0, off));
      bm1 = fmaxf(bm1, __shfl_xor_sync(0xffffffffu, bm1, off));
    }
    const float mn0 = fmaxf(m0, bm0), mn1 = fmaxf(m1, bm1);
    const float z0 = mn0 == -CUDART_INF_F ? 0.f : mn0, z1 = mn1 == -CUDART_INF_F ? 0.f : mn1;      // a block may lie before the window
    const float a0 = exp2f((m0 - z0) * kLog2e), a1 = exp2f((m1 - z1) * kLog2e);
    const float p00 = exp2f((s[0] - z0) * kLog2e), p01 = exp2f((s[1] - z1) * kLog2e);
    const float p10 = exp2f((s[2] - z0) * kLog2e), p11 = exp2f((s[3] - z1) * kLog2e);
    l0 = l0 * a0 + (p00 + p10);
    l1 = l1 * a1 + (p01 + p11);
    m0 = mn0;
    m1 = mn1;
    const uint32_t pb0 = movmatrix_trans(pack_bf16(p00, p01)), pb1 = movmatrix_trans(pack_bf16(p10, p11));
    // A operand V^T: rows d, columns keys, from the row-major block
    const uint32_t va = tc::smem_u32(sv + ((lane & 7) + ((lane >> 4) << 3)) * PV + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int dm = 0; dm < NV; ++dm) {
      if (dm >= nv) break;
      uint32_t vf[4];
      ldsm4_trans(vf, va + dm * 32);
      o[dm][0] *= a0; o[dm][1] *= a1; o[dm][2] *= a0; o[dm][3] *= a1;
      mma16816(o[dm], vf, pb0, pb1);
    }
    __syncwarp();                                       // the stage is free
  }
  tc::cp_async_wait<0>();
#pragma unroll
  for (int off = 4; off < 32; off <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, off);
    l1 += __shfl_xor_sync(0xffffffffu, l1, off);
  }
  __syncthreads();                                      // the rings become the merge buffer
  float* sm_o = reinterpret_cast<float*>(ring);         // [4][8][DV]
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int h = 2 * tq + e;
    if (h >= nh) continue;
    if (g == 0) { sm_m[warp][h] = e ? m1 : m0; sm_l[warp][h] = e ? l1 : l0; }
#pragma unroll
    for (int dm = 0; dm < NV; ++dm) {
      sm_o[(warp * 8 + h) * DV + 16 * dm + g] = o[dm][e];
      sm_o[(warp * 8 + h) * DV + 16 * dm + g + 8] = o[dm][2 + e];
    }
  }
  __syncthreads();
  auto put = [&](int h, int d, float x) {
    const int col = (h0 + h) * v.vdim + d;
    out[bp > 0 ? Layout<__nv_bfloat16>::x_offset(t, col, bp) : (int64_t)t * ldo + col] = __float2bfloat16_rn(x);
  };
  const int64_t slot0 = (int64_t)unit * nsplit;
  float* part_ml = part;                                // [units][nsplit][8][2], then [units][nsplit][8][vdim]
  float* part_o = part + (int64_t)gridDim.x * nsplit * 16;
  for (int i = tid; i < nh * v.vdim; i += kThreads) {
    const int h = i / v.vdim, d = i - h * v.vdim;
    const float M = fmaxf(fmaxf(sm_m[0][h], sm_m[1][h]), fmaxf(sm_m[2][h], sm_m[3][h]));
    const float Z = M == -CUDART_INF_F ? 0.f : M;
    float acc = 0.f, lsum = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float wgt = exp2f((sm_m[w][h] - Z) * kLog2e);
      if (wgt > 0.f) acc += wgt * sm_o[(w * 8 + h) * DV + d];
      lsum += wgt * sm_l[w][h];
    }
    if (nvalid == 1) { put(h, d, acc / lsum); continue; }
    part_o[((slot0 + blockIdx.y) * 8 + h) * v.vdim + d] = acc;
    if (d == 0) {
      part_ml[((slot0 + blockIdx.y) * 8 + h) * 2] = M;
      part_ml[((slot0 + blockIdx.y) * 8 + h) * 2 + 1] = lsum;
    }
  }
  if (nvalid == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    is_last = atomicAdd(&counters[unit], 1u) == (unsigned)nvalid - 1u;
    if (is_last) counters[unit] = 0u;                   // ready for the next launch
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  // weights of the parts, then their weighted sum
  float* wt = reinterpret_cast<float*>(ring);           // [nvalid][8]
  for (int h = warp; h < nh; h += 4) {
    float M = -CUDART_INF_F;
    for (int sp = lane; sp < nvalid; sp += 32) M = fmaxf(M, __ldcg(part_ml + ((slot0 + sp) * 8 + h) * 2));
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, off));
    float den = 0.f;
    for (int sp = lane; sp < nvalid; sp += 32) {
      const float w = exp2f((__ldcg(part_ml + ((slot0 + sp) * 8 + h) * 2) - M) * kLog2e);
      wt[sp * 8 + h] = w;
      den += w * __ldcg(part_ml + ((slot0 + sp) * 8 + h) * 2 + 1);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) den += __shfl_xor_sync(0xffffffffu, den, off);
    if (lane == 0) sm_l[0][h] = 1.0f / den;
  }
  __syncthreads();
  for (int i = tid; i < nh * v.vdim; i += kThreads) {
    const int h = i / v.vdim, d = i - h * v.vdim;
    float acc = 0.f;
#pragma unroll 8
    for (int sp = 0; sp < nvalid; ++sp) acc += wt[sp * 8 + h] * __ldcg(part_o + ((slot0 + sp) * 8 + h) * v.vdim + d);
    put(h, d, acc * sm_l[0][h]);
  }
}

bool split_ok(int dtype, const WindowView& v) { return dtype == LMB200_BF16 && v.dim <= 256 && v.vdim <= 256; }
int wide_of(const WindowView& v) { const int w = std::max(v.dim, v.vdim); return w <= 64 ? 64 : w <= 128 ? 128 : 256; }

template <int D>
int32_t launch_split(const WindowView& v, const WindowRows& in, int nsplit, float* part, unsigned* counters, void* out, int ldo, int bp, cudaStream_t st) {
  const int hb = (int)ceil_div(v.H / v.G, 8);
  const dim3 grid((unsigned)((int64_t)v.T * v.G * hb), (unsigned)nsplit);
  LMB_CUDA(launch_k(in.in_f32 ? window_split_kernel<D, D, true> : window_split_kernel<D, D, false>, grid, dim3(kThreads), split_smem<D, D>(), st, v, in, nsplit,
                    part, counters, (__nv_bfloat16*)out, ldo, bp));
  return LMB200_OK;
}

}  // namespace

int32_t window_configure() {
#define LMB_CFG(D)                                                                                                                                     \
  LMB_CUDA(cudaFuncSetAttribute(window_split_kernel<D, D, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)split_smem<D, D>()));                \
  LMB_CUDA(cudaFuncSetAttribute(window_split_kernel<D, D, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)split_smem<D, D>()))
  LMB_CFG(64);
  LMB_CFG(128);
  LMB_CFG(256);
#undef LMB_CFG
  return LMB200_OK;
}

template <typename IT, typename WT>
int32_t prep_rows(const WindowView& v, const WindowRows& in, void* q_out, cudaStream_t st) {
  const int64_t warps = (int64_t)v.T * (ceil_div(v.H + (in.k ? v.G : 0), kHeads) + (in.k ? ceil_div(v.G, kHeads) : 0));
  const dim3 grid((unsigned)ceil_div(warps, 8));
  if (v.dim <= 64) LMB_CUDA(launch_k(window_prep_rows_kernel<IT, WT, 1>, grid, dim3(256), 0, st, v, in, (WT*)q_out));
  else if (v.dim <= 128) LMB_CUDA(launch_k(window_prep_rows_kernel<IT, WT, 2>, grid, dim3(256), 0, st, v, in, (WT*)q_out));
  else LMB_CUDA(launch_k(window_prep_rows_kernel<IT, WT, 4>, grid, dim3(256), 0, st, v, in, (WT*)q_out));
  return LMB200_OK;
}

int32_t window_prep(Ctx* ctx, int dtype, const WindowView& v, const WindowRows& in, void* q_out, cudaStream_t st) {
  if (v.rot_interleaved && v.dim % 2 == 0 && v.dim <= 256 && in.q_pitch % 2 == 0 && in.k_pitch % 2 == 0 && v.k_ld % 2 == 0) {
    ctx->launches++;
    if (dtype != LMB200_BF16) return prep_rows<float, float>(v, in, q_out, st);
    return in.in_f32 ? prep_rows<float, __nv_bfloat16>(v, in, q_out, st) : prep_rows<__nv_bfloat16, __nv_bfloat16>(v, in, q_out, st);
  }
  const int units = v.H + (in.k ? 2 * v.G : 0);
  const dim3 grid((unsigned)ceil_div((int64_t)v.T * units, 8));
  if (dtype != LMB200_BF16)
    LMB_CUDA(launch_k(window_prep_kernel<float, float>, grid, dim3(256), 0, st, v, in, (float*)q_out));
  else if (in.in_f32)
    LMB_CUDA(launch_k(window_prep_kernel<float, __nv_bfloat16>, grid, dim3(256), 0, st, v, in, (__nv_bfloat16*)q_out));
  else
    LMB_CUDA(launch_k(window_prep_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, st, v, in, (__nv_bfloat16*)q_out));
  ctx->launches++;
  return LMB200_OK;
}

WindowPlan window_plan(const Ctx* ctx, int dtype, const WindowView& v, int T, int ctx_len) {
  WindowPlan pl;
  if (!split_ok(dtype, v)) return pl;
  const int64_t units = (int64_t)T * v.G * ceil_div(v.H / v.G, 8);
  const int keys = (v.window > 0 ? std::min(ctx_len, v.window) : ctx_len) + 15;
  const int64_t slots = (int64_t)ctx->sm_count * (wide_of(v) <= 64 ? 4 : wide_of(v) <= 128 ? 2 : 1);
  double best = 1e30;
  for (int ns = 1; ns <= std::max(1, std::min(64, (int)ceil_div(keys, 64))); ++ns) {       // waves of CTAs x (keys of one + its fixed cost)
    const double cost = (double)ceil_div(units * ns, slots) * (double)(round_up(ceil_div(keys, ns), 64) + (ns > 1 ? 160 : 96));
    if (cost < best) { best = cost; pl.nsplit = ns; }
  }
  pl.part_floats = pl.nsplit > 1 ? units * pl.nsplit * 8 * (2 + v.vdim) : 0;
  pl.n_counters = (int)units;
  return pl;
}

int32_t window_attend(Ctx* ctx, int dtype, const WindowView& v, const WindowRows& in, const WindowPlan& plan, float* part, unsigned* counters, void* out,
                      int ldo, int bp, cudaStream_t st) {
  LMB_REQUIRE(v.T >= 1 && v.G >= 1 && v.H % v.G == 0, "attention: %d tokens, %d heads over %d", v.T, v.H, v.G);
  if (plan.nsplit >= 1) {
    switch (wide_of(v)) {
      case 64: LMB_TRY(launch_split<64>(v, in, plan.nsplit, part, counters, out, ldo, bp, st)); break;
      case 128: LMB_TRY(launch_split<128>(v, in, plan.nsplit, part, counters, out, ldo, bp, st)); break;
      default: LMB_TRY(launch_split<256>(v, in, plan.nsplit, part, counters, out, ldo, bp, st));
    }
  } else {
    const size_t smem = (size_t)(v.dim + v.vdim + kSimple) * 4;
    LMB_REQUIRE(smem <= 48 * 1024 && v.T <= 65535, "attention: heads of %d x %d, %d tokens", v.dim, v.vdim, v.T);
    const dim3 grid((unsigned)v.H, (unsigned)v.T);
    if (dtype == LMB200_BF16)
      LMB_CUDA(launch_k(window_simple_kernel<__nv_bfloat16>, grid, dim3(kSimple), smem, st, v, (const __nv_bfloat16*)in.q, (__nv_bfloat16*)out, ldo, bp));
    else
      LMB_CUDA(launch_k(window_simple_kernel<float>, grid, dim3(kSimple), smem, st, v, (const float*)in.q, (float*)out, ldo, bp));
  }
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
