// Kernels of the channel-wise gated delta rule (see delta.cuh).
#include "activations.cuh"
#include "delta.cuh"
#include "pdl.cuh"
#include "tc.cuh"

namespace lmb {
namespace {

constexpr float kUnitEps = 1e-6f;
constexpr int kRun = 8;                  // tokens a warp of the convolution walks over

__device__ __forceinline__ float warp_sum(float x) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) x += __shfl_xor_sync(0xffffffffu, x, off);
  return x;
}
template <typename T> struct Pair;
template <> struct Pair<float> { typedef float2 V; };
template <> struct Pair<__nv_bfloat16> { typedef __nv_bfloat162 V; };
__device__ __forceinline__ float2 pair_f32(float2 v) { return v; }
__device__ __forceinline__ float2 pair_f32(__nv_bfloat162 v) { return __bfloat1622float2(v); }
__device__ __forceinline__ float conv_silu(float x, float) { return silu_f32(x); }
__device__ __forceinline__ float conv_silu(float x, __nv_bfloat16) { return __fdividef(x, 1.0f + __expf(-x)); }      // rounded to bf16 next
__device__ __forceinline__ void put_pair(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void put_pair(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

// a warp: one head (of q, then k, then v) over kRun packed rows; lane: channel pairs.  The rows before the current one stay in registers.
template <typename T, int NP, int MAXT>
__global__ void __launch_bounds__(256) delta_conv_kernel(const DeltaView v, T* __restrict__ out, float* __restrict__ rq, float* __restrict__ rk) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, units = 2 * v.G + v.H;
  const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int u = (int)(id % units);
  const int64_t first = id / units * kRun;
  if (first >= v.total) return;
  const int kind = u < v.G ? 0 : u < 2 * v.G ? 1 : 2;
  const int a = kind == 0 ? u : kind == 1 ? u - v.G : u - 2 * v.G;
  const int width = kind == 2 ? v.vdim : v.dim, C = 2 * v.G * v.dim + v.H * v.vdim;
  const int c0 = (kind == 0 ? 0 : kind == 1 ? v.G * v.dim : 2 * v.G * v.dim) + a * width;      // channel of the head
  const T* src = reinterpret_cast<const T*>(kind == 0 ? v.q : kind == 1 ? v.k : v.v) + a * width;
  const int pitch = kind == 0 ? v.q_pitch : kind == 1 ? v.k_pitch : v.v_pitch;
  const bool even = ((width | pitch | C | c0) & 1) == 0;
  auto raw = [&](int64_t t, int c) {
    const T* p = src + t * pitch + c;
    if (even) return pair_f32(*reinterpret_cast<const typename Pair<T>::V*>(p));
    return make_float2(to_f32(p[0]), c + 1 < width ? to_f32(p[1]) : 0.f);
  };
  float2 w[MAXT][NP], h[MAXT > 1 ? MAXT - 1 : 1][NP];
#pragma unroll
  for (int j = 0; j < MAXT; ++j)
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int c = 2 * (lane + 32 * i);
      const float* p = v.conv + (int64_t)j * C + c0 + c;
      w[j][i] = j < v.taps && c < width ? make_float2(p[0], c + 1 < width ? p[1] : 0.f) : make_float2(0.f, 0.f);
    }
  // few taps: all rows of the run, and the ones before it, are in flight at once
  constexpr bool kAhead = MAXT <= 4;
  constexpr int kBack = kAhead ? MAXT - 1 : 0, kRows = kAhead ? kRun : 1;
  const int n = (int)min((int64_t)kRun, v.total - first);
  // lane r: row first - (MAXT - 1) + r
  const int64_t mine = first - (MAXT - 1) + lane;
  const bool have = lane < n + MAXT - 1 && mine >= 0;
  const int my_seq = have ? v.seq[mine] : -1, my_pos = have ? v.pos[mine] : 0;
  typename Pair<T>::V ahead[kBack + kRows][NP];
  if (kAhead && even) {
#pragma unroll
    for (int r = 0; r < kBack + kRows; ++r)
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int c = 2 * (lane + 32 * i);
        const int64_t t = first - kBack + r;
        if (t >= 0 && r < kBack + n && c < width) ahead[r][i] = *reinterpret_cast<const typename Pair<T>::V*>(src + t * pitch + c);
      }
  }
  // the rows before packed row first + r, of sequence s at position p
  auto history = [&](int r, int s, int p, auto x_of) {
#pragma unroll
    for (int j = 1; j < MAXT; ++j) {
      const bool packed = __shfl_sync(0xffffffffu, my_seq, r + MAXT - 1 - j) == s;        // the row before is in this call too
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int c = 2 * (lane + 32 * i);
        float2 x = make_float2(0.f, 0.f);
        if (j < v.taps && p - j >= 0 && c < width) {
          if (packed) x = x_of(r - j, i, c);
          else {
            const float* q = v.ring + ((int64_t)s * v.taps + (p - j) % v.taps) * C + c0 + c;
            x = make_float2(q[0], c + 1 < width ? q[1] : 0.f);
          }
        }
        h[j - 1][i] = x;
      }
    }
  };
  auto token = [&](int r, auto x_of) {
    const int64_t t = first + r;
    float ss = 0.f;
    T* o = out + t * C + c0;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int c = 2 * (lane + 32 * i);
      if (c >= width) continue;
      const float2 x = x_of(r, i, c);
      float2 y = make_float2(w[0][i].x * x.x, w[0][i].y * x.y);
#pragma unroll
      for (int j = 1; j < MAXT; ++j) { y.x = fmaf(w[j][i].x, h[j - 1][i].x, y.x); y.y = fmaf(w[j][i].y, h[j - 1][i].y, y.y); }
#pragma unroll
      for (int j = MAXT - 2; j > 0; --j) h[j][i] = h[j - 1][i];
      h[0][i] = x;
      const T r0 = from_f32<T>(conv_silu(y.x, T())), r1 = from_f32<T>(c + 1 < width ? conv_silu(y.y, T()) : 0.f);
      const float z0 = to_f32(r0), z1 = to_f32(r1);              // the length is that of the stored vector
      ss += z0 * z0 + z1 * z1;
      if (even) put_pair(o + c, make_float2(z0, z1));
      else {
        o[c] = r0;
        if (c + 1 < width) o[c + 1] = r1;
      }
    }
    return ss;
  };
  float my_ss = 0.f;                       // lane r: token r's sum
  const int s0 = __shfl_sync(0xffffffffu, my_seq, MAXT - 1), p0 = __shfl_sync(0xffffffffu, my_pos, MAXT - 1);
  const bool one = __all_sync(0xffffffffu, lane < MAXT - 1 || lane >= n + MAXT - 1 || my_seq == s0);
  if (kAhead && even && one) {
    auto x_of = [&](int r, int i, int) { return pair_f32(ahead[kBack + r][i]); };
    history(0, s0, p0, x_of);
    float ss[kRows];
#pragma unroll
    for (int r = 0; r < kRows; ++r) ss[r] = r < n ? token(r, x_of) : 0.f;
    if (kind < 2) {
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        const float s = warp_sum(ss[r]);
        if (lane == r) my_ss = s;
      }
    }
  } else {
    auto x_of = [&](int r, int, int c) { return raw(first + r, c); };
    int last = -1;
#pragma unroll 1
    for (int r = 0; r < n; ++r) {
      const int s = __shfl_sync(0xffffffffu, my_seq, r + MAXT - 1), p = __shfl_sync(0xffffffffu, my_pos, r + MAXT - 1);
      if (s != last) history(r, s, p, x_of);
      last = s;
      const float y = warp_sum(token(r, x_of));
      if (lane == r) my_ss = y;
    }
  }
  if (kind < 2 && lane < n) {
    const float f = 1.0f / sqrtf(my_ss + kUnitEps);
    if (kind == 0) rq[(first + lane) * v.G + a] = f / sqrtf((float)v.dim);
    else rk[(first + lane) * v.G + a] = f;
  }
}

// the last raw inputs of every sequence's portion into its ring
template <typename T>
__global__ void __launch_bounds__(256) delta_ring_kernel(const DeltaView v) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y, j = blockIdx.z, C = 2 * v.G * v.dim + v.H * v.vdim;
  const int n = v.len[s];
  if (j >= n) return;
  const int64_t t = v.start[s] + n - 1 - j;
  const int p = v.pos0[s] + n - 1 - j;
  const int kd = v.G * v.dim;
  for (int c = blockIdx.x * 256 + threadIdx.x; c < C; c += gridDim.x * 256) {
    const T x = c < kd ? reinterpret_cast<const T*>(v.q)[t * v.q_pitch + c]
                       : c < 2 * kd ? reinterpret_cast<const T*>(v.k)[t * v.k_pitch + c - kd] : reinterpret_cast<const T*>(v.v)[t * v.v_pitch + c - 2 * kd];
    v.ring[((int64_t)s * v.taps + p % v.taps) * C + c] = to_f32(x);
  }
}

// One CTA per (value head, sequence).  Thread (c, w): value columns 4 c .., rows w, w + W, ... of the state.  One pass over the state per
// token gives both S^T k and S^T q after the decay; with u the written value, o = S^T q + (k . q) u and S <- S + k u^T.  KEEP: the state
// lies in shared memory over all tokens (one bulk copy brings it while the inputs are prepared); else it is read twice per token.
constexpr int kStep = 256;
constexpr size_t kKeepMax = 100 * 1024;

struct StepShape {
  int V4, blocks, W, parts;
  bool quad;                             // a warp covers 8 column groups x 4 rows: shuffles add four rows, few partial sums meet in shared memory
};
__host__ __device__ inline StepShape step_shape(int vdim) {
  StepShape p;
  p.V4 = (vdim + 3) >> 2;
  p.blocks = p.V4 >> 3;
  p.quad = (p.V4 & 7) == 0 && (kStep / 32) % p.blocks == 0;
  p.W = p.quad ? kStep / 32 / p.blocks * 4 : kStep / p.V4;
  p.parts = p.quad ? p.W / 4 : p.W;
  return p;
}
__host__ __device__ inline size_t step_vectors(int dim, const StepShape& p) {        // floats
  return (size_t)(3 * ((dim + 3) & ~3) + 8 * p.V4 + p.parts * 8 * p.V4);
}

template <typename IT, typename OT, bool RAW, bool KEEP>
__global__ void __launch_bounds__(kStep, 3) delta_step_kernel(const DeltaView v, int* err) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[kStep / 32], s_dot[3];
  __shared__ __align__(8) uint64_t full;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = v.dim, V = v.vdim;
  const StepShape sh = step_shape(V);
  const int V4 = sh.V4, W = sh.W, parts = sh.parts;
  const int gq = v.H / v.G, a = h / gq;
  float* qs = sm;
  float* ks = qs + ((D + 3) & ~3);
  float* gs = ks + ((D + 3) & ~3);
  float* vs = gs + ((D + 3) & ~3);         // [4 V4] v, then o
  float* us = vs + 4 * V4;                 // [4 V4]
  float* os = us + 4 * V4;                 // [parts][2][4 V4]
  float4* const state = reinterpret_cast<float4*>(v.state) + ((int64_t)b * v.H + h) * D * V4;
  float4* const S = KEEP ? reinterpret_cast<float4*>(sm + step_vectors(D, sh)) : state;
  const int c = sh.quad ? (warp % sh.blocks) * 8 + (lane & 7) : tid % V4, w = sh.quad ? warp / sh.blocks * 4 + (lane >> 3) : tid / V4;
  if (KEEP && tid == 0) {
    tc::mbar_init(&full, 1);
    tc::mbar_init_fence();
  }
  pdl_launch_dependents();
  pdl_wait();
  const int n = v.len[b], t0 = v.start[b], p0 = v.pos0[b];
  if (n <= 0) return;
  if (KEEP && tid == 0) {
    tc::mbar_expect_tx(&full, (uint32_t)(D * V4 * 16));
    tc::bulk_g2s(S, state, (uint32_t)(D * V4 * 16), &full);
  }
  bool dead = false;
  for (int it = 0; it < n; ++it) {
    const int64_t t = t0 + it;
    if (RAW) {
      const int C = 2 * v.G * D + v.H * V, now = p0 % v.taps, items = 3 * D + 4 * V4;
      float* ring = v.ring + (int64_t)b * v.taps * C;
      const bool owner = h == a * gq;
      // two elements of q, k, log g or v per round; all of their loads go out before any is used
      for (int i0 = tid; i0 < items; i0 += 2 * kStep) {
        float x[2], tap[2][4], wgt[2][4];
        int kind[2], di[2], ch[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + e * kStep;
          kind[e] = i >= items ? 4 : i < 3 * D ? i / D : 3;
          di[e] = i - min(kind[e], 3) * D;
          ch[e] = 0;
          x[e] = 0.f;
          if (kind[e] == 4 || (kind[e] == 3 && di[e] >= V)) continue;
          if (kind[e] == 2) {
            x[e] = v.decay[t * v.decay_pitch + h * D + di[e]];
            tap[e][0] = v.a_log[h];
            tap[e][1] = v.dt_bias[h * D + di[e]];
            continue;
          }
          const int col = kind[e] == 3 ? h * V + di[e] : a * D + di[e];
          ch[e] = kind[e] == 0 ? col : kind[e] == 1 ? v.G * D + col : 2 * v.G * D + col;
          x[e] = reinterpret_cast<const float*>(kind[e] == 0 ? v.q : kind[e] == 1 ? v.k : v.v)[t * (kind[e] == 0 ? v.q_pitch : kind[e] == 1 ? v.k_pitch : v.v_pitch) + col];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            wgt[e][j] = j < v.taps ? v.conv[(int64_t)j * C + ch[e]] : 0.f;
            tap[e][j] = j > 0 && j < v.taps && p0 - j >= 0 ? ring[(now - j < 0 ? now - j + v.taps : now - j) * C + ch[e]] : 0.f;
          }
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (kind[e] == 4) continue;
          if (kind[e] == 2) { gs[di[e]] = expf(log_decay_f32(x[e], tap[e][0], tap[e][1])); continue; }
          if (kind[e] == 3 && di[e] >= V) { vs[di[e]] = 0.f; continue; }
          float y = wgt[e][0] * x[e];
#pragma unroll
          for (int j = 1; j < 4; ++j) y = fmaf(wgt[e][j], tap[e][j], y);
          for (int j = 4; j < v.taps; ++j)
            if (p0 - j >= 0) y = fmaf(v.conv[(int64_t)j * C + ch[e]], ring[(p0 - j) % v.taps * C + ch[e]], y);
          if (kind[e] == 3 || owner) ring[now * C + ch[e]] = x[e];          // a slot no tap of this token reads
          (kind[e] == 0 ? qs : kind[e] == 1 ? ks : vs)[di[e]] = to_f32(from_f32<IT>(silu_f32(y)));
        }
      }
    } else {
      const IT* q = reinterpret_cast<const IT*>(v.q) + t * v.q_pitch + a * D;
      const IT* k = reinterpret_cast<const IT*>(v.k) + t * v.k_pitch + a * D;
      const IT* x = reinterpret_cast<const IT*>(v.v) + t * v.v_pitch + h * V;
      for (int d = tid; d < D; d += kStep) {
        qs[d] = to_f32(q[d]);
        ks[d] = to_f32(k[d]);
        gs[d] = expf(v.decay[t * v.decay_pitch + h * D + d]);
      }
      for (int d = tid; d < 4 * V4; d += kStep) vs[d] = d < V ? to_f32(x[d]) : 0.f;
    }
    const float beta = sigmoid_f32(v.b[t * v.b_pitch + h]);
    __syncthreads();
    if (KEEP && it == 0) tc::mbar_wait(&full, 0, dead, err);
    // the vectors stay unscaled in shared memory; their scales multiply the sums
    if (warp < 3) {
      float x = 0.f;
      for (int d = lane; d < D; d += 32) x += warp == 0 ? qs[d] * qs[d] : warp == 1 ? ks[d] * ks[d] : qs[d] * ks[d];
      x = warp_sum(x);
      if (lane == 0) s_dot[warp] = x;
    }
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
    if (w < W) {
#pragma unroll 4
      for (int d = w; d < D; d += W) {
        float4 x = S[(int64_t)d * V4 + c];
        const float g = gs[d], kd = ks[d], qd = qs[d];
        x.x *= g; x.y *= g; x.z *= g; x.w *= g;
        ak.x = fmaf(kd, x.x, ak.x); ak.y = fmaf(kd, x.y, ak.y); ak.z = fmaf(kd, x.z, ak.z); ak.w = fmaf(kd, x.w, ak.w);
        aq.x = fmaf(qd, x.x, aq.x); aq.y = fmaf(qd, x.y, aq.y); aq.z = fmaf(qd, x.z, aq.z); aq.w = fmaf(qd, x.w, aq.w);
      }
      if (sh.quad) {
#pragma unroll
        for (int off = 8; off < 32; off <<= 1) {
          ak.x += __shfl_xor_sync(0xffffffffu, ak.x, off); ak.y += __shfl_xor_sync(0xffffffffu, ak.y, off);
          ak.z += __shfl_xor_sync(0xffffffffu, ak.z, off); ak.w += __shfl_xor_sync(0xffffffffu, ak.w, off);
          aq.x += __shfl_xor_sync(0xffffffffu, aq.x, off); aq.y += __shfl_xor_sync(0xffffffffu, aq.y, off);
          aq.z += __shfl_xor_sync(0xffffffffu, aq.z, off); aq.w += __shfl_xor_sync(0xffffffffu, aq.w, off);
        }
      }
      if (!sh.quad || lane < 8) {
        const int part = sh.quad ? w >> 2 : w;
        *reinterpret_cast<float4*>(os + (part * 2) * 4 * V4 + 4 * c) = ak;
        *reinterpret_cast<float4*>(os + (part * 2 + 1) * 4 * V4 + 4 * c) = aq;
      }
    }
    __syncthreads();
    float rq, rk;
    if (RAW) { rq = 1.0f / sqrtf(s_dot[0] + kUnitEps) / sqrtf((float)D); rk = 1.0f / sqrtf(s_dot[1] + kUnitEps); }
    else { rq = v.rq[t * v.G + a]; rk = v.rk[t * v.G + a]; }
    const float kq = s_dot[2] * rq * rk;
    float ss = 0.f;
    for (int d = tid; d < 4 * V4; d += kStep) {
      float x = 0.f, y = 0.f;
      for (int j = 0; j < parts; ++j) { x += os[(j * 2) * 4 * V4 + d]; y += os[(j * 2 + 1) * 4 * V4 + d]; }
      const float u = d < V ? beta * (vs[d] - x * rk) : 0.f, o = y * rq + kq * u;
      us[d] = u * rk;                      // the key's scale on the way into the state
      vs[d] = o;
      if (d < V) ss += o * o;
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int j = 0; j < kStep / 32; ++j) tot += red[j];
    const float inv = 1.0f / sqrtf(tot / (float)V + v.eps);
    if (w < W) {
      const float4 u = *reinterpret_cast<const float4*>(us + 4 * c);
      const bool leave = it == n - 1;
#pragma unroll 4
      for (int d = w; d < D; d += W) {
        float4 x = S[(int64_t)d * V4 + c];
        const float g = gs[d], kd = ks[d];
        x.x = fmaf(kd, u.x, g * x.x); x.y = fmaf(kd, u.y, g * x.y); x.z = fmaf(kd, u.z, g * x.z); x.w = fmaf(kd, u.w, g * x.w);
        if (KEEP && leave) state[(int64_t)d * V4 + c] = x;
        else S[(int64_t)d * V4 + c] = x;
      }
    }
    OT* out = reinterpret_cast<OT*>(v.out);
    for (int d = tid; d < V; d += kStep) {
      const int col = h * V + d;
      const float gate = RAW ? sigmoid_f32(reinterpret_cast<const float*>(v.gate)[t * v.gate_pitch + col])
                             : to_f32(reinterpret_cast<const IT*>(v.gate)[t * v.gate_pitch + col]);
      out[v.bp > 0 ? Layout<OT>::x_offset((int)t, col, v.bp) : t * v.ldo + col] = from_f32<OT>(vs[d] * inv * v.norm[d] * gate);
    }
    __syncthreads();                       // vs, ks, gs and os are rewritten by the next token
  }
}

int32_t check(const DeltaView& v) {
  LMB_REQUIRE(v.G >= 1 && v.H % v.G == 0 && v.dim <= 256 && v.vdim <= 256 && v.taps >= 1 && v.taps <= 16, "delta rule: %d heads of %d x %d over %d, %d taps",
              v.H, v.dim, v.vdim, v.G, v.taps);
  return LMB200_OK;
}

template <typename T>
int32_t conv_launch(const DeltaView& v, T* out, float* rq, float* rk, cudaStream_t st) {
  const dim3 grid((unsigned)ceil_div(ceil_div(v.total, kRun) * (2 * v.G + v.H), 8));
  const int width = v.dim > v.vdim ? v.dim : v.vdim;
  if (v.taps <= 4) LMB_CUDA(launch_k(width <= 128 ? delta_conv_kernel<T, 2, 4> : delta_conv_kernel<T, 4, 4>, grid, dim3(256), 0, st, v, out, rq, rk));
  else LMB_CUDA(launch_k(width <= 128 ? delta_conv_kernel<T, 2, 16> : delta_conv_kernel<T, 4, 16>, grid, dim3(256), 0, st, v, out, rq, rk));
  const int C = 2 * v.G * v.dim + v.H * v.vdim;
  LMB_CUDA(launch_k(delta_ring_kernel<T>, dim3((unsigned)ceil_div(C, 256), (unsigned)v.B, (unsigned)v.taps), dim3(256), 0, st, v));
  return LMB200_OK;
}

}  // namespace

int32_t delta_configure() {
  typedef __nv_bfloat16 bf16;
  LMB_CUDA(cudaFuncSetAttribute(delta_step_kernel<bf16, bf16, true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kKeepMax));
  LMB_CUDA(cudaFuncSetAttribute(delta_step_kernel<bf16, bf16, false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kKeepMax));
  LMB_CUDA(cudaFuncSetAttribute(delta_step_kernel<float, float, false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kKeepMax));
  LMB_TRY(delta_chunk_configure());
  return delta_tc_configure();
}

int32_t delta_conv(Ctx* ctx, int dtype, const DeltaView& v, void* out, float* rq, float* rk, cudaStream_t st) {
  LMB_TRY(check(v));
  LMB_TRY(dtype == LMB200_BF16 ? conv_launch<__nv_bfloat16>(v, (__nv_bfloat16*)out, rq, rk, st) : conv_launch<float>(v, (float*)out, rq, rk, st));
  ctx->launches += 2;
  return LMB200_OK;
}

int32_t delta_steps(Ctx* ctx, int dtype, const DeltaView& v, cudaStream_t st) {
  LMB_TRY(check(v));
  const StepShape sh = step_shape(v.vdim);
  const size_t vectors = step_vectors(v.dim, sh) * 4, whole = vectors + (size_t)v.dim * sh.V4 * 16;
  const bool keep = whole <= kKeepMax, bf = dtype == LMB200_BF16;
  const size_t smem = keep ? whole : vectors;
  const dim3 grid((unsigned)v.H, (unsigned)v.B);
  typedef __nv_bfloat16 bf16;
  if (bf && v.raw) LMB_CUDA(launch_k(keep ? delta_step_kernel<bf16, bf16, true, true> : delta_step_kernel<bf16, bf16, true, false>, grid, dim3(kStep), smem, st, v, ctx->dev_err));
  else if (bf) LMB_CUDA(launch_k(keep ? delta_step_kernel<bf16, bf16, false, true> : delta_step_kernel<bf16, bf16, false, false>, grid, dim3(kStep), smem, st, v, ctx->dev_err));
  else {
    LMB_REQUIRE(!v.raw, "delta rule: float32 models prepare their rows");
    LMB_CUDA(launch_k(keep ? delta_step_kernel<float, float, false, true> : delta_step_kernel<float, float, false, false>, grid, dim3(kStep), smem, st, v, ctx->dev_err));
  }
  ctx->launches++;
  return LMB200_OK;
}

}  // namespace lmb
