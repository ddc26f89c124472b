// The gated delta rule with ONE decay per head (delta_rule.cu has one per key channel):
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;   y = o / rms(o) * w * silu(gate)
//
// q, k and v come through a short causal convolution per channel and silu; q and k are then unit vectors per head (q
// also times q_mult); beta = sigmoid(b), g = exp(-exp(A_log) softplus(a + dt_bias)).  Everything after the projections is
// float.
//
// What a request keeps: S [heads, value channels, key channels] (float), and the last `taps` rows of q | k | v before the
// convolution as a RING over positions: position p's row lies at place p % taps.  A token reads the taps - 1 places
// before its own and writes its own, so blocks that share a request's channels need not wait for one another, and what
// lies before the sequence's start is known by its position alone.
//
//   delta_head_step     single tokens: everything above in one kernel, a cluster of blocks per (request, head)
//   delta_head_prepare  portions: a warp per (head of q / k / v, run of tokens) -> float rows of q, k, v and per head g and
//                       beta (the recurrence itself is delta_rule.cu's)
//   conv_ring_write     portions: their last rows into the ring, after delta_head_prepare has read it
#include "cluster_common.cuh"

using namespace ccb;

namespace {

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

struct HeadDelta {
  int ld, oq, ok, ov, ob, oa, og;   // columns of the projections' rows: q, k (G dk), v (H dv), b, a (H), gate (H dv)
  int G, H, dk, dv, taps;
  const float* conv_w;              // [taps, C], tap-major, C = 2 G dk + H dv
  const float* A_log;
  const float* dt_bias;
  const int *positions, *entry_of_token, *cu_q, *state_slot;
  float q_mult, unit_eps;
  int n_slots;
};

// The row of position p in the ring of a slot.
template <typename T>
__device__ __forceinline__ size_t ring_at(int slot, int p, int taps, int C) {
  return ((size_t)slot * taps + p % taps) * C;
}

template <typename T> struct Row4;   // four neighbouring elements as they are stored
template <> struct Row4<float> {
  using Raw = float4;
  static __device__ __forceinline__ Raw load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ Raw zero() { return make_float4(0.f, 0.f, 0.f, 0.f); }
  static __device__ __forceinline__ float4 value(Raw r) { return r; }
  static __device__ __forceinline__ void store(float* p, Raw r) { *reinterpret_cast<float4*>(p) = r; }
};
template <> struct Row4<__nv_bfloat16> {
  using Raw = uint2;
  static __device__ __forceinline__ Raw load(const __nv_bfloat16* p) { return *reinterpret_cast<const uint2*>(p); }
  static __device__ __forceinline__ Raw zero() { return make_uint2(0u, 0u); }
  static __device__ __forceinline__ float4 value(Raw r) {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, Raw r) { *reinterpret_cast<uint2*>(p) = r; }
};

__device__ __forceinline__ void fma4(float4& a, const float4 x, const float4 y) {
  a.x = fmaf(x.x, y.x, a.x); a.y = fmaf(x.y, y.y, a.y); a.z = fmaf(x.z, y.z, a.z); a.w = fmaf(x.w, y.w, a.w);
}
__device__ __forceinline__ float dot4(const float4 a, const float4 b) {
  return (a.x * b.x + a.y * b.y) + (a.z * b.z + a.w * b.w);
}
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f(x); }
__device__ __forceinline__ float4 silu4(const float4 x) { return make_float4(silu_f(x.x), silu_f(x.y), silu_f(x.z), silu_f(x.w)); }

constexpr int kStepWarps = 4, kStepThreads = 32 * kStepWarps;
constexpr int kStepCols = 8;   // columns of S a warp holds at once where a column takes all its lanes

// Single tokens.  A cluster of blocks (.x) per (head, request): each redoes the head's q and k and owns a run of
// `cols` value channels, i.e. columns of S; the sum of squares that the output's norm divides by is made over the cluster.
// VEC: dk, dv and cols multiples of 4, dk <= 128 X, rows and columns aligned: four channels or key rows a lane, and the
// block's columns of S are asked for before anything else (an earlier step wrote them: they need not wait for the
// projection before this kernel).
template <typename T, bool VEC, int X>
__global__ void __launch_bounds__(kStepThreads)
delta_head_step_kernel(const T* __restrict__ proj, T* __restrict__ ring, float* __restrict__ state,
                       const float* __restrict__ w, float eps, T* __restrict__ y, int ldy, int cols, const HeadDelta a) {
  extern __shared__ __align__(16) float sm[];   // q [dkp], k [dkp], v [cols], o [cols]
  __shared__ float red[3 * kStepWarps + 32];
  __shared__ float slots[kMaxClusterBlocks];
  __shared__ float gates[2];
  cluster_arrive();
  const int h = blockIdx.y, e = blockIdx.z;
  const int dk = a.dk, dv = a.dv, dkp = (dk + 3) & ~3, C = 2 * a.G * dk + a.H * dv;
  const int per_kv = a.H / a.G, kvh = h / per_kv;
  float *q_s = sm, *k_s = q_s + dkp, *v_s = k_s + dkp, *o_s = v_s + ((cols + 3) & ~3);
  const int c_lo = blockIdx.x * cols, n_cols = max(0, min(dv, c_lo + cols) - c_lo);
  const int slot = a.state_slot[e];   // (written by a copy before the step's first kernel)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const bool live = slot >= 0 && slot < a.n_slots;
  float* S = state + (((size_t)(live ? slot : 0) * a.H + h) * dv + c_lo) * dk;

  int lpc = 1;   // lanes a column
  while (lpc < 32 && lpc * 4 < dk) lpc *= 2;
  const int cpw = 32 / lpc, li = lane & (lpc - 1), my_col = warp * cpw + lane / lpc, stride = kStepWarps * cpw;
  float4 s[kStepCols][X];
  auto fetch = [&](int base) {
#pragma unroll
    for (int u = 0; u < kStepCols; ++u) {
      const int c = base + my_col + u * stride;
#pragma unroll
      for (int x = 0; x < X; ++x) {
        const int r = 4 * li + 128 * x;
        if (live && c < n_cols && r < dk) s[u][x] = *reinterpret_cast<const float4*>(S + (size_t)c * dk + r);
      }
    }
  };
  if (VEC) fetch(0);
  ccb::pdl_begin();
  if (live) {
    const int t = a.cu_q[e], pos = a.positions[t];
    const T* row = proj + (size_t)t * a.ld;
    const bool owns_kv = blockIdx.x == 0 && h % per_kv == 0;   // this block writes its group's q and k channels to the ring
    float ssq = 0.f, ssk = 0.f;
    constexpr int W = VEC ? 4 : 1;
    for (int i = W * threadIdx.x; i < 2 * dk + n_cols; i += W * kStepThreads) {
      const bool is_q = i < dk, is_v = i >= 2 * dk;
      const int l = is_v ? i - 2 * dk : (is_q ? i : i - dk);
      const int hd = is_v ? h * dv + c_lo : kvh * dk;
      const int c = (is_v ? 2 * a.G * dk : (is_q ? 0 : a.G * dk)) + hd + l;
      const int col = (is_v ? a.ov : (is_q ? a.oq : a.ok)) + hd + l;
      if constexpr (VEC) {
        using R4 = Row4<T>;
        const typename R4::Raw now = R4::load(row + col);
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        // four taps at a time, their loads in flight together; tap j multiplies the input taps - 1 - j tokens back
        for (int j0 = 0; j0 < a.taps; j0 += 4) {
          typename R4::Raw x[4];
          float4 cw[4];
#pragma unroll
          for (int jj = 0; jj < 4; ++jj) {
            const int j = j0 + jj, p = pos - (a.taps - 1 - j);
            const bool on = j < a.taps && p >= 0;
            x[jj] = on ? (p == pos ? now : R4::load(ring + ring_at<T>(slot, p, a.taps, C) + c)) : R4::zero();
            cw[jj] = on ? *reinterpret_cast<const float4*>(a.conv_w + (size_t)j * C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int jj = 0; jj < 4; ++jj) fma4(acc, cw[jj], R4::value(x[jj]));
        }
        if (a.taps > 1 && (is_v || owns_kv)) R4::store(ring + ring_at<T>(slot, pos, a.taps, C) + c, now);
        acc = silu4(acc);
        *reinterpret_cast<float4*>((is_v ? v_s : (is_q ? q_s : k_s)) + l) = acc;
        if (is_q) ssq += dot4(acc, acc);
        else if (!is_v) ssk += dot4(acc, acc);
      } else {
        const T now = row[col];
        float acc = 0.f;
        for (int j = 0; j < a.taps; ++j) {
          const int p = pos - (a.taps - 1 - j);
          if (p < 0) continue;
          acc = fmaf(a.conv_w[(size_t)j * C + c], p == pos ? to_f32(now) : to_f32(ring[ring_at<T>(slot, p, a.taps, C) + c]), acc);
        }
        if (a.taps > 1 && (is_v || owns_kv)) ring[ring_at<T>(slot, pos, a.taps, C) + c] = now;
        acc = silu_f(acc);
        (is_v ? v_s : (is_q ? q_s : k_s))[l] = acc;
        if (is_q) ssq += acc * acc;
        else if (!is_v) ssk += acc * acc;
      }
    }
    if (threadIdx.x == kStepThreads - 1) {
      gates[0] = expf(-expf(a.A_log[h]) * softplus_f(to_f32(row[a.oa + h]) + a.dt_bias[h]));
      gates[1] = sigmoid_f(to_f32(row[a.ob + h]));
    }
    ssq = warp_sum(ssq);
    ssk = warp_sum(ssk);
    if (lane == 0) red[warp] = ssq, red[kStepWarps + warp] = ssk;
    __syncthreads();
    float tq = 0.f, tk = 0.f;
#pragma unroll
    for (int i = 0; i < kStepWarps; ++i) tq += red[i], tk += red[kStepWarps + i];
    const float fq = a.q_mult / sqrtf(tq + a.unit_eps), fk = 1.0f / sqrtf(tk + a.unit_eps);
    float kq = 0.f;
    for (int i = threadIdx.x; i < dk; i += kStepThreads) {
      const float q = q_s[i] * fq, k = k_s[i] * fk;
      q_s[i] = q;
      k_s[i] = k;
      kq = fmaf(k, q, kq);
    }
    kq = warp_sum(kq);
    if (lane == 0) red[2 * kStepWarps + warp] = kq;
    __syncthreads();
    kq = 0.f;
#pragma unroll
    for (int i = 0; i < kStepWarps; ++i) kq += red[2 * kStepWarps + i];
    const float g = gates[0], beta = gates[1];
    // a column of S (one value channel): S^T k and S^T q of the decayed state, then the write; the read-out after the
    // write is (g S)^T q + u (k . q)
    if constexpr (VEC) {
      for (int base = 0; base < n_cols; base += kStepCols * stride) {
        if (base > 0) fetch(base);
#pragma unroll
        for (int u = 0; u < kStepCols; ++u) {
          const int c = base + my_col + u * stride;
          float dotk = 0.f, dotq = 0.f;
#pragma unroll
          for (int x = 0; x < X; ++x) {
            const int r = 4 * li + 128 * x;
            if (c < n_cols && r < dk) {
              float4& z = s[u][x];
              z.x *= g; z.y *= g; z.z *= g; z.w *= g;
              dotk += dot4(z, *reinterpret_cast<const float4*>(k_s + r));
              dotq += dot4(z, *reinterpret_cast<const float4*>(q_s + r));
            }
          }
          for (int o = lpc >> 1; o > 0; o >>= 1) {
            dotk += __shfl_xor_sync(0xffffffffu, dotk, o);
            dotq += __shfl_xor_sync(0xffffffffu, dotq, o);
          }
          if (c < n_cols) {
            const float put = beta * (v_s[c] - dotk);
#pragma unroll
            for (int x = 0; x < X; ++x) {
              const int r = 4 * li + 128 * x;
              if (r < dk) {
                fma4(s[u][x], *reinterpret_cast<const float4*>(k_s + r), make_float4(put, put, put, put));
                *reinterpret_cast<float4*>(S + (size_t)c * dk + r) = s[u][x];
              }
            }
            if (li == 0) o_s[c] = fmaf(put, kq, dotq);
          }
        }
      }
    } else {
      for (int c = warp; c < n_cols; c += kStepWarps) {
        float dotk = 0.f, dotq = 0.f;
        for (int r = lane; r < dk; r += 32) {
          const float z = g * S[(size_t)c * dk + r];
          dotk = fmaf(z, k_s[r], dotk);
          dotq = fmaf(z, q_s[r], dotq);
        }
        dotk = warp_sum(dotk);
        dotq = warp_sum(dotq);
        const float put = beta * (v_s[c] - dotk);
        for (int r = lane; r < dk; r += 32) S[(size_t)c * dk + r] = fmaf(k_s[r], put, g * S[(size_t)c * dk + r]);
        if (lane == 0) o_s[c] = fmaf(put, kq, dotq);
      }
    }
    __syncthreads();
  }
  float ss = 0.f;
  if (live)
    for (int i = threadIdx.x; i < n_cols; i += kStepThreads) ss += o_s[i] * o_s[i];
  ss = cluster_sum(block_sum<kStepThreads>(ss, red), slots);   // (every block of the cluster, whether its request is live or not)
  if (!live) return;
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  const int t = a.cu_q[e];
  for (int i = threadIdx.x; i < n_cols; i += kStepThreads) {
    const int c = h * dv + c_lo + i;
    y[(size_t)t * ldy + c] = from_f32<T>(o_s[i] * inv * w[c_lo + i] * silu_f(to_f32(proj[(size_t)t * a.ld + a.og + c])));
  }
}

// The convolution's activation in portions: the accurate form in 32 bits; where inputs and results of the projection are
// bfloat16 anyway, the fast exponential and division (a few units of the last place of a float).
template <typename T> __device__ __forceinline__ float4 silu4_of(const float4 x) { return silu4(x); }
template <> __device__ __forceinline__ float4 silu4_of<__nv_bfloat16>(const float4 x) {
  return make_float4(__fdividef(x.x, 1.f + __expf(-x.x)), __fdividef(x.y, 1.f + __expf(-x.y)),
                     __fdividef(x.z, 1.f + __expf(-x.z)), __fdividef(x.w, 1.f + __expf(-x.w)));
}

constexpr int kPrepWarps = 4;

// Rows row0 .. row_end - 1 of the step, one a block.  The form that takes every size.
template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32)
delta_head_prepare_kernel(const T* __restrict__ proj, const T* __restrict__ ring, float* __restrict__ qn,
                          float* __restrict__ kn, float* __restrict__ vv, float* __restrict__ gg, float* __restrict__ bb,
                          int row0, const HeadDelta a) {
  ccb::pdl_begin();
  const int t = row0 + blockIdx.x;
  const int e = a.entry_of_token[t];
  if (e < 0) return;
  const int slot = a.state_slot[e];
  if (slot < 0 || slot >= a.n_slots) return;
  const int lt = t - a.cu_q[e], pos = a.positions[t];
  const int G = a.G, H = a.H, dk = a.dk, dv = a.dv, C = 2 * G * dk + H * dv;
  const int lane = threadIdx.x & 31;
  const int u = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
  if (u >= 2 * G + H) return;
  auto conv = [&](int c, int col) {
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
      const int back = a.taps - 1 - j, p = pos - back;
      if (p < 0) continue;
      const T x = lt >= back ? proj[(size_t)(t - back) * a.ld + col] : ring[ring_at<T>(slot, p, a.taps, C) + c];
      acc = fmaf(a.conv_w[(size_t)j * C + c], to_f32(x), acc);
    }
    return silu_f(acc);
  };
  if (u < 2 * G) {
    const bool is_q = u < G;
    const int head = is_q ? u : u - G;
    const int c0 = (is_q ? 0 : G * dk) + head * dk, col0 = (is_q ? a.oq : a.ok) + head * dk;
    float* dst = (is_q ? qn : kn) + ((size_t)t * G + head) * dk;
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) {
      const float v = conv(c0 + i, col0 + i);
      dst[i] = v;
      ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    const float f = (is_q ? a.q_mult : 1.0f) / sqrtf(ss + a.unit_eps);
    for (int i = lane; i < dk; i += 32) dst[i] *= f;   // (each lane rescales what it wrote itself)
  } else {
    const int head = u - 2 * G;
    for (int i = lane; i < dv; i += 32)
      vv[((size_t)t * H + head) * dv + i] = conv(2 * G * dk + head * dv + i, a.ov + head * dv + i);
    if (lane == 0) {
      const T* row = proj + (size_t)t * a.ld;
      gg[(size_t)t * H + head] = expf(-expf(a.A_log[head]) * softplus_f(to_f32(row[a.oa + head]) + a.dt_bias[head]));
      bb[(size_t)t * H + head] = sigmoid_f(to_f32(row[a.ob + head]));
    }
  }
}

// The same with four channels a lane and kRun neighbouring rows a warp: the taps' weights are loaded once for all of them,
// a row once for all the taps it meets, and all are in flight together.  dk, dv multiples of 4, dk <= 128 X, TAPS taps.
constexpr int kRun = 4;

template <typename T, int TAPS, int X>
__global__ void __launch_bounds__(kPrepWarps * 32, sizeof(T) == 2 && X == 1 ? 7 : 3)   // (latency: warps count)
delta_head_prepare_run_kernel(const T* __restrict__ proj, const T* __restrict__ ring, float* __restrict__ qn,
                              float* __restrict__ kn, float* __restrict__ vv, float* __restrict__ gg,
                              float* __restrict__ bb, int row0, int row_end, const HeadDelta a) {
  using R4 = Row4<T>;
  ccb::pdl_begin();
  const int t0 = row0 + blockIdx.x * kRun;
  const int G = a.G, H = a.H, dk = a.dk, dv = a.dv, C = 2 * G * dk + H * dv;
  const int lane = threadIdx.x & 31;
  const int u = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
  if (u >= 2 * G + H) return;
  const bool is_q = u < G, is_v = u >= 2 * G;
  const int head = is_v ? u - 2 * G : (is_q ? u : u - G), width = is_v ? dv : dk;
  const int c0 = (is_v ? 2 * G * dk : (is_q ? 0 : G * dk)) + head * width;
  const int col0 = (is_v ? a.ov : (is_q ? a.oq : a.ok)) + head * width;
  float* dst = (is_v ? vv : (is_q ? qn : kn)) + head * width;
  const int ldd = (is_v ? H : G) * width;
  // what the rows' requests are: a lane a row, handed round below
  int m_slot = -1, m_lt = 0, m_pos = 0;
  if (lane < kRun && t0 + lane < row_end) {
    const int e = a.entry_of_token[t0 + lane];
    m_pos = a.positions[t0 + lane];
    if (e >= 0) {
      m_slot = a.state_slot[e];
      m_lt = t0 + lane - a.cu_q[e];
      if (m_slot >= a.n_slots) m_slot = -1;
    }
  }
  for (int i0 = 0; i0 < width; i0 += 128 * X) {   // (one round for q and k)
    typename R4::Raw raw[X][kRun];
    float4 cw[X][TAPS], win[X][TAPS];   // win: the row's own input last, those before it
#pragma unroll
    for (int x = 0; x < X; ++x) {
      const int i = i0 + 4 * lane + 128 * x;
#pragma unroll
      for (int r = 0; r < kRun; ++r)
        raw[x][r] = i < width && t0 + r < row_end ? R4::load(proj + (size_t)(t0 + r) * a.ld + col0 + i) : R4::zero();
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        cw[x][j] = i < width ? *reinterpret_cast<const float4*>(a.conv_w + (size_t)j * C + c0 + i)
                             : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int r = 0; r < kRun; ++r) {
      const int t = t0 + r;
      const int slot = __shfl_sync(0xffffffffu, m_slot, r), lt = __shfl_sync(0xffffffffu, m_lt, r);
      const int pos = __shfl_sync(0xffffffffu, m_pos, r);
      if (slot < 0) continue;   // no such row, or a row that pads the step (the same for every lane)
#pragma unroll
      for (int x = 0; x < X; ++x) {
        const int i = i0 + 4 * lane + 128 * x;
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) {
          if (r > 0 && lt > 0) {
            win[x][j] = win[x][j + 1];
            continue;
          }
          // the run's first row, or a request's: what lies before it, from the step, the ring, or nowhere
          const int back = TAPS - 1 - j;
          typename R4::Raw in = R4::zero();
          if (i < width && pos >= back)
            in = lt >= back ? R4::load(proj + (size_t)(t - back) * a.ld + col0 + i)
                            : R4::load(ring + ring_at<T>(slot, pos - back, TAPS, C) + c0 + i);
          win[x][j] = R4::value(in);
        }
        win[x][TAPS - 1] = R4::value(raw[x][r]);
      }
      float4 v[X];
      float ss = 0.f;
#pragma unroll
      for (int x = 0; x < X; ++x) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < TAPS; ++j) fma4(acc, cw[x][j], win[x][j]);
        v[x] = silu4_of<T>(acc);
        ss += dot4(v[x], v[x]);   // (zeros beyond the head's channels)
      }
      float f = 1.f;
      if (!is_v) f = (is_q ? a.q_mult : 1.0f) / sqrtf(warp_sum(ss) + a.unit_eps);
#pragma unroll
      for (int x = 0; x < X; ++x) {
        const int i = i0 + 4 * lane + 128 * x;
        if (i < width)
          *reinterpret_cast<float4*>(dst + (size_t)t * ldd + i) = make_float4(v[x].x * f, v[x].y * f, v[x].z * f, v[x].w * f);
      }
    }
  }
  if (is_v && lane < kRun && t0 + lane < row_end) {   // a lane a row
    const int t = t0 + lane;
    const T* row = proj + (size_t)t * a.ld;
    gg[(size_t)t * H + head] = expf(-expf(a.A_log[head]) * softplus_f(to_f32(row[a.oa + head]) + a.dt_bias[head]));
    bb[(size_t)t * H + head] = sigmoid_f(to_f32(row[a.ob + head]));
  }
}

// Entries entry0 ..: the rows of their last min(n, taps) tokens to the ring.
template <typename T>
__global__ void conv_ring_write_kernel(const T* __restrict__ proj, T* __restrict__ ring, int entry0, const HeadDelta a) {
  ccb::pdl_begin();
  const int e = entry0 + blockIdx.y;
  const int slot = a.state_slot[e];
  const int G = a.G, dk = a.dk, C = 2 * G * dk + a.H * a.dv;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (slot < 0 || slot >= a.n_slots || c >= C) return;
  const int col = c < G * dk ? a.oq + c : (c < 2 * G * dk ? a.ok + (c - G * dk) : a.ov + (c - 2 * G * dk));
  const int r0 = a.cu_q[e], n = a.cu_q[e + 1] - r0;
  for (int i = max(0, n - a.taps); i < n; ++i)
    ring[ring_at<T>(slot, a.positions[r0 + i], a.taps, C) + c] = proj[(size_t)(r0 + i) * a.ld + col];
}

bool sizes_ok(const HeadDelta& a) {
  return a.G > 0 && a.H > 0 && a.H % a.G == 0 && a.dk > 0 && a.dv > 0 && a.taps >= 1;
}

HeadDelta head_delta(int ld, const int* offsets, int G, int H, int dk, int dv, int taps, const float* conv_w,
                     const float* A_log, const float* dt_bias, const int* positions, const int* entry_of_token,
                     const int* cu_q, const int* state_slot, float q_mult, float unit_eps, int n_slots) {
  HeadDelta a;
  a.ld = ld; a.oq = offsets[0]; a.ok = offsets[1]; a.ov = offsets[2]; a.ob = offsets[3]; a.oa = offsets[4]; a.og = offsets[5];
  a.G = G; a.H = H; a.dk = dk; a.dv = dv; a.taps = taps; a.conv_w = conv_w; a.A_log = A_log; a.dt_bias = dt_bias;
  a.positions = positions; a.entry_of_token = entry_of_token; a.cu_q = cu_q; a.state_slot = state_slot;
  a.q_mult = q_mult; a.unit_eps = unit_eps; a.n_slots = n_slots;
  return a;
}

}  // namespace

// `offsets` (host memory, here and below): the first columns of q, k, v, b, a and the gate in the rows of proj.
// The first n_entries entries, which bring one token each: ring and state move on, y [T, >= H dv] gets their rows.
CCB_API int ccb_delta_head_step(const void* proj, int ld, const int* offsets, const float* conv_w, int taps, void* ring,
                                float* state, const float* A_log, const float* dt_bias, const float* w, float eps,
                                const int* positions, const int* cu_q, const int* state_slot, void* y, int ldy,
                                int n_entries, int G, int H, int dk, int dv, int n_slots, float q_mult, float unit_eps,
                                int dtype, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  const HeadDelta a = head_delta(ld, offsets, G, H, dk, dv, taps, conv_w, A_log, dt_bias, positions, nullptr, cu_q,
                                 state_slot, q_mult, unit_eps, n_slots);
  if (!sizes_ok(a) || n_entries > 65535 || ldy < H * dv) return CCB_REFUSE_SIZE;
  // about 32 value channels a block, at most eight blocks a head
  int n_blocks = (dv + 31) / 32;
  if (n_blocks > kMaxClusterBlocks) n_blocks = kMaxClusterBlocks;
  const int cols = ((dv + n_blocks - 1) / n_blocks + 3) & ~3;
  n_blocks = (dv + cols - 1) / cols;
  const size_t smem = (size_t)(2 * ((dk + 3) & ~3) + 2 * cols) * sizeof(float);
  if (smem > 44 * 1024) return CCB_REFUSE_SIZE;
  const int esz = dtype == CCB_F32 ? 4 : 2;
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && dk <= 256 && ld % 4 == 0 && a.oq % 4 == 0 && a.ok % 4 == 0 && a.ov % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring)) % (4 * esz) == 0 &&
                   ((reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(conv_w)) & 15) == 0;
#define CCB_STEP(TT, VV, XX)                                                                                          \
  ccb_launch_cluster(true, n_blocks, delta_head_step_kernel<TT, VV, XX>, dim3(n_blocks, H, n_entries),                \
                     dim3(kStepThreads), smem, stream, (const TT*)proj, (TT*)ring, state, w, eps, (TT*)y, ldy, cols, a)
#define CCB_STEP_X(TT)                                                                                                \
  do {                                                                                                                \
    if (!vec) CCB_STEP(TT, false, 1);                                                                                 \
    else if (dk <= 128) CCB_STEP(TT, true, 1);                                                                        \
    else CCB_STEP(TT, true, 2);                                                                                       \
  } while (0)
  if (dtype == CCB_F32) CCB_STEP_X(float);
  else if (dtype == CCB_BF16) CCB_STEP_X(__nv_bfloat16);
  else return CCB_REFUSE_DTYPE;
#undef CCB_STEP_X
#undef CCB_STEP
  return ccb_launch_status();
}

// Rows row0 .. row0 + rows - 1 of the step (those of its portions): qn, kn [T, G, dk], vv [T, H, dv], gg, bb [T, H].
CCB_API int ccb_delta_head_prepare(const void* proj, int ld, const int* offsets, const float* conv_w, int taps,
                                   const void* ring, const float* A_log, const float* dt_bias, const int* positions,
                                   const int* entry_of_token, const int* cu_q, const int* state_slot, float* qn,
                                   float* kn, float* vv, float* gg, float* bb, int row0, int rows, int G, int H, int dk,
                                   int dv, int n_slots, float q_mult, float unit_eps, int dtype, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const HeadDelta a = head_delta(ld, offsets, G, H, dk, dv, taps, conv_w, A_log, dt_bias, positions, entry_of_token,
                                 cu_q, state_slot, q_mult, unit_eps, n_slots);
  if (!sizes_ok(a) || row0 < 0) return CCB_REFUSE_SIZE;
  const dim3 grid(rows, (2 * G + H + kPrepWarps - 1) / kPrepWarps);
  const int esz = dtype == CCB_F32 ? 4 : 2;
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && dk <= 256 && ld % 4 == 0 && a.oq % 4 == 0 && a.ok % 4 == 0 && a.ov % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring)) % (4 * esz) == 0 &&
                   ((reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn) | reinterpret_cast<uintptr_t>(vv) |
                     reinterpret_cast<uintptr_t>(conv_w)) & 15) == 0;
#define CCB_RUN(TT, TAPS, XX)                                                                                         \
  ccb_launch(delta_head_prepare_run_kernel<TT, TAPS, XX>, run_grid, dim3(kPrepWarps * 32), 0, stream, (const TT*)proj, \
             (const TT*)ring, qn, kn, vv, gg, bb, row0, row0 + rows, a)
#define CCB_RUN_X(TT, TAPS)                                                                                           \
  do {                                                                                                                \
    if (dk <= 128) CCB_RUN(TT, TAPS, 1);                                                                              \
    else CCB_RUN(TT, TAPS, 2);                                                                                        \
  } while (0)
#define CCB_PREP(TT)                                                                                                  \
  do {                                                                                                                \
    if (!vec || taps > 4)                                                                                             \
      ccb_launch(delta_head_prepare_kernel<TT>, grid, dim3(kPrepWarps * 32), 0, stream, (const TT*)proj, (const TT*)ring, \
                 qn, kn, vv, gg, bb, row0, a);                                                                        \
    else if (taps == 1) CCB_RUN_X(TT, 1);                                                                             \
    else if (taps == 2) CCB_RUN_X(TT, 2);                                                                             \
    else if (taps == 3) CCB_RUN_X(TT, 3);                                                                             \
    else CCB_RUN_X(TT, 4);                                                                                            \
  } while (0)
  const dim3 run_grid((rows + kRun - 1) / kRun, grid.y);
  if (dtype == CCB_F32) CCB_PREP(float);
  else if (dtype == CCB_BF16) CCB_PREP(__nv_bfloat16);
  else return CCB_REFUSE_DTYPE;
#undef CCB_RUN
#undef CCB_RUN_X
#undef CCB_PREP
  return ccb_launch_status();
}

// Entries entry0 .. entry0 + n_entries - 1, after ccb_delta_head_prepare.
CCB_API int ccb_conv_ring_write(const void* proj, int ld, const int* offsets, int taps, void* ring, const int* positions,
                                const int* cu_q, const int* state_slot, int entry0, int n_entries, int G, int H, int dk,
                                int dv, int n_slots, int dtype, cudaStream_t stream) {
  if (n_entries <= 0 || taps <= 1) return 0;
  const HeadDelta a = head_delta(ld, offsets, G, H, dk, dv, taps, nullptr, nullptr, nullptr, positions, nullptr, cu_q,
                                 state_slot, 1.f, 0.f, n_slots);
  if (!sizes_ok(a) || n_entries > 65535) return CCB_REFUSE_SIZE;
  const dim3 grid((2 * G * dk + H * dv + 255) / 256, n_entries);
  if (dtype == CCB_F32)
    ccb_launch(conv_ring_write_kernel<float>, grid, dim3(256), 0, stream, (const float*)proj, (float*)ring, entry0, a);
  else if (dtype == CCB_BF16)
    ccb_launch(conv_ring_write_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)proj,
               (__nv_bfloat16*)ring, entry0, a);
  else
    return CCB_REFUSE_DTYPE;
  return ccb_launch_status();
}
