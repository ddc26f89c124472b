// Matrix memories whose decay is ONE number per head and token (retention with a fixed decay; the matrix memory of an
// extended LSTM with exponential gates): what comes before and after their recurrence
//
//   S <- a_t S + b_t k_t v_t^T;   o_t = S^T q_t            (the plain form of the kernel in delta_rule.cu)
//
//   memory_prepare   a block per token: float rows of q, k, v from a projection's rows; q and k optionally rotated (the
//                    first rot_dims coordinates of a head, pairs (i, i + rot_dims / 2), angle position * inv_freq[i]),
//                    then times a constant each; optionally a further value column of ones, whose memory is the
//                    running sum n of the keys: n . q is then one more column of o
//   memory_rotate_split  the same q and k, rotated, as two bfloat16 each: the rounding and what it left
//   memory_gates     a block per (request, head): the gates of an exponentially gated memory from their
//                    pre-activations, i = cap tanh((zi + bi) / cap), f = log sigmoid(cap tanh((zf + bf) / cap)), and
//                    the running maximum m_t = max(f_t + m_(t-1), i_t) over the step's tokens (256 at a time: the maps
//                    m -> max(m + F, I) compose, so lanes and warps take a prefix scan of them).  Leaves, per token,
//                    a_t = exp(f_t + m_(t-1) - m_t), b_t = exp(i_t - m_t) (or their logarithms) and exp(-m_t); m is
//                    state of the request
//   memory_output    a warp per (token, head): o over its normaliser max(|n . q|, exp(-m)) + den_eps where there is
//                    one, over its root mean square, times a weight (one per channel of all heads, optional), times
//                    sigmoid(gate) or silu(gate)
//   memory_step      requests that bring ONE token: all of this and the recurrence in one kernel, a block per
//                    (request, head)
//
// Everything is float between the loads and the stores.
#include "common.cuh"
#include <math_constants.h>

using namespace ccb;

namespace {

__device__ __forceinline__ float sigmoid_of(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_of(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

constexpr int kPrepThreads = 256;

struct MemoryRows {
  int ld, oq, ok, ov;      // row stride of the projection, columns of q, k and v
  int H, dk, dv;
  int rot_dims;            // 0: no rotation
  int ones;                // 1: a value column of ones after the dv others
  float q_mult, k_mult;
};

template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
memory_prepare_kernel(const T* __restrict__ proj, const float* __restrict__ inv_freq, const int* __restrict__ positions,
                      float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ vv, const MemoryRows a) {
  ccb::pdl_begin();
  extern __shared__ float2 cs[];   // [rot_dims / 2]
  const int t = blockIdx.x;
  const int half = a.rot_dims >> 1;
  if (half > 0) {
    const float fpos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += kPrepThreads) {
      float sn, c;
      sincosf(fpos * inv_freq[i], &sn, &c);
      cs[i] = make_float2(c, sn);
    }
    __syncthreads();
  }
  const T* row = proj + (size_t)t * a.ld;
  const int qk = a.H * a.dk, vout = a.dv + a.ones;
  const int begin = blockIdx.y * kPrepThreads + threadIdx.x, step = gridDim.y * kPrepThreads;
  // an element of q and of k together: a rotated pair needs its partner only
  for (int c = begin; c < qk; c += step) {
    const int i = c % a.dk;
    float q = to_f32(row[a.oq + c]), k = to_f32(row[a.ok + c]);
    if (i < a.rot_dims) {
      const bool first = i < half;
      const int pc = first ? c + half : c - half;
      const float qp = to_f32(row[a.oq + pc]), kp = to_f32(row[a.ok + pc]);
      const float2 r = cs[first ? i : i - half];
      q = first ? q * r.x - qp * r.y : q * r.x + qp * r.y;
      k = first ? k * r.x - kp * r.y : k * r.x + kp * r.y;
    }
    qn[(size_t)t * qk + c] = q * a.q_mult;
    kn[(size_t)t * qk + c] = k * a.k_mult;
  }
  for (int c = begin; c < a.H * vout; c += step) {
    const int h = c / vout, i = c - h * vout;
    vv[(size_t)t * a.H * vout + c] = i < a.dv ? to_f32(row[a.ov + h * a.dv + i]) : 1.f;
  }
}

// What the rounding of a rotated q and k to bfloat16 leaves, beside the rounding itself: hi + lo is the float to about
// 2^-17 (operands of the chunked form of the recurrence, memory_chunks.cu).
__global__ void __launch_bounds__(kPrepThreads)
memory_rotate_split_kernel(const __nv_bfloat16* __restrict__ proj, const float* __restrict__ inv_freq,
                           const int* __restrict__ positions, __nv_bfloat16* __restrict__ q_hi,
                           __nv_bfloat16* __restrict__ q_lo, __nv_bfloat16* __restrict__ k_hi,
                           __nv_bfloat16* __restrict__ k_lo, const MemoryRows a) {
  ccb::pdl_begin();
  extern __shared__ float2 cs[];
  const int t = blockIdx.x;
  const int half = a.rot_dims >> 1;
  if (half > 0) {
    const float fpos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += kPrepThreads) {
      float sn, c;
      sincosf(fpos * inv_freq[i], &sn, &c);
      cs[i] = make_float2(c, sn);
    }
    __syncthreads();
  }
  const __nv_bfloat16* row = proj + (size_t)t * a.ld;
  const int qk = a.H * a.dk, rest = (a.dk - a.rot_dims) / 2;
  // two neighbouring pairs of one head at a time (rotated ones first, then the coordinates that pass in twos)
  const int per_head = a.dk / 4, total = 2 * a.H * per_head;   // (dk and rot_dims are multiples of 4)
  for (int c = threadIdx.x; c < total; c += kPrepThreads) {
    const bool is_k = c >= a.H * per_head;
    const int u = is_k ? c - a.H * per_head : c;
    const int h = u / per_head, i = 2 * (u - h * per_head);
    const bool turns = i < half;
    const int i0 = turns ? i : a.rot_dims + (i - half), i1 = turns ? i + half : a.rot_dims + (i - half) + rest;
    const __nv_bfloat16* src = row + (is_k ? a.ok : a.oq) + h * a.dk;
    float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + i0));
    float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + i1));
    if (turns) {
      const float2 r0 = cs[i], r1 = cs[i + 1];
      const float2 x2 = make_float2(x.x * r0.x - y.x * r0.y, x.y * r1.x - y.y * r1.y);
      y = make_float2(y.x * r0.x + x.x * r0.y, y.y * r1.x + x.y * r1.y);
      x = x2;
    }
    const float mult = is_k ? a.k_mult : a.q_mult;
    const size_t at = (size_t)t * qk + h * a.dk;
#pragma unroll
    for (int s = 0; s < 2; ++s) {
      const float fx = (s ? y.x : x.x) * mult, fy = (s ? y.y : x.y) * mult;
      const __nv_bfloat162 hi = __floats2bfloat162_rn(fx, fy);
      const float2 f = __bfloat1622float2(hi);
      *reinterpret_cast<__nv_bfloat162*>((is_k ? k_hi : q_hi) + at + (s ? i1 : i0)) = hi;
      *reinterpret_cast<__nv_bfloat162*>((is_k ? k_lo : q_lo) + at + (s ? i1 : i0)) = __floats2bfloat162_rn(fx - f.x, fy - f.y);
    }
  }
}

constexpr int kGateWarps = 8;

// z [T, ldz] float: H pre-activations of the input gate, then H of the forget gate.  A block per (request, head), 32
// tokens a warp: the lanes' scan, the warps' whole maps through shared memory.
__global__ void __launch_bounds__(kGateWarps * 32)
memory_gates_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ bi, const float* __restrict__ bf,
                    float cap, float* __restrict__ m_state, const int* __restrict__ cu_q,
                    const int* __restrict__ state_slot, float* __restrict__ decay, float* __restrict__ put,
                    float* __restrict__ floor_, int entry0, int H, int max_slots, int logs) {
  ccb::pdl_begin();
  __shared__ float2 maps[2][kGateWarps];
  const int e = entry0 + blockIdx.y, h = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int slot = state_slot[e];
  if (slot < 0 || slot >= max_slots) return;
  const int r0 = cu_q[e], n = cu_q[e + 1] - r0;
  if (n <= 0) return;
  float m = m_state[(size_t)slot * H + h];   // m_(t-1) before the tokens at hand
  const float b_i = bi[h], b_f = bf[h];
  float zi = 0.f, zf = 0.f;
  auto fetch = [&](int t) {
    if (t < n) {
      const float* row = z + (size_t)(r0 + t) * ldz;
      zi = row[h];
      zf = row[H + h];
    }
  };
  fetch(threadIdx.x);
  int turn = 0;
  for (int t0 = 0; t0 < n; t0 += kGateWarps * 32, turn ^= 1) {
    const int t = t0 + threadIdx.x;
    float gi = -CUDART_INF_F, gf = 0.f;   // (tokens past the end leave m as it is)
    if (t < n) {
      gi = soft_cap(zi + b_i, cap);
      gf = log_sigmoid_of(soft_cap(zf + b_f, cap));
    }
    fetch(t + kGateWarps * 32);
    float F = gf, I = gi;   // the map of the warp's tokens up to t: m -> max(m + F, I)
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pF = __shfl_up_sync(0xffffffffu, F, o), pI = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(pI + F, I);
        F += pF;
      }
    }
    if (lane == 31) maps[turn][warp] = make_float2(F, I);
    __syncthreads();
    float m_end = m;
#pragma unroll
    for (int w = 0; w < kGateWarps; ++w) {
      if (w == warp) m = m_end;   // before this warp's tokens
      m_end = fmaxf(m_end + maps[turn][w].x, maps[turn][w].y);
    }
    const float m_t = fmaxf(m + F, I);
    float m_before = __shfl_up_sync(0xffffffffu, m_t, 1);
    if (lane == 0) m_before = m;
    if (t < n) {
      const size_t at = (size_t)(r0 + t) * H + h;
      const float la = gf + m_before - m_t, lb = gi - m_t;
      decay[at] = logs ? la : expf(la);
      put[at] = logs ? lb : expf(lb);
      floor_[at] = expf(-m_t);
    }
    m = m_end;
  }
  if (threadIdx.x == 0) m_state[(size_t)slot * H + h] = m;
}

template <typename T>
__global__ void __launch_bounds__(256)
memory_output_kernel(T* __restrict__ y, const float* __restrict__ o, const float* __restrict__ floor_, float den_eps,
                     const T* __restrict__ gate, int ldg, int silu_gate, const float* __restrict__ w, int rows, int H,
                     int dv, float eps) {
  ccb::pdl_begin();
  const int unit = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= rows * H) return;
  const int lane = threadIdx.x & 31;
  const int t = unit / H, h = unit - t * H;
  const int ldo = dv + (floor_ ? 1 : 0);
  const float* src = o + (size_t)unit * ldo;
  float over = 1.f;
  if (floor_) over = 1.0f / (fmaxf(fabsf(src[dv]), floor_[unit]) + den_eps);
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) {
    const float x = src[i] * over;
    ss += x * x;
  }
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  const T* gr = gate + (size_t)t * ldg + (size_t)h * dv;
  T* dst = y + (size_t)unit * dv;
  for (int i = lane; i < dv; i += 32) {
    const float g = to_f32(gr[i]);
    float x = src[i] * over * inv;
    if (w) x *= w[h * dv + i];
    dst[i] = from_f32<T>(x * (silu_gate ? g * sigmoid_of(g) : sigmoid_of(g)));
  }
}

constexpr int kStepThreads = 512;

struct StepArgs {
  MemoryRows rows;
  int og;                    // column of the output gate
  const float* z;            // gate pre-activations (input gates at zi, forget gates at zf of a row), or null
  int ldz, zi, zf;
  const float *bi, *bf;
  float cap;
  float* m_state;            // [slots, H]
  const float* decay;        // without z: the constant decay of each head
  float* state;              // [slots, H, dv + ones, dk]
  const float* inv_freq;
  const int *positions, *cu_q, *state_slot;
  const float* w;            // [H dv] or null
  float eps, den_eps;
  int silu_gate, max_slots, ldy;
};

// VEC: dk a multiple of 4, the state's rows read 16 bytes a lane by the fewest lanes (a power of two) that hold one.
template <typename TI, typename TO, bool VEC>
__global__ void __launch_bounds__(kStepThreads)
memory_step_kernel(const TI* __restrict__ proj, TO* __restrict__ y, const StepArgs a) {
  extern __shared__ float sm[];   // q [dk], k [dk] (padded to 4), v and o [dvo] each
  __shared__ float red[32];
  __shared__ float gates[3];      // a_t, b_t, exp(-m)
  const MemoryRows& R = a.rows;
  const int h = blockIdx.x, e = blockIdx.y;
  const int dk = R.dk, dv = R.dv, dvo = dv + R.ones, dkp = (dk + 3) & ~3;
  float *q_s = sm, *k_s = q_s + dkp, *v_s = k_s + dkp, *o_s = v_s + dvo;
  const int slot = a.state_slot[e];
  const bool live = slot >= 0 && slot < a.max_slots;
  float* S = a.state + ((size_t)(live ? slot : 0) * R.H + h) * dvo * dk;
  // the memory was written by an earlier step: it may come into L2 while the projection before this kernel still runs
  if (live)
    for (int i = threadIdx.x * 32; i < dvo * dk; i += kStepThreads * 32)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(S + i));
  ccb::pdl_begin();
  if (!live) return;
  const int t = a.cu_q[e];
  const TI* row = proj + (size_t)t * R.ld;
  const int half = R.rot_dims >> 1;
  for (int i = threadIdx.x; i < 2 * dk; i += kStepThreads) {
    const bool is_k = i >= dk;
    const int c = is_k ? i - dk : i;
    const TI* src = row + (is_k ? R.ok : R.oq) + h * dk;
    float x = to_f32(src[c]);
    if (c < R.rot_dims) {
      const bool first = c < half;
      const int p = first ? c : c - half;
      float sn, cn;
      sincosf((float)a.positions[t] * a.inv_freq[p], &sn, &cn);
      const float other = to_f32(src[first ? c + half : c - half]);
      x = first ? x * cn - other * sn : x * cn + other * sn;
    }
    (is_k ? k_s : q_s)[c] = x * (is_k ? R.k_mult : R.q_mult);
  }
  for (int i = threadIdx.x; i < dvo; i += kStepThreads) v_s[i] = i < dv ? to_f32(row[R.ov + h * dv + i]) : 1.f;
  if (threadIdx.x == kStepThreads - 1) {
    if (a.z != nullptr) {
      const float* zr = a.z + (size_t)t * a.ldz;
      const float gi = soft_cap(zr[a.zi + h] + a.bi[h], a.cap);
      const float gf = log_sigmoid_of(soft_cap(zr[a.zf + h] + a.bf[h], a.cap));
      float* ms = a.m_state + (size_t)slot * R.H + h;
      const float m0 = *ms, m = fmaxf(gf + m0, gi);
      *ms = m;
      gates[0] = expf(gf + m0 - m);
      gates[1] = expf(gi - m);
      gates[2] = expf(-m);
    } else {
      gates[0] = a.decay[h];
      gates[1] = 1.f;
      gates[2] = 0.f;
    }
  }
  __syncthreads();
  const float ga = gates[0], gb = gates[1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (VEC) {
    int lpc = 1;                       // lanes a column
    while (lpc < 32 && lpc * 4 < dk) lpc *= 2;
    const int cpw = 32 / lpc, li = lane & (lpc - 1);
    const int stride = (kStepThreads / 32) * cpw;
    constexpr int U = 4;
    for (int c0 = warp * cpw + lane / lpc; c0 - lane / lpc < dvo; c0 += stride * U) {   // (whole warps go on together)
      float4 s[U][2];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * stride;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 4 * li + 128 * x;
          if (c < dvo && r < dk) s[u][x] = *reinterpret_cast<const float4*>(S + (size_t)c * dk + r);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * stride;
        const float v = c < dvo ? gb * v_s[c] : 0.f;
        float dot = 0.f;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 4 * li + 128 * x;
          if (c < dvo && r < dk) {
            const float4 k = *reinterpret_cast<const float4*>(k_s + r), q = *reinterpret_cast<const float4*>(q_s + r);
            float4 w = s[u][x];
            w.x = fmaf(k.x, v, ga * w.x); w.y = fmaf(k.y, v, ga * w.y);
            w.z = fmaf(k.z, v, ga * w.z); w.w = fmaf(k.w, v, ga * w.w);
            *reinterpret_cast<float4*>(S + (size_t)c * dk + r) = w;
            dot += (w.x * q.x + w.y * q.y) + (w.z * q.z + w.w * q.w);
          }
        }
        for (int o = lpc >> 1; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
        if (li == 0 && c < dvo) o_s[c] = dot;
      }
    }
  } else {
    for (int c = warp; c < dvo; c += kStepThreads / 32) {
      const float v = gb * v_s[c];
      float dot = 0.f;
      for (int r = lane; r < dk; r += 32) {
        const float w = fmaf(k_s[r], v, ga * S[(size_t)c * dk + r]);
        S[(size_t)c * dk + r] = w;
        dot += w * q_s[r];
      }
      dot = warp_sum(dot);
      if (lane == 0) o_s[c] = dot;
    }
  }
  __syncthreads();
  const float over = a.z != nullptr && R.ones ? 1.0f / (fmaxf(fabsf(o_s[dv]), gates[2]) + a.den_eps) : 1.f;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dv; i += kStepThreads) {
    const float x = o_s[i] * over;
    ss += x * x;
  }
  ss = block_sum<kStepThreads>(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)dv + a.eps);
  for (int i = threadIdx.x; i < dv; i += kStepThreads) {
    const float g = to_f32(row[a.og + h * dv + i]);
    float x = o_s[i] * over * inv;
    if (a.w) x *= a.w[h * dv + i];
    y[(size_t)t * a.ldy + h * dv + i] = from_f32<TO>(x * (a.silu_gate ? g * sigmoid_of(g) : sigmoid_of(g)));
  }
}

}  // namespace

CCB_API int ccb_memory_prepare(const void* proj, int ld, int oq, int ok, int ov, const float* inv_freq, int rot_dims,
                               const int* positions, float* qn, float* kn, float* vv, int rows, int H, int dk, int dv,
                               float q_mult, float k_mult, int ones, int dtype, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dk <= 0 || dv <= 0 || rot_dims < 0 || rot_dims > dk || (rot_dims & 1) || ones < 0 || ones > 1)
    return CCB_REFUSE_SIZE;
  if (rot_dims > 0 && (inv_freq == nullptr || positions == nullptr)) return CCB_REFUSE_ARG;
  const MemoryRows a{ld, oq, ok, ov, H, dk, dv, rot_dims, ones, q_mult, k_mult};
  // few rows: a row over several blocks, so that its loads are in flight together
  int parts = 1;
  const int widest = H * (dk > dv + ones ? dk : dv + ones);
  while (rows * parts < 148 && parts * kPrepThreads < widest) parts *= 2;
  const size_t smem = (size_t)(rot_dims / 2) * sizeof(float2);
  const dim3 grid(rows, parts);
  if (dtype == CCB_F32)
    ccb_launch(memory_prepare_kernel<float>, grid, dim3(kPrepThreads), smem, stream, (const float*)proj, inv_freq,
               positions, qn, kn, vv, a);
  else if (dtype == CCB_BF16)
    ccb_launch(memory_prepare_kernel<__nv_bfloat16>, grid, dim3(kPrepThreads), smem, stream, (const __nv_bfloat16*)proj,
               inv_freq, positions, qn, kn, vv, a);
  else
    return CCB_REFUSE_DTYPE;
  return ccb_launch_status();
}

// bfloat16 rows; dk and rot_dims multiples of 4.
CCB_API int ccb_memory_rotate_split(const void* proj, int ld, int oq, int ok, const float* inv_freq, int rot_dims,
                                    const int* positions, void* q_hi, void* q_lo, void* k_hi, void* k_lo, int rows, int H,
                                    int dk, float q_mult, float k_mult, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dk <= 0 || dk % 4 || rot_dims < 0 || rot_dims > dk || rot_dims % 4 || ld % 2 || oq % 2 || ok % 2)
    return CCB_REFUSE_SIZE;
  if ((rot_dims > 0 && (inv_freq == nullptr || positions == nullptr)) || (reinterpret_cast<uintptr_t>(proj) & 3))
    return CCB_REFUSE_ARG;
  const MemoryRows a{ld, oq, ok, 0, H, dk, 0, rot_dims, 0, q_mult, k_mult};
  ccb_launch(memory_rotate_split_kernel, dim3(rows), dim3(kPrepThreads), (size_t)(rot_dims / 2) * sizeof(float2), stream,
             (const __nv_bfloat16*)proj, inv_freq, positions, (__nv_bfloat16*)q_hi, (__nv_bfloat16*)q_lo,
             (__nv_bfloat16*)k_hi, (__nv_bfloat16*)k_lo, a);
  return ccb_launch_status();
}

// Entries entry0 .. entry0 + n_entries - 1.  logs: decay and put are left as their logarithms.
CCB_API int ccb_memory_gates(const float* z, int ldz, const float* bi, const float* bf, float cap, float* m_state,
                             const int* cu_q, const int* state_slot, float* decay, float* put, float* floor_, int entry0,
                             int n_entries, int H, int max_slots, int logs, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || ldz < 2 * H || !(cap > 0.f) || n_entries > 65535) return CCB_REFUSE_SIZE;
  ccb_launch(memory_gates_kernel, dim3(H, n_entries), dim3(kGateWarps * 32), 0, stream, z, ldz, bi, bf, cap, m_state, cu_q,
             state_slot, decay, put, floor_, entry0, H, max_slots, logs);
  return ccb_launch_status();
}

// The first n_entries entries, which bring one token each.  z null: the constant decays; y in out_dtype.
CCB_API int ccb_memory_step(const void* proj, int ld, int oq, int ok, int ov, int og, const float* z, int ldz, int zi, int zf,
                            const float* bi, const float* bf, float cap, float* m_state, const float* decay, float* state,
                            const float* inv_freq, int rot_dims, const int* positions, const int* cu_q,
                            const int* state_slot, const float* w, float eps, float den_eps, int silu_gate, void* y, int ldy,
                            int n_entries, int H, int dk, int dv, int ones, int max_slots, float q_mult, float k_mult,
                            int in_dtype, int out_dtype, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || dk <= 0 || dk > 256 || dv <= 0 || rot_dims < 0 || rot_dims > dk || (rot_dims & 1) || ones < 0 || ones > 1 ||
      n_entries > 65535 || ldy < H * dv)
    return CCB_REFUSE_SIZE;
  if ((rot_dims > 0 && (inv_freq == nullptr || positions == nullptr)) || (z == nullptr ? decay == nullptr : m_state == nullptr))
    return CCB_REFUSE_ARG;
  StepArgs a;
  a.rows = MemoryRows{ld, oq, ok, ov, H, dk, dv, rot_dims, ones, q_mult, k_mult};
  a.og = og;
  a.z = z; a.ldz = ldz; a.zi = zi; a.zf = zf; a.bi = bi; a.bf = bf; a.cap = cap; a.m_state = m_state; a.decay = decay;
  a.state = state; a.inv_freq = inv_freq; a.positions = positions; a.cu_q = cu_q; a.state_slot = state_slot; a.w = w;
  a.eps = eps; a.den_eps = den_eps; a.silu_gate = silu_gate; a.max_slots = max_slots; a.ldy = ldy;
  const size_t smem = (size_t)(2 * ((dk + 3) & ~3) + 2 * (dv + ones)) * sizeof(float);
  if (smem > 48 * 1024) return CCB_REFUSE_SIZE;
  const bool vec = dk % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define CCB_STEP(TI, TO, VV)                                                                                            \
  ccb_launch_ex(true, memory_step_kernel<TI, TO, VV>, dim3(H, n_entries), dim3(kStepThreads), smem, stream, (const TI*)proj, \
                (TO*)y, a)
  if (in_dtype == CCB_F32 && out_dtype == CCB_F32) {
    if (vec) CCB_STEP(float, float, true); else CCB_STEP(float, float, false);
  } else if (in_dtype == CCB_F32 && out_dtype == CCB_BF16) {
    if (vec) CCB_STEP(float, __nv_bfloat16, true); else CCB_STEP(float, __nv_bfloat16, false);
  } else if (in_dtype == CCB_BF16 && out_dtype == CCB_BF16) {
    if (vec) CCB_STEP(__nv_bfloat16, __nv_bfloat16, true); else CCB_STEP(__nv_bfloat16, __nv_bfloat16, false);
  } else {
    return CCB_REFUSE_DTYPE;
  }
#undef CCB_STEP
  return ccb_launch_status();
}

// o float [rows, H, dv] or, with floor_ (exp(-m) [rows, H]), [rows, H, dv + 1] whose last column is n . q.
CCB_API int ccb_memory_output(void* y, const float* o, const float* floor_, float den_eps, const void* gate, int ldg,
                              int silu_gate, const float* w, int rows, int H, int dv, float eps, int dtype,
                              cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dv <= 0) return CCB_REFUSE_SIZE;
  const int units = rows * H;
  const dim3 grid((units + 7) / 8);
  if (dtype == CCB_F32)
    ccb_launch(memory_output_kernel<float>, grid, dim3(256), 0, stream, (float*)y, o, floor_, den_eps, (const float*)gate,
               ldg, silu_gate, w, rows, H, dv, eps);
  else if (dtype == CCB_BF16)
    ccb_launch(memory_output_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (__nv_bfloat16*)y, o, floor_, den_eps,
               (const __nv_bfloat16*)gate, ldg, silu_gate, w, rows, H, dv, eps);
  else
    return CCB_REFUSE_DTYPE;
  return ccb_launch_status();
}
