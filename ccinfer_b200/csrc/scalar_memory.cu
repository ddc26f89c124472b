// Matrix memories whose decay is ONE number per head and token (retention with a fixed decay; the matrix memory of an
// extended LSTM with exponential gates): what comes before and after their recurrence
//
//   S <- a_t S + b_t k_t v_t^T;   o_t = S^T q_t            (the plain form of the kernel in delta_rule.cu)
//
//   memory_prepare   a block per token: float rows of q, k, v from a projection's rows; q and k optionally rotated (the
//                    first rot_dims coordinates of a head, pairs (i, i + rot_dims / 2), angle position * inv_freq[i]),
//                    then times a constant each; optionally a further value column of ones, whose memory is the
//                    running sum n of the keys: n . q is then one more column of o
//   memory_gates     a warp per (request, head): the gates of an exponentially gated memory from their
//                    pre-activations, i = cap tanh((zi + bi) / cap), f = log sigmoid(cap tanh((zf + bf) / cap)), and
//                    the running maximum m_t = max(f_t + m_(t-1), i_t) over the step's tokens (32 at a time: the maps
//                    m -> max(m + F, I) compose, so the lanes take a prefix scan of them).  Leaves, per token,
//                    a_t = exp(f_t + m_(t-1) - m_t), b_t = exp(i_t - m_t), exp(-m_t); m is state of the request
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

// z [T, ldz] float: H pre-activations of the input gate, then H of the forget gate.
__global__ void __launch_bounds__(128)
memory_gates_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ bi, const float* __restrict__ bf,
                    float cap, float* __restrict__ m_state, const int* __restrict__ cu_q,
                    const int* __restrict__ state_slot, float* __restrict__ decay, float* __restrict__ put,
                    float* __restrict__ floor_, int n_entries, int H, int max_slots) {
  ccb::pdl_begin();
  const int unit = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= n_entries * H) return;
  const int e = unit / H, h = unit - e * H;
  const int lane = threadIdx.x & 31;
  const int slot = state_slot[e];
  if (slot < 0 || slot >= max_slots) return;
  const int r0 = cu_q[e], n = cu_q[e + 1] - r0;
  if (n <= 0) return;
  float m = m_state[(size_t)slot * H + h];   // m_(t-1) before the 32 tokens at hand
  const float b_i = bi[h], b_f = bf[h];
  for (int t0 = 0; t0 < n; t0 += 32) {
    const int t = t0 + lane;
    float gi = -CUDART_INF_F, gf = 0.f;   // (lanes past the end leave m as it is)
    if (t < n) {
      const float* row = z + (size_t)(r0 + t) * ldz;
      gi = soft_cap(row[h] + b_i, cap);
      gf = log_sigmoid_of(soft_cap(row[H + h] + b_f, cap));
    }
    float F = gf, I = gi;   // the map of tokens t0 .. t: m -> max(m + F, I)
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pF = __shfl_up_sync(0xffffffffu, F, o), pI = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(pI + F, I);
        F += pF;
      }
    }
    const float m_t = fmaxf(m + F, I);
    float m_before = __shfl_up_sync(0xffffffffu, m_t, 1);
    if (lane == 0) m_before = m;
    if (t < n) {
      const size_t at = (size_t)(r0 + t) * H + h;
      decay[at] = expf(gf + m_before - m_t);
      put[at] = expf(gi - m_t);
      floor_[at] = expf(-m_t);
    }
    m = __shfl_sync(0xffffffffu, m_t, min(n - t0, 32) - 1);
  }
  if (lane == 0) m_state[(size_t)slot * H + h] = m;
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

CCB_API int ccb_memory_gates(const float* z, int ldz, const float* bi, const float* bf, float cap, float* m_state,
                             const int* cu_q, const int* state_slot, float* decay, float* put, float* floor_,
                             int n_entries, int H, int max_slots, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || ldz < 2 * H || !(cap > 0.f)) return CCB_REFUSE_SIZE;
  ccb_launch(memory_gates_kernel, dim3((n_entries * H + 3) / 4), dim3(128), 0, stream, z, ldz, bi, bf, cap, m_state, cu_q,
             state_slot, decay, put, floor_, n_entries, H, max_slots);
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
