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
//   delta_head_step     single tokens: everything above in one kernel, a block per (request, head)
//   delta_head_prepare  portions: a warp per (token, head of q / k / v) -> float rows of q, k, v and per head g and beta
//                       (the recurrence itself is delta_rule.cu's)
//   conv_ring_write     portions: their last rows into the ring, after delta_head_prepare has read it
#include "common.cuh"

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

constexpr int kStepThreads = 256;

// VEC: dk a multiple of 4 up to 256 (a column of S is read 16 bytes a lane).
template <typename T, bool VEC>
__global__ void __launch_bounds__(kStepThreads)
delta_head_step_kernel(const T* __restrict__ proj, T* __restrict__ ring, float* __restrict__ state,
                       const float* __restrict__ w, float eps, T* __restrict__ y, int ldy, const HeadDelta a) {
  extern __shared__ float sm[];   // q [dkp], k [dkp], v [dv], o [dv]
  __shared__ float red[96];
  __shared__ float gates[2];
  const int h = blockIdx.x, e = blockIdx.y;
  const int dk = a.dk, dv = a.dv, dkp = (dk + 3) & ~3, C = 2 * a.G * dk + a.H * dv;
  const int per_kv = a.H / a.G, kvh = h / per_kv;
  float *q_s = sm, *k_s = q_s + dkp, *v_s = k_s + dkp, *o_s = v_s + dv;
  const int slot = a.state_slot[e];
  const bool live = slot >= 0 && slot < a.n_slots;
  float* S = state + ((size_t)(live ? slot : 0) * a.H + h) * dv * dk;
  // the state was written by an earlier step: it may come into L2 while the projection before this kernel still runs
  if (live)
    for (int i = threadIdx.x * 32; i < dv * dk; i += kStepThreads * 32)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(S + i));
  ccb::pdl_begin();
  if (!live) return;
  const int t = a.cu_q[e], pos = a.positions[t];
  const T* row = proj + (size_t)t * a.ld;
  const bool owns_kv = h % per_kv == 0;   // this block's head writes the q and k channels of its group to the ring
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x; i < 2 * dk + dv; i += kStepThreads) {
    const bool is_q = i < dk, is_v = i >= 2 * dk;
    const int l = is_v ? i - 2 * dk : (is_q ? i : i - dk);
    const int c = is_v ? 2 * a.G * dk + h * dv + l : (is_q ? 0 : a.G * dk) + kvh * dk + l;
    const int col = is_v ? a.ov + h * dv + l : (is_q ? a.oq : a.ok) + kvh * dk + l;
    const T now = row[col];
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {   // tap j multiplies the input taps - 1 - j tokens back
      const int p = pos - (a.taps - 1 - j);
      if (p < 0) continue;
      const float x = p == pos ? to_f32(now) : to_f32(ring[ring_at<T>(slot, p, a.taps, C) + c]);
      acc = fmaf(a.conv_w[(size_t)j * C + c], x, acc);
    }
    if (a.taps > 1 && (is_v || owns_kv)) ring[ring_at<T>(slot, pos, a.taps, C) + c] = now;
    const float x = acc * sigmoid_f(acc);
    if (is_v) v_s[l] = x;
    else if (is_q) q_s[l] = x, ssq += x * x;
    else k_s[l] = x, ssk += x * x;
  }
  if (threadIdx.x == kStepThreads - 1) {
    gates[0] = expf(-expf(a.A_log[h]) * softplus_f(to_f32(row[a.oa + h]) + a.dt_bias[h]));
    gates[1] = sigmoid_f(to_f32(row[a.ob + h]));
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int kWarps = kStepThreads / 32;
  ssq = warp_sum(ssq);
  ssk = warp_sum(ssk);
  if (lane == 0) red[warp] = ssq, red[32 + warp] = ssk;
  __syncthreads();
  float tq = 0.f, tk = 0.f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) tq += red[i], tk += red[32 + i];
  const float fq = a.q_mult / sqrtf(tq + a.unit_eps), fk = 1.0f / sqrtf(tk + a.unit_eps);
  float kq = 0.f;
  for (int i = threadIdx.x; i < dk; i += kStepThreads) {
    const float q = q_s[i] * fq, k = k_s[i] * fk;
    q_s[i] = q;
    k_s[i] = k;
    kq = fmaf(k, q, kq);
  }
  kq = warp_sum(kq);
  if (lane == 0) red[64 + warp] = kq;
  __syncthreads();
  kq = 0.f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) kq += red[64 + i];
  const float g = gates[0], beta = gates[1];
  // a column of S (one value channel) at a time: S^T k and S^T q of the decayed state, then the write; the read-out after
  // the write is (g S)^T q + u (k . q)
  if (VEC) {
    int lpc = 1;                       // lanes a column
    while (lpc < 32 && lpc * 4 < dk) lpc *= 2;
    const int cpw = 32 / lpc, li = lane & (lpc - 1);
    const int stride = kWarps * cpw;
    constexpr int U = 4;
    for (int base = warp * cpw; base < dv; base += stride * U) {   // (whole warps go on together)
      float4 s[U][2];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = base + lane / lpc + u * stride;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 4 * li + 128 * x;
          if (c < dv && r < dk) s[u][x] = *reinterpret_cast<const float4*>(S + (size_t)c * dk + r);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = base + lane / lpc + u * stride;
        float dotk = 0.f, dotq = 0.f;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 4 * li + 128 * x;
          if (c < dv && r < dk) {
            const float4 k = *reinterpret_cast<const float4*>(k_s + r), q = *reinterpret_cast<const float4*>(q_s + r);
            float4& z = s[u][x];
            z.x *= g; z.y *= g; z.z *= g; z.w *= g;
            dotk += (z.x * k.x + z.y * k.y) + (z.z * k.z + z.w * k.w);
            dotq += (z.x * q.x + z.y * q.y) + (z.z * q.z + z.w * q.w);
          }
        }
        for (int o = lpc >> 1; o > 0; o >>= 1) {
          dotk += __shfl_xor_sync(0xffffffffu, dotk, o);
          dotq += __shfl_xor_sync(0xffffffffu, dotq, o);
        }
        if (c < dv) {
          const float put = beta * (v_s[c] - dotk);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int r = 4 * li + 128 * x;
            if (r < dk) {
              const float4 k = *reinterpret_cast<const float4*>(k_s + r);
              float4 z = s[u][x];
              z.x = fmaf(k.x, put, z.x); z.y = fmaf(k.y, put, z.y); z.z = fmaf(k.z, put, z.z); z.w = fmaf(k.w, put, z.w);
              *reinterpret_cast<float4*>(S + (size_t)c * dk + r) = z;
            }
          }
          if (li == 0) o_s[c] = fmaf(put, kq, dotq);
        }
      }
    }
  } else {
    for (int c = warp; c < dv; c += kWarps) {
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
  float ss = 0.f;
  for (int i = threadIdx.x; i < dv; i += kStepThreads) ss += o_s[i] * o_s[i];
  ss = block_sum<kStepThreads>(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  for (int i = threadIdx.x; i < dv; i += kStepThreads) {
    const float z = to_f32(row[a.og + h * dv + i]);
    y[(size_t)t * ldy + h * dv + i] = from_f32<T>(o_s[i] * inv * w[i] * (z * sigmoid_f(z)));
  }
}

constexpr int kPrepWarps = 4;

template <typename T> __device__ __forceinline__ void load4(const T* p, float* v);
template <> __device__ __forceinline__ void load4<float>(const float* p, float* v) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
template <> __device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float* v) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}

// Rows row0 .. of the step.  W: neighbouring channels a lane takes at once (4 where sizes and strides allow it).
template <typename T, int W>
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

  auto conv = [&](int c, int col, float* out) {
    float acc[W];
#pragma unroll
    for (int i = 0; i < W; ++i) acc[i] = 0.f;
    for (int j = 0; j < a.taps; ++j) {
      const int back = a.taps - 1 - j, p = pos - back;
      if (p < 0) continue;
      float x[W], cw[W];
      const T* src = lt >= back ? proj + (size_t)(t - back) * a.ld + col : ring + ring_at<T>(slot, p, a.taps, C) + c;
      if (W == 4) {
        load4<T>(src, x);
        load4<float>(a.conv_w + (size_t)j * C + c, cw);
      } else {
        x[0] = to_f32(src[0]);
        cw[0] = a.conv_w[(size_t)j * C + c];
      }
#pragma unroll
      for (int i = 0; i < W; ++i) acc[i] = fmaf(cw[i], x[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < W; ++i) out[i] = acc[i] * sigmoid_f(acc[i]);
  };
  auto put = [&](float* dst, const float* v) {
    if (W == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    else dst[0] = v[0];
  };

  if (u < 2 * G) {
    const bool is_q = u < G;
    const int head = is_q ? u : u - G;
    const int c0 = (is_q ? 0 : G * dk) + head * dk, col0 = (is_q ? a.oq : a.ok) + head * dk;
    float* dst = (is_q ? qn : kn) + ((size_t)t * G + head) * dk;
    float ss = 0.f;
    if (W == 4) {   // (key sizes up to 256: what a lane holds stays in registers)
      float v[2][W];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const int i = 4 * lane + 128 * m;
        if (i < dk) {
          conv(c0 + i, col0 + i, v[m]);
#pragma unroll
          for (int x = 0; x < W; ++x) ss = fmaf(v[m][x], v[m][x], ss);
        }
      }
      ss = warp_sum(ss);
      const float f = (is_q ? a.q_mult : 1.0f) / sqrtf(ss + a.unit_eps);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const int i = 4 * lane + 128 * m;
        if (i < dk) {
#pragma unroll
          for (int x = 0; x < W; ++x) v[m][x] *= f;
          put(dst + i, v[m]);
        }
      }
    } else {
      for (int i = lane; i < dk; i += 32) {
        float v[W];
        conv(c0 + i, col0 + i, v);
        dst[i] = v[0];
        ss = fmaf(v[0], v[0], ss);
      }
      ss = warp_sum(ss);
      const float f = (is_q ? a.q_mult : 1.0f) / sqrtf(ss + a.unit_eps);
      for (int i = lane; i < dk; i += 32) dst[i] *= f;   // (each lane rescales what it wrote itself)
    }
  } else {
    const int head = u - 2 * G;
    const int c0 = 2 * G * dk + head * dv;
    float* dst = vv + ((size_t)t * H + head) * dv;
    for (int i = W * lane; i < dv; i += 32 * W) {
      float v[W];
      conv(c0 + i, a.ov + head * dv + i, v);
      put(dst + i, v);
    }
    if (lane == 0) {
      const T* row = proj + (size_t)t * a.ld;
      gg[(size_t)t * H + head] = expf(-expf(a.A_log[head]) * softplus_f(to_f32(row[a.oa + head]) + a.dt_bias[head]));
      bb[(size_t)t * H + head] = sigmoid_f(to_f32(row[a.ob + head]));
    }
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
  const size_t smem = (size_t)(2 * ((dk + 3) & ~3) + 2 * dv) * sizeof(float);
  if (smem > 44 * 1024) return CCB_REFUSE_SIZE;
  const bool vec = dk % 4 == 0 && dk <= 256 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define CCB_STEP(TT, VV)                                                                                             \
  ccb_launch_ex(true, delta_head_step_kernel<TT, VV>, dim3(H, n_entries), dim3(kStepThreads), smem, stream,          \
                (const TT*)proj, (TT*)ring, state, w, eps, (TT*)y, ldy, a)
  if (dtype == CCB_F32) {
    if (vec) CCB_STEP(float, true); else CCB_STEP(float, false);
  } else if (dtype == CCB_BF16) {
    if (vec) CCB_STEP(__nv_bfloat16, true); else CCB_STEP(__nv_bfloat16, false);
  } else {
    return CCB_REFUSE_DTYPE;
  }
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
#define CCB_PREP(TT, WW)                                                                                             \
  ccb_launch(delta_head_prepare_kernel<TT, WW>, grid, dim3(kPrepWarps * 32), 0, stream, (const TT*)proj,             \
             (const TT*)ring, qn, kn, vv, gg, bb, row0, a)
  if (dtype == CCB_F32) {
    if (vec) CCB_PREP(float, 4); else CCB_PREP(float, 1);
  } else if (dtype == CCB_BF16) {
    if (vec) CCB_PREP(__nv_bfloat16, 4); else CCB_PREP(__nv_bfloat16, 1);
  } else {
    return CCB_REFUSE_DTYPE;
  }
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
