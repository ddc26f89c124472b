// Queries and keys of attention layers whose norm runs over the whole projection: from the rows of the q | k product
// to the queries and the cached keys and values in one kernel.
//
//   u = conv(row)                   a causal convolution over time per channel (optional; w tap-major [taps, C]):
//                                   u[t, c] = sum_j w[j, c] * row[t - taps + 1 + j, c]
//   v = u of the key channels       the values are the keys as they leave the convolution
//   q = u / rms(u of all q channels) * wq,   k = u / rms(u of all k channels) * wk
//   q, k rotated in pairs (j, j + hd / 2) of each head by position * inv_freq[j]
//   q -> q_out [T, nq, hd];   k, v -> their page
//
// The channels are C = (nq + nkv) * hd, q heads first.  The means over the projection are over nq * n_real and
// nkv * n_real channels (heads that are laid out in a larger size than their own carry zero rows, which add nothing).
// Rows of the request from before this step come from its state [slot, taps - 1, C], as in short_conv.cu; a request
// that brings ONE token has its state moved on here (conv_state_rows does it for the others, afterwards).
// Everything between the loads and the stores is float.
//
// A block per token.  A unit of work is 8 channels i .. i + 7 of a head's first half and their partners i + hd / 2:
// a thread holds its units in registers from the convolution over the norm to the rotation.
#include "common.cuh"

using namespace ccb;

namespace {

constexpr int kMaxTaps = 16;

__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 x = __bfloat1622float2(h[i]);
    f[2 * i] = x.x;
    f[2 * i + 1] = x.y;
  }
}
__device__ __forceinline__ void store8(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) {
  uint4 v;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = v;
}

struct QkRows {
  int row_stride, taps, nq, nkv, hd, n_real, page_size, num_slots, n_entries, max_slots;
  float eps;
};

template <typename T, int NU, int kThreads>
__global__ void __launch_bounds__(kThreads)
qk_rows_kernel(const T* __restrict__ in, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
               const float* __restrict__ conv_w, T* __restrict__ state, const float* __restrict__ q_w,
               const float* __restrict__ k_w, const float* __restrict__ inv_freq, const int* __restrict__ positions,
               const int* __restrict__ slot_map, const int* __restrict__ entry_of_token, const int* __restrict__ cu_q,
               const int* __restrict__ state_slot, const QkRows a, int* status) {
  ccb::pdl_begin();
  __shared__ float2 cs_table[128];
  __shared__ float red[64];
  const int t = blockIdx.x;
  const int half = a.hd >> 1;
  const int upu = half >> 3;                       // units per head
  const int units = (a.nq + a.nkv) * upu, q_units = a.nq * upu;
  const int C = (a.nq + a.nkv) * a.hd;
  const int e = entry_of_token[t];
  const bool live = e >= 0 && e < a.n_entries;
  if (inv_freq != nullptr) {
    const float fpos = live ? (float)positions[t] : 0.f;
    for (int i = threadIdx.x; i < half; i += kThreads) {
      float sn, cs;
      sincosf(fpos * inv_freq[i], &sn, &cs);
      cs_table[i] = make_float2(cs, sn);
    }
  }
  int r0 = t, n = 1, cslot = -1;
  if (live) {
    r0 = cu_q[e];
    n = cu_q[e + 1] - r0;
    if (state != nullptr) {
      cslot = state_slot[e];
      if (cslot >= a.max_slots) {
        if (threadIdx.x == 0) set_status(status, CCB_ST_BAD_SLOT);
        cslot = -1;
      }
    }
  }
  int kslot = live ? slot_map[t] : -1;
  if (kslot >= a.num_slots) {
    if (threadIdx.x == 0) set_status(status, CCB_ST_BAD_SLOT);
    kslot = -1;
  }
  const int keep = a.taps - 1, li = t - r0;
  T* st = (cslot >= 0 && keep > 0) ? state + (size_t)cslot * keep * C : nullptr;

  float x0[NU][8], x1[NU][8];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int m = 0; m < NU; ++m) {
    const int u = threadIdx.x + m * kThreads;
    if (u < units) {
      const int head = u / upu, i = (u - head * upu) * 8;
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        float* x = s == 0 ? x0[m] : x1[m];
        const int c = head * a.hd + i + s * half;
        const T* own = in + (size_t)t * a.row_stride + c;
        if (conv_w == nullptr || !live) {
          load8(own, x);
        } else {
#pragma unroll
          for (int k = 0; k < 8; ++k) x[k] = 0.f;
          for (int j = 0; j < a.taps; ++j) {
            const int mrow = li - keep + j;   // row of the request relative to the step's first one
            float uu[8], w[8];
            if (mrow >= 0) load8(in + (size_t)(r0 + mrow) * a.row_stride + c, uu);
            else if (st != nullptr) load8(st + (size_t)(keep + mrow) * C + c, uu);
            else continue;
            load8(conv_w + (size_t)j * C + c, w);
#pragma unroll
            for (int k = 0; k < 8; ++k) x[k] = fmaf(w[k], uu[k], x[k]);
          }
          if (n == 1 && st != nullptr) {   // the state moves on by this one row (nobody else touches these channels)
            for (int k = 0; k + 1 < keep; ++k) {
              float mv[8];
              load8(st + (size_t)(k + 1) * C + c, mv);
              store8(st + (size_t)k * C + c, mv);
            }
            float mv[8];
            load8(own, mv);
            store8(st + (size_t)(keep - 1) * C + c, mv);
          }
        }
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(x[k], x[k], ss);
        if (u < q_units) sq += ss; else sk += ss;
      }
    }
  }
  // both sums over the block (the barriers also publish the angles)
  {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) red[warp] = sq, red[32 + warp] = sk;
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) sq += red[w], sk += red[32 + w];
  }
  const float inv_q = q_w ? 1.0f / sqrtf(sq / (float)(a.nq * a.n_real) + a.eps) : 1.f;
  const float inv_k = k_w ? 1.0f / sqrtf(sk / (float)(a.nkv * a.n_real) + a.eps) : 1.f;
  const int page = kslot >= 0 ? kslot / a.page_size : 0, off = kslot >= 0 ? kslot - page * a.page_size : 0;
#pragma unroll
  for (int m = 0; m < NU; ++m) {
    const int u = threadIdx.x + m * kThreads;
    if (u < units) {
      const int head = u / upu, i = (u - head * upu) * 8;
      const bool is_q = u < q_units;
      T* dst;
      if (is_q) {
        dst = q_out + ((size_t)t * a.nq + head) * a.hd + i;
      } else {
        if (kslot < 0) continue;   // a padding row: nothing is cached
        const size_t at = (((size_t)page * a.nkv + (head - a.nq)) * a.page_size + off) * a.hd + i;
        store8(v_cache + at, x0[m]);
        store8(v_cache + at + half, x1[m]);
        dst = k_cache + at;
      }
      const float* w = is_q ? q_w : k_w;
      const float inv = is_q ? inv_q : inv_k;
      if (w != nullptr) {
        const int wc = (is_q ? head : head - a.nq) * a.hd + i;
        float w0[8], w1[8];
        load8(w + wc, w0);
        load8(w + wc + half, w1);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          x0[m][k] = x0[m][k] * inv * w0[k];
          x1[m][k] = x1[m][k] * inv * w1[k];
        }
      }
      if (inv_freq != nullptr) {
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const float2 c = cs_table[i + k];
          const float ra = x0[m][k] * c.x - x1[m][k] * c.y;
          x1[m][k] = x1[m][k] * c.x + x0[m][k] * c.y;
          x0[m][k] = ra;
        }
      }
      store8(dst, x0[m]);
      store8(dst + half, x1[m]);
    }
  }
}

template <typename T>
int launch_rows(const void* in, void* q_out, void* k_cache, void* v_cache, const float* conv_w, void* state,
                const float* q_w, const float* k_w, const float* inv_freq, const int* positions, const int* slot_map,
                const int* entry_of_token, const int* cu_q, const int* state_slot, const QkRows& a, int rows, int* status,
                cudaStream_t stream) {
  const int units = (a.nq + a.nkv) * (a.hd >> 4);
#define CCB_QK(NU, TH)                                                                                               \
  ccb_launch(qk_rows_kernel<T, NU, TH>, dim3(rows), dim3(TH), 0, stream, (const T*)in, (T*)q_out, (T*)k_cache,        \
             (T*)v_cache, conv_w, (T*)state, q_w, k_w, inv_freq, positions, slot_map, entry_of_token, cu_q, state_slot, \
             a, status)
  if (units <= 128) CCB_QK(1, 128);
  else if (units <= 256) CCB_QK(1, 256);
  else if (units <= 512) CCB_QK(1, 512);
  else if (units <= 1024) CCB_QK(2, 512);
  else if (units <= 2048) CCB_QK(4, 512);
  else return CCB_REFUSE_SIZE;
#undef CCB_QK
  return ccb_launch_status();
}

}  // namespace

// in [T, row_stride]: the q | k product.  conv_w null: no convolution (taps 1).  q_w [nq * hd], k_w [nkv * hd] (float,
// null: no norm); n_real: the channels of a head that count in the norm's mean.  hd a multiple of 16 up to 256, at
// most 32,768 channels.
CCB_API int ccb_qk_rows(const void* in, int row_stride, void* q_out, void* k_cache, void* v_cache, const float* conv_w,
                        int taps, void* state, const float* q_w, const float* k_w, float eps, int n_real,
                        const float* inv_freq, const int* positions, const int* slot_map, const int* entry_of_token,
                        const int* cu_q, const int* state_slot, int rows, int n_entries, int max_slots, int nq, int nkv,
                        int hd, int page_size, int num_slots, int dtype, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || hd <= 0 || hd % 16 || hd > 256 || page_size <= 0 || taps < 1 ||
      taps > kMaxTaps || n_real <= 0 || n_real > hd || row_stride < (nq + nkv) * hd || row_stride % 8)
    return CCB_REFUSE_SIZE;
  if ((conv_w == nullptr && taps != 1) || (taps > 1 && state == nullptr) || k_cache == nullptr || v_cache == nullptr)
    return CCB_REFUSE_ARG;
  const auto bits = [](const void* p) { return reinterpret_cast<uintptr_t>(p); };
  if ((bits(in) | bits(q_out) | bits(k_cache) | bits(v_cache) | bits(conv_w) | bits(state) | bits(q_w) | bits(k_w)) & 15)
    return CCB_REFUSE_ARG;
  const QkRows a{row_stride, taps, nq, nkv, hd, n_real, page_size, num_slots, n_entries, max_slots, eps};
  if (dtype == CCB_F32)
    return launch_rows<float>(in, q_out, k_cache, v_cache, conv_w, state, q_w, k_w, inv_freq, positions, slot_map,
                              entry_of_token, cu_q, state_slot, a, rows, status, stream);
  if (dtype == CCB_BF16)
    return launch_rows<__nv_bfloat16>(in, q_out, k_cache, v_cache, conv_w, state, q_w, k_w, inv_freq, positions, slot_map,
                                      entry_of_token, cu_q, state_slot, a, rows, status, stream);
  return CCB_REFUSE_DTYPE;
}
