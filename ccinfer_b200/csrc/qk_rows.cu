// Queries and keys of attention layers whose norm runs over the whole projection: from the rows of the q | k product
// to the queries and the cached keys and values in one kernel.
//
//   u = conv(row)                   a causal convolution over time per channel (optional; w tap-major [taps, C] in the
//                                   storage type):
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
// A block takes a token, or several one after another.  A unit of work is 8 channels i .. i + 7 of a head's first half
// and their partners i + hd / 2: a thread holds its units in registers from the convolution over the norm to the
// rotation.
#include "common.cuh"

using namespace ccb;

namespace {

constexpr int kMaxTaps = 16;
constexpr int kMaxThreads = 512;

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

// Eight elements as they lie in memory.
template <typename T> struct Raw;
template <> struct Raw<float> { float4 a, b; };
template <> struct Raw<__nv_bfloat16> { uint4 a; };
__device__ __forceinline__ Raw<float> zero_raw(float) { return {make_float4(0.f, 0.f, 0.f, 0.f), make_float4(0.f, 0.f, 0.f, 0.f)}; }
__device__ __forceinline__ Raw<__nv_bfloat16> zero_raw(__nv_bfloat16) { return {make_uint4(0u, 0u, 0u, 0u)}; }
template <typename T> __device__ __forceinline__ Raw<T> load_raw(const T* p) { return *reinterpret_cast<const Raw<T>*>(p); }
template <typename T> __device__ __forceinline__ void store_raw(T* p, const Raw<T>& r) { *reinterpret_cast<Raw<T>*>(p) = r; }
template <typename T> __device__ __forceinline__ void unpack8(const Raw<T>& r, float* f) {
  load8(reinterpret_cast<const T*>(&r), f);
}

// TAPS > 0: that many taps, every row and weight of a unit asked for before any is used; 0: any number, in a loop (or
// no convolution).  A block takes `per_block` tokens one after another.  MANY: many tokens, so the registers of a thread
// are kept to what lets three or four blocks share an SM (a unit's halves one after the other, the taps' weights from L1);
// else the weights of the convolution are in registers before the kernel waits for its predecessor.
template <typename T, int NU, int TAPS, bool MANY>
__global__ void __launch_bounds__(kMaxThreads, MANY ? 2 : 1)
qk_rows_kernel(const T* __restrict__ in, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
               const T* __restrict__ conv_w, T* __restrict__ state, const float* __restrict__ q_w,
               const float* __restrict__ k_w, const float* __restrict__ inv_freq, const int* __restrict__ positions,
               const int* __restrict__ slot_map, const int* __restrict__ entry_of_token, const int* __restrict__ cu_q,
               const int* __restrict__ state_slot, const QkRows a, int rows, int per_block, int* status) {
  __shared__ float2 cs_table[2][128];
  __shared__ float red[2][64];
  constexpr bool kHeld = NU == 1 && TAPS > 0 && !MANY;
  const int threads = blockDim.x;
  const int half = a.hd >> 1;
  const int upu = half >> 3;                       // units per head
  const int units = (a.nq + a.nkv) * upu, q_units = a.nq * upu;
  const int C = (a.nq + a.nkv) * a.hd;
  Raw<T> held[kHeld ? 2 * TAPS : 1];
  if (kHeld && threadIdx.x < units) {              // (weights need not wait for the kernel before this one)
    const int head = threadIdx.x / upu, c = head * a.hd + (threadIdx.x - head * upu) * 8;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      held[2 * j] = load_raw(conv_w + (size_t)j * C + c);
      held[2 * j + 1] = load_raw(conv_w + (size_t)j * C + c + half);
    }
  }
  ccb::pdl_begin();
  const int t_end = min(rows, ((int)blockIdx.x + 1) * per_block);
  for (int t = blockIdx.x * per_block, turn = 0; t < t_end; ++t, turn ^= 1) {
    const int e = entry_of_token[t];
    const bool live = e >= 0 && e < a.n_entries;
    if (inv_freq != nullptr) {
      const float fpos = live ? (float)positions[t] : 0.f;
      for (int i = threadIdx.x; i < half; i += threads) {
        float sn, cs;
        sincosf(fpos * inv_freq[i], &sn, &cs);
        cs_table[turn][i] = make_float2(cs, sn);
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
    const bool moves = n == 1 && st != nullptr;   // the state moves on by this one row (nobody else touches it)

    float x[NU][2][8];
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int m = 0; m < NU; ++m) {
      const int u = threadIdx.x + m * threads;
      if (u < units) {
        const int head = u / upu, c0 = head * a.hd + (u - head * upu) * 8;
        if (TAPS > 0 && MANY && live) {
          constexpr int TP = TAPS > 0 ? TAPS : 1;
#pragma unroll
          for (int s = 0; s < 2; ++s) {
            const int c = c0 + s * half;
            Raw<T> raw[TP], w[TP];
#pragma unroll
            for (int j = 0; j < TP; ++j) {
              const int mrow = li - (TP - 1) + j;
              const T* src = mrow >= 0 ? in + (size_t)(r0 + mrow) * a.row_stride + c
                                       : (st != nullptr ? st + (size_t)(TP - 1 + mrow) * C + c : nullptr);
              raw[j] = src != nullptr ? load_raw(src) : zero_raw(T());
              w[j] = load_raw(conv_w + (size_t)j * C + c);
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) x[m][s][k] = 0.f;
#pragma unroll
            for (int j = 0; j < TP; ++j) {
              float uu[8], ww[8];
              unpack8(raw[j], uu);
              unpack8(w[j], ww);
#pragma unroll
              for (int k = 0; k < 8; ++k) x[m][s][k] = fmaf(ww[k], uu[k], x[m][s][k]);
            }
            if (moves) {
#pragma unroll
              for (int j = 0; j + 1 < TP; ++j) store_raw(st + (size_t)j * C + c, raw[j + 1]);
            }
          }
        } else if (TAPS > 0 && live) {
          constexpr int TP = TAPS > 0 ? TAPS : 1;
          Raw<T> raw[2 * TP];
#pragma unroll
          for (int j = 0; j < TP; ++j) {
            const int mrow = li - (TP - 1) + j;   // row of the request relative to the step's first one
            const T* src = mrow >= 0 ? in + (size_t)(r0 + mrow) * a.row_stride + c0
                                     : (st != nullptr ? st + (size_t)(TP - 1 + mrow) * C + c0 : nullptr);
            raw[2 * j] = src != nullptr ? load_raw(src) : zero_raw(T());
            raw[2 * j + 1] = src != nullptr ? load_raw(src + half) : zero_raw(T());
          }
#pragma unroll
          for (int s = 0; s < 2; ++s) {
#pragma unroll
            for (int k = 0; k < 8; ++k) x[m][s][k] = 0.f;
#pragma unroll
            for (int j = 0; j < TP; ++j) {
              float uu[8], w[8];
              unpack8(raw[2 * j + s], uu);
              if (kHeld) unpack8(held[kHeld ? 2 * j + s : 0], w);
              else load8(conv_w + (size_t)j * C + c0 + s * half, w);
#pragma unroll
              for (int k = 0; k < 8; ++k) x[m][s][k] = fmaf(w[k], uu[k], x[m][s][k]);
            }
          }
          if (moves) {
#pragma unroll
            for (int j = 0; j + 1 < TP; ++j) {
              store_raw(st + (size_t)j * C + c0, raw[2 * j + 2]);
              store_raw(st + (size_t)j * C + c0 + half, raw[2 * j + 3]);
            }
          }
        } else {
#pragma unroll
          for (int s = 0; s < 2; ++s) {
            const int c = c0 + s * half;
            const T* own = in + (size_t)t * a.row_stride + c;
            if (conv_w == nullptr || !live) {
              load8(own, x[m][s]);
              continue;
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) x[m][s][k] = 0.f;
            for (int j = 0; j < a.taps; ++j) {
              const int mrow = li - keep + j;
              float uu[8], w[8];
              if (mrow >= 0) load8(in + (size_t)(r0 + mrow) * a.row_stride + c, uu);
              else if (st != nullptr) load8(st + (size_t)(keep + mrow) * C + c, uu);
              else continue;
              load8(conv_w + (size_t)j * C + c, w);
#pragma unroll
              for (int k = 0; k < 8; ++k) x[m][s][k] = fmaf(w[k], uu[k], x[m][s][k]);
            }
            if (moves) {
              for (int k = 0; k + 1 < keep; ++k) store_raw(st + (size_t)k * C + c, load_raw(st + (size_t)(k + 1) * C + c));
              store_raw(st + (size_t)(keep - 1) * C + c, load_raw(own));
            }
          }
        }
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(x[m][0][k], x[m][0][k], fmaf(x[m][1][k], x[m][1][k], ss));
        if (u < q_units) sq += ss; else sk += ss;
      }
    }
    {   // both sums over the block (the barrier also publishes the angles; two sets of buffers in turn)
      const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      if (lane == 0) red[turn][warp] = sq, red[turn][32 + warp] = sk;
      __syncthreads();
      sq = sk = 0.f;
      for (int w = 0; w < threads / 32; ++w) sq += red[turn][w], sk += red[turn][32 + w];
    }
    const float inv_q = q_w ? 1.0f / sqrtf(sq / (float)(a.nq * a.n_real) + a.eps) : 1.f;
    const float inv_k = k_w ? 1.0f / sqrtf(sk / (float)(a.nkv * a.n_real) + a.eps) : 1.f;
    const int page = kslot >= 0 ? kslot / a.page_size : 0, off = kslot >= 0 ? kslot - page * a.page_size : 0;
#pragma unroll
    for (int m = 0; m < NU; ++m) {
      const int u = threadIdx.x + m * threads;
      if (u < units) {
        const int head = u / upu, i = (u - head * upu) * 8;
        const bool is_q = u < q_units;
        T* dst;
        if (is_q) {
          dst = q_out + ((size_t)t * a.nq + head) * a.hd + i;
        } else {
          if (kslot < 0) continue;   // a padding row: nothing is cached
          const size_t at = (((size_t)page * a.nkv + (head - a.nq)) * a.page_size + off) * a.hd + i;
          store8(v_cache + at, x[m][0]);
          store8(v_cache + at + half, x[m][1]);
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
            x[m][0][k] = x[m][0][k] * inv * w0[k];
            x[m][1][k] = x[m][1][k] * inv * w1[k];
          }
        }
        if (inv_freq != nullptr) {
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const float2 c = cs_table[turn][i + k];
            const float ra = x[m][0][k] * c.x - x[m][1][k] * c.y;
            x[m][1][k] = x[m][1][k] * c.x + x[m][0][k] * c.y;
            x[m][0][k] = ra;
          }
        }
        store8(dst, x[m][0]);
        store8(dst + half, x[m][1]);
      }
    }
  }
}

template <typename T, int NU>
int launch_rows(const void* in, void* q_out, void* k_cache, void* v_cache, const void* conv_w, void* state,
                const float* q_w, const float* k_w, const float* inv_freq, const int* positions, const int* slot_map,
                const int* entry_of_token, const int* cu_q, const int* state_slot, const QkRows& a, int rows, int* status,
                cudaStream_t stream) {
  const int units = (a.nq + a.nkv) * (a.hd >> 4);
  const int threads = ((units + NU - 1) / NU + 31) / 32 * 32;
  // many tokens: as many a block as three blocks on every SM leave, so that the weights are fetched once for all of them
  const bool many = rows > 2 * 148 && NU == 1;
  const int per_block = rows <= 2 * 148 ? 1 : (rows + 3 * 148 - 1) / (3 * 148);
  const dim3 grid((rows + per_block - 1) / per_block);
#define CCB_QK(TP)                                                                                                    \
  if (many) CCB_QKM(TP, (NU == 1)); else CCB_QKM(TP, false)
#define CCB_QKM(TP, MM)                                                                                               \
  ccb_launch_ex(true, qk_rows_kernel<T, NU, TP, MM>, grid, dim3(threads), 0, stream, (const T*)in, (T*)q_out, (T*)k_cache, \
                (T*)v_cache, (const T*)conv_w, (T*)state, q_w, k_w, inv_freq, positions, slot_map, entry_of_token, cu_q, \
                state_slot, a, rows, per_block, status)
  if (conv_w != nullptr && a.taps == 2) { CCB_QK(2); }
  else if (conv_w != nullptr && a.taps == 3) { CCB_QK(3); }
  else if (conv_w != nullptr && a.taps == 4) { CCB_QK(4); }
  else { CCB_QK(0); }
#undef CCB_QKM
#undef CCB_QK
  return ccb_launch_status();
}

template <typename T>
int pick_units(const void* in, void* q_out, void* k_cache, void* v_cache, const void* conv_w, void* state,
               const float* q_w, const float* k_w, const float* inv_freq, const int* positions, const int* slot_map,
               const int* entry_of_token, const int* cu_q, const int* state_slot, const QkRows& a, int rows, int* status,
               cudaStream_t stream) {
  const int units = (a.nq + a.nkv) * (a.hd >> 4);
#define CCB_QKN(NU)                                                                                                    \
  return launch_rows<T, NU>(in, q_out, k_cache, v_cache, conv_w, state, q_w, k_w, inv_freq, positions, slot_map,        \
                            entry_of_token, cu_q, state_slot, a, rows, status, stream)
  if (units <= kMaxThreads) CCB_QKN(1);
  if (units <= 2 * kMaxThreads) CCB_QKN(2);
  if (units <= 4 * kMaxThreads) CCB_QKN(4);
#undef CCB_QKN
  return CCB_REFUSE_SIZE;
}

}  // namespace

// in [T, row_stride]: the q | k product.  conv_w (storage type) null: no convolution (taps 1).  q_w [nq * hd],
// k_w [nkv * hd] (float, null: no norm); n_real: the channels of a head that count in the norm's mean.  hd a multiple of 16 up to 256, at
// most 32,768 channels.
CCB_API int ccb_qk_rows(const void* in, int row_stride, void* q_out, void* k_cache, void* v_cache, const void* conv_w,
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
    return pick_units<float>(in, q_out, k_cache, v_cache, conv_w, state, q_w, k_w, inv_freq, positions, slot_map,
                              entry_of_token, cu_q, state_slot, a, rows, status, stream);
  if (dtype == CCB_BF16)
    return pick_units<__nv_bfloat16>(in, q_out, k_cache, v_cache, conv_w, state, q_w, k_w, inv_freq, positions, slot_map,
                                      entry_of_token, cu_q, state_slot, a, rows, status, stream);
  return CCB_REFUSE_DTYPE;
}
