// What stands between two sublayers, in one pass over a row: the norm(s) on the output of the sublayer that ends,
// the sum into the residual stream, and the norm that reads the stream next.
//
//   d = delta                                                              one sublayer's output, or of a pair
//     = ca * unit(delta) * wa + cb * unit(delta_b) * wb                    unit(x) = x / sqrt(mean(x^2) + eps)
//   h <- h + mult * post(d) [+ add];      y = next(h)
//
// `post` and `next` are each nothing, an RMS norm  unit(x) * w,  or a layer norm
//   (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b
// whose variance is taken from the deviations (two passes over the registers, not E[x^2] - mean^2).  With `next`
// nothing, y holds the stream's own rows.  Every part is optional; with row_idx only those rows are read, nothing is
// written to h, and y holds them in the order of row_idx.  The stream and every sum are float; delta and y are of
// the storage type.
//
//   norm_chain_vec    D a multiple of 4 up to 8,192 with aligned rows: everything a row needs (with few rows the
//                     weights too) is asked for at once with 16-byte loads and stays in registers between the sums
//   norm_chain_row    any D whose row fits shared memory
#include "common.cuh"

using namespace ccb;

struct NormStage {
  int kind;          // 0: nothing, 1: RMS, 2: layer norm
  const float* w;
  const float* b;    // layer norm only
  float eps;
};

struct NormPair {
  const void* second;   // null: no pair
  const float* wa;
  const float* wb;
  float ca, cb, eps;
};

namespace {

template <typename T> struct V4;
template <> struct V4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct V4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 r;
    r.x = *reinterpret_cast<const uint32_t*>(&a);
    r.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
  }
};

__device__ __forceinline__ float sum4(const float4 v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float ssq4(const float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

// Two sums over the block at once (see block_sum).
template <int kThreads>
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) red[warp] = a, red[32 + warp] = b;
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) t.x += red[w], t.y += red[32 + w];
  return t;
}

// Normalises x[NV] (the row's pieces this thread holds) in place.  kHeld: the weights are in w and b; else they are
// loaded where they are needed.
template <int NV, int kThreads, bool kHeld>
__device__ __forceinline__ void apply_stage(const NormStage& st, float4* x, const float4* w, const float4* b, int nvec,
                                            int D, float* red) {
  if (st.kind == 0) return;
  float mean = 0.f;
  if (st.kind == 2) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (threadIdx.x + j * kThreads < nvec) s += sum4(x[j]);
    mean = block_sum<kThreads>(s, red) / (float)D;
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j)
    if (threadIdx.x + j * kThreads < nvec) {
      x[j].x -= mean; x[j].y -= mean; x[j].z -= mean; x[j].w -= mean;
      ss += ssq4(x[j]);
    }
  ss = block_sum<kThreads>(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)D + st.eps);
#pragma unroll
  for (int j = 0; j < NV; ++j)
    if (threadIdx.x + j * kThreads < nvec) {
      const int i = 4 * (threadIdx.x + j * kThreads);
      const float4 wj = kHeld ? w[j] : V4<float>::load(st.w + i);
      x[j].x = x[j].x * inv * wj.x; x[j].y = x[j].y * inv * wj.y;
      x[j].z = x[j].z * inv * wj.z; x[j].w = x[j].w * inv * wj.w;
      if (st.kind == 2) {
        const float4 bj = kHeld ? b[j] : V4<float>::load(st.b + i);
        x[j].x += bj.x; x[j].y += bj.y; x[j].z += bj.z; x[j].w += bj.w;
      }
    }
}

// kAhead: the weights are asked for with the row (few rows: latency); else each when it is needed (many rows: fewer
// registers, more blocks on an SM).
template <typename T, int NV, int kThreads, bool kAhead, bool kPair>
__global__ void __launch_bounds__(kThreads)
norm_chain_vec_kernel(T* __restrict__ y, float* __restrict__ h, const T* __restrict__ delta, const NormPair pair,
                      const NormStage post, float mult, const float* __restrict__ add, const NormStage next,
                      const int* __restrict__ row_idx, int n_src_rows, int D, int* status) {
  __shared__ float red[64];
  const int r = blockIdx.x;
  const int nvec = D >> 2;
  float4 pw[NV], pb[NV], nw[NV], nb[NV];
  auto load_stage = [&](const NormStage& st, float4* w, float4* b) {
    if (st.kind == 0) return;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = threadIdx.x + j * kThreads;
      if (i < nvec) {
        w[j] = V4<float>::load(st.w + 4 * i);
        if (st.kind == 2) b[j] = V4<float>::load(st.b + 4 * i);
      }
    }
  };
  if (kAhead) {   // weights are nobody's output: they need not wait for the kernel before this one
    load_stage(post, pw, pb);
    load_stage(next, nw, nb);
  }
  ccb::pdl_begin();
  const int src = row_idx ? row_idx[r] : r;
  T* yr = y ? y + (size_t)r * D : nullptr;
  if (src < 0 || src >= n_src_rows) {
    if (threadIdx.x == 0) set_status(status, CCB_ST_BAD_ROW);
    if (yr)
      for (int i = threadIdx.x; i < nvec; i += kThreads) V4<T>::store(yr + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  float* hr = h + (size_t)src * D;
  const float* ar = add ? add + (size_t)src * D : nullptr;
  float4 v[NV], d[NV];
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = threadIdx.x + j * kThreads;
    if (i < nvec) {
      v[j] = V4<float>::load(hr + 4 * i);
      if (delta) d[j] = V4<T>::load(delta + (size_t)src * D + 4 * i);
    }
  }
  if (kPair) {
    const T* br = static_cast<const T*>(pair.second) + (size_t)src * D;
    float4 e[NV], wa[NV], wb[NV];
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = threadIdx.x + j * kThreads;
      if (i < nvec) {
        e[j] = V4<T>::load(br + 4 * i);
        if (kAhead) {
          wa[j] = V4<float>::load(pair.wa + 4 * i);
          wb[j] = V4<float>::load(pair.wb + 4 * i);
        }
        sa += ssq4(d[j]);
        sb += ssq4(e[j]);
      }
    }
    const float2 s2 = block_sum2<kThreads>(sa, sb, red);
    const float fa = pair.ca / sqrtf(s2.x / (float)D + pair.eps), fb = pair.cb / sqrtf(s2.y / (float)D + pair.eps);
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (threadIdx.x + j * kThreads < nvec) {
        const int i = 4 * (threadIdx.x + j * kThreads);
        const float4 a = kAhead ? wa[j] : V4<float>::load(pair.wa + i), b = kAhead ? wb[j] : V4<float>::load(pair.wb + i);
        d[j].x = d[j].x * fa * a.x + e[j].x * fb * b.x;
        d[j].y = d[j].y * fa * a.y + e[j].y * fb * b.y;
        d[j].z = d[j].z * fa * a.z + e[j].z * fb * b.z;
        d[j].w = d[j].w * fa * a.w + e[j].w * fb * b.w;
      }
  }
  if (delta) apply_stage<NV, kThreads, kAhead>(post, d, pw, pb, nvec, D, red);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = threadIdx.x + j * kThreads;
    if (i < nvec) {
      if (delta) {
        v[j].x += mult * d[j].x; v[j].y += mult * d[j].y; v[j].z += mult * d[j].z; v[j].w += mult * d[j].w;
      }
      if (ar) {
        const float4 a = V4<float>::load(ar + 4 * i);
        v[j].x += a.x; v[j].y += a.y; v[j].z += a.z; v[j].w += a.w;
      }
      if ((delta || ar) && row_idx == nullptr) V4<float>::store(hr + 4 * i, v[j]);
    }
  }
  if (yr == nullptr) return;
  apply_stage<NV, kThreads, kAhead>(next, v, nw, nb, nvec, D, red);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = threadIdx.x + j * kThreads;
    if (i < nvec) V4<T>::store(yr + 4 * i, v[j]);
  }
}

constexpr int kRowThreads = 256;

// x[D] in shared memory, each thread its own elements d = threadIdx.x, + kRowThreads, ...
__device__ __forceinline__ void row_stage(const NormStage& st, float* x, int D, float* red) {
  if (st.kind == 0) return;
  float mean = 0.f;
  if (st.kind == 2) {
    float s = 0.f;
    for (int d = threadIdx.x; d < D; d += kRowThreads) s += x[d];
    mean = block_sum<kRowThreads>(s, red) / (float)D;
  }
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += kRowThreads) {
    const float c = x[d] - mean;
    x[d] = c;
    ss += c * c;
  }
  ss = block_sum<kRowThreads>(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)D + st.eps);
  for (int d = threadIdx.x; d < D; d += kRowThreads) {
    const float n = x[d] * inv * st.w[d];
    x[d] = st.kind == 2 ? n + st.b[d] : n;
  }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
norm_chain_row_kernel(T* __restrict__ y, float* __restrict__ h, const T* __restrict__ delta, const NormPair pair,
                      const NormStage post, float mult, const float* __restrict__ add, const NormStage next,
                      const int* __restrict__ row_idx, int n_src_rows, int D, int* status) {
  ccb::pdl_begin();
  extern __shared__ float x[];
  __shared__ float red[64];
  const int r = blockIdx.x;
  const int src = row_idx ? row_idx[r] : r;
  T* yr = y ? y + (size_t)r * D : nullptr;
  if (src < 0 || src >= n_src_rows) {
    if (threadIdx.x == 0) set_status(status, CCB_ST_BAD_ROW);
    if (yr)
      for (int d = threadIdx.x; d < D; d += kRowThreads) yr[d] = from_f32<T>(0.f);
    return;
  }
  float* hr = h + (size_t)src * D;
  const T* dr = delta ? delta + (size_t)src * D : nullptr;
  const float* ar = add ? add + (size_t)src * D : nullptr;
  if (dr) {
    for (int d = threadIdx.x; d < D; d += kRowThreads) x[d] = to_f32(dr[d]);
    if (pair.second != nullptr) {
      const T* br = static_cast<const T*>(pair.second) + (size_t)src * D;
      float sa = 0.f, sb = 0.f;
      for (int d = threadIdx.x; d < D; d += kRowThreads) {
        const float e = to_f32(br[d]);
        sa += x[d] * x[d];
        sb += e * e;
      }
      const float2 s2 = block_sum2<kRowThreads>(sa, sb, red);
      const float fa = pair.ca / sqrtf(s2.x / (float)D + pair.eps), fb = pair.cb / sqrtf(s2.y / (float)D + pair.eps);
      for (int d = threadIdx.x; d < D; d += kRowThreads)
        x[d] = x[d] * fa * pair.wa[d] + to_f32(br[d]) * fb * pair.wb[d];
    }
    row_stage(post, x, D, red);
  }
  for (int d = threadIdx.x; d < D; d += kRowThreads) {
    float v = hr[d];
    if (dr) v += mult * x[d];
    if (ar) v += ar[d];
    if ((dr || ar) && row_idx == nullptr) hr[d] = v;
    x[d] = v;
  }
  if (yr == nullptr) return;
  row_stage(next, x, D, red);
  for (int d = threadIdx.x; d < D; d += kRowThreads) yr[d] = from_f32<T>(x[d]);
}

template <typename T>
int launch_chain(void* y, float* h, const void* delta, const NormPair& pair, const NormStage& post, float mult,
                 const float* add, const NormStage& next, const int* row_idx, int rows, int n_src_rows, int D, bool vec,
                 int* status, cudaStream_t stream) {
#define CCB_CHAIN(NV, TH, AH)                                                                                      \
  if (pair.second != nullptr)                                                                                       \
    ccb_launch_ex(AH, norm_chain_vec_kernel<T, NV, TH, AH, true>, dim3(rows), dim3(TH), 0, stream, (T*)y, h, (const T*)delta, \
               pair, post, mult, add, next, row_idx, n_src_rows, D, status);                                          \
  else                                                                                                              \
    ccb_launch_ex(AH, norm_chain_vec_kernel<T, NV, TH, AH, false>, dim3(rows), dim3(TH), 0, stream, (T*)y, h, (const T*)delta, \
               pair, post, mult, add, next, row_idx, n_src_rows, D, status)
  if (vec && D <= 8192) {
    if (rows <= 148) {
      if (D <= 512) { CCB_CHAIN(1, 128, true); }
      else if (D <= 1024) { CCB_CHAIN(1, 256, true); }
      else if (D <= 2048) { CCB_CHAIN(1, 512, true); }
      else if (D <= 4096) { CCB_CHAIN(2, 512, true); }
      else { CCB_CHAIN(4, 512, false); }
    } else {
      if (D <= 512) { CCB_CHAIN(1, 128, false); }
      else if (D <= 1024) { CCB_CHAIN(1, 256, false); }
      else if (D <= 2048) { CCB_CHAIN(2, 256, false); }
      else if (D <= 4096) { CCB_CHAIN(4, 256, false); }
      else { CCB_CHAIN(4, 512, false); }
    }
    return ccb_launch_status();
  }
#undef CCB_CHAIN
  const size_t smem = (size_t)D * sizeof(float);
  if (smem > 200 * 1024) return CCB_REFUSE_SIZE;
  cudaFuncSetAttribute(norm_chain_row_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ccb_launch(norm_chain_row_kernel<T>, dim3(rows), dim3(kRowThreads), smem, stream, (T*)y, h, (const T*)delta, pair,
             post, mult, add, next, row_idx, n_src_rows, D, status);
  return ccb_launch_status();
}

}  // namespace

// *_kind 0: no such norm (its pointers are ignored), 1: RMS (w), 2: layer norm (w and b).  delta_b null: no pair.
CCB_API int ccb_norm_chain(void* y, float* h, const void* delta, const void* delta_b, const float* wa, const float* wb,
                           float ca, float cb, float eps_pair, int post_kind, const float* post_w, const float* post_b,
                           float post_eps, float mult, const float* add, int next_kind, const float* next_w,
                           const float* next_b, float next_eps, const int* row_idx, int rows, int n_src_rows, int D,
                           int dtype, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (D <= 0 || n_src_rows <= 0) return CCB_REFUSE_SIZE;
  if (h == nullptr || (delta_b != nullptr && (delta == nullptr || wa == nullptr || wb == nullptr)) || post_kind < 0 ||
      post_kind > 2 || next_kind < 0 || next_kind > 2 || (post_kind > 0 && post_w == nullptr) ||
      (post_kind == 2 && post_b == nullptr) || (next_kind > 0 && (next_w == nullptr || y == nullptr)) ||
      (next_kind == 2 && next_b == nullptr))
    return CCB_REFUSE_ARG;
  const NormPair pair{delta_b, wa, wb, ca, cb, eps_pair};
  const NormStage post{delta != nullptr ? post_kind : 0, post_w, post_b, post_eps}, next{next_kind, next_w, next_b, next_eps};
  const auto bits = [](const void* p) { return reinterpret_cast<uintptr_t>(p); };
  uintptr_t all = bits(y) | bits(h) | bits(delta) | bits(add);
  if (delta_b != nullptr) all |= bits(delta_b) | bits(wa) | bits(wb);
  if (post.kind > 0) all |= bits(post_w);
  if (post.kind == 2) all |= bits(post_b);
  if (next_kind > 0) all |= bits(next_w);
  if (next_kind == 2) all |= bits(next_b);
  const bool vec = D % 4 == 0 && (all & 15) == 0;
  if (dtype == CCB_F32)
    return launch_chain<float>(y, h, delta, pair, post, mult, add, next, row_idx, rows, n_src_rows, D, vec, status, stream);
  if (dtype == CCB_BF16)
    return launch_chain<__nv_bfloat16>(y, h, delta, pair, post, mult, add, next, row_idx, rows, n_src_rows, D, vec, status,
                                       stream);
  return CCB_REFUSE_DTYPE;
}
