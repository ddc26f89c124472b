// A residual stream kept as S copies x_1 .. x_S (hyper-connections): what stands between two sublayers, in one pass
// over a token's rows.
//
//   x_t <- sum_s mix[s, t] x_s + out[t] * d      d = the output of the sublayer that ends (mix is [from, to])
//   u    = sum_t in[t] x_t                       what the next sublayer reads, before its norm
//   y    = u / sqrt(mean(u^2) + eps) * w         its RMS norm, in the storage type
//
// Every part is optional: without `mix` the copies stay as they are; without x_out nothing is written back (the
// last sum of a step, of which only some rows are wanted: row_idx); without `in` u is the plain sum of the copies.
// `shared`: all copies are equal and x holds them once ([T, D]), as they are right after the embedding.
// d is a row of the storage type, or with pair_pos the sum of the rows of the token's chosen experts
// (pair_rows[pair_pos[t * top + k]], float, in the order of k).
//
// `table`: the copies come straight from the embedding: x = table[ids[t]] * scale is written to x_out ([T, D]) and y
// is the first sublayer's norm.
//
//   streams_vec   D a multiple of 4 up to 8,192 with aligned rows: 16-byte accesses, u stays in registers.  Few rows: a
//                 cluster of up to eight blocks shares a row (the copies of one row alone are tens of kilobytes), and
//                 their sums of squares meet through distributed shared memory
//   streams_row   any D whose row fits shared memory
//
// Everything is float but d, y and the table.
#include "cluster_common.cuh"

using namespace ccb;

namespace {

constexpr int kMaxStreams = 16;
constexpr int kClusterMaxRows = 64;   // up to this many rows a cluster shares each

struct StreamsArgs {
  const float* x;          // [rows, S, D], or [rows, D] with `shared`
  float* x_out;            // [rows, S, D] (with a table [rows, D]) or null
  const void* delta;       // [rows, D] or null
  const float* pair_rows;  // [pairs, D] or null
  const int* pair_pos;     // [rows, top]
  const float* mix;        // [S, S] or null
  const float* out;        // [S]
  const float* in;         // [S] or null
  const float* w;          // [D]
  const int* row_idx;
  const void* table;
  const int* ids;
  const int* pending;
  int S, D, top, shared, n_src_rows, n_pair_rows, vocab, n_pending;
  float eps, scale;
  int* status;
};

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

__device__ __forceinline__ void axpy4(float4& a, float f, const float4 v) {
  a.x = fmaf(f, v.x, a.x); a.y = fmaf(f, v.y, a.y); a.z = fmaf(f, v.z, a.z); a.w = fmaf(f, v.w, a.w);
}

// The token of row t (-1 - s stands for the token last sampled for request slot s), or -1 if it is none.
__device__ __forceinline__ int token_of(const StreamsArgs& a, int t) {
  int id = a.ids[t];
  if (id < 0 && a.pending != nullptr && -1 - id < a.n_pending) id = a.pending[-1 - id];
  return id >= 0 && id < a.vocab ? id : -1;
}

// SS: copies (0: a.S of them, a loop).  kAhead: the norm's weight is asked for before the row.  kCluster: the blocks of a
// cluster share a row, side by side (NV 1).
template <typename T, int SS, int NV, int kThreads, bool kAhead, bool kCluster>
__global__ void __launch_bounds__(kThreads)
streams_vec_kernel(T* __restrict__ y, const StreamsArgs a) {
  constexpr int SM = SS > 0 ? SS : kMaxStreams;
  const int S = SS > 0 ? SS : a.S;
  __shared__ float red[32];
  __shared__ float slots[kMaxClusterBlocks];
  __shared__ float coef[kMaxStreams * kMaxStreams + 2 * kMaxStreams];   // mix, out, in
  static_assert(!kCluster || NV == 1, "a block of a cluster holds one run of columns");
  int r = blockIdx.x, base = 0;
  if constexpr (kCluster) {
    cluster_arrive();
    const int n = (int)cooperative_groups::this_cluster().num_blocks();
    r = blockIdx.x / n;
    base = (blockIdx.x % n) * kThreads;
  }
  const int first = base + threadIdx.x;   // this thread's vectors of four columns: first, first + kThreads, ...
  const int D = a.D, nvec = D >> 2;
  float* mix_s = coef;
  float* out_s = coef + kMaxStreams * kMaxStreams;
  float* in_s = out_s + kMaxStreams;
  // weights are nobody's output: they need not wait for the kernel before this one
  for (int i = threadIdx.x; i < S * S; i += kThreads) mix_s[i] = a.mix ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += kThreads) {
    out_s[i] = a.out ? a.out[i] : 0.f;
    in_s[i] = a.in ? a.in[i] : 1.f;
  }
  float4 w[NV];
  if (kAhead && y != nullptr) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = first + j * kThreads;
      if (i < nvec) w[j] = V4<float>::load(a.w + 4 * i);
    }
  }
  ccb::pdl_begin();
  __syncthreads();
  const int src = a.row_idx ? a.row_idx[r] : r;
  T* yr = y ? y + (size_t)r * D : nullptr;
  const bool bad = src < 0 || src >= a.n_src_rows;
  if (bad) {
    if (threadIdx.x == 0) set_status(a.status, CCB_ST_BAD_ROW);
    if (yr)
      for (int i = first; i < nvec; i += (kCluster ? nvec : kThreads))
        V4<T>::store(yr + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    if constexpr (!kCluster) return;
  }
  float4 u[NV];
#pragma unroll
  for (int j = 0; j < NV; ++j) u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
  if (kCluster && bad) {
    // (the blocks of a cluster meet below, whatever their row)
  } else
  if (a.table != nullptr) {
    const int id = token_of(a, src);
    if (id < 0 && threadIdx.x == 0) set_status(a.status, CCB_ST_BAD_TOKEN);
    float sum = 0.f;
    for (int s = 0; s < S; ++s) sum += in_s[s];
    const T* er = static_cast<const T*>(a.table) + (size_t)(id < 0 ? 0 : id) * D;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = first + j * kThreads;
      if (i < nvec) {
        float4 v = V4<T>::load(er + 4 * i);
        const float f = id < 0 ? 0.f : a.scale;
        v.x *= f; v.y *= f; v.z *= f; v.w *= f;
        V4<float>::store(a.x_out + (size_t)src * D + 4 * i, v);
        u[j] = make_float4(v.x * sum, v.y * sum, v.z * sum, v.w * sum);
      }
    }
  } else {
    const size_t row = (size_t)src * S * D;
    const float* xr = a.shared ? a.x + (size_t)src * D : a.x + row;
    const T* dr = a.delta ? static_cast<const T*>(a.delta) + (size_t)src * D : nullptr;
    const int* pp = a.pair_rows ? a.pair_pos + (size_t)src * a.top : nullptr;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = first + j * kThreads;
      if (i >= nvec) continue;
      float4 x[SM], d = make_float4(0.f, 0.f, 0.f, 0.f);
      if (a.shared) {
        x[0] = V4<float>::load(xr + 4 * i);
#pragma unroll
        for (int s = 1; s < SM; ++s) x[s] = x[0];
      } else {
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) x[s] = V4<float>::load(xr + (size_t)s * D + 4 * i);
      }
      if (dr) d = V4<T>::load(dr + 4 * i);
      if (pp) {
#pragma unroll 4
        for (int k = 0; k < a.top; ++k) {
          const int p = pp[k];
          if (p >= 0 && p < a.n_pair_rows) axpy4(d, 1.f, V4<float>::load(a.pair_rows + (size_t)p * D + 4 * i));
        }
      }
      float4 uj = make_float4(0.f, 0.f, 0.f, 0.f);
      if (a.mix != nullptr) {
#pragma unroll
        for (int t = 0; t < SM; ++t) {
          if (t >= S) continue;
          const float o = out_s[t];
          float4 n = make_float4(o * d.x, o * d.y, o * d.z, o * d.w);
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (s < S) axpy4(n, mix_s[s * S + t], x[s]);
          if (a.x_out) V4<float>::store(a.x_out + row + (size_t)t * D + 4 * i, n);
          axpy4(uj, in_s[t], n);
        }
      } else {
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) axpy4(uj, in_s[s], x[s]);
      }
      u[j] = uj;
    }
  }
  if constexpr (!kCluster) {
    if (yr == nullptr) return;
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j)
    if (first + j * kThreads < nvec)
      ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
  ss = block_sum<kThreads>(ss, red);
  if constexpr (kCluster) {
    ss = cluster_sum(ss, slots);
    if (yr == nullptr || bad) return;
  }
  const float inv = 1.0f / sqrtf(ss / (float)D + a.eps);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = first + j * kThreads;
    if (i >= nvec) continue;
    const float4 wj = kAhead ? w[j] : V4<float>::load(a.w + 4 * i);
    V4<T>::store(yr + 4 * i, make_float4(u[j].x * inv * wj.x, u[j].y * inv * wj.y, u[j].z * inv * wj.z,
                                         u[j].w * inv * wj.w));
  }
}

constexpr int kRowThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kRowThreads) streams_row_kernel(T* __restrict__ y, const StreamsArgs a) {
  ccb::pdl_begin();
  extern __shared__ float u[];
  __shared__ float red[32];
  const int r = blockIdx.x, D = a.D, S = a.S;
  const int src = a.row_idx ? a.row_idx[r] : r;
  T* yr = y ? y + (size_t)r * D : nullptr;
  if (src < 0 || src >= a.n_src_rows) {
    if (threadIdx.x == 0) set_status(a.status, CCB_ST_BAD_ROW);
    if (yr)
      for (int i = threadIdx.x; i < D; i += kRowThreads) yr[i] = from_f32<T>(0.f);
    return;
  }
  const size_t row = (size_t)src * S * D;
  const float* xr = a.x ? (a.shared ? a.x + (size_t)src * D : a.x + row) : nullptr;
  const int id = a.table ? token_of(a, src) : 0;
  if (id < 0 && threadIdx.x == 0) set_status(a.status, CCB_ST_BAD_TOKEN);
  float ss = 0.f;
  for (int i = threadIdx.x; i < D; i += kRowThreads) {
    float x[kMaxStreams], d = 0.f;
    if (a.table != nullptr) {
      const float v = id < 0 ? 0.f : to_f32(static_cast<const T*>(a.table)[(size_t)id * D + i]) * a.scale;
      a.x_out[(size_t)src * D + i] = v;
      for (int s = 0; s < S; ++s) x[s] = v;
    } else {
      for (int s = 0; s < S; ++s) x[s] = a.shared ? xr[i] : xr[(size_t)s * D + i];
    }
    if (a.delta) d = to_f32(static_cast<const T*>(a.delta)[(size_t)src * D + i]);
    if (a.pair_rows)
      for (int k = 0; k < a.top; ++k) {
        const int p = a.pair_pos[(size_t)src * a.top + k];
        if (p >= 0 && p < a.n_pair_rows) d += a.pair_rows[(size_t)p * D + i];
      }
    float v = 0.f;
    for (int t = 0; t < S; ++t) {
      float n = x[t];
      if (a.mix != nullptr) {
        n = a.out[t] * d;
        for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], x[s], n);
        if (a.x_out) a.x_out[row + (size_t)t * D + i] = n;
      }
      v = fmaf(a.in ? a.in[t] : 1.f, n, v);
    }
    u[i] = v;
    ss += v * v;
  }
  if (yr == nullptr) return;
  ss = block_sum<kRowThreads>(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)D + a.eps);
  for (int i = threadIdx.x; i < D; i += kRowThreads) yr[i] = from_f32<T>(u[i] * inv * a.w[i]);
}

template <typename T, int SS>
void launch_vec(void* y, const StreamsArgs& a, int rows, cudaStream_t stream) {
#define CCB_STREAMS(NV, TH, AH)                                                                                       \
  ccb_launch_ex(AH, streams_vec_kernel<T, SS, NV, TH, AH, false>, dim3(rows), dim3(TH), 0, stream, (T*)y, a)
  const int D = a.D;
  if (D > 512 && rows <= kClusterMaxRows) {   // 512 or 1,024 columns a block
    const int threads = D <= 4096 ? 128 : 256, n = (D / 4 + threads - 1) / threads;
    if (threads == 128)
      ccb_launch_cluster(true, n, streams_vec_kernel<T, SS, 1, 128, true, true>, dim3(rows * n), dim3(128), 0, stream, (T*)y, a);
    else
      ccb_launch_cluster(true, n, streams_vec_kernel<T, SS, 1, 256, true, true>, dim3(rows * n), dim3(256), 0, stream, (T*)y, a);
    return;
  }
  if (rows <= 148) {
    if (D <= 512) CCB_STREAMS(1, 128, true);
    else if (D <= 1024) CCB_STREAMS(1, 256, true);
    else if (D <= 2048) CCB_STREAMS(1, 512, true);
    else if (D <= 4096) CCB_STREAMS(2, 512, true);
    else CCB_STREAMS(4, 512, false);
  } else {
    if (D <= 512) CCB_STREAMS(1, 128, false);
    else if (D <= 1024) CCB_STREAMS(1, 256, false);
    else if (D <= 2048) CCB_STREAMS(2, 256, false);
    else if (D <= 4096) CCB_STREAMS(4, 256, false);
    else CCB_STREAMS(4, 512, false);
  }
#undef CCB_STREAMS
}

template <typename T>
int launch_streams(void* y, const StreamsArgs& a, int rows, bool vec, cudaStream_t stream) {
  if (vec && a.D <= 8192) {
    switch (a.S) {
      case 1: launch_vec<T, 1>(y, a, rows, stream); break;
      case 2: launch_vec<T, 2>(y, a, rows, stream); break;
      case 3: launch_vec<T, 3>(y, a, rows, stream); break;
      case 4: launch_vec<T, 4>(y, a, rows, stream); break;
      default: launch_vec<T, 0>(y, a, rows, stream); break;
    }
    return ccb_launch_status();
  }
  const size_t smem = (size_t)a.D * sizeof(float);
  if (smem > 200 * 1024) return CCB_REFUSE_SIZE;
  cudaFuncSetAttribute(streams_row_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ccb_launch(streams_row_kernel<T>, dim3(rows), dim3(kRowThreads), smem, stream, (T*)y, a);
  return ccb_launch_status();
}

}  // namespace

// rows: rows of y (with row_idx as many as there are indices).  mix and out come together; x_out may be x itself
// (each place is read before it is written) except with `shared`.
CCB_API int ccb_streams_step(void* y, const float* x, float* x_out, const void* delta, const float* pair_rows,
                             const int* pair_pos, int top, int n_pair_rows, const float* mix, const float* out,
                             const float* in, const float* w, float eps, const int* row_idx, int rows, int n_src_rows,
                             int S, int D, int shared, const void* table, const int* ids, float scale, int vocab,
                             const int* pending, int n_pending, int dtype, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (S <= 0 || S > kMaxStreams || D <= 0 || n_src_rows <= 0) return CCB_REFUSE_SIZE;
  if ((y != nullptr && w == nullptr) || (mix == nullptr) != (out == nullptr) ||
      (mix == nullptr && table == nullptr && x_out != nullptr) || (mix == nullptr && (delta || pair_rows)) ||
      (x_out != nullptr && row_idx != nullptr) || (pair_rows != nullptr && (pair_pos == nullptr || top <= 0)) ||
      (table == nullptr && x == nullptr) ||
      (table != nullptr && (ids == nullptr || x_out == nullptr || mix != nullptr || vocab <= 0)) ||
      (shared && x_out != nullptr && x_out == x))
    return CCB_REFUSE_ARG;
  StreamsArgs a;
  a.x = x; a.x_out = x_out; a.delta = delta; a.pair_rows = pair_rows; a.pair_pos = pair_pos; a.mix = mix; a.out = out;
  a.in = in; a.w = w; a.row_idx = row_idx; a.table = table; a.ids = ids; a.pending = pending; a.S = S; a.D = D;
  a.top = top; a.shared = shared; a.n_src_rows = n_src_rows; a.n_pair_rows = n_pair_rows; a.vocab = vocab;
  a.n_pending = n_pending; a.eps = eps; a.scale = scale; a.status = status;
  const auto bits = [](const void* p) { return reinterpret_cast<uintptr_t>(p); };
  const bool vec = D % 4 == 0 && ((bits(y) | bits(x) | bits(x_out) | bits(delta) | bits(pair_rows) | bits(w) |
                                   bits(table)) & 15) == 0;
  if (dtype == CCB_F32) return launch_streams<float>(y, a, rows, vec, stream);
  if (dtype == CCB_BF16) return launch_streams<__nv_bfloat16>(y, a, rows, vec, stream);
  return CCB_REFUSE_DTYPE;
}
