// Shared device helpers of the ccinfer_b200 kernels (sm_100a).
//
// Every kernel family is instantiated for two element types: float (the true
// 32-bit path) and __nv_bfloat16 (the serving path).  Arithmetic is always
// done in float; only loads and stores see the storage type.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <utility>

#define CCB_API extern "C" __attribute__((visibility("default")))

// dtype codes of the C interface
enum { CCB_F32 = 0, CCB_BF16 = 1 };

// bits of the device status word (set by kernels, never cleared by them)
enum {
  CCB_ST_BAD_TOKEN = 1,   // token id outside [0, vocab)
  CCB_ST_BAD_SLOT = 2,    // cache slot outside the pool
  CCB_ST_BAD_PAGE = 4,    // block-table entry outside the pool where a key was needed
  CCB_ST_BAD_ROW = 8,     // row index outside the batch
  CCB_ST_WAIT_TIMEOUT = 16  // a bounded mbarrier wait gave up
};

namespace ccb {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of kThreads (a multiple of 32, at most 1024) in a fixed
// order: lanes by butterfly, then the warps' partial sums one after another.
// Every thread gets the result.  `red` holds at least 32 floats.
template <int kThreads>
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  v = warp_sum(v);
  __syncthreads();  // red may still be read from an earlier call
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) total += red[w];
  return total;
}

// Programmatic dependent launch.  A kernel launched with the attribute may start while its predecessor in
// the stream still runs; `pdl_wait` blocks until the predecessor has completed and its writes are visible,
// `pdl_trigger` lets the successor start early in turn.  Without the attribute both are no-ops.
// Every kernel calls pdl_begin() (or the two halves, with read-only prefetching of weights in between)
// before it touches memory that another kernel may have written.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
// Kernels without weights to prefetch: wait for the predecessor, then let the successor start (a product
// then streams its first weight tiles while this kernel runs).  The order matters: a kernel that let its
// successor in BEFORE its predecessor had finished would put three kernels on the device at once, and a
// product's blocks, resident but waiting, would keep the predecessor's last blocks from being scheduled.
__device__ __forceinline__ void pdl_begin() {
  pdl_wait();
  pdl_trigger();
}

// Sum of a row of `n` partial sums by one warp, every lane with the result; the order of the additions is
// fixed (by lane, then a shuffle tree).  The loads are asked for together, not one after the other's use.
__device__ __forceinline__ float row_ssq(const float* row, int n, int lane) {
  float ss = 0.f;
  if ((n & 3) == 0 && (reinterpret_cast<uintptr_t>(row) & 15) == 0) {
    const float4* row4 = reinterpret_cast<const float4*>(row);
#pragma unroll 4
    for (int p = lane; p < (n >> 2); p += 32) {
      const float4 v = __ldcg(row4 + p);
      ss += (v.x + v.y) + (v.z + v.w);
    }
  } else {
#pragma unroll 4
    for (int p = lane; p < n; p += 32) ss += __ldcg(row + p);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  return ss;
}

// The gated activation of a feed-forward, as the epilogue of its gate|up product:
//   g * sigmoid(g * (alpha + cubic * g^2)) * u
// where with limit > 0 g and u are first g' = min(g, limit), u' = clamp(u, -limit, limit) + shift.
//   silu(g) * u:     limit 0, alpha 1, cubic 0
//   clamped:         limit, alpha and shift of the model's choosing, cubic 0
//   gelu(g) * u with the tanh form 0.5 g (1 + tanh(sqrt(2 / pi) (g + 0.044715 g^3))):  since 0.5 (1 + tanh(z)) =
//                    sigmoid(2 z), alpha = 2 sqrt(2 / pi) and cubic = 0.044715 alpha
struct CcbGluAct {
  float limit, alpha, shift, cubic;
};

__device__ __forceinline__ float glu_act(const CcbGluAct a, float g, float u) {
  if (a.limit > 0.f) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit) + a.shift;
  }
  return g / (1.f + __expf(-g * fmaf(a.cubic, g * g, a.alpha))) * u;
}

// The same with the accurate exponential (kernels of their own, the 32-bit path).
__device__ __forceinline__ float glu_act_exact(const CcbGluAct a, float g, float u) {
  if (a.limit > 0.f) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit) + a.shift;
  }
  return g / (1.f + expf(-g * fmaf(a.cubic, g * g, a.alpha))) * u;
}

// What an attention kernel takes beside keys and values (all optional):
//   chunk  > 0: a query at position p sees only keys from floor(p / chunk) * chunk on (runs of `chunk` positions
//          counted from the start of the sequence), on top of a window if there is one;
//   sink   float [q heads]: one more term exp(sink[h]) in the softmax denominator of head h, with no key and no
//          value, not scaled, counted once per query;
//   gate   [tokens, gate_stride] in the compute type: head h's result is multiplied by sigmoid(gate[t, h]);
//   keep   > 0: the first `keep` keys of the sequence are seen by every later query, whatever the window and the
//          chunk leave out.
struct AttnExtra {
  int chunk;
  const float* sink;
  const void* gate;
  int gate_stride;
  int keep;
};

// The first key position a query at position p sees (both bounds are non-decreasing in p).
__device__ __forceinline__ int first_visible_key(int p, int window, int chunk) {
  int j0 = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
  if (chunk > 0) {
    const int c0 = (p / chunk) * chunk;
    j0 = c0 > j0 ? c0 : j0;
  }
  return j0;
}

// Whether a query at position p whose window (or chunk) starts at key lo sees key j.
__device__ __forceinline__ bool key_visible(int j, int lo, int p, int keep) {
  return j <= p && (j >= lo || j < keep);
}

// The tiles of `tile_keys` keys that a walk over the keys of a query (or of a tile of queries whose first window
// starts at key j0) visits: those of the keys that are always seen, then those from the window's first one on.
// They are counted in one run of numbers first .. last (the window's last tile): from `window` on a number is the
// tile itself, below it the tiles count from 0.  Without kept keys, or where the window reaches them, the two are
// the same.
struct KeyTiles {
  int first, window;
  __device__ __forceinline__ KeyTiles(int j0, int keep, int tile_keys) {
    window = j0 / tile_keys;
    const int kept = (keep + tile_keys - 1) / tile_keys;
    first = window - (kept < window ? kept : window);
  }
  __device__ __forceinline__ int tile(int n) const { return n >= window ? n : n - first; }
};

// The sink's term folded into a finished softmax of head h (maximum mm, sum ll, natural exponent): ll becomes the
// whole denominator, and the weighted values are to be multiplied by the factor returned.  A row that saw no key
// (mm = -inf, a padded row) is left as it is.
__device__ __forceinline__ float attn_sink_fold(const AttnExtra& ex, int h, float mm, float& ll) {
  if (ex.sink == nullptr || mm == -INFINITY) return 1.f;
  const float sk = ex.sink[h];
  const float m2 = fmaxf(mm, sk);
  const float f = __expf(mm - m2);
  ll = ll * f + __expf(sk - m2);
  return f;
}

template <typename T>
__device__ __forceinline__ float attn_gate(const AttnExtra& ex, int t, int h) {
  if (ex.gate == nullptr) return 1.f;
  const float z = to_f32(static_cast<const T*>(ex.gate)[(size_t)t * ex.gate_stride + h]);
  return 1.f / (1.f + expf(-z));
}

__device__ __forceinline__ void set_status(int* status, int bit) {
  if (status != nullptr) atomicOr(status, bit);
}

}  // namespace ccb

// Host side: every launcher returns the CUDA error code of its launch (0 = ok)
// or a negative number for an argument it refuses.
#define CCB_REFUSE_SIZE (-2)
#define CCB_REFUSE_DTYPE (-3)
#define CCB_REFUSE_ARG (-4)

static inline int ccb_launch_status() { return (int)cudaGetLastError(); }

// One switch per kernel family (ccb_set_pdl of its shared object; kernels.set_pdl tells every loaded family and every
// family loaded later): launch kernels with programmatic stream serialization.
extern int g_ccb_pdl;

// `early`: this kernel gains from starting before its predecessor has finished (it prefetches weights).
template <typename... KArgs, typename... Args>
static inline void ccb_launch_ex(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                 cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  if (g_ccb_pdl && (early || g_ccb_pdl > 1)) {
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
  }
  cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);  // the error is read by ccb_launch_status()
}

template <typename... KArgs, typename... Args>
static inline void ccb_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args&&... args) {
  ccb_launch_ex(false, kernel, grid, block, smem, stream, static_cast<Args&&>(args)...);
}
