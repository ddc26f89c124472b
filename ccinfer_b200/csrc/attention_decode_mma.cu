// Decode attention on tensor cores (bfloat16, head size 64 or 128): single query tokens over paged keys.
//
// Same result as ccb_attention_split (s_j = q.k_j * scale over the visible keys, online softmax, o = P v;
// 7QiC/ccInfer: src/kernel/attention/decode_attn.cu:417-473), other machinery: a block serves ALL q heads
// of one kv head (up to 16: they are the 16 rows of an m16n8k16 tile, so keys and values are read once per
// group), keys and values of 64 positions at a time travel global -> shared memory through a three-stage
// cp.async pipeline (the copy of tile i+2 is in flight while tile i is multiplied, which is what keeps HBM
// busy), each of the 4 warps takes 16 of the 64 keys: S = Q K^T and O += P V by mma.sync, softmax in float
// registers.  The warps' partial results are merged through shared memory, the splits' through scratch
// memory and attention_merge, both in a fixed order.
#include "common.cuh"
#include "mma_common.cuh"
#include <math_constants.h>

using namespace ccb;

namespace {

constexpr int kTileKeys = 64;
constexpr int kStages = 3;
constexpr int kThreads = 128;

template <int HD>
__global__ void __launch_bounds__(kThreads)
attention_decode_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                            const __nv_bfloat16* __restrict__ v_cache, __nv_bfloat16* __restrict__ out,
                            float* __restrict__ part_acc, float* __restrict__ part_ml,
                            const int* __restrict__ positions, const int* __restrict__ entry_of_token,
                            const int* __restrict__ block_table, int bt_stride, int n_entries, int row0, int nq,
                            int nkv, int page_size, int num_pages, int window, float scale, int num_splits,
                            AttnExtra ex, int* status) {
  ccb::pdl_begin();
  constexpr int CH = HD / 8;            // 16-byte chunks per row
  constexpr int KS = HD / 16;           // k steps of q.k, and pairs of 8-wide output blocks of P v
  constexpr int TILE_ELEMS = kTileKeys * HD;
  extern __shared__ __align__(128) unsigned char smem_raw[];
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* v_s = k_s + kStages * TILE_ELEMS;

  const int G = nq / nkv;
  const int gchunks = (G + 15) / 16;
  const int r = blockIdx.x, t = row0 + r;
  const int kvh = blockIdx.y / gchunks, gc = blockIdx.y - kvh * gchunks;
  const int split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gid = lane >> 2, tig = lane & 3;
  const int h0 = kvh * G + gc * 16;
  const int n_heads = min(16, G - gc * 16);

  const int b = entry_of_token[t];
  const int p = positions[t];
  const bool padded = b < 0 || b >= n_entries || p < 0;

  float o[2 * KS][4];
#pragma unroll
  for (int i = 0; i < 2 * KS; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.f, l1 = 0.f;

  if (!padded) {
    // q as A fragments: rows = heads of the group (zero beyond n_heads)
    uint32_t qa[KS][4];
    {
      const __nv_bfloat16* q0 = q + ((size_t)t * nq + h0 + gid) * HD;
      const __nv_bfloat16* q1 = q0 + (size_t)8 * HD;
      const bool v0 = gid < n_heads, v1 = gid + 8 < n_heads;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const int c = ks * 16 + 2 * tig;
        qa[ks][0] = v0 ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
        qa[ks][1] = v1 ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
        qa[ks][2] = v0 ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
        qa[ks][3] = v1 ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
      }
    }
    const int* bt = block_table + (size_t)b * bt_stride;
    const int page_shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;
    const int j0 = first_visible_key(p, window, ex.chunk);
    const KeyTiles kt(j0, ex.keep, kTileKeys);
    const int first_tile = kt.first, last_tile = p / kTileKeys;
    const int n_tiles = last_tile - first_tile + 1;
    const int per_split = (n_tiles + num_splits - 1) / num_splits;
    const int my_first = first_tile + split * per_split;
    const int my_tiles = min(my_first + per_split, last_tile + 1) - my_first;

    // Two threads share a key row: one page lookup and one address per thread and tile, then 16-byte copies of
    // alternating chunks, so that a pair of lanes always asks for one whole 32-byte sector.
    static_assert(kThreads == 2 * kTileKeys, "two threads per key row");
    const int ld_row = tid >> 1, ld_half = tid & 1;
    auto issue = [&](int tile, int stage) {
      __nv_bfloat16* ks_ = k_s + stage * TILE_ELEMS;
      __nv_bfloat16* vs_ = v_s + stage * TILE_ELEMS;
      const int j = kt.tile(tile) * kTileKeys + ld_row;
      bool valid = key_visible(j, j0, p, ex.keep);
      size_t src = 0;
      if (valid) {
        const int lp = page_shift >= 0 ? (j >> page_shift) : (j / page_size);
        const int page = lp < bt_stride ? bt[lp] : -1;
        if (page < 0 || page >= num_pages) {
          set_status(status, CCB_ST_BAD_PAGE);
          valid = false;
        } else {
          src = (((size_t)page * nkv + kvh) * page_size + (j - lp * page_size)) * HD;
        }
      }
      const __nv_bfloat16* ksrc = k_cache + src;
      const __nv_bfloat16* vsrc = v_cache + src;
      const uint32_t kdst = smem_u32(ks_ + ld_row * HD), vdst = smem_u32(vs_ + ld_row * HD);
      const int sw = ld_row & 7;
#pragma unroll
      for (int i = 0; i < CH / 2; ++i) {
        const int c = 2 * i + ld_half;
        const uint32_t off = (uint32_t)((c ^ sw) << 4);
        cp_async16(kdst + off, ksrc + c * 8, valid);
        cp_async16(vdst + off, vsrc + c * 8, valid);
      }
    };

#pragma unroll
    for (int s = 0; s < kStages - 1; ++s) {
      if (s < my_tiles) issue(my_first + s, s);
      cp_async_commit();
    }
    for (int it = 0; it < my_tiles; ++it) {
      cp_async_wait<kStages - 2>();
      __syncthreads();
      if (it + kStages - 1 < my_tiles) issue(my_first + it + kStages - 1, (it + kStages - 1) % kStages);
      cp_async_commit();
      const __nv_bfloat16* ks_ = k_s + (it % kStages) * TILE_ELEMS;
      const __nv_bfloat16* vs_ = v_s + (it % kStages) * TILE_ELEMS;

      // S[16 heads, 16 keys of this warp] = Q K^T
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      {
        const int krow = warp * 16 + (lane & 7) + 8 * (lane >> 4);
        const int kchunk = (lane >> 3) & 1;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          uint32_t b00, b01, b10, b11;
          ldmatrix_x4(b00, b01, b10, b11, smem_u32(ks_ + swz<HD>(krow, 2 * ks + kchunk)));
          mma_bf16_16816(s[0], qa[ks], b00, b01);
          mma_bf16_16816(s[1], qa[ks], b10, b11);
        }
      }
      // mask, online softmax (rows gid and gid + 8)
      const int jbase = kt.tile(my_first + it) * kTileKeys + warp * 16 + 2 * tig;
      float mx0 = -CUDART_INF_F, mx1 = -CUDART_INF_F;
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = jbase + nb * 8 + e;
          const bool vis = key_visible(j, j0, p, ex.keep);
          s[nb][e] = vis ? s[nb][e] * scale : -CUDART_INF_F;
          s[nb][2 + e] = vis ? s[nb][2 + e] * scale : -CUDART_INF_F;
          mx0 = fmaxf(mx0, s[nb][e]);
          mx1 = fmaxf(mx1, s[nb][2 + e]);
        }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
      // a row that has seen no key yet keeps max -inf: its probabilities are 0 and nothing is rescaled
      const float c0 = mn0 == -CUDART_INF_F ? 1.f : __expf(m0 - mn0);
      const float c1 = mn1 == -CUDART_INF_F ? 1.f : __expf(m1 - mn1);
      const float sub0 = mn0 == -CUDART_INF_F ? 0.f : mn0, sub1 = mn1 == -CUDART_INF_F ? 0.f : mn1;
      m0 = mn0;
      m1 = mn1;
      float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[nb][e] = __expf(s[nb][e] - sub0);          // exp(-inf) = 0 for masked keys
          s[nb][2 + e] = __expf(s[nb][2 + e] - sub1);
          ps0 += s[nb][e];
          ps1 += s[nb][2 + e];
        }
      l0 = l0 * c0 + ps0;   // per-lane partial sums; the four lanes of a row are added at the end
      l1 = l1 * c1 + ps1;
#pragma unroll
      for (int i = 0; i < 2 * KS; ++i) {
        o[i][0] *= c0; o[i][1] *= c0;
        o[i][2] *= c1; o[i][3] *= c1;
      }
      // O += P V
      uint32_t pa[4];
      pa[0] = pack_bf16(s[0][0], s[0][1]);
      pa[1] = pack_bf16(s[0][2], s[0][3]);
      pa[2] = pack_bf16(s[1][0], s[1][1]);
      pa[3] = pack_bf16(s[1][2], s[1][3]);
      {
        const int vrow = warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1);
        const int vchunk = lane >> 4;
#pragma unroll
        for (int nn = 0; nn < KS; ++nn) {
          uint32_t b00, b01, b10, b11;
          ldmatrix_x4_trans(b00, b01, b10, b11, smem_u32(vs_ + swz<HD>(vrow, 2 * nn + vchunk)));
          mma_bf16_16816(o[2 * nn], pa, b00, b01);
          mma_bf16_16816(o[2 * nn + 1], pa, b10, b11);
        }
      }
    }
    cp_async_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  }
  __syncthreads();  // every copy has landed and every warp is done with the tiles: reuse the memory

  float* o_s = reinterpret_cast<float*>(smem_raw);  // [4 warps][16 rows][HD]
  float* m_s = o_s + 4 * 16 * HD;                   // [4][16]
  float* l_s = m_s + 64;
#pragma unroll
  for (int i = 0; i < 2 * KS; ++i) {
    const int d = i * 8 + 2 * tig;
    float* dst0 = o_s + ((size_t)(warp * 16 + gid)) * HD + d;
    float* dst1 = o_s + ((size_t)(warp * 16 + gid + 8)) * HD + d;
    dst0[0] = o[i][0]; dst0[1] = o[i][1];
    dst1[0] = o[i][2]; dst1[1] = o[i][3];
  }
  if (tig == 0) {
    m_s[warp * 16 + gid] = m0;
    m_s[warp * 16 + gid + 8] = m1;
    l_s[warp * 16 + gid] = l0;
    l_s[warp * 16 + gid + 8] = l1;
  }
  __syncthreads();
  for (int idx = tid; idx < n_heads * HD; idx += kThreads) {
    const int row = idx / HD, d = idx - row * HD;
    float mm = -CUDART_INF_F;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, m_s[w * 16 + row]);
    float a = 0.f, ll = 0.f;
    if (mm != -CUDART_INF_F) {
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float f = __expf(m_s[w * 16 + row] - mm);
        a += o_s[(size_t)(w * 16 + row) * HD + d] * f;
        ll += l_s[w * 16 + row] * f;
      }
    }
    const int h = h0 + row;
    if (num_splits == 1) {
      a *= attn_sink_fold(ex, h, mm, ll);
      if (mm != -CUDART_INF_F) a *= attn_gate<__nv_bfloat16>(ex, t, h);
      out[((size_t)t * nq + h) * HD + d] = __float2bfloat16_rn(ll > 0.f ? a / ll : 0.f);
    } else {
      const size_t slot = ((size_t)r * nq + h) * num_splits + split;
      part_acc[slot * HD + d] = a;
      if (d == 0) {
        part_ml[slot * 2] = mm;
        part_ml[slot * 2 + 1] = ll;
      }
    }
  }
}

__global__ void attention_merge_bf16_kernel(__nv_bfloat16* __restrict__ out, const float* __restrict__ part_acc,
                                            const float* __restrict__ part_ml, int row0, int nq, int hd,
                                            int num_splits, AttnExtra ex) {
  ccb::pdl_begin();
  const int r = blockIdx.x, h = blockIdx.y;
  const size_t base = ((size_t)r * nq + h) * num_splits;
  float mm = -CUDART_INF_F;
  for (int s = 0; s < num_splits; ++s) mm = fmaxf(mm, part_ml[(base + s) * 2]);
  __nv_bfloat16* o = out + ((size_t)(row0 + r) * nq + h) * hd;
  if (mm == -CUDART_INF_F) {
    for (int d = threadIdx.x; d < hd; d += blockDim.x) o[d] = __float2bfloat16_rn(0.f);
    return;
  }
  float ll = 0.f;
  for (int s = 0; s < num_splits; ++s) ll += part_ml[(base + s) * 2 + 1] * __expf(part_ml[(base + s) * 2] - mm);
  const float fold = attn_sink_fold(ex, h, mm, ll) * attn_gate<__nv_bfloat16>(ex, row0 + r, h);
  for (int d = threadIdx.x; d < hd; d += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < num_splits; ++s) a += part_acc[(base + s) * hd + d] * __expf(part_ml[(base + s) * 2] - mm);
    o[d] = __float2bfloat16_rn(a * fold / ll);
  }
}

template <int HD>
int launch(const void* q, const void* k_cache, const void* v_cache, void* out, float* part_acc, float* part_ml,
           const int* positions, const int* entry_of_token, const int* block_table, int bt_stride, int n_entries,
           int row0, int n_rows, int nq, int nkv, int page_size, int num_pages, int window, float scale,
           int num_splits, AttnExtra ex, int* status, cudaStream_t stream) {
  const int G = nq / nkv, gchunks = (G + 15) / 16;
  const size_t smem = (size_t)2 * kStages * kTileKeys * HD * sizeof(__nv_bfloat16);
  static bool configured = false;  // per process and head size; the attribute belongs to the function
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attention_decode_mma_kernel<HD>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  dim3 grid(n_rows, nkv * gchunks, num_splits);
  ccb_launch(attention_decode_mma_kernel<HD>, grid, kThreads, smem, stream, 
      (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, (__nv_bfloat16*)out,
      part_acc, part_ml, positions, entry_of_token, block_table, bt_stride, n_entries, row0, nq, nkv, page_size,
      num_pages, window, scale, num_splits, ex, status);
  int rc = ccb_launch_status();
  if (rc != 0 || num_splits == 1) return rc;
  ccb_launch(attention_merge_bf16_kernel, dim3(n_rows, nq), 128, 0, stream, (__nv_bfloat16*)out, part_acc, part_ml, row0,
                                                                     nq, HD, num_splits, ex);
  return ccb_launch_status();
}

}  // namespace

// bfloat16 only, head size 64 or 128 (others: CCB_REFUSE_SIZE, use ccb_attention_split).  Scratch as for
// ccb_attention_split: n_rows * nq * num_splits * (hd + 2) floats, unused with one split.  chunk, sink, gate,
// gate_stride: see AttnExtra (0 / null: none).
CCB_API int ccb_attention_decode_mma(const void* q, const void* k_cache, const void* v_cache, void* out,
                                     float* part_acc, float* part_ml, const int* positions,
                                     const int* entry_of_token, const int* block_table, int bt_stride,
                                     int n_entries, int row0, int n_rows, int nq, int nkv, int hd, int page_size,
                                     int num_pages, int window, float scale, int num_splits, int chunk, int keep,
                                     const float* sink, const void* gate, int gate_stride, int* status,
                                     cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (chunk < 0 || keep < 0 || (gate != nullptr && gate_stride < nq)) return CCB_REFUSE_ARG;
  const AttnExtra ex{chunk, sink, gate, gate_stride, keep};
  if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || page_size <= 0 || bt_stride <= 0 || num_splits <= 0 ||
      num_splits > 64)
    return CCB_REFUSE_SIZE;
  if (num_splits > 1 && (part_acc == nullptr || part_ml == nullptr)) return CCB_REFUSE_ARG;
  if (hd == 128)
    return launch<128>(q, k_cache, v_cache, out, part_acc, part_ml, positions, entry_of_token, block_table,
                       bt_stride, n_entries, row0, n_rows, nq, nkv, page_size, num_pages, window, scale, num_splits,
                       ex, status, stream);
  if (hd == 64)
    return launch<64>(q, k_cache, v_cache, out, part_acc, part_ml, positions, entry_of_token, block_table,
                      bt_stride, n_entries, row0, n_rows, nq, nkv, page_size, num_pages, window, scale, num_splits,
                      ex, status, stream);
  return CCB_REFUSE_SIZE;
}
