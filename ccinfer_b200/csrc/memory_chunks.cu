// The recurrence of a matrix memory with one decay per head and token,
//
//   S <- a_t S + b_t k_t v_t^T;   o_t = S^T q_t * q_mult,
//
// over a request's portion of a prompt in chunks of 64 tokens on tensor cores (bfloat16 operands, float sums).  With
// c_t the sum of log a over the chunk up to t and S0 the memory before the chunk,
//
//   o_t = exp(c_t) S0^T q_t + sum_{s <= t} exp(c_t - c_s + log b_s) (q_t . k_s) v_s
//   S   = exp(c_64) S0 + sum_s exp(c_64 - c_s + log b_s) k_s v_s^T
//
// so a chunk is four small products, and only S is carried from chunk to chunk.  What the model computes in 32 bits
// stays so to about 2^-17: the logarithms, their sums and the exponentials are float; the memory lives in float
// registers for the whole portion; and every float that must become an operand (the memory, the weighted scores, the
// weighted values, queries and keys that were rotated) goes in as TWO bfloat16, its rounding and what the rounding
// left, each with a product of its own.  Queries, keys and values straight from a projection are bfloat16 already.
//
// A block: one request, one head, a slice of 8 NB value columns; four warps.  A warp takes 16 query rows of the chunk
// for the read-out and DK / 4 key channels of S for the update.  With a column of ones after the values (a running sum
// of the keys: n . q is one more column of o) the first slice takes it as one more block of eight columns.
// The next chunk's rows arrive through cp.async while this one is computed; two barriers a chunk.
#include "common.cuh"
#include "mma_common.cuh"
#include <math_constants.h>

using namespace ccb;

namespace {

constexpr int kChunk = 64;
constexpr int kThreads = 128;

struct ChunkArgs {
  const __nv_bfloat16 *q, *q_lo, *k, *k_lo, *v;
  int ldqk, ldv;              // row strides (q and k in one; q_lo, k_lo as q and k)
  const float* log_a;         // [tokens, H]
  const float* log_b;         // [tokens, H] or null: zero
  float* state;               // [slots, H, dvo, DK]
  float* out;                 // [tokens, H, dvo]
  const int *cu_q, *state_slot;
  int entry0, H, dv, dvo, max_slots;
  float q_mult;
};

// bfloat16 pair of (x, y) and of what their rounding left
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(x - f.x, y - f.y);
}

template <int DK, int NB, bool SPLIT, bool ONES>
__global__ void __launch_bounds__(kThreads)
memory_chunks_kernel(const ChunkArgs a) {
  ccb::pdl_begin();
  constexpr int BN = 8 * NB, VP = BN + 8;      // columns of the slice, pitch of its rows in shared memory (elements)
  constexpr int NT = NB + (ONES ? 1 : 0);      // blocks of eight columns
  constexpr int KS = DK / 16;
  constexpr int MT = DK / 64;                  // 16-row tiles of S a warp owns
  constexpr int TILE = kChunk * DK, VT = kChunk * VP;
  constexpr int QK = SPLIT ? 4 : 2;            // tiles of a stage: q, k (, their second halves)
  extern __shared__ __align__(128) unsigned char smem_raw[];
  __nv_bfloat16* tiles = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [2][QK][64][DK], swizzled
  __nv_bfloat16* v_s = tiles + 2 * QK * TILE;                          // [2][64][VP]
  __nv_bfloat16* s_hi = v_s + 2 * VT;                                  // [DK][VP]
  __nv_bfloat16* s_lo = s_hi + DK * VP;
  __nv_bfloat16* w_hi = s_lo + DK * VP;                                // [64][VP]
  __nv_bfloat16* w_lo = w_hi + VT;
  float* gates = reinterpret_cast<float*>(w_lo + VT);                  // [2][4][64]: c_t, exp(c_t), log b - c, weights

  const int e = a.entry0 + blockIdx.z, h = blockIdx.y, slice = blockIdx.x;
  const int slot = a.state_slot[e];
  const int r0 = a.cu_q[e], n = a.cu_q[e + 1] - r0;
  if (slot < 0 || slot >= a.max_slots || n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gid = lane >> 2, tig = lane & 3;
  const int col0 = slice * BN;
  const bool ones = ONES && slice == 0;
  const int nt = NB + (ones ? 1 : 0);

  auto issue = [&](int chunk, int st) {
    const int t0 = chunk * kChunk;
    __nv_bfloat16* dst = tiles + st * QK * TILE;
    const __nv_bfloat16* src[4] = {a.q, a.k, a.q_lo, a.k_lo};
#pragma unroll
    for (int x = 0; x < QK; ++x)
#pragma unroll
      for (int i = 0; i < kChunk * (DK / 8) / kThreads; ++i) {
        const int idx = tid + kThreads * i;
        const int row = idx / (DK / 8), c = idx % (DK / 8);
        const bool ok = t0 + row < n;
        cp_async16(smem_u32(dst + x * TILE + swz<DK>(row, c)),
                   src[x] + (size_t)(r0 + t0 + (ok ? row : 0)) * a.ldqk + h * DK + c * 8, ok);
      }
#pragma unroll
    for (int i = 0; i < (kChunk * NB + kThreads - 1) / kThreads; ++i) {
      const int idx = tid + kThreads * i;
      const int row = idx / NB, c = idx % NB;
      const bool ok = t0 + row < n;
      cp_async16(smem_u32(v_s + st * VT + row * VP + c * 8),
                 a.v + (size_t)(r0 + t0 + (ok ? row : 0)) * a.ldv + h * a.dv + col0 + c * 8, ok);
    }
    cp_async_commit();
  };

  // The gates of a chunk, two tokens a lane of warp 0: loaded one chunk ahead, summed and left in shared memory.
  float la[2], lb[2];
  auto load_gates = [&](int chunk) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = chunk * kChunk + 2 * lane + i;
      const bool ok = t < n;
      la[i] = ok ? a.log_a[(size_t)(r0 + t) * a.H + h] : 0.f;
      lb[i] = ok ? (a.log_b ? a.log_b[(size_t)(r0 + t) * a.H + h] : 0.f) : -CUDART_INF_F;
    }
  };
  auto write_gates = [&](int st) {
    float* g = gates + st * 4 * kChunk;
    float sum = la[0] + la[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float p = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += p;
    }
    const float total = __shfl_sync(0xffffffffu, sum, 31);
    const float c1 = sum, c0 = sum - la[1];
    g[2 * lane] = c0;
    g[2 * lane + 1] = c1;
    g[kChunk + 2 * lane] = expf(c0);
    g[kChunk + 2 * lane + 1] = expf(c1);
    g[2 * kChunk + 2 * lane] = lb[0] - c0;
    g[2 * kChunk + 2 * lane + 1] = lb[1] - c1;
    g[3 * kChunk + 2 * lane] = expf(total + (lb[0] - c0));
    g[3 * kChunk + 2 * lane + 1] = expf(total + (lb[1] - c1));
  };

  issue(0, 0);
  if (warp == 0) {
    load_gates(0);
    write_gates(0);
    load_gates(1);
  }
  // the column of ones beside the values (and zeros after it): the same in both stages, for good
  for (int i = tid; i < 2 * kChunk * 8; i += kThreads)
    v_s[(i >> 3) * VP + BN + (i & 7)] = __float2bfloat16_rn((i & 7) == 0 && ones ? 1.f : 0.f);
  for (int i = tid; i < kChunk * 8; i += kThreads) {
    w_hi[(i >> 3) * VP + BN + (i & 7)] = __float2bfloat16_rn(0.f);
    w_lo[(i >> 3) * VP + BN + (i & 7)] = __float2bfloat16_rn(0.f);
  }

  // S: rows (key channels) m0 .. of the warp, columns of the slice; the accumulator layout of the update's product
  float S[MT][NT][4];
  float* sp = a.state + ((size_t)slot * a.H + h) * a.dvo * DK;
  auto column = [&](int nb, int c) { return nb < NB ? col0 + nb * 8 + c : (c == 0 ? a.dv : -1); };
  auto store_s = [&]() {   // the memory as two bfloat16, rows of key channels
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nb = 0; nb < NT; ++nb) {
        if (nb >= nt) continue;
        const int row = (warp * MT + mt) * 16 + gid, c = nb * 8 + 2 * tig;
        uint32_t hi, lo;
        split2(S[mt][nb][0], S[mt][nb][1], hi, lo);
        *reinterpret_cast<uint32_t*>(s_hi + row * VP + c) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + row * VP + c) = lo;
        split2(S[mt][nb][2], S[mt][nb][3], hi, lo);
        *reinterpret_cast<uint32_t*>(s_hi + (row + 8) * VP + c) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + (row + 8) * VP + c) = lo;
      }
  };
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nb = 0; nb < NT; ++nb)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int row = (warp * MT + mt) * 16 + gid + 8 * (x >> 1);
        const int c = nb < nt ? column(nb, 2 * tig + (x & 1)) : -1;
        S[mt][nb][x] = c >= 0 ? sp[(size_t)c * DK + row] : 0.f;
      }
  store_s();

  // rows of an operand whose k runs over rows of shared memory with pitch VP: block pair p (16 columns), 16 k from k0;
  // the last single block reads its own columns twice
  const int trow = (lane & 7) + 8 * ((lane >> 3) & 1);
  auto load_b = [&](const __nv_bfloat16* base, int k0, int nb, bool single, uint32_t* b) {
    const int c = nb * 8 + (single ? 0 : 8 * (lane >> 4));
    ldmatrix_x4_trans(b[0], b[1], b[2], b[3], smem_u32(base + (k0 + trow) * VP + c));
  };

  const int chunks = (n + kChunk - 1) / kChunk;
  for (int ch = 0; ch < chunks; ++ch) {
    const int st = ch & 1;
    cp_async_wait<0>();
    __syncthreads();   // the chunk's rows and gates are there; everybody is done with the chunk before
    if (ch + 1 < chunks) issue(ch + 1, st ^ 1);
    if (warp == 0 && ch + 1 < chunks) {
      write_gates(st ^ 1);
      load_gates(ch + 2);
    }
    const __nv_bfloat16 *qt = tiles + st * QK * TILE, *kt = qt + TILE, *ql = qt + 2 * TILE, *kl = qt + 3 * TILE;
    const __nv_bfloat16* vt = v_s + st * VT;
    const float *gc = gates + st * 4 * kChunk, *ga = gc + kChunk, *gb = ga + kChunk, *gw = gb + kChunk;

    {   // the values times their weights in the chunk's contribution to S
      const int row = tid >> 1, part = (tid & 1) * (BN / 2);
      const float w = gw[row];
#pragma unroll
      for (int c = 0; c < BN / 2; c += 2) {
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(vt + row * VP + part + c);
        const float2 f = __bfloat1622float2(x);
        uint32_t hi, lo;
        split2(f.x * w, f.y * w, hi, lo);
        *reinterpret_cast<uint32_t*>(w_hi + row * VP + part + c) = hi;
        *reinterpret_cast<uint32_t*>(w_lo + row * VP + part + c) = lo;
      }
      if (ones && (tid & 1) == 0) {
        const __nv_bfloat16 hi = __float2bfloat16_rn(w);
        w_hi[row * VP + BN] = hi;
        w_lo[row * VP + BN] = __float2bfloat16_rn(w - __bfloat162float(hi));
      }
    }

    // read-out of rows warp * 16 ..: first S0^T q and the raw scores q . k of the keys up to the rows' own block
    float acc[NT][4], s[2 * 4][4];
#pragma unroll
    for (int nb = 0; nb < NT; ++nb) acc[nb][0] = acc[nb][1] = acc[nb][2] = acc[nb][3] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const int arow = warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1), achunk = lane >> 4;
    const int krow = (lane & 7) + 8 * (lane >> 4), kchunk = (lane >> 3) & 1;
#pragma unroll 2
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t qa[4], qb[4];
      ldmatrix_x4(qa[0], qa[1], qa[2], qa[3], smem_u32(qt + swz<DK>(arow, 2 * ks + achunk)));
      if (SPLIT) ldmatrix_x4(qb[0], qb[1], qb[2], qb[3], smem_u32(ql + swz<DK>(arow, 2 * ks + achunk)));
#pragma unroll
      for (int nb = 0; nb < NT; nb += 2) {
        if (nb >= nt) continue;
        const bool single = nb + 1 >= NT;
        uint32_t bh[4], bl[4];
        load_b(s_hi, ks * 16, nb, single, bh);
        load_b(s_lo, ks * 16, nb, single, bl);
        mma_bf16_16816(acc[nb], qa, bh[0], bh[1]);
        mma_bf16_16816(acc[nb], qa, bl[0], bl[1]);
        if (SPLIT) mma_bf16_16816(acc[nb], qb, bh[0], bh[1]);
        if (!single) {
          mma_bf16_16816(acc[nb + 1 < NT ? nb + 1 : nb], qa, bh[2], bh[3]);
          mma_bf16_16816(acc[nb + 1 < NT ? nb + 1 : nb], qa, bl[2], bl[3]);
          if (SPLIT) mma_bf16_16816(acc[nb + 1 < NT ? nb + 1 : nb], qb, bh[2], bh[3]);
        }
      }
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np > warp) continue;
        uint32_t b[4];
        ldmatrix_x4(b[0], b[1], b[2], b[3], smem_u32(kt + swz<DK>(np * 16 + krow, 2 * ks + kchunk)));
        mma_bf16_16816(s[2 * np], qa, b[0], b[1]);
        mma_bf16_16816(s[2 * np + 1], qa, b[2], b[3]);
        if (SPLIT) {
          mma_bf16_16816(s[2 * np], qb, b[0], b[1]);
          mma_bf16_16816(s[2 * np + 1], qb, b[2], b[3]);
          ldmatrix_x4(b[0], b[1], b[2], b[3], smem_u32(kl + swz<DK>(np * 16 + krow, 2 * ks + kchunk)));
          mma_bf16_16816(s[2 * np], qa, b[0], b[1]);
          mma_bf16_16816(s[2 * np + 1], qa, b[2], b[3]);
        }
      }
    }
    const int t_lo = warp * 16 + gid, t_hi = t_lo + 8;
    const float a_lo = ga[t_lo] * a.q_mult, a_hi = ga[t_hi] * a.q_mult;
    const float c_lo = gc[t_lo], c_hi = gc[t_hi];
#pragma unroll
    for (int nb = 0; nb < NT; ++nb) {
      acc[nb][0] *= a_lo; acc[nb][1] *= a_lo;
      acc[nb][2] *= a_hi; acc[nb][3] *= a_hi;
    }
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np > warp) continue;
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float* x = s[2 * np + half];
        const int j = np * 16 + half * 8 + 2 * tig;
        const float b0 = gb[j], b1 = gb[j + 1];
        x[0] = j <= t_lo ? x[0] * (__expf(c_lo + b0) * a.q_mult) : 0.f;
        x[1] = j + 1 <= t_lo ? x[1] * (__expf(c_lo + b1) * a.q_mult) : 0.f;
        x[2] = j <= t_hi ? x[2] * (__expf(c_hi + b0) * a.q_mult) : 0.f;
        x[3] = j + 1 <= t_hi ? x[3] * (__expf(c_hi + b1) * a.q_mult) : 0.f;
        split2(x[0], x[1], ph[2 * half], pl[2 * half]);
        split2(x[2], x[3], ph[2 * half + 1], pl[2 * half + 1]);
      }
#pragma unroll
      for (int nb = 0; nb < NT; nb += 2) {
        if (nb >= nt) continue;
        const bool single = nb + 1 >= NT;
        uint32_t b[4];
        load_b(vt, np * 16, nb, single, b);
        mma_bf16_16816(acc[nb], ph, b[0], b[1]);
        mma_bf16_16816(acc[nb], pl, b[0], b[1]);
        if (!single) {
          mma_bf16_16816(acc[nb + 1 < NT ? nb + 1 : nb], ph, b[2], b[3]);
          mma_bf16_16816(acc[nb + 1 < NT ? nb + 1 : nb], pl, b[2], b[3]);
        }
      }
    }
    const int left = n - ch * kChunk;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int t = x == 0 ? t_lo : t_hi;
      if (t < left) {
        float* o = a.out + ((size_t)(r0 + ch * kChunk + t) * a.H + h) * a.dvo;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
          o[col0 + nb * 8 + 2 * tig] = acc[nb][2 * x];
          o[col0 + nb * 8 + 2 * tig + 1] = acc[nb][2 * x + 1];
        }
        if (ones && tig == 0) o[a.dv] = acc[NT - 1][2 * x];
      }
    }
    __syncthreads();   // everybody has read S0, and the weighted values are complete

    const float keep = ga[kChunk - 1];   // exp(c_64)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nb = 0; nb < NT; ++nb)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[mt][nb][x] *= keep;
#pragma unroll
    for (int ks = 0; ks < kChunk / 16; ++ks) {
      // keys as the A operand, transposed: rows are key channels, k are tokens
      uint32_t ka[MT][4], kb[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const int token = ks * 16 + (lane & 7) + 8 * (lane >> 4);
        const int c8 = (warp * MT + mt) * 2 + ((lane >> 3) & 1);
        ldmatrix_x4_trans(ka[mt][0], ka[mt][1], ka[mt][2], ka[mt][3], smem_u32(kt + swz<DK>(token, c8)));
        if (SPLIT) ldmatrix_x4_trans(kb[mt][0], kb[mt][1], kb[mt][2], kb[mt][3], smem_u32(kl + swz<DK>(token, c8)));
      }
#pragma unroll
      for (int nb = 0; nb < NT; nb += 2) {
        if (nb >= nt) continue;
        const bool single = nb + 1 >= NT;
        uint32_t bh[4], bl[4];
        load_b(w_hi, ks * 16, nb, single, bh);
        load_b(w_lo, ks * 16, nb, single, bl);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16_16816(S[mt][nb], ka[mt], bh[0], bh[1]);
          mma_bf16_16816(S[mt][nb], ka[mt], bl[0], bl[1]);
          if (SPLIT) mma_bf16_16816(S[mt][nb], kb[mt], bh[0], bh[1]);
          if (!single) {
            mma_bf16_16816(S[mt][nb + 1 < NT ? nb + 1 : nb], ka[mt], bh[2], bh[3]);
            mma_bf16_16816(S[mt][nb + 1 < NT ? nb + 1 : nb], ka[mt], bl[2], bl[3]);
            if (SPLIT) mma_bf16_16816(S[mt][nb + 1 < NT ? nb + 1 : nb], kb[mt], bh[2], bh[3]);
          }
        }
      }
    }
    if (ch + 1 < chunks) store_s();
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nb = 0; nb < NT; ++nb)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int row = (warp * MT + mt) * 16 + gid + 8 * (x >> 1);
        const int c = nb < nt ? column(nb, 2 * tig + (x & 1)) : -1;
        if (c >= 0) sp[(size_t)c * DK + row] = S[mt][nb][x];
      }
}

template <int DK, int NB, bool SPLIT, bool ONES>
int launch_chunks(const ChunkArgs& a, int n_entries, cudaStream_t stream) {
  constexpr int VP = 8 * NB + 8;
  constexpr size_t smem = (size_t)(2 * (SPLIT ? 4 : 2) * kChunk * DK + 2 * kChunk * VP + 2 * DK * VP + 2 * kChunk * VP) * 2 +
                          2 * 4 * kChunk * sizeof(float);
  static_assert(smem <= 227 * 1024, "shared memory of a block");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(memory_chunks_kernel<DK, NB, SPLIT, ONES>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  ccb_launch(memory_chunks_kernel<DK, NB, SPLIT, ONES>, dim3(a.dv / (8 * NB), a.H, n_entries), dim3(kThreads), smem, stream,
             a);
  return ccb_launch_status();
}

template <int DK, int NB>
int pick_chunks(const ChunkArgs& a, int n_entries, cudaStream_t stream) {
  const bool split = a.q_lo != nullptr, ones = a.dvo > a.dv;
  if (split) return ones ? launch_chunks<DK, NB, true, true>(a, n_entries, stream) : launch_chunks<DK, NB, true, false>(a, n_entries, stream);
  return ones ? launch_chunks<DK, NB, false, true>(a, n_entries, stream) : launch_chunks<DK, NB, false, false>(a, n_entries, stream);
}

}  // namespace

// Key sizes 64 and 128, value sizes that are multiples of 16 (others: CCB_REFUSE_SIZE).  q, k (and q_lo, k_lo: what the
// rounding of q and k to bfloat16 left, or null) [tokens, ldqk] with head h at column h * dk; v [tokens, ldv] with head
// h at column h * dv; log_a, log_b (null: zero) float [tokens, H]; state float [slots, H, dvo, dk] and out float
// [tokens, H, dvo] with dvo = dv, or dv + 1 for a last value column of ones.  Entries entry0 .. entry0 + n_entries - 1.
CCB_API int ccb_memory_chunks(const void* q, const void* q_lo, const void* k, const void* k_lo, int ldqk, const void* v,
                              int ldv, const float* log_a, const float* log_b, float* state, float* out, const int* cu_q,
                              const int* state_slot, int entry0, int n_entries, int H, int dk, int dv, int dvo,
                              int max_slots, float q_mult, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || (dk != 64 && dk != 128) || dv <= 0 || dv % 16 || (dvo != dv && dvo != dv + 1) || ldqk % 8 || ldv % 8)
    return CCB_REFUSE_SIZE;
  if ((q_lo == nullptr) != (k_lo == nullptr) || log_a == nullptr) return CCB_REFUSE_ARG;
  const auto bits = [](const void* p) { return reinterpret_cast<uintptr_t>(p); };
  if ((bits(q) | bits(q_lo) | bits(k) | bits(k_lo) | bits(v)) & 15) return CCB_REFUSE_ARG;
  const __nv_bfloat16 *qp = (const __nv_bfloat16*)q, *qlp = (const __nv_bfloat16*)q_lo, *kp = (const __nv_bfloat16*)k,
                      *klp = (const __nv_bfloat16*)k_lo, *vp = (const __nv_bfloat16*)v;
  const ChunkArgs a{qp, qlp, kp, klp, vp, ldqk, ldv, log_a, log_b, state, out, cu_q, state_slot, entry0, H, dv, dvo,
                    max_slots, q_mult};
  // slices of 32 columns where they give enough blocks, else of 16
  const bool wide = dv % 32 == 0 && (long long)(dv / 32) * H * n_entries >= 96;
  if (dk == 128) return wide ? pick_chunks<128, 4>(a, n_entries, stream) : pick_chunks<128, 2>(a, n_entries, stream);
  return wide ? pick_chunks<64, 4>(a, n_entries, stream) : pick_chunks<64, 2>(a, n_entries, stream);
}
