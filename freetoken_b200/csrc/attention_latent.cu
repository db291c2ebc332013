// Attention over cached latent rows: every query head reads ONE row of d values per key, whose first
// `rank` values are also the value (absorbed latent attention, rows of any width up to 1,024).
//
// Queries are the rows of [T * nq, d] (token-major, then head).  A CTA owns RT = 16 * MT consecutive
// rows of one segment - the heads of a decoded token, or of a few neighbouring tokens of a short prompt
// portion - and one split of the keys, and walks key tiles of 64 rows, each fetched ONCE (cp.async, 16-byte
// pieces, up to three stages) and used twice: as keys and, its first `rank` columns, as values.
//
//   S[RT, 64]    = Q K^T   eight warps: two groups of 32 keys x four interleaved quarters of d, partial
//                          products of mma.sync m16n8k16 left in shared memory (float32)
//   softmax      : RT rows x 64 keys spread over the 256 threads (16 / MT threads a row): the four
//                          partial scores are added in order, scaled, masked by absolute position; running
//                          max and sum in float32 per row; P rounded to bfloat16 into shared memory
//   O[RT, rank] += P V     each warp owns CB blocks of 16 value columns for all 64 keys (ldmatrix.trans on
//                          the same tile), accumulators in registers
// With splits > 1 every CTA leaves an unnormalised partial (o, max, sum); latent_merge combines the
// splits in ascending order.
//
// The reference has no latent attention; its split-KV decode kernel
// (python/freetoken/kernel/triton/attention.py:147-349) is the pattern of the splits.
#include "common.cuh"
#include "mma_utils.cuh"

namespace ft {

struct LatentAttnArgs {
  const __nv_bfloat16* q;       // [T * nq, d]
  __nv_bfloat16* out;           // flat row r at r * ldo, `rank` values
  float* part_o;                // [tiles * RT, splits, rank]
  float* part_ml;               // [tiles * RT, splits, 2]
  const __nv_bfloat16* pages;   // [pages, P, d]
  const int* tile_seg;          // [tiles]
  const int* tile_row;          // [tiles] first flat row inside the segment
  const int* seg_q_start;
  const int* seg_pos0;
  const int* block_table;
  long long page_stride, ldo;
  int nq, d, rank, P, table_width, window, splits, split_keys, stages;
  float scale_log2;
};

constexpr int LT_KEYS = 64, LT_THREADS = 256, LT_PLD = LT_KEYS + 8;

template <int CB, int MT>
__global__ void __launch_bounds__(LT_THREADS) attn_latent_kernel(LatentAttnArgs a) {
  constexpr int RT = 16 * MT;
  constexpr int TPR = 16 / MT;                 // threads per row in the softmax
  constexpr int KPT = LT_KEYS / TPR;           // keys per thread there
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int dp = (a.d + 15) & ~15, ld = dp + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);            // [RT][ld]
  __nv_bfloat16* sK = sQ + RT * ld;                                          // [stages][64][ld]
  __nv_bfloat16* sP = sK + (size_t)a.stages * LT_KEYS * ld;                  // [RT][72]
  float* sS = reinterpret_cast<float*>(sP + RT * LT_PLD);                    // [4 quarters][RT][64]
  float* sAlpha = sS + 4 * RT * LT_KEYS;                                     // [RT]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_wait();

  const int seg = a.tile_seg[blockIdx.x], row0 = a.tile_row[blockIdx.x];
  const int split = blockIdx.y;
  const int seg_begin = a.seg_q_start[seg];
  const int rows = min(RT, (a.seg_q_start[seg + 1] - seg_begin) * a.nq - row0);
  const int pos0 = a.seg_pos0[seg];
  const long long flat0 = (long long)seg_begin * a.nq + row0;
  const int* table = a.block_table + (size_t)seg * a.table_width;
  const int pos_first = pos0 + row0 / a.nq, pos_last = pos0 + (row0 + rows - 1) / a.nq;
  const int k_lo = max(first_visible(pos_first, a.window, 0), split * a.split_keys);
  const int k_end = min(pos_last + 1, (split + 1) * a.split_keys);
  const int k_begin = k_lo / LT_KEYS * LT_KEYS;
  const int ntiles = k_end > k_lo ? (k_end - k_begin + LT_KEYS - 1) / LT_KEYS : 0;
  const int chunks = a.d >> 3;

  // A warp fetches rows warp, warp + 8, ... of a tile.  Lanes 0..7 look their row's place up (all at once);
  // rows outside the visible keys repeat a valid one (masked later).
  auto locate = [&](int tile) -> const __nv_bfloat16* {
    const int j = min(max(k_begin + tile * LT_KEYS + warp + 8 * (lane & 7), k_lo), pos_last);
    return a.pages + (size_t)table[j / a.P] * a.page_stride + (size_t)(j % a.P) * a.d;
  };
  auto load_tile = [&](const __nv_bfloat16* mine, int stage) {
    __nv_bfloat16* dst = sK + (size_t)stage * LT_KEYS * ld + warp * ld;
#pragma unroll
    for (int i = 0; i < LT_KEYS / 8; ++i) {
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(__shfl_sync(0xffffffffu, (unsigned long long)mine, i));
      for (int c = lane; c < chunks; c += 32) cp_async16(dst + i * 8 * ld + c * 8, src + c * 8);
    }
  };

  // rows of 8 more values than a multiple of 16: the pad of every row counts as zeros
  if (dp != a.d)
    for (int r = tid; r < RT + a.stages * LT_KEYS; r += LT_THREADS)
      *reinterpret_cast<uint4*>((r < RT ? sQ + r * ld : sK + (size_t)(r - RT) * ld) + a.d) = make_uint4(0u, 0u, 0u, 0u);
  for (int s = 0; s < a.stages - 1; ++s) {
    if (s < ntiles) load_tile(locate(s), s);
    cp_async_commit();
  }
  const __nv_bfloat16* ahead = a.stages - 1 < ntiles ? locate(a.stages - 1) : nullptr;    // the next tile to fetch
  for (int r = warp; r < RT; r += LT_THREADS / 32)
    for (int c = lane; c < chunks; c += 32) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < rows) v = *reinterpret_cast<const uint4*>(a.q + (flat0 + r) * a.d + c * 8);
      *reinterpret_cast<uint4*>(sQ + r * ld + c * 8) = v;
    }

  float o[MT][CB][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int c = 0; c < CB; ++c)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[m][c][n][i] = 0.f;
  // this thread's row and keys in the softmax
  const int srow = tid / TPR, skey = (tid % TPR) * KPT;
  const int spos = pos0 + (row0 + srow) / a.nq;
  const int slo = max(k_lo, first_visible(spos, a.window, 0));
  const int shi = srow < rows ? min(spos, k_end - 1) : -1;         // last key this row sees here
  float m_run = -INFINITY, l_run = 0.f;
  const int quarter = warp & 3, kgroup = warp >> 2;
  const int g = lane >> 2, t4 = lane & 3;
  const int nks = dp >> 4;

  for (int tile = 0; tile < ntiles; ++tile) {
    if (a.stages > 2) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();                            // the tile has landed (stages > 1); everybody is done with tile - 1
    const int pre = tile + a.stages - 1;
    if (pre < ntiles) load_tile(ahead, pre % a.stages);
    cp_async_commit();
    if (pre + 1 < ntiles) ahead = locate(pre + 1);
    if (a.stages == 1) {
      cp_async_wait<0>();
      __syncthreads();
    }
    const __nv_bfloat16* tk = sK + (size_t)(tile % a.stages) * LT_KEYS * ld;

    // ---- partial scores: 32 keys, every fourth k-step of 16
    {
      float s[MT][4][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) s[m][n][i] = 0.f;
      const __nv_bfloat16* kr = tk + (size_t)(kgroup * 32 + (lane & 7) + ((lane >> 4) << 3)) * ld + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* qr = sQ + (size_t)(lane & 15) * ld + (lane >> 4) * 8;
#pragma unroll 3
      for (int ks = quarter; ks < nks; ks += 4) {
        unsigned kf[2][4];
        ldsm_x4(kf[0], kr + ks * 16);
        ldsm_x4(kf[1], kr + 16 * ld + ks * 16);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          unsigned qf[4];
          ldsm_x4(qf, qr + m * 16 * ld + ks * 16);
#pragma unroll
          for (int n = 0; n < 4; ++n) mma16816(s[m][n], qf, kf[n >> 1][(n & 1) * 2], kf[n >> 1][(n & 1) * 2 + 1]);
        }
      }
      float* dst = sS + (size_t)quarter * RT * LT_KEYS + kgroup * 32;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          *reinterpret_cast<float2*>(dst + (m * 16 + g) * LT_KEYS + n * 8 + 2 * t4) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(dst + (m * 16 + g + 8) * LT_KEYS + n * 8 + 2 * t4) = make_float2(s[m][n][2], s[m][n][3]);
        }
    }
    __syncthreads();

    // ---- softmax of this thread's KPT keys of its row
    {
      const int j0 = k_begin + tile * LT_KEYS + skey;
      float v[KPT];
#pragma unroll
      for (int i = 0; i < KPT; i += 4) {
        const float* src = sS + (size_t)srow * LT_KEYS + skey + i;
        float4 x = *reinterpret_cast<const float4*>(src);
#pragma unroll
        for (int p = 1; p < 4; ++p) {
          const float4 y = *reinterpret_cast<const float4*>(src + (size_t)p * RT * LT_KEYS);
          x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        }
        v[i] = x.x; v[i + 1] = x.y; v[i + 2] = x.z; v[i + 3] = x.w;
      }
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        v[i] = (j0 + i >= slo && j0 + i <= shi) ? v[i] * a.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      // the running max only moves when it would grow by more than 2^8 (exp2 of the rest stays far
      // inside float32 and bfloat16 range): most tiles then leave the accumulators alone
      const float m_new = mx > m_run + 8.f ? mx : m_run;
      const float alpha = m_run == -INFINITY ? 0.f : fast_exp2(m_run - m_new);
      const float base = m_new == -INFINITY ? 0.f : m_new;
      float sum = 0.f;
      unsigned pk[KPT / 2];
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float p0 = fast_exp2(v[i] - base), p1 = fast_exp2(v[i + 1] - base);
        sum += p0 + p1;
        pk[i / 2] = pack_bf16(p0, p1);
      }
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
      l_run = l_run * alpha + sum;
      if (tid % TPR == 0) sAlpha[srow] = m_new == m_run ? 1.f : alpha;
      m_run = m_new;
#pragma unroll
      for (int i = 0; i < KPT / 2; i += 2)
        *reinterpret_cast<uint2*>(sP + (size_t)srow * LT_PLD + skey + 2 * i) = make_uint2(pk[i], pk[i + 1]);
    }
    __syncthreads();

    // ---- O += P V on this warp's columns
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = sAlpha[m * 16 + g], a1 = sAlpha[m * 16 + g + 8];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int c = 0; c < CB; ++c)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            o[m][c][n][0] *= a0; o[m][c][n][1] *= a0; o[m][c][n][2] *= a1; o[m][c][n][3] *= a1;
          }
      }
    }
    if (warp * CB * 16 < a.rank) {
      const __nv_bfloat16* vr = tk + (size_t)((lane & 7) + (((lane >> 3) & 1) << 3)) * ld + (lane >> 4) * 8 + warp * CB * 16;
#pragma unroll
      for (int kk = 0; kk < LT_KEYS / 16; ++kk) {
        unsigned pa[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          ldsm_x4(pa[m], sP + (size_t)(m * 16 + (lane & 15)) * LT_PLD + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int c = 0; c < CB; ++c) {
          if ((warp * CB + c) * 16 < a.rank) {
            unsigned vf[4];
            ldsm_x4_t(vf, vr + (size_t)kk * 16 * ld + c * 16);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma16816(o[m][c][0], pa[m], vf[0], vf[1]);
              mma16816(o[m][c][1], pa[m], vf[2], vf[3]);
            }
          }
        }
      }
    }
  }
  cp_async_wait<0>();

  // ---- epilogue
  __syncthreads();
  float* sInv = sAlpha;
  if (tid % TPR == 0) {
    sInv[srow] = l_run > 0.f ? 1.f / l_run : 0.f;
    if (a.splits > 1 && srow < rows) {
      const size_t pi = ((size_t)blockIdx.x * RT + srow) * a.splits + split;
      a.part_ml[pi * 2] = m_run;                // log2 domain
      a.part_ml[pi * 2 + 1] = l_run;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int c = 0; c < CB; ++c)
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int col = (warp * CB + c) * 16 + n * 8 + 2 * t4;
        if (col >= a.rank) continue;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int r = m * 16 + g + 8 * h;
          if (r >= rows) continue;
          const float x = o[m][c][n][2 * h], y = o[m][c][n][2 * h + 1];
          if (a.splits == 1) {
            const float inv = sInv[r];
            *reinterpret_cast<unsigned*>(a.out + (flat0 + r) * a.ldo + col) = pack_bf16(x * inv, y * inv);
          } else {
            const size_t pi = ((size_t)blockIdx.x * RT + r) * a.splits + split;
            *reinterpret_cast<float2*>(a.part_o + pi * a.rank + col) = make_float2(x, y);
          }
        }
      }
}

// out row = sum_s o_s 2^(m_s - m) / sum_s l_s 2^(m_s - m), splits ascending; a block per row
__global__ void __launch_bounds__(128) latent_merge_kernel(LatentAttnArgs a, int rt) {
  pdl_wait();
  const int tile = blockIdx.x, r = blockIdx.y;
  const int seg = a.tile_seg[tile], row0 = a.tile_row[tile];
  const int seg_begin = a.seg_q_start[seg];
  if (r >= (a.seg_q_start[seg + 1] - seg_begin) * a.nq - row0) return;
  const size_t base = ((size_t)tile * rt + r) * a.splits;
  float m = -INFINITY;
  for (int s = 0; s < a.splits; ++s) m = fmaxf(m, a.part_ml[(base + s) * 2]);
  float l = 0.f;
  for (int s = 0; s < a.splits; ++s) {
    const float ms = a.part_ml[(base + s) * 2];
    l += ms == -INFINITY ? 0.f : a.part_ml[(base + s) * 2 + 1] * fast_exp2(ms - m);
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  __nv_bfloat16* out = a.out + ((long long)seg_begin * a.nq + row0 + r) * a.ldo;
  for (int c = threadIdx.x * 4; c < a.rank; c += blockDim.x * 4) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < a.splits; ++s) {
      const float ms = a.part_ml[(base + s) * 2];
      if (ms == -INFINITY) continue;
      const float f = fast_exp2(ms - m);
      const float4 v = *reinterpret_cast<const float4*>(a.part_o + (base + s) * a.rank + c);
      acc.x += v.x * f; acc.y += v.y * f; acc.z += v.z * f; acc.w += v.w * f;
    }
    *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16(acc.x * inv, acc.y * inv), pack_bf16(acc.z * inv, acc.w * inv));
  }
}

static size_t latent_smem(int d, int mt, int stages) {
  const size_t ld = ((d + 15) & ~15) + 8, rt = 16 * mt;
  return (rt * ld + stages * LT_KEYS * ld + rt * LT_PLD) * 2 + (4 * rt * LT_KEYS + rt) * 4;
}

template <int CB, int MT>
int launch_latent(const LatentAttnArgs& a, int tiles, cudaStream_t stream) {
  const size_t smem = latent_smem(a.d, MT, a.stages);
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<CB, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  cudaError_t e = launch_pdl(attn_latent_kernel<CB, MT>, dim3(tiles, a.splits), dim3(LT_THREADS), smem, stream, a);
  return e == cudaSuccess ? FT_OK : (int)e;
}

template <int MT>
int launch_latent_by_rank(const LatentAttnArgs& a, int tiles, cudaStream_t stream) {
  if (a.rank <= 128) return launch_latent<1, MT>(a, tiles, stream);
  if (a.rank <= 256) return launch_latent<2, MT>(a, tiles, stream);
  if (a.rank <= 512) return launch_latent<4, MT>(a, tiles, stream);
  return launch_latent<8, MT>(a, tiles, stream);
}

constexpr size_t LT_SMEM_MAX = 227 * 1024;

}  // namespace ft

using namespace ft;

extern "C" {

// Stages of the key ring and CTAs per SM for rows of d values and row tiles of 16 * mt (0: does not fit).
int ft_attn_latent_stages(int d, int mt) {
  for (int s = 3; s >= 1; --s)
    if (latent_smem(d, mt, s) <= LT_SMEM_MAX) return s;
  return 0;
}
int ft_attn_latent_ctas_per_sm(int d, int mt) {
  const int s = ft_attn_latent_stages(d, mt);
  if (s == 0) return 0;
  const int by_smem = (int)((size_t)(228 * 1024) / (latent_smem(d, mt, s) + 1024));
  return by_smem < 1 ? 1 : (by_smem > 2 ? 2 : by_smem);
}

// bfloat16; d and rank multiples of 8, rank <= d <= 1024; mt 1 or 2 (row tiles of 16 or 32 flat rows, as
// listed in tile_seg / tile_row); window <= 0: none.  part_o / part_ml are needed when splits > 1.
int ft_attn_latent(const void* q, void* out, long long ldo, float* part_o, float* part_ml, const void* pages,
                   const int* tile_seg, const int* tile_row, const int* seg_q_start, const int* seg_pos0,
                   const int* block_table, long long page_stride, int nq, int d, int rank, int P, int table_width,
                   int window, int tiles, int mt, int splits, int split_keys, float scale, cudaStream_t stream) {
  if (tiles <= 0) return FT_OK;
  if ((d & 7) || (rank & 7) || rank <= 0 || rank > d || d > 1024 || (mt != 1 && mt != 2) || splits < 1 ||
      split_keys < LT_KEYS || split_keys % LT_KEYS || (ldo & 7) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15) ||
      ((uintptr_t)pages & 15) || (page_stride & 7) || P <= 0 || (splits > 1 && (!part_o || !part_ml)))
    return FT_ERR_SHAPE;
  const int stages = ft_attn_latent_stages(d, mt);
  if (stages == 0) return FT_ERR_SHAPE;
  LatentAttnArgs a{(const __nv_bfloat16*)q, (__nv_bfloat16*)out, part_o, part_ml, (const __nv_bfloat16*)pages,
                   tile_seg, tile_row, seg_q_start, seg_pos0, block_table, page_stride, ldo, nq, d, rank, P,
                   table_width, window, splits, split_keys, stages, scale * 1.4426950408889634f};
  const int rc = mt == 1 ? launch_latent_by_rank<1>(a, tiles, stream) : launch_latent_by_rank<2>(a, tiles, stream);
  if (rc != FT_OK) return rc;
  if (splits > 1) launch_pdl(latent_merge_kernel, dim3(tiles, 16 * mt), dim3(128), 0, stream, a, 16 * mt);
  FT_LAUNCH_CHECK();
  return FT_OK;
}

}  // extern "C"
