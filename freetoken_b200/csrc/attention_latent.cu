// Attention over cached latent rows: every query head reads ONE row of d values per key, whose first
// `rank` values are also the value (absorbed latent attention, rows of any width up to 1,024).
//
// Queries are the rows of [T * nq, d] (token-major, then head).  A CTA owns RT = 16 * MT consecutive
// rows of one segment - the heads of a decoded token, or of a few neighbouring tokens of a short prompt
// portion - and one split of the keys, and walks key tiles of 64 rows, each fetched ONCE (cp.async in 16-byte
// pieces into padded shared-memory rows, up to three stages; pages of any size) and used twice: as keys and,
// its first `rank` columns, as values.
//
//   warps 8-11   producers: 16 rows of every tile each; a row's page is looked up one tile ahead (the
//                lookup's latency, not the copies, was most of a tile's time when the other warps did it)
//   warps 0-7    S[RT, 64] = Q K^T: two groups of 32 keys x four interleaved quarters of d, Q's fragments in
//                registers (re-read from shared memory they cost as much bandwidth as the keys); partial
//                products of mma.sync m16n8k16 are left in shared memory (float32)
//                softmax: RT rows x 64 keys spread over the 256 threads: the four partial scores are added
//                in order, scaled, masked by absolute position; running max and sum in float32 per row; P
//                rounded to bfloat16 into shared memory
//                O[RT, rank] += P V: a warp owns CB blocks of 16 value columns for all 64 keys
//                (ldmatrix.trans on the same tile), accumulators in registers
// Every mbarrier wait is bounded (about two seconds): on expiry the CTA leaves a code in `status`, waits
// (bounded) for its copies and returns.
// With splits > 1 every CTA leaves an unnormalised partial (o, max, sum); latent_merge combines the
// splits in ascending order.
//
// The reference has no latent attention; its split-KV decode kernel
// (python/freetoken/kernel/triton/attention.py:147-349) is the pattern of the splits.
#include "common.cuh"
#include "mma_utils.cuh"
#include "tcgen05.cuh"

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
  int* status;
  long long page_stride, ldo;
  int nq, d, rank, P, table_width, window, splits, split_keys, stages;
  float scale_log2;
};

constexpr int LT_KEYS = 64, LT_PLD = LT_KEYS + 8, LT_SLD = LT_KEYS + 8, LT_STAGES = 3, LT_THREADS = 384, LT_PRODUCERS = 128;

// Arrives on `bar` when this thread's copies so far have landed.
__device__ __forceinline__ void cp_async_arrive(unsigned long long* bar) {
  asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}

// The consumer warps' own barrier, and the same with a vote.
__device__ __forceinline__ void consumer_sync() { asm volatile("barrier.cta.sync.aligned 1, 256;" ::: "memory"); }
__device__ __forceinline__ bool consumer_sync_and(bool mine) {
  unsigned all;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\t"
               "barrier.cta.red.and.pred.aligned q, 1, 256, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
               : "=r"(all) : "r"((unsigned)mine) : "memory");
  return all != 0;
}

// NKS: k-steps of 16 a quarter owns (rows are filled up with zeros to 64 * NKS values in shared memory, so that
// no step needs a guard); CB: blocks of 16 value columns a warp owns
template <int NKS, int CB, int MT>
__global__ void __launch_bounds__(LT_THREADS) attn_latent_kernel(LatentAttnArgs a) {
  constexpr int RT = 16 * MT;
  constexpr int TPR = 256 / RT;                // threads per row in the softmax
  constexpr int KPT = LT_KEYS / TPR;           // keys per thread there (4 or 8)
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int dp = 64 * NKS, ld = dp + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);            // [RT][ld]
  __nv_bfloat16* sK = sQ + RT * ld;                                          // [stages][64][ld]
  __nv_bfloat16* sP = sK + (size_t)a.stages * LT_KEYS * ld;                  // [RT][72]
  float* sS = reinterpret_cast<float*>(sP + RT * LT_PLD);                    // [4 quarters][RT][72]
  float* sAlpha = sS + 4 * RT * LT_SLD;                                      // [RT]
  __shared__ __align__(8) unsigned long long full[LT_STAGES], empty[LT_STAGES];
  __shared__ int gave_up;
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

  if (tid == 0) {
    gave_up = 0;
    for (int s = 0; s < LT_STAGES; ++s) {
      mbar_init(&full[s], LT_PRODUCERS);
      mbar_init(&empty[s], 8);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  // the fill of every row counts as zeros, of a key row too (a copy never writes it)
  for (int r = warp; r < RT + a.stages * LT_KEYS; r += LT_THREADS / 32)
    for (int c = chunks + lane; c < dp / 8; c += 32)
      *reinterpret_cast<uint4*>((r < RT ? sQ + r * ld : sK + (size_t)(r - RT) * ld) + c * 8) = make_uint4(0u, 0u, 0u, 0u);
  for (int r = warp; r < RT; r += LT_THREADS / 32)
    for (int c = lane; c < chunks; c += 32) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < rows) v = *reinterpret_cast<const uint4*>(a.q + (flat0 + r) * a.d + c * 8);
      *reinterpret_cast<uint4*>(sQ + r * ld + c * 8) = v;
    }
  __syncthreads();

  if (warp >= 8) {
    // 16 rows a warp, four at a time: eight lanes a row, 128 bytes of it per copy instruction.  Rows outside
    // the visible keys repeat a valid one (masked later)
    const int row = (warp - 8) * 16 + (lane >> 3), piece = lane & 7;
    auto key_of = [&](int tile, int i) { return min(max(k_begin + tile * LT_KEYS + row + 4 * i, k_lo), pos_last); };
    int page[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) page[i] = ntiles > 0 ? table[key_of(0, i) / a.P] : 0;
    for (int tile = 0; tile < ntiles; ++tile) {
      const int stage = tile % a.stages;
      const __nv_bfloat16* src[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        src[i] = a.pages + (size_t)page[i] * a.page_stride + (size_t)(key_of(tile, i) % a.P) * a.d;
        if (tile + 1 < ntiles) page[i] = table[key_of(tile + 1, i) / a.P];      // not used before the next round
      }
      bool ok = mbar_wait(&empty[stage], ((unsigned)(tile / a.stages) & 1u) ^ 1u, &gave_up);
      if (!__all_sync(0xffffffffu, ok)) {
        if (lane == 0) atomicCAS(a.status, 0, FT_ST_LATENT_PRODUCER);
        gave_up = 1;
        break;
      }
      __nv_bfloat16* dst = sK + ((size_t)stage * LT_KEYS + row) * ld;
#pragma unroll 3
      for (int c = piece; c < chunks; c += 8) {
#pragma unroll
        for (int i = 0; i < 4; ++i) cp_async16(dst + 4 * i * ld + c * 8, src[i] + c * 8);
      }
      cp_async_arrive(&full[stage]);
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    return;
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
  unsigned qf[MT][NKS][4];                     // this quarter's fragments of Q
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NKS; ++i)
      ldsm_x4(qf[m][i], sQ + (size_t)(m * 16 + (lane & 15)) * ld + (lane >> 4) * 8 + (quarter + 4 * i) * 16);
  bool ok = true;

  for (int tile = 0; tile < ntiles; ++tile) {
    const bool landed = mbar_wait(&full[tile % a.stages], (unsigned)(tile / a.stages) & 1u, &gave_up);
    const __nv_bfloat16* tk = sK + (size_t)(tile % a.stages) * LT_KEYS * ld;

    // ---- partial scores: this group's 32 keys, every fourth k-step of 16
    {
      float s[MT][4][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) s[m][n][i] = 0.f;
      const __nv_bfloat16* kr = tk + (size_t)(kgroup * 32 + (lane & 7) + ((lane >> 4) << 3)) * ld + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int i = 0; i < NKS; ++i) {
        unsigned kf[2][4];
        ldsm_x4(kf[0], kr + (quarter + 4 * i) * 16);
        ldsm_x4(kf[1], kr + 16 * ld + (quarter + 4 * i) * 16);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 4; ++n) mma16816(s[m][n], qf[m][i], kf[n >> 1][(n & 1) * 2], kf[n >> 1][(n & 1) * 2 + 1]);
      }
      float* dst = sS + (size_t)quarter * RT * LT_SLD + kgroup * 32;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          *reinterpret_cast<float2*>(dst + (m * 16 + g) * LT_SLD + n * 8 + 2 * t4) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(dst + (m * 16 + g + 8) * LT_SLD + n * 8 + 2 * t4) = make_float2(s[m][n][2], s[m][n][3]);
        }
    }
    ok = consumer_sync_and(landed);             // all scores are there (and whether every warp saw the tile)
    if (!ok) {
      if (tid == 0) atomicCAS(a.status, 0, FT_ST_LATENT_TILE);
      gave_up = 1;
      break;
    }

    // ---- softmax of this thread's KPT keys of its row
    {
      const int j0 = k_begin + tile * LT_KEYS + skey;
      float v[KPT];
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float* src = sS + (size_t)srow * LT_SLD + skey + i;
        float2 x = *reinterpret_cast<const float2*>(src);
#pragma unroll
        for (int p = 1; p < 4; ++p) {
          const float2 y = *reinterpret_cast<const float2*>(src + (size_t)p * RT * LT_SLD);
          x.x += y.x; x.y += y.y;
        }
        v[i] = x.x; v[i + 1] = x.y;
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
      for (int i = 0; i < KPT / 2; ++i) *reinterpret_cast<unsigned*>(sP + (size_t)srow * LT_PLD + skey + 2 * i) = pk[i];
    }
    consumer_sync();

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
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[tile % a.stages]);
  }
  if (!ok) return;

  // ---- epilogue
  consumer_sync();
  float* sInv = sAlpha;
  if (tid % TPR == 0) {
    sInv[srow] = l_run > 0.f ? 1.f / l_run : 0.f;
    if (a.splits > 1 && srow < rows) {
      const size_t pi = ((size_t)blockIdx.x * RT + srow) * a.splits + split;
      a.part_ml[pi * 2] = m_run;                // log2 domain
      a.part_ml[pi * 2 + 1] = l_run;
    }
  }
  consumer_sync();
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

// k-steps of a quarter for rows of d values: the sizes the kernel is built for
static int latent_nks(int d) { return d <= 128 ? 2 : d <= 192 ? 3 : d <= 256 ? 4 : d <= 320 ? 5 : d <= 576 ? 9 : 16; }
static size_t latent_smem(int d, int mt, int stages) {
  const size_t ld = 64 * latent_nks(d) + 8, rt = 16 * mt;
  return (rt * ld + stages * LT_KEYS * ld + rt * LT_PLD) * 2 + (4 * rt * LT_SLD + rt) * 4;
}

template <int NKS, int CB, int MT>
int launch_latent(const LatentAttnArgs& a, int tiles, cudaStream_t stream) {
  const size_t smem = latent_smem(a.d, MT, a.stages);
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<NKS, CB, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  cudaError_t e = launch_pdl(attn_latent_kernel<NKS, CB, MT>, dim3(tiles, a.splits), dim3(LT_THREADS), smem, stream, a);
  return e == cudaSuccess ? FT_OK : (int)e;
}

template <int MT>
int launch_latent_by_size(const LatentAttnArgs& a, int tiles, cudaStream_t stream) {
  switch (latent_nks(a.d)) {
    case 2: return launch_latent<2, 1, MT>(a, tiles, stream);
    case 3: return a.rank <= 128 ? launch_latent<3, 1, MT>(a, tiles, stream) : launch_latent<3, 2, MT>(a, tiles, stream);
    case 4: return launch_latent<4, 2, MT>(a, tiles, stream);
    case 5: return a.rank <= 256 ? launch_latent<5, 2, MT>(a, tiles, stream) : launch_latent<5, 4, MT>(a, tiles, stream);
    case 9: if (a.rank <= 512) return launch_latent<9, 4, MT>(a, tiles, stream);
  }
  if constexpr (MT == 1) return latent_nks(a.d) == 16 ? launch_latent<16, 8, 1>(a, tiles, stream)
                                                      : launch_latent<9, 8, 1>(a, tiles, stream);
  return FT_ERR_SHAPE;
}

constexpr size_t LT_SMEM_MAX = 227 * 1024 - 64;      // beside the static part

}  // namespace ft

using namespace ft;

extern "C" {

// Stages of the key ring and CTAs per SM for rows of d values and row tiles of 16 * mt (0: does not fit).
int ft_attn_latent_stages(int d, int mt) {
  for (int s = LT_STAGES; s >= 1; --s)
    if (latent_smem(d, mt, s) <= LT_SMEM_MAX) return s;
  return 0;
}
int ft_attn_latent_ctas_per_sm(int d, int mt) {
  const int s = ft_attn_latent_stages(d, mt);
  if (s == 0) return 0;
  const int by_smem = (int)((size_t)(228 * 1024) / (latent_smem(d, mt, s) + 1024));
  return by_smem < 1 ? 1 : (by_smem > 2 ? 2 : by_smem);
}

// bfloat16; d and rank multiples of 8, rank <= d <= 1024; mt 1 or 2 (row tiles of 16 or 32 flat rows - 32
// for d <= 576 and rank <= 512 -, as listed in tile_seg / tile_row); window <= 0: none.  part_o / part_ml are needed when splits > 1.
int ft_attn_latent(const void* q, void* out, long long ldo, float* part_o, float* part_ml, const void* pages,
                   const int* tile_seg, const int* tile_row, const int* seg_q_start, const int* seg_pos0,
                   const int* block_table, int* status, long long page_stride, int nq, int d, int rank, int P,
                   int table_width, int window, int tiles, int mt, int splits, int split_keys, float scale, cudaStream_t stream) {
  if (tiles <= 0) return FT_OK;
  if ((d & 7) || (rank & 7) || rank <= 0 || rank > d || d > 1024 || (mt != 1 && mt != 2) || splits < 1 ||
      split_keys < LT_KEYS || split_keys % LT_KEYS || (ldo & 7) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15) ||
      ((uintptr_t)pages & 15) || (page_stride & 7) || P <= 0 || (splits > 1 && (!part_o || !part_ml)))
    return FT_ERR_SHAPE;
  const int stages = ft_attn_latent_stages(d, mt);
  if (stages == 0) return FT_ERR_SHAPE;
  LatentAttnArgs a{(const __nv_bfloat16*)q, (__nv_bfloat16*)out, part_o, part_ml, (const __nv_bfloat16*)pages,
                   tile_seg, tile_row, seg_q_start, seg_pos0, block_table, status, page_stride, ldo, nq, d, rank, P,
                   table_width, window, splits, split_keys, stages, scale * 1.4426950408889634f};
  const int rc = mt == 1 ? launch_latent_by_size<1>(a, tiles, stream) : launch_latent_by_size<2>(a, tiles, stream);
  if (rc != FT_OK) return rc;
  if (splits > 1) launch_pdl(latent_merge_kernel, dim3(tiles, 16 * mt), dim3(128), 0, stream, a, 16 * mt);
  FT_LAUNCH_CHECK();
  return FT_OK;
}

}  // extern "C"
