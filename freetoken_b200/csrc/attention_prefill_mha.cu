// Prompt attention over keys and values that lie in plain rows instead of cache pages, with a key of
// two parts: `dk` values of the head's own and `rot` values that all heads share.  This is latent
// attention in its expanded form: for a prompt portion it is cheaper to make every head's keys and
// values from the cached latents once (one library product per layer) and to score dk + rot values than
// to score the whole latent for every head.
//
//   latent_gather   cached rows [latent | rotated key part] of the portions' contexts -> plain rows
//   (library)       rows x [Wuk ; Wuv]^T -> [rows, heads * dk | heads * dv]
//   attn_prefill_mha  causal softmax((q . k + q_rot . k_rot) scale) v on tcgen05
//
// attn_prefill_mha: a CTA owns 128 query tokens of one segment and one head and walks the key tiles of
// 64 rows from the first visible key to its diagonal.  Roles, barriers and the softmax are those of
// attention_prefill_tc.cu (S = Q K^T into one of two TMEM buffers, a softmax thread per query row, P over
// S in TMEM, O += P V with P from TMEM, the next tile's S issued before this tile's O); different here:
// operands are 3-D maps over plain rows (a row past the end, and a column past a head's size, reads as
// zero, so any head size that is a multiple of 8 works), a K tile is the head's blocks of 64 columns
// followed by the shared part's, and the V ring has one or two stages, whichever lets two CTAs share an SM.
//
// Every mbarrier wait is bounded (about two seconds): on expiry the CTA writes a code into `status`,
// stops issuing work, waits (bounded) for its copies, frees its TMEM and returns.
//
// Reference: tiled extend kernel, python/freetoken/kernel/triton/attention.py:469-758.
#include <cuda.h>

#include <cstring>

#include "common.cuh"
#include "mma_utils.cuh"
#include "tcgen05.cuh"

namespace ft {

constexpr int MQ = 128;                 // query rows per CTA (UMMA M)
constexpr int MK = 64;                  // keys per tile
constexpr int MQB = MQ * 128;           // bytes of one 64-column block of Q
constexpr int MKB = MK * 128;           // bytes of one 64-column block of K or V
constexpr int MHA_BARRIERS = 16;

struct MhaArgs {
  __nv_bfloat16* out;        // [T, heads * dv]
  const int* tile_seg;       // [tiles]
  const int* tile_q0;        // [tiles] first token of the tile inside its segment
  const int* tile_row0;      // [tiles] plain row of the segment's key 0 (may be negative: see window)
  const int* seg_q_start;
  const int* seg_pos0;
  int* status;
  int heads, dk, rot, dv, window;
  int kblocks, rblocks, vblocks, vstages;
  float scale_log2;
};

__global__ void __launch_bounds__(192, 2) attn_prefill_mha_kernel(const __grid_constant__ CUtensorMap tm_q,
                                                                  const __grid_constant__ CUtensorMap tm_k,
                                                                  const __grid_constant__ CUtensorMap tm_r,
                                                                  const __grid_constant__ CUtensorMap tm_v, MhaArgs a) {
  // no static shared memory: the dynamic part then starts on the 1,024-byte boundary that the swizzle needs,
  // and no byte is lost to rounding (two CTAs share an SM's 228 KB)
  extern __shared__ __align__(1024) unsigned char sm[];
  const int nb = a.kblocks + a.rblocks, vs = a.vstages;
  const int k_bytes = nb * MKB, v_bytes = a.vblocks * MKB;
  unsigned char* sQ = sm;
  unsigned char* sKr = sQ + nb * MQB;                  // K ring [2]
  unsigned char* sVr = sKr + 2 * k_bytes;              // V ring [vs]
  unsigned long long* bars = reinterpret_cast<unsigned long long*>(sVr + vs * v_bytes);
  unsigned long long *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7,
                     *s_full = bars + 9, *p_full = bars + 11, *pv_done = bars + 13;
  unsigned* tmem_slot = reinterpret_cast<unsigned*>(bars + 14);
  volatile int* gave_up = reinterpret_cast<volatile int*>(bars + 15);
  constexpr unsigned TMEM_COLS = 256u;                 // O: up to 128 columns, then S/P: 2 x 64

  if (smem_u32(sm) & 1023u) {                          // cannot happen with the layout above; checked, not assumed
    if (threadIdx.x == 0) atomicCAS(a.status, 0, FT_ST_MHA_SMEM_BASE);
    return;
  }
  const int tile_index = gridDim.x - 1 - blockIdx.x;   // backwards: most keys first
  const int q0 = a.tile_q0[tile_index], seg = a.tile_seg[tile_index], row0 = a.tile_row0[tile_index];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y;
  const int seg_begin = a.seg_q_start[seg];
  const int rows = min(MQ, a.seg_q_start[seg + 1] - seg_begin - q0);
  const int tok0 = seg_begin + q0;
  const int pos_first = a.seg_pos0[seg] + q0;
  const int tile0 = first_visible(pos_first, a.window, 0) / MK;
  const int ntiles = (pos_first + rows - 1) / MK + 1 - tile0;

  if (threadIdx.x == 0) {
    *gave_up = 0;
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 4);
    }
    mbar_init(pv_done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)),
                 "r"(TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const unsigned tmem_base = *tmem_slot;
  const unsigned tmem_o = tmem_base, tmem_s = tmem_base + 128;

  if (warp == 0) {
    if (lane == 0) {
      const int qcol = head * (a.dk + a.rot);
      mbar_expect_tx(q_full, nb * MQB);
      for (int b = 0; b < nb; ++b)
        tma_load_2d(sQ + b * MQB, &tm_q, b < a.kblocks ? qcol + b * 64 : qcol + a.dk + (b - a.kblocks) * 64, tok0, q_full);
      // K runs one tile ahead of V: K_j is wanted a whole softmax earlier than V_j
      int k_issued = 0, v_issued = 0;
      for (int j = 0; j <= ntiles; ++j) {
        if (j < ntiles) {
          const int s = j & 1;
          if (!mbar_wait(&k_empty[s], (((unsigned)j >> 1) & 1u) ^ 1u, gave_up)) {
            atomicCAS(a.status, 0, FT_ST_MHA_PRODUCER);
            *gave_up = 1;
            break;
          }
          const int row = row0 + (tile0 + j) * MK;
          mbar_expect_tx(&k_full[s], k_bytes);
          for (int b = 0; b < a.kblocks; ++b)
            tma_load_3d(sKr + s * k_bytes + b * MKB, &tm_k, b * 64, head, row, &k_full[s]);
          for (int b = 0; b < a.rblocks; ++b)
            tma_load_2d(sKr + s * k_bytes + (a.kblocks + b) * MKB, &tm_r, b * 64, row, &k_full[s]);
          ++k_issued;
        }
        if (j > 0) {
          const int i = j - 1, s = i % vs;
          if (!mbar_wait(&v_empty[s], (((unsigned)(i / vs)) & 1u) ^ 1u, gave_up)) {
            atomicCAS(a.status, 0, FT_ST_MHA_PRODUCER);
            *gave_up = 1;
            break;
          }
          const int row = row0 + (tile0 + i) * MK;
          mbar_expect_tx(&v_full[s], v_bytes);
          for (int b = 0; b < a.vblocks; ++b)
            tma_load_3d(sVr + s * v_bytes + b * MKB, &tm_v, b * 64, head, row, &v_full[s]);
          ++v_issued;
        }
      }
      if (*gave_up) {
        // let copies already in flight land before the CTA (and its shared memory) goes away
        const unsigned long long start = global_ns();
        while (!mbar_try(q_full, 0) && global_ns() - start < 100000000ull) {}
        for (int j = k_issued > 2 ? k_issued - 2 : 0; j < k_issued; ++j) {
          const unsigned long long t0 = global_ns();
          while (!mbar_try(&k_full[j & 1], ((unsigned)j >> 1) & 1u) && global_ns() - t0 < 100000000ull) {}
        }
        for (int j = v_issued > vs ? v_issued - vs : 0; j < v_issued; ++j) {
          const unsigned long long t0 = global_ns();
          while (!mbar_try(&v_full[j % vs], (unsigned)(j / vs) & 1u) && global_ns() - t0 < 100000000ull) {}
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // instruction descriptors: D f32, A/B bf16, M = 128; S: N = 64, both K-major; O: N = whole blocks of
      // 64 value columns (those past dv hold zeros), B (= V) MN-major
      const unsigned n_o = (unsigned)(a.vblocks * 64);
      const unsigned idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(MK >> 3) << 17) |
                               ((unsigned)(MQ >> 4) << 24);
      const unsigned idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((n_o >> 3) << 17) |
                               ((unsigned)(MQ >> 4) << 24);
      bool ok = mbar_wait(q_full, 0, gave_up);
      if (!ok) { atomicCAS(a.status, 0, FT_ST_MHA_MMA_Q); *gave_up = 1; }
      const unsigned sQa = smem_u32(sQ);
      const int ksteps = (a.dk + 15) >> 4, rsteps = (a.rot + 15) >> 4;
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1;
        if (!mbar_wait(&k_full[s], ((unsigned)j >> 1) & 1u, gave_up)) {
          atomicCAS(a.status, 0, FT_ST_MHA_MMA_K);
          *gave_up = 1;
          return false;
        }
        tc_fence_after();
        const unsigned sK = smem_u32(sKr + s * k_bytes);
        for (int kk = 0; kk < ksteps + rsteps; ++kk) {
          const int step = kk < ksteps ? kk : kk - ksteps;
          const unsigned block = (unsigned)((kk < ksteps ? 0 : a.kblocks) + (step >> 2)), in = (unsigned)(step & 3) * 32u;
          tc_mma(tmem_s + (unsigned)(s * MK), sw128_desc(sQa + block * MQB + in), sw128_desc(sK + block * MKB + in),
                 idesc_s, kk > 0);
        }
        tc_commit(&s_full[s]);
        tc_commit(&k_empty[s]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        const int s = j & 1, v = j % vs;
        // the next tile's S goes first: it runs under this tile's softmax.  Its buffer held P of tile j-1,
        // read by an O product issued before it (MMAs run in order)
        if (j + 1 < ntiles && !issue_s(j + 1)) break;
        if (!mbar_wait(&p_full[s], ((unsigned)j >> 1) & 1u, gave_up) ||
            !mbar_wait(&v_full[v], (unsigned)(j / vs) & 1u, gave_up)) {
          atomicCAS(a.status, 0, FT_ST_MHA_MMA_PV);
          *gave_up = 1;
          break;
        }
        tc_fence_after();
        const unsigned sV = smem_u32(sVr + v * v_bytes);
#pragma unroll
        for (int kk = 0; kk < MK / 16; ++kk)
          tc_mma_ts(tmem_o, tmem_s + (unsigned)(s * MK + kk * 8), sw128_mn_desc(sV + kk * 16 * 128, MKB, 1024),
                    idesc_o, (j | kk) != 0);
        tc_commit(&v_empty[v]);
        tc_commit(pv_done);
      }
    }
  } else {
    // softmax: TMEM lane = query row; this warp may touch lanes 32*(warp%4) .. +31
    const int lane_base = (warp & 3) * 32;
    const int r = lane_base + lane;
    const int my_pos = pos_first + r;
    const unsigned lane_bits = (unsigned)lane_base << 16;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    const int my_lo = first_visible(my_pos, a.window, 0);
    const int last_lo = first_visible(pos_first + rows - 1, a.window, 0);      // no row's first key lies later
    for (int j = 0; j < ntiles; ++j) {
      const unsigned tmem_sj = tmem_s + (unsigned)((j & 1) * MK) + lane_bits;
      ok = mbar_wait(&s_full[j & 1], ((unsigned)j >> 1) & 1u, gave_up);
      if (!ok && lane == 0) { atomicCAS(a.status, 0, FT_ST_MHA_SOFTMAX_S); *gave_up = 1; }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      tc_fence_after();
      unsigned lo[32], hi[32];
      tc_ld32(tmem_sj, lo);
      tc_ld32(tmem_sj + 32, hi);
      tc_ld_wait();
      const int key0 = (tile0 + j) * MK;
      if (key0 < last_lo) {
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          if (key0 + c < my_lo) lo[c] = 0xff800000u;
          if (key0 + 32 + c < my_lo) hi[c] = 0xff800000u;
        }
      }
      if (key0 + MK - 1 > pos_first) {
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          if (key0 + c > my_pos) lo[c] = 0xff800000u;
          if (key0 + 32 + c > my_pos) hi[c] = 0xff800000u;
        }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 32; ++c)
        mx4[c & 3] = fmaxf(mx4[c & 3], fmaxf(__uint_as_float(lo[c]), __uint_as_float(hi[c])));
      const float cand = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * a.scale_log2;
      // the running max only moves when it would grow by more than 2^8 (see attention_prefill_tc.cu)
      const float m_new = cand > m + 8.f ? cand : m;
      if (j > 0 && __any_sync(0xffffffffu, m_new != m)) {
        ok = mbar_wait(pv_done, (unsigned)(j - 1) & 1u, gave_up);
        if (!ok && lane == 0) { atomicCAS(a.status, 0, FT_ST_MHA_SOFTMAX_PV); *gave_up = 1; }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        tc_fence_after();
        const float alpha = (m == -INFINITY) ? 0.f : fast_exp2(m - m_new);
#pragma unroll 1
        for (int c0 = 0; c0 < a.dv; c0 += 32) {
          unsigned o[32];
          tc_ld32(tmem_o + lane_bits + c0, o);
          tc_ld_wait();
#pragma unroll
          for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
          tc_st32(tmem_o + lane_bits + c0, o);
        }
        tc_st_wait();
        l *= alpha;
      }
      m = m_new;
      const float neg_m = (m_new == -INFINITY) ? 0.f : -m_new;
      const float2 sc2 = make_float2(a.scale_log2, a.scale_log2), nm2 = make_float2(neg_m, neg_m);
      float2 sum2[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      unsigned pk[32];
#pragma unroll
      for (int c = 0; c < 16; ++c) {
        const float2 x0 = __ffma2_rn(make_float2(__uint_as_float(lo[2 * c]), __uint_as_float(lo[2 * c + 1])), sc2, nm2);
        const float2 x1 = __ffma2_rn(make_float2(__uint_as_float(hi[2 * c]), __uint_as_float(hi[2 * c + 1])), sc2, nm2);
        const float2 p01 = make_float2(fast_exp2(x0.x), fast_exp2(x0.y));
        const float2 p23 = make_float2(fast_exp2(x1.x), fast_exp2(x1.y));
        sum2[c & 3] = __fadd2_rn(sum2[c & 3], __fadd2_rn(p01, p23));
        pk[c] = pack_bf16(p01.x, p01.y);
        pk[16 + c] = pack_bf16(p23.x, p23.y);
      }
      const float2 s01 = __fadd2_rn(__fadd2_rn(sum2[0], sum2[1]), __fadd2_rn(sum2[2], sum2[3]));
      tc_st32(tmem_sj, pk);
      tc_st_wait();
      l += s01.x + s01.y;
      if (j == ntiles - 1 && j > 0) {
        // pins the phase of pv_done before the final wait (attention_prefill_tc.cu says why)
        ok = mbar_wait(pv_done, (unsigned)(j - 1) & 1u, gave_up);
        if (!ok && lane == 0) { atomicCAS(a.status, 0, FT_ST_MHA_SOFTMAX_PV); *gave_up = 1; }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    if (ok) {
      ok = mbar_wait(pv_done, (unsigned)(ntiles - 1) & 1u, gave_up);
      if (!ok && lane == 0) { atomicCAS(a.status, 0, FT_ST_MHA_SOFTMAX_LAST); *gave_up = 1; }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
    }
    if (ok) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = a.out + ((size_t)(tok0 + r) * a.heads + head) * a.dv;
#pragma unroll 1
      for (int c0 = 0; c0 < a.dv; c0 += 32) {
        unsigned o[32];
        tc_ld32(tmem_o + lane_bits + c0, o);
        tc_ld_wait();
        if (r < rows) {
#pragma unroll
          for (int c = 0; c < 32; c += 8) {
            if (c0 + c >= a.dv) continue;
            uint4 v;
            v.x = pack_bf16(__uint_as_float(o[c]) * inv, __uint_as_float(o[c + 1]) * inv);
            v.y = pack_bf16(__uint_as_float(o[c + 2]) * inv, __uint_as_float(o[c + 3]) * inv);
            v.z = pack_bf16(__uint_as_float(o[c + 4]) * inv, __uint_as_float(o[c + 5]) * inv);
            v.w = pack_bf16(__uint_as_float(o[c + 6]) * inv, __uint_as_float(o[c + 7]) * inv);
            *reinterpret_cast<uint4*>(orow + c0 + c) = v;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
  }
}

// Cached rows of d values -> plain rows.  Eight blocks (a warp per row) copy the 64 rows of keys key0[b] .. of segment
// seg[b] to plain rows row0[b] ..; keys the segment does not have, and keys before the first that
// its first token sees (their pages may be another request's by now), become zeros.
__global__ void __launch_bounds__(256) latent_gather_kernel(const __nv_bfloat16* __restrict__ pages,
                                                            __nv_bfloat16* __restrict__ dst, const int* __restrict__ seg,
                                                            const int* __restrict__ key0, const int* __restrict__ row0,
                                                            const int* __restrict__ seg_kv_len,
                                                            const int* __restrict__ seg_pos0,
                                                            const int* __restrict__ block_table, long long page_stride,
                                                            int d, int P, int table_width, int window) {
  pdl_wait();
  const int s = seg[blockIdx.x], k0 = key0[blockIdx.x], r0 = row0[blockIdx.x];
  const int len = seg_kv_len[s], lo = first_visible(seg_pos0[s], window, 0);
  const int* table = block_table + (size_t)s * table_width;
  const int chunks = d >> 3;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  {
    const int r = blockIdx.y * 8 + warp;               // a warp per row
    const int j = k0 + r;
    const __nv_bfloat16* src = j >= lo && j < len ? pages + (size_t)table[j / P] * page_stride + (size_t)(j % P) * d : nullptr;
    for (int c = lane; c < chunks; c += 32) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (src) v = *reinterpret_cast<const uint4*>(src + c * 8);
      *reinterpret_cast<uint4*>(dst + (size_t)(r0 + r) * d + c * 8) = v;
    }
  }
}

typedef CUresult (*MhaEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static MhaEncodeFn mha_encode() {
  static MhaEncodeFn fn = nullptr;
  if (!fn) {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = (MhaEncodeFn)p;
  }
  return fn;
}

constexpr size_t MHA_SM_SHARED = 228 * 1024, MHA_CTA_RESERVED = 1024, MHA_CTA_MAX = 227 * 1024;
static size_t mha_smem(int nb, int vblocks, int vstages) {
  return (size_t)nb * MQB + 2 * (size_t)nb * MKB + (size_t)vstages * vblocks * MKB + MHA_BARRIERS * 8;
}
// two V stages, unless one lets two CTAs share an SM and two do not
static int mha_vstages(int nb, int vblocks) {
  const bool two = 2 * (mha_smem(nb, vblocks, 2) + MHA_CTA_RESERVED) <= MHA_SM_SHARED;
  const bool one = 2 * (mha_smem(nb, vblocks, 1) + MHA_CTA_RESERVED) <= MHA_SM_SHARED;
  return !two && one ? 1 : 2;
}

}  // namespace ft

using namespace ft;

extern "C" {

// Tensor map over bfloat16 rows: `heads` = 0: 2-D [rows, cols], boxes of `box_rows` rows by 64 columns; else
// 3-D [rows, heads, cols] with heads `head_stride` elements apart, boxes of box_rows rows of one head by 64
// columns.  Columns past `cols` and rows past `rows` read as zeros.  `out` receives 128 bytes.
int ft_mha_map(void* out, const void* base, long long rows, long long cols, long long heads, long long row_stride,
               long long head_stride, int box_rows) {
  MhaEncodeFn fn = mha_encode();
  if (!fn) return -201;
  if ((row_stride & 7) || (head_stride & 7) || ((uintptr_t)base & 15) || rows <= 0 || cols <= 0 ||
      (box_rows != MQ && box_rows != MK))
    return FT_ERR_SHAPE;
  CUtensorMap map;
  const int dims_n = heads ? 3 : 2;
  cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)(heads ? heads : rows), (cuuint64_t)rows};
  cuuint64_t strides[2] = {(cuuint64_t)(heads ? head_stride : row_stride) * 2, (cuuint64_t)row_stride * 2};
  cuuint32_t box[3] = {64, (cuuint32_t)(heads ? 1 : box_rows), (cuuint32_t)box_rows};
  cuuint32_t es[3] = {1, 1, 1};
  CUresult rc = fn(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, dims_n, (void*)base, dims, strides, box, es,
                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (rc != CUDA_SUCCESS) return -202;
  memcpy(out, &map, sizeof(map));
  return FT_OK;
}

int ft_latent_gather(const void* pages, void* dst, const int* seg, const int* key0, const int* row0,
                     const int* seg_kv_len, const int* seg_pos0, const int* block_table, long long page_stride, int d,
                     int P, int table_width, int window, int blocks, cudaStream_t stream) {
  if (blocks <= 0) return FT_OK;
  if (d <= 0 || (d & 7) || (page_stride & 7) || ((uintptr_t)pages & 15) || ((uintptr_t)dst & 15) || P <= 0)
    return FT_ERR_SHAPE;
  launch_pdl(latent_gather_kernel, dim3(blocks, MK / 8), dim3(256), 0, stream, (const __nv_bfloat16*)pages,
             (__nv_bfloat16*)dst, seg, key0, row0, seg_kv_len, seg_pos0, block_table, page_stride, d, P, table_width,
             window);
  FT_LAUNCH_CHECK();
  return FT_OK;
}

// bfloat16.  Query rows [T, heads * (dk + rot)] through map_q (boxes of 128 rows), keys and values through
// 3-D maps over plain rows, the shared key part through a 2-D one (boxes of 64 rows; unused when rot = 0).
// dk, rot, dv multiples of 8; the blocks of 64 columns of dk and of rot together at most 4, dv at most 128.
int ft_attn_prefill_mha(const void* map_q, const void* map_k, const void* map_r, const void* map_v, void* out,
                        const int* tile_seg, const int* tile_q0, const int* tile_row0, const int* seg_q_start,
                        const int* seg_pos0, int* status, int heads, int dk, int rot, int dv, int window, int tiles,
                        float scale, cudaStream_t stream) {
  if (tiles <= 0) return FT_OK;
  const int kb = (dk + 63) / 64, rb = (rot + 63) / 64, vb = (dv + 63) / 64;
  if (heads <= 0 || heads > 65535 || dk <= 0 || rot < 0 || dv <= 0 || (dk & 7) || (rot & 7) || (dv & 7) || kb + rb > 4 ||
      vb > 2 || ((uintptr_t)out & 15))
    return FT_ERR_SHAPE;
  CUtensorMap mq, mk, mr, mv;
  memcpy(&mq, map_q, sizeof(mq));
  memcpy(&mk, map_k, sizeof(mk));
  memcpy(&mr, rot ? map_r : map_k, sizeof(mr));
  memcpy(&mv, map_v, sizeof(mv));
  const int vs = mha_vstages(kb + rb, vb);
  const size_t smem = mha_smem(kb + rb, vb, vs);
  if (smem > MHA_CTA_MAX) return FT_ERR_SHAPE;
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_prefill_mha_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  MhaArgs a{(__nv_bfloat16*)out, tile_seg, tile_q0, tile_row0, seg_q_start, seg_pos0, status, heads, dk, rot, dv,
            window, kb, rb, vb, vs, scale * 1.4426950408889634f};
  attn_prefill_mha_kernel<<<dim3(tiles, heads), 192, smem, stream>>>(mq, mk, mr, mv, a);
  FT_LAUNCH_CHECK();
  return FT_OK;
}

}  // extern "C"
