// Time mixing with a decay per key channel and a bonus for the current token (the recurrence of RWKV), and
// the mix of every token's input with the previous token's in front of it.
//
//   token_shift       out[m][t, c] = x[t, c] + (x[t-1, c] - x[t, c]) mu[m, c]   for M mixes of one input; the
//                     previous token of a segment's first token lives in the request's state slot (zeros at
//                     the start of a sequence), which takes the segment's last input afterwards
//   time_mixing_scan  per head, state S (D x P):  w_t = exp(-exp(a_t + w0)),
//                     o_t = (S + diag(u) k_t v_t^T)^T r_t,   then  S <- diag(w_t) S + k_t v_t^T
//
// Everything behind the projections is float32 whatever the activation type.  A token's result depends on its
// own request alone, and every token performs the same operations in the same order however the request was
// cut into steps.
#include "common.cuh"

namespace ft {

__device__ __forceinline__ void load_piece(const float* p, float (&v)[1]) { v[0] = p[0]; }
__device__ __forceinline__ void load_piece(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(p[0]); }
__device__ __forceinline__ void load_piece(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load_piece(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load_piece(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void store_piece(float* p, const float (&v)[1]) { p[0] = v[0]; }
__device__ __forceinline__ void store_piece(__nv_bfloat16* p, const float (&v)[1]) { p[0] = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void store_piece(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_piece(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store_piece(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = raw;
}

// ------------------------------------------------------------------ token shift
struct ShiftArgs {
  const void* x;           // [T, ldx]
  const float* mu;         // [M, W]
  void* out;               // [M, T, W]
  float* state;            // slot s: state + s * slot_stride, the last input of its request [W]
  const int* token_seg;    // [T]
  const int* seg_slot;     // [S]
  const int* seg_q_start;  // [S + 1]
  long long ldx, slot_stride;
  int T, W, M;
};

// A thread owns VEC neighbouring columns of RUN consecutive tokens: their inputs stay in registers while the
// mixes' factors are fetched one after the other, once per RUN tokens.  The thread of a segment's first token
// is the only one that reads the slot, and it alone replaces the slot's contents, after its read.
template <typename AT, int VEC, int RUN>
__global__ void __launch_bounds__(128) token_shift_kernel(ShiftArgs a) {
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= a.W) return;
  const AT* x = (const AT*)a.x;
  float cur[RUN][VEC], step[RUN][VEC];                 // x_t and x_{t-1} - x_t
  const int t0 = blockIdx.x * RUN;
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int t = t0 + i;
    if (t >= a.T) break;
    const int seg = a.token_seg[t], q0 = a.seg_q_start[seg];
    load_piece(x + (size_t)t * a.ldx + c, cur[i]);
    if (t == q0) {
      float* slot = a.state + (size_t)a.seg_slot[seg] * a.slot_stride + c;
      load_piece(slot, step[i]);
      float last[VEC];
      load_piece(x + (size_t)(a.seg_q_start[seg + 1] - 1) * a.ldx + c, last);
      store_piece(slot, last);
    } else {
      load_piece(x + (size_t)(t - 1) * a.ldx + c, step[i]);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) step[i][j] -= cur[i][j];
  }
  for (int m = 0; m < a.M; ++m) {
    float mu[VEC];
    load_piece(a.mu + (size_t)m * a.W + c, mu);
    AT* out = (AT*)a.out + ((size_t)m * a.T + t0) * a.W + c;
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      if (t0 + i >= a.T) break;
      float y[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) y[j] = fmaf(step[i][j], mu[j], cur[i][j]);
      store_piece(out + (size_t)i * a.W, y);
    }
  }
}

// ------------------------------------------------------------------------- scan
// A column of a head's state is shared by LPC lanes; lane l holds rows (LPC j + l) 4 .. + 3 for j < RPL / 4, so
// that the lanes read consecutive pieces of r, k, w (and of the state, which is kept value by value: [P][D]).  A
// warp owns 32 / LPC columns, a block of 8 warps 256 / LPC.  Tokens come in chunks of 8: every warp fetches one
// token of a later chunk into registers while the block works through the current chunk in shared memory and puts
// the next one into the other of two buffers afterwards: one barrier a chunk.  The decay's exponentials and the bonus
// u . (r k) are formed on the way into shared memory.  The read-out's partial sums of the 8 tokens are added over the
// lanes together, each lane ending with the total of one token: 8 shuffles a chunk.
constexpr int TM_WARPS = 8;
constexpr int TM_THREADS = 32 * TM_WARPS;
constexpr int TM_CHUNK = 8;
static_assert(TM_CHUNK == TM_WARPS, "a warp stages a token");

struct TimeMixArgs {
  const void *r, *k, *v;   // row t: r + t * ld, head h's D values at h * D (v: h * P)
  const float* decay;      // [T, ld_decay] a_t: channel n of head h at h * D + n
  const float *w0, *u;     // [heads * D]
  float* state;            // slot s: state + s * slot_stride, [heads][P][D]
  float* o;                // [T, heads * P]
  const int* seg_slot;
  const int* seg_q_start;
  long long ld, ld_decay, slot_stride;
  int heads, P, D, vec;    // vec: state rows may be read in 16-byte pieces
};

constexpr int time_mix_buffer(int RPL, int LPC) { return TM_CHUNK * (3 * LPC * RPL + TM_THREADS / LPC + 1); }

template <typename AT, int RPL, int LPC>
__global__ void __launch_bounds__(TM_THREADS) time_mixing_kernel(TimeMixArgs a) {
  constexpr int DP = LPC * RPL;                        // rows, filled up
  constexpr int NE = DP / 32;                          // channels a lane stages per token
  constexpr int CPW = 32 / LPC, COLS = TM_WARPS * CPW; // columns of a warp, of a block
  constexpr int LOG = LPC == 8 ? 3 : 4;
  constexpr int PER = time_mix_buffer(RPL, LPC);
  static_assert((LPC == 8 || LPC == 16) && DP % 32 == 0 && TM_CHUNK * COLS <= TM_THREADS, "lanes, rows, columns");
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, l = lane & (LPC - 1);
  const int head = blockIdx.y, seg = blockIdx.z;
  const int D = a.D, P = a.P;
  const int q0 = a.seg_q_start[seg], q1 = a.seg_q_start[seg + 1];
  if (q1 <= q0) return;
  const int cb = warp * CPW + (lane >> LOG);           // this lane's column inside the block
  const int col = blockIdx.x * COLS + cb;
  float* st = a.state + (size_t)a.seg_slot[seg] * a.slot_stride + ((size_t)head * P + col) * D;
  const AT* rp = (const AT*)a.r + (size_t)head * D;
  const AT* kp = (const AT*)a.k + (size_t)head * D;
  const AT* vp = (const AT*)a.v + (size_t)head * P;
  const float* dp = a.decay + (size_t)head * D;

  float S[RPL];
#pragma unroll
  for (int j = 0; j < RPL / 4; ++j) {
    const int n = (LPC * j + l) * 4;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col < P && n < D) {
      if (a.vec) f = *reinterpret_cast<const float4*>(st + n);
      else {
        f.x = st[n];
        if (n + 1 < D) f.y = st[n + 1];
        if (n + 2 < D) f.z = st[n + 2];
        if (n + 3 < D) f.w = st[n + 3];
      }
    }
    S[4 * j] = f.x; S[4 * j + 1] = f.y; S[4 * j + 2] = f.z; S[4 * j + 3] = f.w;
  }
  float w0[NE], u[NE];
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int n = lane + 32 * e;
    w0[e] = n < D ? a.w0[(size_t)head * D + n] : 0.f;
    u[e] = n < D ? a.u[(size_t)head * D + n] : 0.f;
  }

  // this warp stages token `warp` of a chunk, the first TM_CHUNK * COLS threads one value of v each; two chunks
  // are on their way in registers, so that a load from device memory has a whole chunk's time and more
  struct Staged {
    AT r[NE], k[NE], v;
    float d[NE];
  } even, odd;
  const int vt = threadIdx.x / COLS, vc = threadIdx.x % COLS;
  auto fetch = [&](int t0, Staged& x) {
    const int nt = min(TM_CHUNK, q1 - t0);             // may be 0 or less: nothing is read
    const size_t t = t0 + warp;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int n = lane + 32 * e;
      const bool in = warp < nt && n < D;
      x.r[e] = in ? rp[t * a.ld + n] : from_float<AT>(0.f);
      x.k[e] = in ? kp[t * a.ld + n] : from_float<AT>(0.f);
      x.d[e] = in ? dp[t * a.ld_decay + n] : 0.f;
    }
    const int c = blockIdx.x * COLS + vc;
    x.v = (vt < nt && c < P) ? vp[(size_t)(t0 + vt) * a.ld + c] : from_float<AT>(0.f);
  };
  auto put = [&](float* buf, const Staged& x) {
    float* rs = buf;
    float* ks = rs + TM_CHUNK * DP;
    float* ws = ks + TM_CHUNK * DP;
    float* vs = ws + TM_CHUNK * DP;
    float* bs = vs + TM_CHUNK * COLS;
    float bonus = 0.f;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int n = lane + 32 * e;
      const float rv = to_float(x.r[e]), kv = to_float(x.k[e]);
      rs[warp * DP + n] = rv;
      ks[warp * DP + n] = kv;
      ws[warp * DP + n] = expf(-expf(x.d[e] + w0[e]));
      bonus = fmaf(rv * kv, u[e], bonus);
    }
    bonus = warp_sum(bonus);
    if (lane == 0) bs[warp] = bonus;
    if (vt < TM_CHUNK) vs[threadIdx.x] = to_float(x.v);
  };

  struct Row {
    float4 r[RPL / 4], k[RPL / 4], w[RPL / 4];
    float v;
  };
  // one chunk: works through tokens t0 .. from buffer `turn`, puts the next chunk (`x`) into the other one and
  // fetches the chunk two further on in its place
  auto chunk = [&](int t0, int turn, Staged& x) {
    const int nt = min(TM_CHUNK, q1 - t0);
    const float* rs = sm + turn * PER;
    const float* ks = rs + TM_CHUNK * DP;
    const float* ws = ks + TM_CHUNK * DP;
    const float* vs = ws + TM_CHUNK * DP;
    const float* bs = vs + TM_CHUNK * COLS;
    float part[TM_CHUNK];
    auto load_row = [&](int tt, Row& row) {
      row.v = vs[tt * COLS + cb];
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {
        const int n = tt * DP + (LPC * j + l) * 4;
        row.r[j] = *reinterpret_cast<const float4*>(rs + n);
        row.k[j] = *reinterpret_cast<const float4*>(ks + n);
        row.w[j] = *reinterpret_cast<const float4*>(ws + n);
      }
    };
    auto token = [&](const Row& row) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {
        acc = fmaf(S[4 * j], row.r[j].x, acc);
        acc = fmaf(S[4 * j + 1], row.r[j].y, acc);
        acc = fmaf(S[4 * j + 2], row.r[j].z, acc);
        acc = fmaf(S[4 * j + 3], row.r[j].w, acc);
        S[4 * j] = fmaf(row.w[j].x, S[4 * j], row.k[j].x * row.v);
        S[4 * j + 1] = fmaf(row.w[j].y, S[4 * j + 1], row.k[j].y * row.v);
        S[4 * j + 2] = fmaf(row.w[j].z, S[4 * j + 2], row.k[j].z * row.v);
        S[4 * j + 3] = fmaf(row.w[j].w, S[4 * j + 3], row.k[j].w * row.v);
      }
      return acc;
    };
    if (nt == TM_CHUNK) {
      Row cur, ahead;                                  // the next token's row is on its way meanwhile
      load_row(0, cur);
#pragma unroll
      for (int tt = 0; tt < TM_CHUNK; ++tt) {
        if (tt + 1 < TM_CHUNK) load_row(tt + 1, ahead);
        part[tt] = token(cur);
        cur = ahead;
      }
    } else {
#pragma unroll
      for (int tt = 0; tt < TM_CHUNK; ++tt) {
        part[tt] = 0.f;
        if (tt < nt) {
          Row cur;
          load_row(tt, cur);
          part[tt] = token(cur);
        }
      }
    }
    // lane l of a column's ends with the total of token l >> (LOG - 3)
    int mask = LPC / 2;
#pragma unroll
    for (int w = TM_CHUNK / 2; w >= 1; w >>= 1) {
      const bool upper = l & mask;
#pragma unroll
      for (int i = 0; i < w; ++i) {
        const float send = upper ? part[i] : part[i + w];
        const float keep = upper ? part[i + w] : part[i];
        part[i] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
      }
      mask >>= 1;
    }
    if constexpr (LOG == 4) part[0] += __shfl_xor_sync(0xffffffffu, part[0], 1);
    const int tok = l >> (LOG - 3);
    if ((l & (LPC / 8 - 1)) == 0 && tok < nt && col < P)
      a.o[(size_t)(t0 + tok) * a.heads * P + (size_t)head * P + col] = fmaf(bs[tok], vs[tok * COLS + cb], part[0]);
    if (t0 + TM_CHUNK < q1) {
      put(sm + (turn ^ 1) * PER, x);
      fetch(t0 + 3 * TM_CHUNK, x);
    }
    __syncthreads();
  };

  fetch(q0, even);
  fetch(q0 + TM_CHUNK, odd);
  put(sm, even);
  fetch(q0 + 2 * TM_CHUNK, even);
  __syncthreads();
  for (int t0 = q0; t0 < q1; t0 += 2 * TM_CHUNK) {
    chunk(t0, 0, odd);
    if (t0 + TM_CHUNK < q1) chunk(t0 + TM_CHUNK, 1, even);
  }
#pragma unroll
  for (int j = 0; j < RPL / 4; ++j) {
    const int n = (LPC * j + l) * 4;
    if (col < P && n < D) {
      if (a.vec) *reinterpret_cast<float4*>(st + n) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
      else {
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (n + i < D) st[n + i] = S[4 * j + i];
      }
    }
  }
}

// Segments of one token each (a decode step): what it costs is reading and writing the states, so a lane holds
// its rows of r, k and w in registers, made once, and streams CPL columns of the state, all loads in flight
// together, without shared memory.  Sums run in the order of the kernel above: a token's result does not depend on
// which of the two it took.
template <typename AT, int RPL, int LPC, int CPL>
__global__ void __launch_bounds__(128) time_mixing_step_kernel(TimeMixArgs a) {
  constexpr int NE = LPC * RPL / 32, NJ = RPL / 4;
  constexpr int CPW = 32 / LPC;
  constexpr int LOG = LPC == 8 ? 3 : 4;
  static_assert(CPL <= LPC, "a lane per column when they are added up");
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, l = lane & (LPC - 1);
  const int head = blockIdx.y, seg = blockIdx.z;
  const int D = a.D, P = a.P;
  const int col0 = (blockIdx.x * 4 + warp) * CPL * CPW + (lane >> LOG);       // columns col0 + c * CPW
  if ((blockIdx.x * 4 + warp) * CPL * CPW >= P) return;                        // the whole warp leaves
  const size_t t = a.seg_q_start[seg];
  float* st = a.state + (size_t)a.seg_slot[seg] * a.slot_stride + (size_t)head * P * D;
  const AT* rp = (const AT*)a.r + t * a.ld + (size_t)head * D;
  const AT* kp = (const AT*)a.k + t * a.ld + (size_t)head * D;
  const AT* vp = (const AT*)a.v + t * a.ld + (size_t)head * P;
  const float* dp = a.decay + t * a.ld_decay + (size_t)head * D;
  const float* w0 = a.w0 + (size_t)head * D;
  const float* up = a.u + (size_t)head * D;

  float4 S[CPL][NJ];
#pragma unroll
  for (int c = 0; c < CPL; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int col = col0 + c * CPW, n = (LPC * j + l) * 4;
      S[c][j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col < P && n < D) {
        const float* p = st + (size_t)col * D + n;
        if (a.vec) S[c][j] = *reinterpret_cast<const float4*>(p);
        else {
          S[c][j].x = p[0];
          if (n + 1 < D) S[c][j].y = p[1];
          if (n + 2 < D) S[c][j].z = p[2];
          if (n + 3 < D) S[c][j].w = p[3];
        }
      }
    }
  float v[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) v[c] = col0 + c * CPW < P ? to_float(vp[col0 + c * CPW]) : 0.f;
  float bonus = 0.f;
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int n = lane + 32 * e;
    if (n < D) bonus = fmaf(to_float(rp[n]) * to_float(kp[n]), up[n], bonus);
  }
  bonus = warp_sum(bonus);
  float part[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) part[c] = 0.f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    float r[4], k[4], w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int n = (LPC * j + l) * 4 + i;
      const bool in = n < D;
      r[i] = in ? to_float(rp[n]) : 0.f;
      k[i] = in ? to_float(kp[n]) : 0.f;
      w[i] = in ? expf(-expf(dp[n] + w0[n])) : 0.f;
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float4& s = S[c][j];
      part[c] = fmaf(s.x, r[0], part[c]);
      part[c] = fmaf(s.y, r[1], part[c]);
      part[c] = fmaf(s.z, r[2], part[c]);
      part[c] = fmaf(s.w, r[3], part[c]);
      s.x = fmaf(w[0], s.x, k[0] * v[c]);
      s.y = fmaf(w[1], s.y, k[1] * v[c]);
      s.z = fmaf(w[2], s.z, k[2] * v[c]);
      s.w = fmaf(w[3], s.w, k[3] * v[c]);
    }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int col = col0 + c * CPW, n = (LPC * j + l) * 4;
      if (col < P && n < D) {
        float* p = st + (size_t)col * D + n;
        if (a.vec) *reinterpret_cast<float4*>(p) = S[c][j];
        else {
          p[0] = S[c][j].x;
          if (n + 1 < D) p[1] = S[c][j].y;
          if (n + 2 < D) p[2] = S[c][j].z;
          if (n + 3 < D) p[3] = S[c][j].w;
        }
      }
    }
  // a column's lanes are added up; the lanes share the columns out among themselves on the way
  int mask = LPC / 2, mine = 0;
#pragma unroll
  for (int w = CPL / 2; w >= 1; w >>= 1) {
    const bool upper = l & mask;
    if (upper) mine += w;
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const float send = upper ? part[i] : part[i + w];
      const float keep = upper ? part[i + w] : part[i];
      part[i] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
    }
    mask >>= 1;
  }
  const int first = 2 * mask - 1;                      // lanes with the same columns differ in these bits
  for (; mask >= 1; mask >>= 1) part[0] += __shfl_xor_sync(0xffffffffu, part[0], mask);
  const int col = col0 + mine * CPW;
  if ((l & first) == 0 && col < P) {
    float vm = v[0];
#pragma unroll
    for (int c = 1; c < CPL; ++c) vm = mine == c ? v[c] : vm;
    a.o[t * a.heads * P + (size_t)head * P + col] = fmaf(bonus, vm, part[0]);
  }
}

template <typename AT, int RPL, int LPC>
static int launch_time_mix_step(const TimeMixArgs& a, int S, cudaStream_t stream) {
  constexpr int MANY = 32 / RPL, FEW = RPL == 4 ? 2 : 1;   // columns a lane: plenty of blocks, or a few
  auto grid = [&](int cpl) { return dim3((a.P + 4 * cpl * (32 / LPC) - 1) / (4 * cpl * (32 / LPC)), a.heads, S); };
  const dim3 many = grid(MANY);
  cudaError_t e;
  if ((long long)many.x * many.y * many.z >= 2 * 148)
    e = launch_pdl(time_mixing_step_kernel<AT, RPL, LPC, MANY>, many, dim3(128), 0, stream, a);
  else
    e = launch_pdl(time_mixing_step_kernel<AT, RPL, LPC, FEW>, grid(FEW), dim3(128), 0, stream, a);
  return e == cudaSuccess ? FT_OK : (int)e;
}

template <typename AT, int RPL, int LPC>
static int launch_time_mix(const TimeMixArgs& a, int S, cudaStream_t stream) {
  const size_t smem = 2 * time_mix_buffer(RPL, LPC) * sizeof(float);
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(time_mixing_kernel<AT, RPL, LPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const int cols = TM_THREADS / LPC;
  const dim3 grid((a.P + cols - 1) / cols, a.heads, S);
  const cudaError_t e = launch_pdl(time_mixing_kernel<AT, RPL, LPC>, grid, dim3(TM_THREADS), smem, stream, a);
  return e == cudaSuccess ? FT_OK : (int)e;
}

}  // namespace ft

using namespace ft;

extern "C" {

int ft_token_shift(const void* x, long long ldx, const float* mu, void* out, float* state, long long slot_stride,
                   const int* token_seg, const int* seg_slot, const int* seg_q_start, int T, int W, int M, int dtype,
                   cudaStream_t stream) {
  if (T <= 0) return FT_OK;
  if (W <= 0 || M <= 0) return FT_ERR_SHAPE;
  ShiftArgs a{x, mu, out, state, token_seg, seg_slot, seg_q_start, ldx, slot_stride, T, W, M};
  const bool aligned = !((uintptr_t)x & 15) && !((uintptr_t)mu & 15) && !((uintptr_t)out & 15) &&
                       !((uintptr_t)state & 15) && !(slot_stride & 3);
  const bool many = T >= 1024;
  constexpr int RUN = 4;
  const unsigned rows = many ? (T + RUN - 1) / RUN : T;
  auto grid = [&](int vec) { return dim3(rows, ((W + vec - 1) / vec + 127) / 128); };
  if (dtype == FT_DTYPE_BF16 && aligned && !(W & 7) && !(ldx & 7)) {
    if (many) launch_pdl(token_shift_kernel<__nv_bfloat16, 8, RUN>, grid(8), dim3(128), 0, stream, a);
    else launch_pdl(token_shift_kernel<__nv_bfloat16, 8, 1>, grid(8), dim3(128), 0, stream, a);
  } else if (dtype == FT_DTYPE_F32 && aligned && !(W & 3) && !(ldx & 3)) {
    if (many) launch_pdl(token_shift_kernel<float, 4, RUN>, grid(4), dim3(128), 0, stream, a);
    else launch_pdl(token_shift_kernel<float, 4, 1>, grid(4), dim3(128), 0, stream, a);
  } else {
    FT_DISPATCH(dtype, AT, {
      if (many) launch_pdl(token_shift_kernel<AT, 1, RUN>, grid(1), dim3(128), 0, stream, a);
      else launch_pdl(token_shift_kernel<AT, 1, 1>, grid(1), dim3(128), 0, stream, a);
    });
  }
  FT_LAUNCH_CHECK();
  return FT_OK;
}

int ft_time_mixing_scan(const void* r, const void* k, const void* v, long long ld, const float* decay,
                        long long ld_decay, const float* w0, const float* u, float* state, long long slot_stride,
                        float* o, const int* seg_slot, const int* seg_q_start, int heads, int P, int D, int S, int T,
                        int dtype, cudaStream_t stream) {
  if (S <= 0) return FT_OK;
  if (heads <= 0 || P <= 0 || D <= 0 || D > 256 || heads > 65535 || S > 65535) return FT_ERR_SHAPE;
  TimeMixArgs a{r, k, v, decay, w0, u, state, o, seg_slot, seg_q_start, ld, ld_decay, slot_stride, heads, P, D, 0};
  a.vec = !(D & 3) && !(slot_stride & 3) && !((uintptr_t)state & 15);
  int rc = FT_OK;
  if (T == S) {                                        // one token a segment
    FT_DISPATCH(dtype, AT, {
      if (D <= 32) rc = launch_time_mix_step<AT, 4, 8>(a, S, stream);
      else if (D <= 64) rc = launch_time_mix_step<AT, 4, 16>(a, S, stream);
      else if (D <= 128) rc = launch_time_mix_step<AT, 8, 16>(a, S, stream);
      else rc = launch_time_mix_step<AT, 16, 16>(a, S, stream);
    });
    if (rc != FT_OK) return rc;
    FT_LAUNCH_CHECK();
    return FT_OK;
  }
  FT_DISPATCH(dtype, AT, {
    if (D <= 32) rc = launch_time_mix<AT, 4, 8>(a, S, stream);
    else if (D <= 64) rc = launch_time_mix<AT, 4, 16>(a, S, stream);
    else if (D <= 128) rc = launch_time_mix<AT, 8, 16>(a, S, stream);
    else rc = launch_time_mix<AT, 16, 16>(a, S, stream);
  });
  if (rc != FT_OK) return rc;
  FT_LAUNCH_CHECK();
  return FT_OK;
}

}  // extern "C"
