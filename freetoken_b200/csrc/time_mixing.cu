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
// token of the NEXT chunk into registers while the block works through the current chunk in shared memory and puts
// it into the other of two buffers afterwards: one barrier a chunk.  The decay's exponentials and the bonus
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

  // this warp stages token `warp` of a chunk, the first TM_CHUNK * COLS threads one value of v each
  AT pr[NE], pk[NE], pv;
  float pd[NE];
  const int vt = threadIdx.x / COLS, vc = threadIdx.x % COLS;
  auto fetch = [&](int t0, int nt) {
    const size_t t = t0 + warp;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int n = lane + 32 * e;
      const bool in = warp < nt && n < D;
      pr[e] = in ? rp[t * a.ld + n] : from_float<AT>(0.f);
      pk[e] = in ? kp[t * a.ld + n] : from_float<AT>(0.f);
      pd[e] = in ? dp[t * a.ld_decay + n] : 0.f;
    }
    const int c = blockIdx.x * COLS + vc;
    pv = (vt < nt && c < P) ? vp[(size_t)(t0 + vt) * a.ld + c] : from_float<AT>(0.f);
  };
  auto put = [&](float* buf) {
    float* rs = buf;
    float* ks = rs + TM_CHUNK * DP;
    float* ws = ks + TM_CHUNK * DP;
    float* vs = ws + TM_CHUNK * DP;
    float* bs = vs + TM_CHUNK * COLS;
    float bonus = 0.f;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int n = lane + 32 * e;
      const float rv = to_float(pr[e]), kv = to_float(pk[e]);
      rs[warp * DP + n] = rv;
      ks[warp * DP + n] = kv;
      ws[warp * DP + n] = expf(-expf(pd[e] + w0[e]));
      bonus = fmaf(rv * kv, u[e], bonus);
    }
    bonus = warp_sum(bonus);
    if (lane == 0) bs[warp] = bonus;
    if (vt < TM_CHUNK) vs[threadIdx.x] = to_float(pv);
  };

  fetch(q0, min(TM_CHUNK, q1 - q0));
  put(sm);
  __syncthreads();
  int turn = 0;
  for (int t0 = q0; t0 < q1; t0 += TM_CHUNK, turn ^= 1) {
    const int nt = min(TM_CHUNK, q1 - t0);
    const int next = min(TM_CHUNK, q1 - t0 - TM_CHUNK);
    if (next > 0) fetch(t0 + TM_CHUNK, next);
    const float* rs = sm + turn * PER;
    const float* ks = rs + TM_CHUNK * DP;
    const float* ws = ks + TM_CHUNK * DP;
    const float* vs = ws + TM_CHUNK * DP;
    const float* bs = vs + TM_CHUNK * COLS;
    float part[TM_CHUNK];
    auto token = [&](int tt) {
      const float v = vs[tt * COLS + cb];
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {
        const int n = tt * DP + (LPC * j + l) * 4;
        const float4 r4 = *reinterpret_cast<const float4*>(rs + n);
        const float4 k4 = *reinterpret_cast<const float4*>(ks + n);
        const float4 w4 = *reinterpret_cast<const float4*>(ws + n);
        acc = fmaf(S[4 * j], r4.x, acc);
        acc = fmaf(S[4 * j + 1], r4.y, acc);
        acc = fmaf(S[4 * j + 2], r4.z, acc);
        acc = fmaf(S[4 * j + 3], r4.w, acc);
        S[4 * j] = fmaf(w4.x, S[4 * j], k4.x * v);
        S[4 * j + 1] = fmaf(w4.y, S[4 * j + 1], k4.y * v);
        S[4 * j + 2] = fmaf(w4.z, S[4 * j + 2], k4.z * v);
        S[4 * j + 3] = fmaf(w4.w, S[4 * j + 3], k4.w * v);
      }
      return acc;
    };
    if (nt == TM_CHUNK) {
#pragma unroll
      for (int tt = 0; tt < TM_CHUNK; ++tt) part[tt] = token(tt);
    } else {
#pragma unroll
      for (int tt = 0; tt < TM_CHUNK; ++tt) part[tt] = tt < nt ? token(tt) : 0.f;
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
    if (next > 0) put(sm + (turn ^ 1) * PER);
    __syncthreads();
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
                        float* o, const int* seg_slot, const int* seg_q_start, int heads, int P, int D, int S,
                        int dtype, cudaStream_t stream) {
  if (S <= 0) return FT_OK;
  if (heads <= 0 || P <= 0 || D <= 0 || D > 256 || heads > 65535 || S > 65535) return FT_ERR_SHAPE;
  TimeMixArgs a{r, k, v, decay, w0, u, state, o, seg_slot, seg_q_start, ld, ld_decay, slot_stride, heads, P, D, 0};
  a.vec = !(D & 3) && !(slot_stride & 3) && !((uintptr_t)state & 15);
  int rc = FT_OK;
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
