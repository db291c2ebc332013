// The norm behind a recurrence: rows of float32 values in equal parts, each divided by its own root mean
// square, times a weight, with a gate silu(z) or sigmoid(z) before or behind it.
#include "common.cuh"

namespace ft {

// a gate's function: 0 silu, 1 sigmoid
__device__ __forceinline__ float gate_f(float v, int kind) {
  const float sg = 1.f / (1.f + expf(-v));
  return kind == 1 ? sg : v * sg;
}

// --------------------------------------------------------------------- gated norm
// A row of `width` float32 values in `groups` equal parts, each divided by its own root mean
// square; times weight[i % weight_len]; a gate silu(z) (or sigmoid(z)) on the values before the norm
// (gate_first) or on the result.  One warp per (token, group).
template <typename AT>
__global__ void __launch_bounds__(128) gated_norm_kernel(const float* __restrict__ y, const AT* __restrict__ z,
                                                         long long ldz, const float* __restrict__ weight,
                                                         int weight_len, AT* __restrict__ out, int T, int width,
                                                         int groups, float eps, int gate_first, int gate_kind) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)T * groups) return;
  const int t = (int)(item / groups), grp = (int)(item % groups);
  const int size = width / groups, base = grp * size;
  const float* row = y + (size_t)t * width + base;
  const AT* gate = z + (size_t)t * ldz + base;
  float ss = 0.f;
  for (int i = lane; i < size; i += 32) {
    float v = row[i];
    if (gate_first) v *= gate_f(to_float(gate[i]), gate_kind);
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)size + eps);
  AT* dst = out + (size_t)t * width + base;
  for (int i = lane; i < size; i += 32) {
    const float gv = gate_f(to_float(gate[i]), gate_kind);
    float v = row[i];
    if (gate_first) v *= gv;
    v = v * inv * weight[(base + i) % weight_len];
    if (!gate_first) v *= gv;
    dst[i] = from_float<AT>(v);
  }
}

// The same norm with TPI threads (8: several small parts a warp, 32, or 128: a block) per (token, group), 16-byte pieces, and every value kept in
// registers between the sum of squares and the scaling: parts of up to 4 * KEEP * TPI values, a
// multiple of 4, rows 16-byte (bfloat16 gate: 8-byte) aligned.
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}

template <typename AT, int TPI, int KEEP>
__global__ void __launch_bounds__(128) gated_norm_vec_kernel(const float* __restrict__ y, const AT* __restrict__ z,
                                                             long long ldz, const float* __restrict__ weight,
                                                             int weight_len, AT* __restrict__ out, int T, int width,
                                                             int groups, float eps, int gate_first, int gate_kind) {
  __shared__ float scratch[33];
  pdl_wait();
  const int sub = threadIdx.x % TPI;
  const long long item = (long long)blockIdx.x * (128 / TPI) + threadIdx.x / TPI;
  const bool live = item < (long long)T * groups;
  if (TPI >= 32 && !live) return;                     // a warp (TPI 32) or the whole block (TPI 128) leaves
  const int t = live ? (int)(item / groups) : 0, grp = live ? (int)(item % groups) : 0;
  const int size = width / groups, base = grp * size, pieces = live ? size >> 2 : 0;
  const float* row = y + (size_t)t * width + base;
  const AT* gate = z + (size_t)t * ldz + base;
  float4 keep[KEEP], gk[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int gi = sub + j * TPI;
    if (gi < pieces) {
      float4 v = ld4(row + 4 * gi);
      const float4 gr = ld4(gate + 4 * gi);
      const float4 gv = make_float4(gate_f(gr.x, gate_kind), gate_f(gr.y, gate_kind), gate_f(gr.z, gate_kind), gate_f(gr.w, gate_kind));
      if (gate_first) { v.x *= gv.x; v.y *= gv.y; v.z *= gv.z; v.w *= gv.w; }
      keep[j] = v;
      gk[j] = gv;
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
  }
  if constexpr (TPI < 32) {
#pragma unroll
    for (int o = TPI / 2; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  } else {
    ss = TPI == 32 ? warp_sum(ss) : block_sum(ss, scratch);
  }
  const float inv = 1.f / sqrtf(ss / (float)size + eps);
  AT* dst = out + (size_t)t * width + base;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int gi = sub + j * TPI;
    if (gi < pieces) {
      const float4 w = ld4(weight + (base + 4 * gi) % weight_len);
      float4 v = keep[j];
      v.x *= inv * w.x; v.y *= inv * w.y; v.z *= inv * w.z; v.w *= inv * w.w;
      if (!gate_first) { v.x *= gk[j].x; v.y *= gk[j].y; v.z *= gk[j].z; v.w *= gk[j].w; }
      st4(dst + 4 * gi, v);
    }
  }
}

}  // namespace ft

using namespace ft;

extern "C" {

int ft_gated_norm(const float* y, const void* z, long long ldz, const float* weight, int weight_len, void* out,
                  int T, int width, int groups, float eps, int gate_first, int gate_kind, int dtype,
                  cudaStream_t stream) {
  if (T <= 0) return FT_OK;
  if (width <= 0 || groups <= 0 || width % groups || weight_len <= 0) return FT_ERR_SHAPE;
  const long long items = (long long)T * groups;
  const int size = width / groups;
  const bool vec = !(size & 3) && !(weight_len & 3) && !(ldz & 3) && !((uintptr_t)y & 15) && !((uintptr_t)z & 15) &&
                   !((uintptr_t)weight & 15) && !((uintptr_t)out & 15);
  if (vec && size <= 16 * 8) {
    FT_DISPATCH(dtype, AT, launch_pdl(gated_norm_vec_kernel<AT, 8, 4>, dim3((unsigned)((items + 15) / 16)), dim3(128), 0, stream,
                                      y, (const AT*)z, ldz, weight, weight_len, (AT*)out, T, width, groups, eps,
                                      gate_first, gate_kind));
    FT_LAUNCH_CHECK();
    return FT_OK;
  }
  if (vec && size <= 16 * 32) {
    FT_DISPATCH(dtype, AT, launch_pdl(gated_norm_vec_kernel<AT, 32, 4>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream,
                                      y, (const AT*)z, ldz, weight, weight_len, (AT*)out, T, width, groups, eps,
                                      gate_first, gate_kind));
    FT_LAUNCH_CHECK();
    return FT_OK;
  }
  if (vec && size <= 16 * 128) {
    FT_DISPATCH(dtype, AT, launch_pdl(gated_norm_vec_kernel<AT, 128, 4>, dim3((unsigned)items), dim3(128), 0, stream, y,
                                      (const AT*)z, ldz, weight, weight_len, (AT*)out, T, width, groups, eps,
                                      gate_first, gate_kind));
    FT_LAUNCH_CHECK();
    return FT_OK;
  }
  if (vec && size <= 64 * 128) {
    FT_DISPATCH(dtype, AT, launch_pdl(gated_norm_vec_kernel<AT, 128, 16>, dim3((unsigned)items), dim3(128), 0, stream, y,
                                      (const AT*)z, ldz, weight, weight_len, (AT*)out, T, width, groups, eps,
                                      gate_first, gate_kind));
    FT_LAUNCH_CHECK();
    return FT_OK;
  }
  const unsigned blocks = (unsigned)((items + 3) / 4);
  FT_DISPATCH(dtype, AT, launch_pdl(gated_norm_kernel<AT>, dim3(blocks), dim3(128), 0, stream, y, (const AT*)z, ldz,
                                    weight, weight_len, (AT*)out, T, width, groups, eps, gate_first, gate_kind));
  FT_LAUNCH_CHECK();
  return FT_OK;
}

}  // extern "C"
