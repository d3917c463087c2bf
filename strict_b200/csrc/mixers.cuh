// Device helpers of the mixers' row kernels: sums of a projection's partial results, activations of its feed-forward columns.
#pragma once
#include "common.cuh"

#ifdef __CUDACC__
namespace mix {

template <typename T>
__device__ __forceinline__ T to_t(float v);
template <>
__device__ __forceinline__ float to_t<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 to_t<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { return f32_to_bf16_bits(lo) | (f32_to_bf16_bits(hi) << 16); }
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float* p, float4 v) { *(float4*)p = v; }
template <>
__device__ __forceinline__ void store4<bf16>(bf16* p, float4 v) { *(uint2*)p = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }

__device__ __forceinline__ float proj(const ProjRows& p, int64_t T, int64_t t, int64_t col) {
  float v = 0.f;
  for (int s = 0; s < p.splits; s++) v += p.in[((int64_t)s * T + t) * p.ld + col];
  return v;
}
// four columns (col and the row stride multiples of 4), every split's load in flight at once
__device__ __forceinline__ float4 proj4(const ProjRows& p, int64_t T, int64_t t, int64_t col) {
  if (p.splits == 1) return *(const float4*)(p.in + t * p.ld + col);
  float4 q[8], v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int s = 0; s < 8; s++)
    if (s < p.splits) q[s] = *(const float4*)(p.in + ((int64_t)s * T + t) * p.ld + col);
#pragma unroll
  for (int s = 0; s < 8; s++)
    if (s < p.splits) { v.x += q[s].x; v.y += q[s].y; v.z += q[s].z; v.w += q[s].w; }
  return v;
}
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// Blocks of 256 threads per row that act_block needs.
__host__ __device__ inline int act_blocks(const ActArgs& a) { return a.kind ? (a.n + 1023) / 1024 : 0; }
// Block `blk` of row t: 1024 values of the activation.
template <typename T>
__device__ __forceinline__ void act_block(const ActArgs& a, const ProjRows& p, int64_t rows, int64_t t, int blk) {
  T* out = (T*)a.out + t * a.ld;
  const int i0 = blk * 1024 + (int)threadIdx.x * 4;
  if (((a.col | a.n) & 3) == 0 && (p.ld & 3) == 0 && (a.ld & 3) == 0) {
    if (i0 >= a.n) return;
    float4 o;
    if (a.kind == 2) {
      const float4 u = proj4(p, rows, t, a.col + 2 * i0), w = proj4(p, rows, t, a.col + 2 * i0 + 4);
      o = make_float4(fmaxf(u.x, 0.f) * u.y, fmaxf(u.z, 0.f) * u.w, fmaxf(w.x, 0.f) * w.y, fmaxf(w.z, 0.f) * w.w);
    } else {
      const float4 u = proj4(p, rows, t, a.col + i0);
      o = make_float4(sb_xielu(u.x, a.pos, a.neg), sb_xielu(u.y, a.pos, a.neg), sb_xielu(u.z, a.pos, a.neg), sb_xielu(u.w, a.pos, a.neg));
    }
    store4<T>(out + i0, o);
    return;
  }
  for (int i = i0; i < i0 + 4 && i < a.n; i++) {
    float v;
    if (a.kind == 2) v = fmaxf(proj(p, rows, t, a.col + 2 * i), 0.f) * proj(p, rows, t, a.col + 2 * i + 1);
    else v = sb_xielu(proj(p, rows, t, a.col + i), a.pos, a.neg);
    out[i] = to_t<T>(v);
  }
}

}  // namespace mix
#endif
