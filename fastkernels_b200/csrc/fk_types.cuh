// Activation element types of the kernels that serve both number formats: bf16
// (uint16_t storage, fp32 arithmetic) and fp32.  All helpers move four elements.
#pragma once

#include "fk_common.cuh"

namespace fk {

#ifdef __CUDACC__

template <typename T>
struct Elem;

template <>
struct Elem<uint16_t> {
  static __device__ __forceinline__ float4 load4(const uint16_t* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
  }
  static __device__ __forceinline__ void store4(uint16_t* p, const float4& f) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f.x, f.y), pack_bf16(f.z, f.w));
  }
  static __device__ __forceinline__ float load(const uint16_t* p) {
    return bf16_bits_to_float(*p);
  }
  static __device__ __forceinline__ void store(uint16_t* p, float f) {
    *p = __bfloat16_as_ushort(__float2bfloat16_rn(f));
  }
};

template <>
struct Elem<float> {
  static __device__ __forceinline__ float4 load4(const float* p) {
    return *reinterpret_cast<const float4*>(p);
  }
  static __device__ __forceinline__ void store4(float* p, const float4& f) {
    *reinterpret_cast<float4*>(p) = f;
  }
  static __device__ __forceinline__ float load(const float* p) { return *p; }
  static __device__ __forceinline__ void store(float* p, float f) { *p = f; }
};

__device__ __forceinline__ float4 operator+(const float4& a, const float4& b) {
  return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
}
__device__ __forceinline__ float4 operator-(const float4& a, const float4& b) {
  return make_float4(a.x - b.x, a.y - b.y, a.z - b.z, a.w - b.w);
}
__device__ __forceinline__ float4 operator*(const float4& a, float s) {
  return make_float4(a.x * s, a.y * s, a.z * s, a.w * s);
}
__device__ __forceinline__ float4 operator*(const float4& a, const float4& b) {
  return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w);
}
__device__ __forceinline__ float sumsq(const float4& v) {
  return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }

// Two values as a high and a low bf16 part each (16 significant bits together).
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t* hi, uint32_t* lo) {
  *hi = pack_bf16(a, b);
  *lo = pack_bf16(a - bf16lo(*hi), b - bf16hi(*hi));
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Sum of N values over the block; every thread gets the sums.  `red` holds
// 2 x 32 x N floats: consecutive calls alternate between its halves (`flip`), so
// one barrier per call is enough.
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float* red, int& flip) {
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = blockDim.x >> 5;
  if (nwarps == 1) return;
  float* r = red + flip * 32 * N;
  flip ^= 1;
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) r[warp * N + i] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < nwarps ? r[lane * N + i] : 0.f);
}

#endif  // __CUDACC__

}  // namespace fk
