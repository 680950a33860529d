// Loads and stores of activations that are bf16 when a model is served in bf16 and fp32 when it is run in 32-bit.
#pragma once
#include "ptx.cuh"

namespace b200 {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float& d, float v) { d = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16& d, float v) { d = __float2bfloat16(v); }

// VEC consecutive elements (1 or 4) <-> fp32 registers; VEC == 4 needs 4-element alignment.
template <int VEC>
__device__ __forceinline__ void load_vec(const float* p, float (&f)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    f[0] = *p;
  }
}
template <int VEC>
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&f)[VEC]) {
  if constexpr (VEC == 4) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    f[0] = __bfloat162float(*p);
  }
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const float (&f)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float (&f)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  else *p = __float2bfloat16(f[0]);
}

template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) Raw {       // VEC elements as they are stored
  T v[VEC];
};

template <typename T>
struct Piece {                    // 8 elements as they are stored
  uint4 v[sizeof(T) / 2];
};
__device__ __forceinline__ void unpack(const Piece<__nv_bfloat16>& r, float (&f)[8]) {
  const float2 a = unpack_bf16x2(r.v[0].x), b = unpack_bf16x2(r.v[0].y), c = unpack_bf16x2(r.v[0].z), d = unpack_bf16x2(r.v[0].w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
__device__ __forceinline__ void unpack(const Piece<float>& r, float (&f)[8]) {
  f[0] = __uint_as_float(r.v[0].x); f[1] = __uint_as_float(r.v[0].y); f[2] = __uint_as_float(r.v[0].z); f[3] = __uint_as_float(r.v[0].w);
  f[4] = __uint_as_float(r.v[1].x); f[5] = __uint_as_float(r.v[1].y); f[6] = __uint_as_float(r.v[1].z); f[7] = __uint_as_float(r.v[1].w);
}
template <typename T>
__device__ __forceinline__ Piece<T> load_piece(const T* p) {
  Piece<T> r;
#pragma unroll
  for (int j = 0; j < (int)sizeof(T) / 2; ++j) r.v[j] = reinterpret_cast<const uint4*>(p)[j];
  return r;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

// Sum over the block (blockDim.x a multiple of 32, at most 1024); every thread receives it.  `red`: 32 floats.
__device__ __forceinline__ float block_total(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}

__device__ __forceinline__ float sigmoid_f(float g) { return 1.f / (1.f + __expf(-g)); }

__device__ __forceinline__ void report_bad_arg(uint32_t* status, uint32_t where) {
  if (status != nullptr) atomicCAS(status, 0u, ERR_BAD_ARG | (where << 8));
}

}  // namespace b200
