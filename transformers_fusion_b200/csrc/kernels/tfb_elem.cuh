// Element-type helpers for kernels that exist in a bf16 and a true fp32 form: scalar and vector loads / stores that
// convert to and from fp32, and block / warp reductions.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

#include "tfb_ptx.cuh"

namespace tfb {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// N consecutive elements (N * sizeof(T) is 16, 8 or one element; the address has that alignment)
template <int N> __device__ __forceinline__ void load_n(const float* p, float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      const float4 u = reinterpret_cast<const float4*>(p)[i];
      f[4 * i] = u.x; f[4 * i + 1] = u.y; f[4 * i + 2] = u.z; f[4 * i + 3] = u.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = p[i];
  }
}
template <int N> __device__ __forceinline__ void load_n(const __nv_bfloat16* p, float (&f)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N / 8; ++i) {
      const uint4 u = reinterpret_cast<const uint4*>(p)[i];
      const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 t = unpack_bf16(w[j]);
        f[8 * i + 2 * j] = t.x;
        f[8 * i + 2 * j + 1] = t.y;
      }
    }
  } else if constexpr (N == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int N> __device__ __forceinline__ void store_n(float* p, const float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i)
      reinterpret_cast<float4*>(p)[i] = make_float4(f[4 * i], f[4 * i + 1], f[4 * i + 2], f[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = f[i];
  }
}
template <int N> __device__ __forceinline__ void store_n(__nv_bfloat16* p, const float (&f)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N / 8; ++i) {
      uint4 u;
      u.x = pack_bf16(f[8 * i], f[8 * i + 1]);
      u.y = pack_bf16(f[8 * i + 2], f[8 * i + 3]);
      u.z = pack_bf16(f[8 * i + 4], f[8 * i + 5]);
      u.w = pack_bf16(f[8 * i + 6], f[8 * i + 7]);
      reinterpret_cast<uint4*>(p)[i] = u;
    }
  } else if constexpr (N == 4) {
    uint2 u;
    u.x = pack_bf16(f[0], f[1]);
    u.y = pack_bf16(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

__device__ __forceinline__ float warp_add(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the block (a multiple of 32 threads); `red` holds 32 floats of shared memory and is free again afterwards.
__device__ __forceinline__ float block_add(float v, float* red) {
  v = warp_add(v);
  const int nw = blockDim.x >> 5;
  if (nw == 1) return v;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = (int(threadIdx.x & 31) < nw) ? red[threadIdx.x & 31] : 0.f;
  v = warp_add(v);
  __syncthreads();
  return v;
}

__device__ __forceinline__ float silu_exact(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
// 0.5 z (1 + tanh(u)) = z sigmoid(2 u), u = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_exact(float z) {
  const float u = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z / (1.f + expf(-2.f * u));
}

// gated feed-forwards: silu(g) u, gelu(g) u (tanh form), or, with g = min(g, limit) and u clamped to +-limit, g sigmoid(1.702 g) (u + 1)
enum { GLU_SILU = 0, GLU_GELU = 1, GLU_CLAMPED = 2 };
template <int ACT>
__device__ __forceinline__ float glu_value(float g, float u, float limit) {
  if constexpr (ACT == GLU_CLAMPED) {
    g = fminf(g, limit);
    return g / (1.f + expf(-1.702f * g)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
  }
  return (ACT == GLU_GELU ? gelu_tanh_exact(g) : silu_exact(g)) * u;
}

// pairs of fp32 in one register pair: one instruction, two IEEE operations
typedef unsigned long long u64;
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
  u64 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
  u64 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ u64 pack2(float lo, float hi) {
  u64 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(u64 v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}

}  // namespace tfb
