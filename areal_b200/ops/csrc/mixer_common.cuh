// Typed access and scalar functions shared by the mixer-stack kernels (activations bf16 or fp32).
#pragma once
#include "common.cuh"

namespace ab2 {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// V consecutive elements (V = 1, 2, 4 or 8; the address is aligned to V elements)
template <int V>
__device__ __forceinline__ void ldv(const float* p, float (&v)[V]) {
  if constexpr (V == 8) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else if constexpr (V == 2) {
    const float2 a = *reinterpret_cast<const float2*>(p);
    v[0] = a.x; v[1] = a.y;
  } else {
    v[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void ldv(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 8) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 x = unpack_bf16(w[i]);
      v[2 * i] = x.x;
      v[2 * i + 1] = x.y;
    }
  } else if constexpr (V == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 x = unpack_bf16(a.x), y = unpack_bf16(a.y);
    v[0] = x.x; v[1] = x.y; v[2] = y.x; v[3] = y.y;
  } else if constexpr (V == 2) {
    const float2 x = unpack_bf16(*reinterpret_cast<const uint32_t*>(p));
    v[0] = x.x; v[1] = x.y;
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void stv(float* p, const float (&v)[V]) {
  if constexpr (V == 8) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  } else if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}
template <int V>
__device__ __forceinline__ void stv(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
  else if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16(v[0], v[1]);
  else *p = __float2bfloat16(v[0]);
}

// Copy of N bytes from global into shared memory that the copying thread alone will read, after its own wait (cp.async.wait_group).
template <int N>
__device__ __forceinline__ void copy_own(void* dst, const void* src) {
  if constexpr (N == 2) *reinterpret_cast<uint16_t*>(dst) = *reinterpret_cast<const uint16_t*>(src);
  else if constexpr (N == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(N) : "memory");
}

// Scalar functions. FAST (beside bf16 activations) takes the hardware exponential, logarithm and division, about 1e-6
// relative to the result's scale; the 32-bit mode takes the math library's.
template <bool FAST>
__device__ __forceinline__ float exp_t(float z) {
  if constexpr (FAST) return fast_exp2(z * 1.4426950408889634f);
  return expf(z);
}
template <bool FAST>
__device__ __forceinline__ float sigmoid_t(float z) {
  if constexpr (FAST) return __fdividef(1.f, 1.f + fast_exp2(fminf(z * -1.4426950408889634f, 80.f)));
  return 1.f / (1.f + expf(-z));
}
template <bool FAST>
__device__ __forceinline__ float silu_t(float z) {
  if constexpr (FAST) return z * sigmoid_t<true>(z);
  return z / (1.f + expf(-z));
}
// exp(z) - 1 for z <= 0
template <bool FAST>
__device__ __forceinline__ float expm1_neg(float z) {
  if constexpr (FAST) {
    const float series = z * (1.f + z * (0.5f + z * (1.f / 6.f + z * (1.f / 24.f + z * (1.f / 120.f)))));
    return z > -0.125f ? series : fast_exp2(z * 1.4426950408889634f) - 1.f;
  }
  return expm1f(z);
}
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_t(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  if constexpr (FAST) return z * sigmoid_t<true>(2.f * u);              // (1 + tanh u) / 2 is the logistic function of 2 u
  return 0.5f * z * (1.f + tanhf(u));
}
__device__ __forceinline__ float softplusf(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// What an attention may have beside queries, keys and values (host side: passed by address, null = none of it).
struct AttnExtra {
  const void *q2 = nullptr, *k2 = nullptr;   // second part of queries [R, Hq, D2] and keys [cache rows, D2]: its product is added before the scale
  const void* gate = nullptr;                // output times sigmoid(gate): [R, Hq] (gate_per_head) or [R, Hq * Dv]
  const float* sink = nullptr;               // per head: a score (scaled as it stands, never capped) that only enters the denominator
  const float* kf = nullptr;                 // factor of every key's scores (what norms a key that is cached as it is): [cache rows, Hkv]
  // elements between rows (and heads); 0: contiguous
  long long ldq = 0, hsq = 0, ldq2 = 0, hsq2 = 0, ldk = 0, ldv = 0, ldk2 = 0, ldo = 0, ldg = 0;
  int D2 = 0, gate_per_head = 0;
  float sink_const = -INFINITY;              // sink of every head without `sink`; minus infinity: none
  float out_scale = 1.f;

  __device__ __forceinline__ float sink_of(int h) const { return sink ? sink[h] : sink_const; }
};

static inline bool aligned_to(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; }

}  // namespace ab2
