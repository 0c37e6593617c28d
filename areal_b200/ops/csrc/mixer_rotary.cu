// Rotated positions of mixer stacks. A table of (cos, sin) per row of the step and frequency is made once per step; the kernels
// that rotate read it:
//   qk_head_norm_append   per-head RMS norms of q and k (optional; with or without weights), rotation, k and v into the paged cache. A
//                         turn keeps a head's length, so norms without weights may as well be taken to follow it. Or the keys go into
//                         the cache as they are (they are the values too) with the number that norms each of them beside them
//   latent_rope_append    norm of the cached latent and rotation of the key part behind it, both into the cache; rotation of the
//                         queries' second part in place
// Pairs are (i, i + half) of the rotated stretch, or (2 i, 2 i + 1) when interleaved.
#include <type_traits>

#include "mixer_common.cuh"

namespace ab2 {

// Angles in double, brought into one turn before the 32-bit functions.
__global__ void __launch_bounds__(256)
rotary_table_kernel(const int* __restrict__ pos, const double* __restrict__ freq, const float* __restrict__ mult, float2* __restrict__ out,
                    long long total, int P) {
  pdl_wait();
  pdl_trigger();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / P;
    const int f = (int)(i - r * P);
    const double turns = (double)pos[r] * freq[f];                  // frequencies in turns per position
    const float a = (float)((turns - rint(turns)) * 6.283185307179586);
    float s, c;
    sincosf(a, &s, &c);
    out[i] = make_float2(c * mult[f], s * mult[f]);
  }
}

struct QkExtra {
  const float* qf;            // [Hq] factors of the queries, or null
  float* kf;                  // [cache rows, Hkv]: keys are stored as they are and their norms' factors here; or null
  int unit;                   // norms without weights
};

// One CTA per row, a warp per head, any sizes.
template <typename T, int V, bool INTERLEAVED>
__global__ void __launch_bounds__(256)
qk_head_norm_append_kernel(const T* __restrict__ z, long long ld, const float* __restrict__ wq, const float* __restrict__ wk,
                           const float2* __restrict__ rot, int ldr, int half, const int* __restrict__ slots, T* __restrict__ q, T* __restrict__ kc,
                           T* __restrict__ vc, int Hq, int Hkv, int D, int nv, float eps, const QkExtra x2) {
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int slot = slots[row];
  const T* src = z + (size_t)row * ld;
  const float2* cs = rot + (size_t)row * ldr;
  float* x = sm + warp * ((D + 3) & ~3);
  for (int u = warp; u < Hq + Hkv; u += nw) {
    if (u >= Hq && slot < 0) break;
    const float* w = u < Hq ? wq : wk;
    float ss = 0.f;
    for (int c = lane * V; c < D; c += 32 * V) {
      float v[V];
      ldv<V>(src + (size_t)u * D + c, v);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += v[e] * v[e];
      stv<V>(x + c, v);
    }
    float rstd = w != nullptr || x2.unit ? 1.f / sqrtf(warp_sum(ss) / D + eps) : 1.f;
    if (u >= Hq && x2.kf != nullptr) {
      if (lane == 0) x2.kf[(size_t)slot * Hkv + u - Hq] = rstd;
      rstd = 1.f;
    }
    if (u < Hq && x2.qf != nullptr) rstd *= x2.qf[u];
    __syncwarp();
    T* dst = u < Hq ? q + ((size_t)row * Hq + u) * D : kc + ((size_t)slot * Hkv + u - Hq) * D;
    auto normed = [&](int c, float (&v)[V]) {
      ldv<V>(x + c, v);
      float g[V];
#pragma unroll
      for (int e = 0; e < V; ++e) g[e] = 1.f;
      if (w != nullptr) ldv<V>(w + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] *= rstd * g[e];
    };
    for (int c = lane * V; c < D; c += 32 * V) {              // V numbers turn together or not at all
      float v[V], o[V];
      normed(c, v);
      if (c < 2 * half) {
        if constexpr (INTERLEAVED && V > 1) {
#pragma unroll
          for (int e = 0; e < V; e += 2) {
            const float2 r = cs[(c + e) >> 1];
            const float a = v[e], b = v[e + 1];
            v[e] = a * r.x - b * r.y;
            v[e + 1] = b * r.x + a * r.y;
          }
        } else {
          const bool first = INTERLEAVED ? !(c & 1) : c < half;
          normed(INTERLEAVED ? c ^ 1 : (first ? c + half : c - half), o);
          const float2* r = cs + (INTERLEAVED ? c >> 1 : (first ? c : c - half));
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const float2 t = r[e];
            v[e] = v[e] * t.x + (first ? -o[e] : o[e]) * t.y;
          }
        }
      }
      stv<V>(dst + c, v);
    }
    __syncwarp();
  }
  if (slot >= 0) {
    const T* sv = src + (size_t)(Hq + Hkv) * D;
    for (int c = threadIdx.x * V; c < nv; c += blockDim.x * V) {
      float v[V];
      ldv<V>(sv + c, v);
      stv<V>(vc + (size_t)slot * nv + c, v);
    }
  }
}

// The same for heads of up to 128 numbers, four to a lane: weights and angles of a lane stay in its registers, partners come
// from another lane, and a warp has several heads on their way.
constexpr int QK_U = 4;

template <typename T, bool INTERLEAVED>
__global__ void __launch_bounds__(256)
qk_head_norm_append_lanes_kernel(const T* __restrict__ z, long long ld, const float* __restrict__ wq, const float* __restrict__ wk,
                                 const float2* __restrict__ rot, int ldr, int half, const int* __restrict__ slots, T* __restrict__ q, T* __restrict__ kc,
                                 T* __restrict__ vc, int Hq, int Hkv, int D, int nv, float eps, const QkExtra x2) {
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, c = lane * 4;
  const int slot = slots[row], heads = slot >= 0 ? Hq + Hkv : Hq;
  const T* src = z + (size_t)row * ld;
  const bool in = c < D, turns = c < 2 * half, first = c < half;
  const int step = half / 4, partner = turns ? (first ? lane + step : lane - step) : lane;
  float gq[4], gk[4];
  float2 cs[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    gq[e] = in && wq != nullptr ? wq[c + e] : 1.f;
    gk[e] = in && wk != nullptr ? wk[c + e] : 1.f;
    cs[e] = make_float2(1.f, 0.f);
    if (turns && (!INTERLEAVED || e < 2)) cs[e] = rot[(size_t)row * ldr + (INTERLEAVED ? (c >> 1) + e : (first ? c : c - half) + e)];
    if (!INTERLEAVED && first) cs[e].y = -cs[e].y;
  }
  for (int u0 = warp; u0 < heads; u0 += QK_U * nw) {
    float v[QK_U][4];
#pragma unroll
    for (int i = 0; i < QK_U; ++i) {
      const int u = u0 + i * nw;
      v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
      if (u < heads && in) ldv<4>(src + (size_t)u * D + c, v[i]);
    }
#pragma unroll
    for (int i = 0; i < QK_U; ++i) {
      const int u = u0 + i * nw;
      if (u >= heads) break;
      const float ss = warp_sum(v[i][0] * v[i][0] + v[i][1] * v[i][1] + v[i][2] * v[i][2] + v[i][3] * v[i][3]);
      const bool is_q = u < Hq;
      float rstd = (is_q ? wq : wk) != nullptr || x2.unit ? 1.f / sqrtf(ss / D + eps) : 1.f;
      if (!is_q && x2.kf != nullptr) {
        if (lane == 0) x2.kf[(size_t)slot * Hkv + u - Hq] = rstd;
        rstd = 1.f;
      }
      if (is_q && x2.qf != nullptr) rstd *= x2.qf[u];
      float x[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = v[i][e] * rstd * (is_q ? gq[e] : gk[e]);
      if constexpr (INTERLEAVED) {
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const float a = x[e], b = x[e + 1];
          x[e] = a * cs[e / 2].x - b * cs[e / 2].y;
          x[e + 1] = b * cs[e / 2].x + a * cs[e / 2].y;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float o = __shfl_sync(0xffffffffu, x[e], partner);
          x[e] = x[e] * cs[e].x + o * cs[e].y;
        }
      }
      if (in) stv<4>((is_q ? q + ((size_t)row * Hq + u) * D : kc + ((size_t)slot * Hkv + u - Hq) * D) + c, x);
    }
  }
  if (slot >= 0) {
    const T* sv = src + (size_t)(Hq + Hkv) * D;
    for (int i = threadIdx.x * 4; i < nv; i += blockDim.x * 4) {
      float v[4];
      ldv<4>(sv + i, v);
      stv<4>(vc + (size_t)slot * nv + i, v);
    }
  }
}

// z rows: queries [H, D + 2 half] | latent [C] | shared key part [2 half] | anything. Cache rows: latent | key part.
template <typename T, int V, bool INTERLEAVED>
__global__ void __launch_bounds__(256)
latent_rope_append_kernel(T* __restrict__ z, long long ld, const float* __restrict__ wc, const float2* __restrict__ rot, int ldr, int half,
                          const int* __restrict__ slots, T* __restrict__ cache, int H, int D, int C, float eps) {
  __shared__ float red[8];
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, slot = slots[row];
  T* src = z + (size_t)row * ld;
  const float2* cs = rot + (size_t)row * ldr;
  auto turn = [&](const T* from, T* to, int i) {
    const int a = INTERLEAVED ? 2 * i : i, b = INTERLEAVED ? 2 * i + 1 : i + half;
    const float u = ldf(from + a), v = ldf(from + b);
    const float2 r = cs[i];
    stf(to + a, u * r.x - v * r.y);
    stf(to + b, v * r.x + u * r.y);
  };
  if constexpr (V == 8 && INTERLEAVED) {                      // four pairs at a time
    const int per = half / 4;
    for (int k = tid; k < H * per; k += 256) {
      const int h = k / per, c = (k - h * per) * 8;
      T* p = src + (size_t)h * (D + 2 * half) + D + c;
      float v[8];
      ldv<8>(p, v);
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        const float2 r = cs[(c + e) >> 1];
        const float a = v[e], b = v[e + 1];
        v[e] = a * r.x - b * r.y;
        v[e + 1] = b * r.x + a * r.y;
      }
      stv<8>(p, v);
    }
  } else {
    for (int k = tid; k < H * half; k += 256) {
      const int h = k / half;
      T* p = src + (size_t)h * (D + 2 * half) + D;
      turn(p, p, k - h * half);
    }
  }
  if (slot < 0) return;
  const T* lat = src + (size_t)H * (D + 2 * half);
  T* dst = cache + (size_t)slot * (C + 2 * half);
  for (int i = tid; i < half; i += 256) turn(lat + C, dst + C, i);
  float ss = 0.f;
  for (int c = tid * V; c < C; c += 256 * V) {
    float v[V];
    ldv<V>(lat + c, v);
    for (int e = 0; e < V; ++e) ss += v[e] * v[e];
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float rstd = 1.f / sqrtf(ss / C + eps);
  for (int c = tid * V; c < C; c += 256 * V) {
    float v[V], w[V];
    ldv<V>(lat + c, v);
    ldv<V>(wc + c, w);
    for (int e = 0; e < V; ++e) v[e] = v[e] * rstd * w[e];
    stv<V>(dst + c, v);
  }
}

}  // namespace ab2

#define AB2_ROT(VV, IL, ...)                                        \
  do {                                                              \
    constexpr int V = VV;                                           \
    if (IL) { constexpr bool INTER = true; __VA_ARGS__; }           \
    else { constexpr bool INTER = false; __VA_ARGS__; }             \
  } while (0)
#define AB2_ROT_TYPED(dt, v8, v4, IL, ...)                                            \
  do {                                                                                \
    if ((dt) == 0) {                                                                  \
      using T = __nv_bfloat16;                                                        \
      if (v8) AB2_ROT(8, IL, __VA_ARGS__); else if (v4) AB2_ROT(4, IL, __VA_ARGS__);  \
      else AB2_ROT(1, IL, __VA_ARGS__);                                               \
    } else {                                                                          \
      using T = float;                                                                \
      if (v4) AB2_ROT(4, IL, __VA_ARGS__); else AB2_ROT(1, IL, __VA_ARGS__);          \
    }                                                                                 \
  } while (0)

extern "C" {
using namespace ab2;

// out [R, P] (cos, sin) times mult; freq [P] double, in turns per position.
int ab2_rotary_table(const int* pos, const double* freq, const float* mult, void* out, int R, int P, void* stream) {
  if (R <= 0 || P <= 0) return 0;
  const long long n = (long long)R * P, g = (n + 255) / 256;
  launch_pdl(rotary_table_kernel, dim3((unsigned)(g < 148 * 8 ? g : 148 * 8)), dim3(256), 0, (cudaStream_t)stream, pos, freq, mult, (float2*)out, n, P);
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

// z rows q [Hq, D] | k [Hkv, D] | v [nv]; q [R, Hq, D], kc [S, Hkv, D], vc [S, nv]; wq / wk [D] or null (no norm); rot: the step's
// table from this mixer's column on, ldr pairs from row to row; the first 2 half numbers of every head turn. slot < 0: nothing cached.
// unit: norms without weights. qf [Hq] or null: factors of the queries. kf [S, Hkv] or null: keys are stored as they are (then no turn), kf
// gets what norms them.
int ab2_qk_head_norm_append(const void* z, long long ld, const float* wq, const float* wk, const void* rot, int ldr, int half, int interleaved,
                            const int* slots, void* q, void* kc, void* vc, int R, int Hq, int Hkv, int D, int nv, float eps, int unit, const float* qf,
                            float* kf, int dt, void* stream) {
  if (R <= 0) return 0;
  if ((half > 0 && rot == nullptr) || (kf && (half > 0 || wk || !unit))) return 11;
  const QkExtra x2{qf, kf, unit};
  const size_t smem = (size_t)8 * ((D + 3) & ~3) * 4;
  if (2 * half > D || half < 0 || smem > 48 * 1024) return 10;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) {
    return D % v == 0 && nv % v == 0 && ld % v == 0 && (interleaved ? 2 * half : half) % v == 0 && aligned_to(z, v * eb) && aligned_to(q, v * eb) &&
           aligned_to(kc, v * eb) && aligned_to(vc, v * eb) && aligned_to(wq, 16) && aligned_to(wk, 16);
  };
  if (D <= 128 && fits(4)) {
    auto go = [&](auto t, auto inter) {
      using T = decltype(t);
      launch_pdl(qk_head_norm_append_lanes_kernel<T, decltype(inter)::value>, dim3(R), dim3(256), 0, (cudaStream_t)stream, (const T*)z, ld, wq, wk,
                 (const float2*)rot, ldr, half, slots, (T*)q, (T*)kc, (T*)vc, Hq, Hkv, D, nv, eps, x2);
    };
    if (dt == 0 && interleaved) go(__nv_bfloat16(), std::true_type());
    else if (dt == 0) go(__nv_bfloat16(), std::false_type());
    else if (interleaved) go(0.f, std::true_type());
    else go(0.f, std::false_type());
    return cudaGetLastError() == cudaSuccess ? 0 : 1;
  }
  AB2_ROT_TYPED(dt, fits(8), fits(4), interleaved, {
    launch_pdl(qk_head_norm_append_kernel<T, V, INTER>, dim3(R), dim3(256), smem, (cudaStream_t)stream, (const T*)z, ld, wq, wk, (const float2*)rot, ldr,
               half, slots, (T*)q, (T*)kc, (T*)vc, Hq, Hkv, D, nv, eps, x2);
  });
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

// z rows q [H, D + 2 half] (turned in place) | latent [C] | key part [2 half]; cache [S, C + 2 half]; wc [C].
int ab2_latent_rope_append(void* z, long long ld, const float* wc, const void* rot, int ldr, int half, int interleaved, const int* slots, void* cache,
                           int R, int H, int D, int C, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  if (half < 1 || C < 1) return 10;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) {
    return C % v == 0 && D % v == 0 && (2 * half) % v == 0 && ld % v == 0 && aligned_to(z, v * eb) && aligned_to(cache, v * eb) && aligned_to(wc, 16);
  };
  AB2_ROT_TYPED(dt, fits(8), fits(4), interleaved, {
    launch_pdl(latent_rope_append_kernel<T, V, INTER>, dim3(R), dim3(256), 0, (cudaStream_t)stream, (T*)z, ld, wc, (const float2*)rot, ldr, half, slots,
               (T*)cache, H, D, C, eps);
  });
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}
}
