// Element-wise gated recurrence whose gates read only the current token (minGRU), on per-request state slots:
//   z = sigmoid(zr + bz);  c = u + 1/2 for u = ur + bu >= 0, else sigmoid(u);  S = (1 - z) S + z c;  out = S * silu(g)
// Gates, candidates and states are fp32; rows of the projections z | u | g and the output are bf16 or fp32.
//
//   min_gru_decode_kernel    single-token rows: one pass over state and row
//   min_gru_portion_kernel   portions: the CTAs of a cluster take 64 rows each, so a tile of channels advances CTAS * 64 rows at a
//                            time with its data read once; inside a CTA every warp scans 8 rows, and (product of 1 - z, state
//                            from zero) is chained over the warps in shared memory and over the CTAs in distributed shared memory
#include <cooperative_groups.h>

#include "mixer_common.cuh"

namespace ab2 {

constexpr int GRU_ROWS = 64, GRU_WARPS = 8, GRU_PER = GRU_ROWS / GRU_WARPS;

template <bool FAST>
__device__ __forceinline__ void gru_values(float zl, float u, float& keep, float& in) {
  keep = sigmoid_t<FAST>(-zl);                                  // 1 - z
  in = sigmoid_t<FAST>(zl) * (u >= 0.f ? u + 0.5f : sigmoid_t<FAST>(u));
}

template <int V>
__device__ __forceinline__ void ld_pair(const float* p, float (&v)[V]) {
  if constexpr (V == 2) { const float2 a = *reinterpret_cast<const float2*>(p); v[0] = a.x; v[1] = a.y; }
  else v[0] = *p;
}
template <int V>
__device__ __forceinline__ void ld_pair(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 2) { const float2 a = unpack_bf16(*reinterpret_cast<const uint32_t*>(p)); v[0] = a.x; v[1] = a.y; }
  else v[0] = __bfloat162float(*p);
}
template <int V>
__device__ __forceinline__ void st_pair(float* p, const float (&v)[V]) {
  if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}
template <int V>
__device__ __forceinline__ void st_pair(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16(v[0], v[1]);
  else *p = __float2bfloat16(v[0]);
}

template <typename T, int V>
__global__ void __launch_bounds__(128)
min_gru_decode_kernel(const T* __restrict__ zug, long long ld, const float* __restrict__ bias, const int* __restrict__ start,
                      const int* __restrict__ state, float* __restrict__ S, T* __restrict__ out, long long ldo, int W) {
  constexpr bool FAST = sizeof(T) == 2;
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= W) return;
  const int slot = state[row];
  float h[V];
#pragma unroll
  for (int v = 0; v < V; ++v) h[v] = 0.f;
  if (slot >= 0) {
    float* st = S + (size_t)slot * W + c;
    const T* r = zug + row * ld + c;
    float z[V], u[V], g[V], bz[V], bu[V];
    ldv<V>(r, z);
    ldv<V>(r + W, u);
    ldv<V>(r + 2 * W, g);
    ldv<V>(bias + c, bz);
    ldv<V>(bias + W + c, bu);
    if (start[row] > 0) ldv<V>(st, h);
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float keep, in;
      gru_values<FAST>(z[v] + bz[v], u[v] + bu[v], keep, in);
      h[v] = keep * h[v] + in;
    }
    stv<V>(st, h);
#pragma unroll
    for (int v = 0; v < V; ++v) h[v] *= silu_t<FAST>(g[v]);
  }
  stv<V>(out + row * ldo + c, h);
}

// CTAS: cluster size along x. A lane has V neighbouring channels, a CTA 32 V.
template <typename T, int V, int CTAS>
__device__ __forceinline__ void min_gru_portion_body(const T* __restrict__ zug, long long ld, const float* __restrict__ bias, const int* __restrict__ cu,
                                                     const int* __restrict__ start, const int* __restrict__ state, int n_dec, float* __restrict__ S,
                                                     T* __restrict__ out, long long ldo, int W) {
  namespace cg = cooperative_groups;
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int C = 32 * V;
  __shared__ float s_end[2][GRU_WARPS][C];              // every warp's (product, state from zero)
  __shared__ float s_cta[2][2][C];                      // this CTA's, for the cluster; two rounds take turns
  __shared__ float s_in[2][C];                          // state before this CTA's rows, state after the round
  pdl_wait();
  pdl_trigger();
  const int e = n_dec + blockIdx.y, rank = blockIdx.x % CTAS, c0 = blockIdx.x / CTAS * C;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, k = lane * V, c = c0 + k;
  const bool in = c < W;                                // (W is a multiple of V)
  const int r0 = cu[e], r1 = cu[e + 1], slot = state[e];
  float bz[V], bu[V], h0[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    bz[v] = in ? bias[c + v] : 0.f;
    bu[v] = in ? bias[W + c + v] : 0.f;
    h0[v] = in && slot >= 0 && start[e] > 0 ? S[(size_t)slot * W + c + v] : 0.f;      // kept by warp 0
  }
  int turn = 0;
  for (int base = r0; base < r1; base += CTAS * GRU_ROWS, turn ^= 1) {
    const int row = base + rank * GRU_ROWS + warp * GRU_PER;
    float a[GRU_PER][V], x[GRU_PER][V], g[GRU_PER][V];
#pragma unroll
    for (int i = 0; i < GRU_PER; ++i) {
#pragma unroll
      for (int v = 0; v < V; ++v) a[i][v] = x[i][v] = g[i][v] = 0.f;
      if (in && row + i < r1) {
        const T* p = zug + (row + i) * ld + c;
        ld_pair<V>(p, a[i]);
        ld_pair<V>(p + W, x[i]);
        ld_pair<V>(p + 2 * W, g[i]);
      }
    }
    // from zero, rows after the portion's end keep the state as it is: a becomes the running product, x the state
#pragma unroll
    for (int i = 0; i < GRU_PER; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float keep = 1.f, add = 0.f;
        if (row + i < r1) gru_values<FAST>(a[i][v] + bz[v], x[i][v] + bu[v], keep, add);
        a[i][v] = i ? a[i - 1][v] * keep : keep;
        x[i][v] = i ? keep * x[i - 1][v] + add : add;
      }
#pragma unroll
    for (int v = 0; v < V; ++v) {
      s_end[0][warp][k + v] = a[GRU_PER - 1][v];
      s_end[1][warp][k + v] = x[GRU_PER - 1][v];
    }
    __syncthreads();
    float P[V], h[V];                                   // of the warps before this one
#pragma unroll
    for (int v = 0; v < V; ++v) {
      P[v] = 1.f;
      h[v] = 0.f;
      for (int w = 0; w < warp; ++w) {
        h[v] = s_end[0][w][k + v] * h[v] + s_end[1][w][k + v];
        P[v] *= s_end[0][w][k + v];
      }
      if (warp == GRU_WARPS - 1) {
        s_cta[turn][0][k + v] = P[v] * a[GRU_PER - 1][v];
        s_cta[turn][1][k + v] = a[GRU_PER - 1][v] * h[v] + x[GRU_PER - 1][v];
      }
    }
    if constexpr (CTAS > 1) cg::this_cluster().sync();
    else __syncthreads();
    if (warp == 0) {
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float q[CTAS], y[CTAS];
#pragma unroll
        for (int i = 0; i < CTAS; ++i) {
          const float* far = &s_cta[turn][0][0];
          if constexpr (CTAS > 1) far = cg::this_cluster().map_shared_rank(far, i);
          q[i] = far[k + v];
          y[i] = far[C + k + v];
        }
#pragma unroll
        for (int i = 0; i < CTAS; ++i) {
          if (i == rank) s_in[0][k + v] = h0[v];
          h0[v] = q[i] * h0[v] + y[i];
        }
        s_in[1][k + v] = h0[v];
      }
    }
    __syncthreads();
#pragma unroll
    for (int v = 0; v < V; ++v) h[v] += P[v] * s_in[0][k + v];           // the state before this warp's rows
#pragma unroll
    for (int i = 0; i < GRU_PER; ++i)
      if (in && row + i < r1) {
        float o[V];
#pragma unroll
        for (int v = 0; v < V; ++v) o[v] = (x[i][v] + a[i][v] * h[v]) * silu_t<FAST>(g[i][v]);
        st_pair<V>(out + (row + i) * ldo + c, o);
      }
  }
  // every CTA of the cluster has read the old state before the first round's barrier
  if (rank == 0 && warp == 0 && in && slot >= 0)
#pragma unroll
    for (int v = 0; v < V; ++v) S[(size_t)slot * W + c + v] = h0[v];
  if constexpr (CTAS > 1) cg::this_cluster().sync();    // nobody leaves while its shared memory is being read
}

#define AB2_GRU_PARAMS                                                                                                                              \
  const T *__restrict__ zug, long long ld, const float *__restrict__ bias, const int *__restrict__ cu, const int *__restrict__ start,               \
      const int *__restrict__ state, int n_dec, float *__restrict__ S, T *__restrict__ out, long long ldo, int W
template <typename T, int V>
__global__ void __launch_bounds__(GRU_WARPS * 32)
min_gru_portion_kernel(AB2_GRU_PARAMS) {
  min_gru_portion_body<T, V, 1>(zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
}
template <typename T, int V, int CTAS>
__global__ void __cluster_dims__(CTAS, 1, 1) __launch_bounds__(GRU_WARPS * 32)
min_gru_portion_cluster_kernel(AB2_GRU_PARAMS) {
  min_gru_portion_body<T, V, CTAS>(zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
}
#undef AB2_GRU_PARAMS

template <typename T>
static int launch_min_gru(const T* zug, long long ld, const float* bias, const int* cu, const int* start, const int* state, int n_dec, int E, int nb,
                          float* S, T* out, long long ldo, int W, cudaStream_t s) {
  if (n_dec > 0) {
    const bool vec = W % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && aligned_to(zug, 4 * sizeof(T)) && aligned_to(out, 4 * sizeof(T)) && aligned_to(bias, 16) &&
                     aligned_to(S, 16);
    if (vec) launch_pdl(min_gru_decode_kernel<T, 4>, dim3((W / 4 + 127) / 128, n_dec), dim3(128), 0, s, zug, ld, bias, start, state, S, out, ldo, W);
    else launch_pdl(min_gru_decode_kernel<T, 1>, dim3((W + 127) / 128, n_dec), dim3(128), 0, s, zug, ld, bias, start, state, S, out, ldo, W);
  }
  if (E > n_dec) {
    const int per = (nb + E - n_dec - 1) / (E - n_dec);       // blocks of 64 rows that a portion has on average
    auto go = [&](auto v) {
      constexpr int V = decltype(v)::value;
      const int tiles = (W + 32 * V - 1) / (32 * V);
      const dim3 th(GRU_WARPS * 32);
      if (per <= 1) launch_pdl(min_gru_portion_kernel<T, V>, dim3(tiles, E - n_dec), th, 0, s, zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
      else if (per <= 4) launch_pdl(min_gru_portion_cluster_kernel<T, V, 4>, dim3(4 * tiles, E - n_dec), th, 0, s, zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
      else launch_pdl(min_gru_portion_cluster_kernel<T, V, 8>, dim3(8 * tiles, E - n_dec), th, 0, s, zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
    };
    if (W % 2 == 0 && ld % 2 == 0 && ldo % 2 == 0 && aligned_to(zug, 2 * sizeof(T)) && aligned_to(out, 2 * sizeof(T))) go(std::integral_constant<int, 2>());
    else go(std::integral_constant<int, 1>());
  }
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Rows z | u | g of W numbers each (ld elements from row to row); bias [2 W] of z, then u; S [slots, W]; out [R, W] (ldo). The first n_dec of
// the E entries have one row each, the others nb blocks of up to 64 rows in all.
int ab2_min_gru(const void* zug, long long ld, const float* bias, const int* cu, const int* start, const int* state, int n_dec, int E, int nb, float* S,
                void* out, long long ldo, int W, int dt, void* stream) {
  if (E <= 0 || W <= 0) return 0;
  if (n_dec > 65535 || E - n_dec > 65535 || n_dec > E) return 11;
  if (dt == 0)
    return launch_min_gru((const __nv_bfloat16*)zug, ld, bias, cu, start, state, n_dec, E, nb, S, (__nv_bfloat16*)out, ldo, W, (cudaStream_t)stream);
  return launch_min_gru((const float*)zug, ld, bias, cu, start, state, n_dec, E, nb, S, (float*)out, ldo, W, (cudaStream_t)stream);
}
}
