// minGRU: an element-wise recurrence with gates made from the token alone, not from the state; on per-request state slots:
//   z = sigmoid(zr + bz);  c = u + 1/2 for u = ur + bu >= 0, else sigmoid(u);  S = (1 - z) S + z c;  out = S * silu(g)
// Gates, candidates and states are fp32; rows of the projections z | u | g and the output are bf16 or fp32.
//
//   min_gru_decode_kernel    single-token rows: one pass over state and row
//   min_gru_portion_kernel   portions: a CTA walks down a tile of channels, 64 rows a round, its data read once and fetched rounds
//                            ahead. Every warp scans 8 rows; (product of 1 - z, state from zero) is chained over the warps in shared
//                            memory. Where entries and tiles are too few to fill the GPU, the CTAs of a cluster take 64 rows
//                            each, chained through distributed shared memory
#include <cooperative_groups.h>

#include <type_traits>

#include "mixer_common.cuh"

namespace ab2 {

__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Biases of a channel, also in base-2 units.
struct GruBias {
  float z, u, z2, u2;
  __device__ __forceinline__ void set(float bz, float bu) {
    z = bz; u = bu;
    z2 = bz * -1.4426950408889634f; u2 = bu * -1.4426950408889634f;
  }
};

// 1 - z and z c from the projections' numbers. FAST: two exponentials of at most 2^60 and one reciprocal of both denominators.
template <bool FAST>
__device__ __forceinline__ void gru_values(float zr, float ur, const GruBias& b, float& keep, float& in) {
  const float u = ur + b.u;
  if constexpr (FAST) {
    const float ez = fast_exp2(fminf(fmaf(zr, -1.4426950408889634f, b.z2), 60.f)), eu = fast_exp2(fminf(fmaf(ur, -1.4426950408889634f, b.u2), 60.f));
    const float dz = 1.f + ez, du = 1.f + eu, r = fast_rcp(dz * du), z = r * du;
    keep = ez * z;
    in = z * (u >= 0.f ? u + 0.5f : r * dz);
  } else {
    const float zl = zr + b.z;
    keep = sigmoid_t<false>(-zl);
    in = sigmoid_t<false>(zl) * (u >= 0.f ? u + 0.5f : sigmoid_t<false>(u));
  }
}

// silu; an infinite exponential gives zero
template <bool FAST>
__device__ __forceinline__ float gru_gate(float g) {
  if constexpr (FAST) return g * fast_rcp(1.f + fast_exp2(g * -1.4426950408889634f));
  return silu_t<false>(g);
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
      GruBias b;
      b.set(bz[v], bu[v]);
      float keep, in;
      gru_values<FAST>(z[v], u[v], b, keep, in);
      h[v] = keep * h[v] + in;
    }
    stv<V>(st, h);
#pragma unroll
    for (int v = 0; v < V; ++v) h[v] *= gru_gate<FAST>(g[v]);
  }
  stv<V>(out + row * ldo + c, h);
}

// A lane has V neighbouring channels, a warp GRU_PER rows, a CTA 32 V channels and GRU_ROWS rows per round; the CTAS CTAs of a cluster
// take consecutive rows. What a thread reads is on its way GRU_STAGES - 1 rounds ahead.
constexpr int GRU_WARPS = 8, GRU_PER = 8, GRU_ROWS = GRU_WARPS * GRU_PER, GRU_STAGES = 3;

template <typename T, int V>
struct GruCfg {
  static constexpr int C = 32 * V, N = V * (int)sizeof(T);
  static constexpr int PIECE = GRU_WARPS * 32 * N;              // one number of every row of every thread
  static constexpr int STAGE = 3 * GRU_PER * PIECE;             // z, u, g
  static constexpr int SMEM = GRU_STAGES * STAGE;
};

template <typename T, int V, int CTAS>
__device__ __forceinline__ void min_gru_portion_body(const T* __restrict__ zug, long long ld, const float* __restrict__ bias, const int* __restrict__ cu,
                                                     const int* __restrict__ start, const int* __restrict__ state, int n_dec, float* __restrict__ S,
                                                     T* __restrict__ out, long long ldo, int W) {
  namespace cg = cooperative_groups;
  using Cfg = GruCfg<T, V>;
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int C = Cfg::C;
  extern __shared__ __align__(16) unsigned char ring[];
  __shared__ float s_end[2][2][GRU_WARPS][C];           // every warp's (product, state from zero); rounds take turns
  __shared__ float s_cta[2][2][C];                      // this CTA's, for the cluster
  __shared__ float s_in[2][C];                          // state before this CTA's rows
  pdl_wait();
  pdl_trigger();
  const int e = n_dec + blockIdx.y, rank = blockIdx.x % CTAS, c0 = blockIdx.x / CTAS * C;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, k = lane * V, c = c0 + k;
  const bool in = c < W;                                // (W is a multiple of V)
  const int r0 = cu[e], r1 = cu[e + 1], slot = state[e];
  GruBias bi[V];
  float h0[V];                                          // state before the round (CTAS > 1: of warp 0 only)
#pragma unroll
  for (int v = 0; v < V; ++v) {
    bi[v].set(in ? bias[c + v] : 0.f, in ? bias[W + c + v] : 0.f);
    h0[v] = in && slot >= 0 && start[e] > 0 ? S[(size_t)slot * W + c + v] : 0.f;
  }
  const int mine = r0 + rank * GRU_ROWS + warp * GRU_PER;
  auto fetch = [&](int round) {
    const int row = mine + round * CTAS * GRU_ROWS;
    unsigned char* dst = ring + round % GRU_STAGES * Cfg::STAGE + tid * Cfg::N;
    auto copy = [&](auto all) {
      const T* p = zug + row * ld + c;
#pragma unroll
      for (int i = 0; i < GRU_PER; ++i, p += ld)
        if (decltype(all)::value || row + i < r1) {
#pragma unroll
          for (int j = 0; j < 3; ++j) copy_own<Cfg::N>(dst + (j * GRU_PER + i) * Cfg::PIECE, p + j * W);
        }
    };
    if (in) {
      if (row + GRU_PER <= r1) copy(std::true_type());
      else copy(std::false_type());
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < GRU_STAGES - 1; ++i) fetch(i);
  int round = 0;
  for (int base = r0; base < r1; base += CTAS * GRU_ROWS, ++round) {
    const int row = mine + base - r0, turn = round & 1;
    fetch(round + GRU_STAGES - 1);
    asm volatile("cp.async.wait_group %0;" ::"n"(GRU_STAGES - 1) : "memory");
    const unsigned char* got = ring + round % GRU_STAGES * Cfg::STAGE + tid * Cfg::N;
    // from zero, rows after the portion's end keep the state as it is: a is the running product, x the state
    float a[GRU_PER][V], x[GRU_PER][V];
    const bool whole = row + GRU_PER <= r1;             // (of the warp)
    auto scan = [&](auto all) {
#pragma unroll
      for (int i = 0; i < GRU_PER; ++i) {
        float z[V], u[V];
        ldv<V>(reinterpret_cast<const T*>(got + i * Cfg::PIECE), z);
        ldv<V>(reinterpret_cast<const T*>(got + (GRU_PER + i) * Cfg::PIECE), u);
#pragma unroll
        for (int v = 0; v < V; ++v) {
          float keep = 1.f, add = 0.f;
          if (decltype(all)::value || row + i < r1) gru_values<FAST>(z[v], u[v], bi[v], keep, add);
          a[i][v] = i ? a[i - 1][v] * keep : keep;
          x[i][v] = i ? keep * x[i - 1][v] + add : add;
        }
      }
    };
    if (whole) scan(std::true_type());
    else scan(std::false_type());
#pragma unroll
    for (int v = 0; v < V; ++v) {
      s_end[turn][0][warp][k + v] = a[GRU_PER - 1][v];
      s_end[turn][1][warp][k + v] = x[GRU_PER - 1][v];
    }
    __syncthreads();
    float h[V];                                         // the state before this warp's rows
    if constexpr (CTAS == 1) {
#pragma unroll
      for (int w = 0; w < GRU_WARPS; ++w)
#pragma unroll
        for (int v = 0; v < V; ++v) {
          if (w == warp) h[v] = h0[v];
          h0[v] = s_end[turn][0][w][k + v] * h0[v] + s_end[turn][1][w][k + v];
        }
    } else {
      float P[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        P[v] = 1.f;
        h[v] = 0.f;
        for (int w = 0; w < warp; ++w) {
          h[v] = s_end[turn][0][w][k + v] * h[v] + s_end[turn][1][w][k + v];
          P[v] *= s_end[turn][0][w][k + v];
        }
        if (warp == GRU_WARPS - 1) {
          s_cta[turn][0][k + v] = P[v] * a[GRU_PER - 1][v];
          s_cta[turn][1][k + v] = a[GRU_PER - 1][v] * h[v] + x[GRU_PER - 1][v];
        }
      }
      cg::this_cluster().sync();
      if (warp == 0) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          float q[CTAS], y[CTAS];
#pragma unroll
          for (int i = 0; i < CTAS; ++i) {
            const float* far = cg::this_cluster().map_shared_rank(&s_cta[turn][0][0], i);
            q[i] = far[k + v];
            y[i] = far[C + k + v];
          }
#pragma unroll
          for (int i = 0; i < CTAS; ++i) {
            if (i == rank) s_in[turn][k + v] = h0[v];
            h0[v] = q[i] * h0[v] + y[i];
          }
        }
      }
      __syncthreads();
#pragma unroll
      for (int v = 0; v < V; ++v) h[v] += P[v] * s_in[turn][k + v];
    }
    auto emit = [&](auto all) {
      T* to = out + row * ldo + c;
#pragma unroll
      for (int i = 0; i < GRU_PER; ++i, to += ldo)
        if (decltype(all)::value || row + i < r1) {
          float o[V];
          ldv<V>(reinterpret_cast<const T*>(got + (2 * GRU_PER + i) * Cfg::PIECE), o);
#pragma unroll
          for (int v = 0; v < V; ++v) o[v] = (x[i][v] + a[i][v] * h[v]) * gru_gate<FAST>(o[v]);
          stv<V>(to, o);
        }
    };
    if (in) {
      if (whole) emit(std::true_type());
      else emit(std::false_type());
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  // (every CTA of the cluster has read the old state before the first round's barrier)
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
                          int ctas, float* S, T* out, long long ldo, int W, cudaStream_t s) {
  if (n_dec > 0) {
    const bool vec = W % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && aligned_to(zug, 4 * sizeof(T)) && aligned_to(out, 4 * sizeof(T)) && aligned_to(bias, 16) &&
                     aligned_to(S, 16);
    if (vec) launch_pdl(min_gru_decode_kernel<T, 4>, dim3((W / 4 + 127) / 128, n_dec), dim3(128), 0, s, zug, ld, bias, start, state, S, out, ldo, W);
    else launch_pdl(min_gru_decode_kernel<T, 1>, dim3((W + 127) / 128, n_dec), dim3(128), 0, s, zug, ld, bias, start, state, S, out, ldo, W);
  }
  int rc = 0;
  if (E > n_dec) {
    const int n = E - n_dec, per = (nb + n - 1) / n;          // blocks of 64 rows that a portion has on average
    auto go = [&](auto v) -> int {
      constexpr int V = decltype(v)::value, SMEM = GruCfg<T, V>::SMEM;
      const int tiles = (W + 32 * V - 1) / (32 * V);
      // as few CTAs per cluster as leave no SM idle
      int k = ctas;
      if (k == 0)
        for (k = 1; k < 8 && 2 * k <= per && (long long)tiles * n * k < 148; k *= 2) {}
      auto run = [&](auto kern, ab2host::DevState& st) -> int {
        if (ab2host::prepare_launch(kern, SMEM, st, nullptr)) return 300;
        launch_pdl(kern, dim3(k * tiles, n), dim3(GRU_WARPS * 32), (size_t)SMEM, s, zug, ld, bias, cu, start, state, n_dec, S, out, ldo, W);
        return 0;
      };
      static ab2host::DevState st1, st2, st4, st8;
      switch (k) {
        case 1: return run(min_gru_portion_kernel<T, V>, st1);
        case 2: return run(min_gru_portion_cluster_kernel<T, V, 2>, st2);
        case 4: return run(min_gru_portion_cluster_kernel<T, V, 4>, st4);
        case 8: return run(min_gru_portion_cluster_kernel<T, V, 8>, st8);
        default: return 12;
      }
    };
    const bool pairs = W % 2 == 0 && ld % 2 == 0 && ldo % 2 == 0 && aligned_to(zug, 2 * sizeof(T)) && aligned_to(out, 2 * sizeof(T));
    if constexpr (sizeof(T) == 2)
      if (pairs) rc = go(std::integral_constant<int, 2>());
    if (sizeof(T) != 2 || !pairs) rc = go(std::integral_constant<int, 1>());
  }
  if (rc) return rc;
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Rows z | u | g of W numbers each (ld elements from row to row); bias [2 W] of z, then u; S [slots, W]; out [R, W] (ldo). The first n_dec of
// the E entries have one row each, the others nb blocks of up to 64 rows in all. ctas: cluster size of the portions (1, 2, 4, 8), 0: by size.
int ab2_min_gru(const void* zug, long long ld, const float* bias, const int* cu, const int* start, const int* state, int n_dec, int E, int nb, int ctas,
                float* S, void* out, long long ldo, int W, int dt, void* stream) {
  if (E <= 0 || W <= 0) return 0;
  if (n_dec > 65535 || E - n_dec > 65535 || n_dec > E) return 11;
  if (dt == 0)
    return launch_min_gru((const __nv_bfloat16*)zug, ld, bias, cu, start, state, n_dec, E, nb, ctas, S, (__nv_bfloat16*)out, ldo, W, (cudaStream_t)stream);
  return launch_min_gru((const float*)zug, ld, bias, cu, start, state, n_dec, E, nb, ctas, S, (float*)out, ldo, W, (cudaStream_t)stream);
}
}
