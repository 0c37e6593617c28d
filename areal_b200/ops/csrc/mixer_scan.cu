// Recurrences of mixer stacks on per-request state slots: the RG-LRU (block-diagonal gates on tensor cores, then a
// blocked linear scan) and the Mamba-2 state update. Gates, decays and states are fp32 throughout.
#include "mixer_common.cuh"

namespace ab2 {

// ------------------------------------------------------------------ RG-LRU gates
// One CTA: 64 rows x 32 channels of one block of the block-diagonal gate matrices, both gates at once (64 product
// columns: 32 of r, 32 of i), so the thread that holds r of a channel also holds its i. The epilogue turns the two
// logits into the decay a = exp(-8 r softplus(lam)) and the input sqrt(1 - a^2) i u. Single-token rows advance their
// state at once; for portions the 64 rows are one block of the scan, and the CTA scans them from zero before it stores
// (running product of a, state from zero).
constexpr int GT_R = 64, GT_C = 32, GT_K = 64;

// Operand stages: bf16 operands are brought in by asynchronous copies, several 64-wide pieces ahead (single-token rows:
// few CTAs, all pieces of a 256-wide block at once); the 32-bit form uses one stage.
template <typename T, bool DECODE>
struct GateCfg {
  static constexpr int LD = sizeof(T) == 2 ? GT_K + 8 : GT_K + 1;          // padded rows: no bank conflicts on fragment reads
  static constexpr int NS = sizeof(T) == 2 ? (DECODE ? 4 : 2) : 1;
  static constexpr int OP_BYTES = (GT_R + 2 * GT_C) * LD * (int)sizeof(T);
};

struct GateEpi {
  const float *gb, *lam, *yb;
  const int *start, *state;
  const int4* blocks;
  float *S, *a, *x, *carry;
  int W, bs, nblk, row0, nb;
};

// decay and scaled input of one channel; nsp = -8 softplus(lam)
template <bool FAST>
__device__ __forceinline__ void gate_values(float zr, float zi, float nsp, float u, float& a, float& xin) {
  const float la = nsp * sigmoid_t<FAST>(zr);
  a = exp_t<FAST>(la);
  xin = sqrtf(-expm1_neg<FAST>(2.f * la)) * sigmoid_t<FAST>(zi) * u;
}

template <typename T, bool DECODE>
__global__ void __launch_bounds__(128)
rglru_gate_kernel(const T* __restrict__ u, const T* __restrict__ y, long long ldy, const T* __restrict__ gw, GateEpi p, T* __restrict__ out, int R) {
  constexpr bool MMA = sizeof(T) == 2;
  constexpr int LD = GateCfg<T, DECODE>::LD, NS = GateCfg<T, DECODE>::NS, OP_BYTES = GateCfg<T, DECODE>::OP_BYTES;
  constexpr int SCAN_BYTES = DECODE ? 0 : 2 * GT_R * (GT_C + 1) * 4;       // a and x of the block, over the operands
  static_assert(NS * OP_BYTES >= SCAN_BYTES, "the scan's values fit over the operand stages");
  extern __shared__ __align__(16) unsigned char s_raw[];     // NS operand stages
  __shared__ float s_par[3][GT_C];                       // r bias, i bias, -8 softplus(lam)
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cpb = (p.bs + GT_C - 1) / GT_C;              // channel tiles per block
  const int blk = blockIdx.x / cpb, c0 = (blockIdx.x % cpb) * GT_C;
  int r0 = blockIdx.y * GT_R;
  if constexpr (!DECODE) {
    const int4 b = p.blocks[blockIdx.y];
    r0 = b.y - p.row0;
    R = r0 + b.z;
  }
  if (tid < GT_C && c0 + tid < p.bs) {
    const int ch = blk * p.bs + c0 + tid;
    s_par[0][tid] = p.gb[ch];
    s_par[1][tid] = p.gb[p.W + ch];
    s_par[2][tid] = -8.f * softplusf(p.lam[ch]);
  }
  const T zero = T(0.f);
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // element q of this thread's 16 results: row and channel of the tile (r in acc[q / 4][q % 4], i four columns on)
  auto rr_of = [&](int q) { return MMA ? warp * 16 + (lane >> 2) + ((q & 3) >> 1) * 8 : (tid >> 3) * 4 + (q & 3); };
  auto c_of = [&](int q) { return MMA ? (q >> 2) * 8 + (lane & 3) * 2 + (q & 1) : (tid & 7) + 8 * (q >> 2); };
  const bool vec = MMA && p.bs % 8 == 0 && p.W % 8 == 0;
  const int nk = (p.bs + GT_K - 1) / GT_K;
  auto copy = [&](int kt) {                                // piece kt of both operands into its stage (vec only)
    if (kt < nk) {
      const uint32_t dA = smem_u32(s_raw) + (kt % NS) * OP_BYTES, dB = dA + GT_R * LD * (int)sizeof(T);
      for (int i = tid; i < GT_R * (GT_K / 8); i += 128) {
        const int r = i / (GT_K / 8), kc = (i % (GT_K / 8)) * 8, k = kt * GT_K + kc;
        const int g = r >> 5, c = c0 + (r & 31);           // 2 x 32 weight rows: as many as there are token rows
        const bool oa = r0 + r < R && k < p.bs, ob = c < p.bs && k < p.bs;
        const T* pa = oa ? u + (size_t)(r0 + r) * p.W + blk * p.bs + k : u;
        const T* pb = ob ? gw + (((size_t)g * p.nblk + blk) * p.bs + c) * p.bs + k : gw;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dA + (r * LD + kc) * (int)sizeof(T)), "l"(pa), "r"(oa ? 16 : 0) : "memory");
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dB + (r * LD + kc) * (int)sizeof(T)), "l"(pb), "r"(ob ? 16 : 0) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (vec)
    for (int kt = 0; kt < NS - 1; ++kt) copy(kt);
  // single-token rows: what the epilogue needs is asked for before the products, all of it at once
  float ev_u[16], ev_y[16], ev_s[16];
  int ev_slot[16];
#pragma unroll
  for (int q = 0; q < 16; ++q) {
    const int row = r0 + rr_of(q), c = c0 + c_of(q), ch = blk * p.bs + c;
    const bool in = row < R && c < p.bs;
    ev_u[q] = in ? ldf(u + (size_t)row * p.W + ch) : 0.f;
    if constexpr (DECODE) {
      ev_slot[q] = in ? p.state[row] : -1;
      ev_y[q] = in ? ldf(y + (size_t)row * ldy + ch) + p.yb[ch] : 0.f;
      ev_s[q] = ev_slot[q] >= 0 && p.start[row] > 0 ? p.S[(size_t)ev_slot[q] * p.W + ch] : 0.f;
    }
  }
  for (int kt = 0; kt < nk; ++kt) {
    const int k0 = kt * GT_K;
    T* sA = reinterpret_cast<T*>(s_raw + (vec ? (kt % NS) * OP_BYTES : 0));
    T* sB = sA + GT_R * LD;
    if (vec) {
      copy(kt + NS - 1);                                   // its stage was read in the previous turn
      asm volatile("cp.async.wait_group %0;" ::"n"(NS - 1) : "memory");
    } else {
      for (int i = tid; i < GT_R * GT_K; i += 128) {
        const int r = i / GT_K, k = i % GT_K;
        sA[r * LD + k] = (r0 + r < R && k0 + k < p.bs) ? u[(size_t)(r0 + r) * p.W + blk * p.bs + k0 + k] : zero;
        const int g = r >> 5, c = c0 + (r & 31);
        sB[r * LD + k] = (c < p.bs && k0 + k < p.bs) ? gw[(((size_t)g * p.nblk + blk) * p.bs + c) * p.bs + k0 + k] : zero;
      }
    }
    __syncthreads();
    if constexpr (MMA) {
      const int gq = lane >> 2, tq = lane & 3;
      const uint32_t* A = reinterpret_cast<const uint32_t*>(sA);
      const uint32_t* B = reinterpret_cast<const uint32_t*>(sB);
      constexpr int LW = LD / 2;
#pragma unroll
      for (int kk = 0; kk < GT_K / 16; ++kk) {
        const int ar = (warp * 16 + gq) * LW + kk * 8 + tq;
        const uint32_t a0 = A[ar], a1 = A[ar + 8 * LW], a2 = A[ar + 4], a3 = A[ar + 8 * LW + 4];
#pragma unroll
        for (int t = 0; t < 8; ++t) {
          const int br = (t * 8 + gq) * LW + kk * 8 + tq;
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                       : "+f"(acc[t][0]), "+f"(acc[t][1]), "+f"(acc[t][2]), "+f"(acc[t][3])
                       : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(B[br]), "r"(B[br + 4]));
        }
      }
    } else {
      // thread = 4 rows x (4 channels of r and the same 4 of i): channels tx + 8 j
      const int tx = tid & 7, ty = tid >> 3;
      for (int k = 0; k < GT_K; ++k) {
        float av[4], bv[8];
#pragma unroll
        for (int i = 0; i < 4; ++i) av[i] = ldf(sA + (ty * 4 + i) * LD + k);
#pragma unroll
        for (int j = 0; j < 8; ++j) bv[j] = ldf(sB + (tx + 8 * j) * LD + k);
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[j][i] += av[i] * bv[j];
      }
    }
    __syncthreads();
  }
  float* s_a = reinterpret_cast<float*>(s_raw);
  float* s_x = s_a + GT_R * (GT_C + 1);
#pragma unroll
  for (int q = 0; q < 16; ++q) {
    const int rr = rr_of(q), c = c_of(q), row = r0 + rr;
    const bool in = row < R && c0 + c < p.bs;
    float a = 1.f, xin = 0.f;
    if (in) gate_values<MMA>(acc[q >> 2][q & 3] + s_par[0][c], acc[(q >> 2) + 4][q & 3] + s_par[1][c], s_par[2][c], ev_u[q], a, xin);
    if constexpr (DECODE) {
      if (in) {
        const int ch = blk * p.bs + c0 + c;
        const float h = a * ev_s[q] + xin;
        if (ev_slot[q] >= 0) p.S[(size_t)ev_slot[q] * p.W + ch] = h;
        stf(out + (size_t)row * p.W + ch, ev_slot[q] >= 0 ? h * gelu_tanh_t<MMA>(ev_y[q]) : 0.f);
      }
    } else {
      s_a[rr * (GT_C + 1) + c] = a;
      s_x[rr * (GT_C + 1) + c] = xin;
    }
  }
  if constexpr (!DECODE) {
    // a warp scans 16 of the 64 rows, a lane one channel; the warps' ends are chained through shared memory
    __shared__ float s_end[2][4][GT_C];
    __syncthreads();
    float pa[16], hx[16], P = 1.f, h = 0.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const int o = (warp * 16 + i) * (GT_C + 1) + lane;
      const float at = s_a[o];
      h = at * h + s_x[o];
      P *= at;
      pa[i] = P;
      hx[i] = h;
    }
    s_end[0][warp][lane] = P;
    s_end[1][warp][lane] = h;
    __syncthreads();
    float Pp = 1.f, hp = 0.f;
    for (int w = 0; w < warp; ++w) {
      hp = s_end[0][w][lane] * hp + s_end[1][w][lane];
      Pp *= s_end[0][w][lane];
    }
    if (c0 + lane < p.bs) {
      const int ch = blk * p.bs + c0 + lane;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const int row = r0 + warp * 16 + i;
        if (row < R) {
          p.a[(size_t)row * p.W + ch] = pa[i] * Pp;
          p.x[(size_t)row * p.W + ch] = hx[i] + pa[i] * hp;
        }
      }
      if (warp == 3) {                                     // rows past the block's end have a = 1, x = 0
        p.carry[(size_t)blockIdx.y * p.W + ch] = pa[15] * Pp;
        p.carry[((size_t)p.nb + blockIdx.y) * p.W + ch] = hx[15] + pa[15] * hp;
      }
    }
  }
}

// The states between the blocks of every portion (carry: product and state of each block, then the state before it),
// and the rows from their block's true start, gated on the way out. Row indices of `blocks` count from the first row of
// the step, a / x / y / out from row0.
__global__ void __launch_bounds__(128)
lru_carry_kernel(const int4* __restrict__ blocks, const int* __restrict__ start, const int* __restrict__ state, float* __restrict__ S,
                 float* __restrict__ carry, int nb, int W) {
  const int c = blockIdx.x * 128 + threadIdx.x, k0 = blockIdx.y;
  const int4 b0 = blocks[k0];
  if (c >= W || !b0.w) return;                            // one CTA row per entry: that of its first block
  float* st = S + (size_t)state[b0.x] * W + c;
  float h = start[b0.x] > 0 ? *st : 0.f;
  bool more = true;
  for (int k = k0; more; k += 8) {
    float A[8], x[8];
    int n = 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {                         // up to eight blocks' values before the chain of products
      const bool in = more && k + i < nb && blocks[k + i].x == b0.x;
      more = in;
      n += in;
      A[i] = in ? carry[(size_t)(k + i) * W + c] : 1.f;
      x[i] = in ? carry[((size_t)nb + k + i) * W + c] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i < n) carry[(size_t)(k + i) * W + c] = h;      // state before the block
      h = A[i] * h + x[i];
    }
  }
  *st = h;
}

template <typename T, int V>
__global__ void __launch_bounds__(128)
lru_apply_kernel(const float* __restrict__ a, const float* __restrict__ x, const int4* __restrict__ blocks, int row0, const float* __restrict__ carry,
                 const T* __restrict__ y, long long ldy, const float* __restrict__ yb, T* __restrict__ out, int W) {
  const int4 b = blocks[blockIdx.y];
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= W) return;
  float h0[V], bias[V];
  ldv<V>(carry + (size_t)blockIdx.y * W + c, h0);
  ldv<V>(yb + c, bias);
  const int r0 = b.y - row0;
#pragma unroll 2
  for (int t = blockIdx.z; t < b.z; t += gridDim.z) {
    const size_t o = (size_t)(r0 + t) * W + c;
    float av[V], xv[V], yv[V];
    ldv<V>(a + o, av);
    ldv<V>(x + o, xv);
    ldv<V>(y + (size_t)(r0 + t) * ldy + c, yv);
#pragma unroll
    for (int v = 0; v < V; ++v) yv[v] = (av[v] * h0[v] + xv[v]) * gelu_tanh_t<sizeof(T) == 2>(yv[v] + bias[v]);
    stv<V>(out + o, yv);
  }
}

// ------------------------------------------------------------------ Mamba-2, token by token
// A warp owns 8 channels p of one head: lane l holds the states n = l, l + 32, ... of each. Serves single-token rows
// (one pass over the state) and any sizes; portions with aligned sizes take the blocked form below.
constexpr int M2_P = 8;

template <typename T, int NL>
__global__ void __launch_bounds__(128)
mamba2_scan_kernel(const T* __restrict__ xbc, long long ldx, const T* __restrict__ dtr, long long ldd, const float* __restrict__ dt_bias,
                   const float* __restrict__ A_log, const float* __restrict__ Dp, const int* __restrict__ cu, const int* __restrict__ start,
                   const int* __restrict__ state, float* __restrict__ S, float* __restrict__ y, int H, int P, int N, int G) {
  pdl_wait();
  pdl_trigger();
  const int e = blockIdx.x, hd = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p0 = (blockIdx.z * 4 + warp) * M2_P;
  if (p0 >= P) return;
  const int np = min(M2_P, P - p0);
  const int inner = H * P, g = hd / (H / G);
  const int r0 = cu[e], r1 = cu[e + 1], slot = state[e];
  if (slot < 0) {
    for (int r = r0; r < r1; ++r)
      if (lane < np) y[(size_t)r * inner + hd * P + p0 + lane] = 0.f;
    return;
  }
  float* Sp = S + (((size_t)slot * H + hd) * P + p0) * N;
  float s[M2_P][NL];
  const bool fresh = start[e] <= 0;
#pragma unroll
  for (int i = 0; i < M2_P; ++i)
#pragma unroll
    for (int j = 0; j < NL; ++j) {
      const int n = lane + 32 * j;
      s[i][j] = (!fresh && i < np && n < N) ? Sp[(size_t)i * N + n] : 0.f;
    }
  const float A = -expf(A_log[hd]), bias = dt_bias[hd], Dh = Dp[hd];
  const T* Bb = xbc + inner + g * N;
  const T* Cb = Bb + G * N;
  const T* xb = xbc + hd * P + p0;
  float bn[NL], cn[NL], xn, dn;
  auto fetch = [&](int r) {
#pragma unroll
    for (int j = 0; j < NL; ++j) {
      const int n = lane + 32 * j;
      bn[j] = n < N ? ldf(Bb + (size_t)r * ldx + n) : 0.f;
      cn[j] = n < N ? ldf(Cb + (size_t)r * ldx + n) : 0.f;
    }
    xn = lane < np ? ldf(xb + (size_t)r * ldx + lane) : 0.f;
    dn = ldf(dtr + (size_t)r * ldd + hd);
  };
  if (r0 < r1) fetch(r0);
  for (int r = r0; r < r1; ++r) {
    float b[NL], c[NL];
#pragma unroll
    for (int j = 0; j < NL; ++j) { b[j] = bn[j]; c[j] = cn[j]; }
    const float x = xn, dt = softplusf(dn + bias);
    if (r + 1 < r1) fetch(r + 1);
    const float dec = expf(A * dt);
    float mine = 0.f;
#pragma unroll
    for (int i = 0; i < M2_P; ++i) {
      const float dx = dt * __shfl_sync(0xffffffffu, x, i);
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < NL; ++j) {
        s[i][j] = dec * s[i][j] + dx * b[j];
        acc += s[i][j] * c[j];
      }
      acc = warp_sum(acc);
      if (lane == i) mine = acc;
    }
    if (lane < np) y[(size_t)r * inner + hd * P + p0 + lane] = mine + Dh * x;
  }
#pragma unroll
  for (int i = 0; i < M2_P; ++i)
#pragma unroll
    for (int j = 0; j < NL; ++j) {
      const int n = lane + 32 * j;
      if (i < np && n < N) Sp[(size_t)i * N + n] = s[i][j];
    }
}

template <typename T, bool DECODE>
static int launch_gates(const void* u, const void* y, long long ldy, const void* gw, const GateEpi& p, void* out, int R, cudaStream_t s) {
  const dim3 grid(p.nblk * ((p.bs + GT_C - 1) / GT_C), DECODE ? (R + GT_R - 1) / GT_R : p.nb);
  if (grid.y > 65535) return 11;
  auto kern = rglru_gate_kernel<T, DECODE>;
  constexpr int SMEM = GateCfg<T, DECODE>::NS * GateCfg<T, DECODE>::OP_BYTES;
  static ab2host::DevState st;
  if (ab2host::prepare_launch(kern, SMEM, st, nullptr)) return 300;
  launch_pdl(kern, grid, dim3(128), (size_t)SMEM, s, (const T*)u, (const T*)y, ldy, (const T*)gw, p, (T*)out, R);
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

template <typename T>
static int launch_lru_prefill(const void* u, const void* y, long long ldy, const void* gw, const GateEpi& p, void* out, cudaStream_t s) {
  if (const int rc = launch_gates<T, false>(u, y, ldy, gw, p, out, 0, s)) return rc;
  lru_carry_kernel<<<dim3((p.W + 127) / 128, p.nb), 128, 0, s>>>(p.blocks, p.start, p.state, p.S, p.carry, p.nb, p.W);
  const bool vec = p.W % 4 == 0 && ldy % 4 == 0 && aligned_to(y, 16) && aligned_to(out, 16) && aligned_to(p.yb, 16);
  if (vec)
    lru_apply_kernel<T, 4><<<dim3((p.W / 4 + 127) / 128, p.nb, 4), 128, 0, s>>>(p.a, p.x, p.blocks, p.row0, p.carry, (const T*)y, ldy, p.yb, (T*)out, p.W);
  else
    lru_apply_kernel<T, 1><<<dim3((p.W + 127) / 128, p.nb, 1), 128, 0, s>>>(p.a, p.x, p.blocks, p.row0, p.carry, (const T*)y, ldy, p.yb, (T*)out, p.W);
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Single-token rows. u [R, W], y [R, W] (row stride ldy), gw [2, n, bs, bs], gb [2, W], S [slots, W].
int ab2_rglru_decode(const void* u, const void* y, long long ldy, const float* yb, const void* gw, const float* gb, const float* lam,
                     const int* start, const int* state, float* S, void* out, int R, int n, int bs, int dt, void* stream) {
  if (R <= 0) return 0;
  GateEpi p{};
  p.gb = gb; p.lam = lam; p.yb = yb; p.start = start; p.state = state; p.S = S; p.W = n * bs; p.bs = bs; p.nblk = n;
  return dt == 0 ? launch_gates<__nv_bfloat16, true>(u, y, ldy, gw, p, out, R, (cudaStream_t)stream)
                 : launch_gates<float, true>(u, y, ldy, gw, p, out, R, (cudaStream_t)stream);
}

// Portions: R rows from row row0 of the step on, in nb blocks. a, x [R, W] and carry [2, nb, W] are scratch.
int ab2_rglru_prefill(const void* u, const void* y, long long ldy, const float* yb, const void* gw, const float* gb, const float* lam,
                      const void* blocks, int nb, int row0, int R, const int* start, const int* state, float* S, float* a, float* x, float* carry,
                      void* out, int n, int bs, int dt, void* stream) {
  if (R <= 0 || nb <= 0) return 0;
  if (nb > 65535) return 11;
  cudaStream_t s = (cudaStream_t)stream;
  GateEpi p{};
  p.gb = gb; p.lam = lam; p.yb = yb; p.start = start; p.state = state; p.S = S; p.W = n * bs; p.bs = bs; p.nblk = n;
  p.blocks = (const int4*)blocks; p.nb = nb; p.row0 = row0; p.a = a; p.x = x; p.carry = carry;
  return dt == 0 ? launch_lru_prefill<__nv_bfloat16>(u, y, ldy, gw, p, out, s) : launch_lru_prefill<float>(u, y, ldy, gw, p, out, s);
}

// Entries 0 .. E - 1, each over its rows. xbc rows: x [H * P] | B [G * N] | C [G * N]; S [slots, H, P, N]; y [rows, H * P] fp32.
int ab2_mamba2_scan(const void* xbc, long long ldx, const void* dtr, long long ldd, const float* dt_bias, const float* A_log, const float* D,
                    const int* cu, const int* start, const int* state, int E, float* S, float* y, int H, int P, int N, int G, int dt, void* stream) {
  if (E <= 0) return 0;
  if (G < 1 || H % G || H > 65535) return 10;
  const dim3 grid(E, H, (P + 4 * M2_P - 1) / (4 * M2_P));
  const int nl = (N + 31) / 32;
#define AB2_M2(TT, NLV)                                                                                                                       \
  launch_pdl(mamba2_scan_kernel<TT, NLV>, grid, dim3(128), 0, (cudaStream_t)stream, (const TT*)xbc, ldx, (const TT*)dtr, ldd, dt_bias, A_log, D, \
             cu, start, state, S, y, H, P, N, G)
#define AB2_M2_N(TT)                                                                                                                   \
  if (nl <= 1) AB2_M2(TT, 1); else if (nl <= 2) AB2_M2(TT, 2); else if (nl <= 4) AB2_M2(TT, 4); else if (nl <= 8) AB2_M2(TT, 8); else if (nl <= 16) AB2_M2(TT, 16); else return 12
  if (dt == 0) { AB2_M2_N(__nv_bfloat16); } else { AB2_M2_N(float); }
#undef AB2_M2_N
#undef AB2_M2
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}
}
