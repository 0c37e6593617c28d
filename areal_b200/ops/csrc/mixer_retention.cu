// Retention: linear attention whose state forgets by a fixed factor a per head,
//   S_t = a S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
// with rotated q and k (halves paired; k scaled after its rotation). States are fp32, [slot][head][channel p of v][n of k].
//
//   retention_decode   single-token rows, any sizes: one pass over the state, then o over its root mean square, gate, factor
//   retention_scan     portions token by token, any sizes (32-bit mode, odd sizes)
//   retention_blocks   portions in blocks of 64 tokens on the tensor cores (bf16): inside a block the outputs are a masked product
//                      (q k^T weighted by powers of a) v; across blocks only the state is carried, in registers
//   head_norm_gate     o over its root mean square per head, times silu(gate) and a factor (after the two above)
// z rows: q [H, N] | k [H, N] | v [H, P] | gate [H, P]. rot: (cos, sin) of the step's rows.
#include "mixer_common.cuh"

namespace ab2 {

struct RetArgs {
  long long ld;                // elements from row to row of z
  const float2* rot;           // ldr pairs from row to row, the first `half` of them used
  int ldr, half;
  const float *decay, *log2_decay;
  float k_scale;
  const int *cu, *start, *state;
  float* S;
  int H, N, P;
};

// element n of a head, rotated
template <typename T>
__device__ __forceinline__ float turned(const T* x, int n, int half, const float2* cs) {
  if (n >= 2 * half) return ldf(x + n);
  const bool first = n < half;
  const float2 r = cs[first ? n : n - half];
  const float u = ldf(x + n), o = ldf(x + (first ? n + half : n - half));
  return first ? u * r.x - o * r.y : u * r.x + o * r.y;
}

// ------------------------------------------------------------------ single-token rows
// A CTA owns a row's head. Lane l of every warp holds the elements n = (32 j + l) W .. + W - 1, j < J, of q, k and a channel's state.
constexpr int RD_CH = 4;       // channels of a warp in flight

template <typename T, int W, int J>
__global__ void __launch_bounds__(256)
retention_decode_kernel(const T* __restrict__ z, const RetArgs p, T* __restrict__ out, long long ldo, float eps, float scale) {
  extern __shared__ float sy[];                       // [P]
  __shared__ float red[8];
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slot = p.state[row], N = p.N, P = p.P;
  T* o = out + row * ldo + (size_t)h * P;
  if (slot < 0) {
    for (int c = tid; c < P; c += 256) stf(o + c, 0.f);
    return;
  }
  const bool fresh = p.start[row] <= 0;
  const T* qg = z + row * p.ld + (size_t)h * N;
  const T* kg = qg + (size_t)p.H * N;
  const T* vg = z + row * p.ld + (size_t)2 * p.H * N + (size_t)h * P;
  const T* gg = vg + (size_t)p.H * P;
  const float2* cs = p.rot + (size_t)row * p.ldr;
  float* Sg = p.S + ((size_t)slot * p.H + h) * P * N;
  float s[RD_CH][J][W];
  auto load = [&](int c0) {
#pragma unroll
    for (int i = 0; i < RD_CH; ++i)
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const int n = (j * 32 + lane) * W;
#pragma unroll
        for (int w = 0; w < W; ++w) s[i][j][w] = 0.f;
        if (!fresh && c0 + i < P && n < N) {
          const float* a = Sg + (size_t)(c0 + i) * N + n;
          if constexpr (W == 4) {
            const float4 v = *reinterpret_cast<const float4*>(a);
            s[i][j][0] = v.x; s[i][j][1] = v.y; s[i][j][2] = v.z; s[i][j][3] = v.w;
          } else {
#pragma unroll
            for (int w = 0; w < W; ++w) s[i][j][w] = a[w];
          }
        }
      }
  };
  const int per = (P + 7) / 8, c_end = min(P, (warp + 1) * per);
  load(warp * per);                                   // on their way while q and k are turned
  float q[J][W], k[J][W];
#pragma unroll
  for (int j = 0; j < J; ++j)
#pragma unroll
    for (int w = 0; w < W; ++w) {
      const int n = (j * 32 + lane) * W + w;
      q[j][w] = n < N ? turned(qg, n, p.half, cs) : 0.f;
      k[j][w] = n < N ? turned(kg, n, p.half, cs) * p.k_scale : 0.f;
    }
  const float a = p.decay[h];
  float ss = 0.f;
  for (int c0 = warp * per; c0 < c_end; c0 += RD_CH) {
    if (c0 != warp * per) load(c0);
#pragma unroll
    for (int i = 0; i < RD_CH; ++i) {
      if (c0 + i >= c_end) break;
      const float v = ldf(vg + c0 + i);
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const int n = (j * 32 + lane) * W;
#pragma unroll
        for (int w = 0; w < W; ++w) {
          s[i][j][w] = a * s[i][j][w] + k[j][w] * v;
          acc += s[i][j][w] * q[j][w];
        }
        if (n < N) {
          float* d = Sg + (size_t)(c0 + i) * N + n;
          if constexpr (W == 4) {
            *reinterpret_cast<float4*>(d) = make_float4(s[i][j][0], s[i][j][1], s[i][j][2], s[i][j][3]);
          } else {
#pragma unroll
            for (int w = 0; w < W; ++w) d[w] = s[i][j][w];
          }
        }
      }
      acc = warp_sum(acc);
      if (lane == 0) sy[c0 + i] = acc;
      ss += acc * acc;
    }
  }
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float f = scale / sqrtf(ss / P + eps);
  for (int c = tid; c < P; c += 256) stf(o + c, sy[c] * f * silu_t<sizeof(T) == 2>(ldf(gg + c)));
}

// ------------------------------------------------------------------ portions, token by token
// A warp owns 8 channels of one head; lane l holds n = l, l + 32, ... of each.
constexpr int RS_CH = 8;

template <typename T, int NL>
__global__ void __launch_bounds__(128)
retention_scan_kernel(const T* __restrict__ z, const RetArgs p, int e0, float* __restrict__ y) {
  const int e = e0 + blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = (blockIdx.z * 4 + warp) * RS_CH, N = p.N, P = p.P;
  const int slot = p.state[e];
  if (c0 >= P || slot < 0) return;
  const int nc = min(RS_CH, P - c0), r0 = p.cu[e], r1 = p.cu[e + 1], first = p.cu[e0];
  float* Sg = p.S + (((size_t)slot * p.H + h) * P + c0) * N;
  const bool fresh = p.start[e] <= 0;
  float s[RS_CH][NL];
#pragma unroll
  for (int i = 0; i < RS_CH; ++i)
#pragma unroll
    for (int j = 0; j < NL; ++j) s[i][j] = (!fresh && i < nc && lane + 32 * j < N) ? Sg[(size_t)i * N + lane + 32 * j] : 0.f;
  const float a = p.decay[h];
  for (int r = r0; r < r1; ++r) {
    const T* qg = z + r * p.ld + (size_t)h * N;
    const T* kg = qg + (size_t)p.H * N;
    const T* vg = z + r * p.ld + (size_t)2 * p.H * N + (size_t)h * P + c0;
    const float2* cs = p.rot + (size_t)r * p.ldr;
    float q[NL], k[NL];
#pragma unroll
    for (int j = 0; j < NL; ++j) {
      const int n = lane + 32 * j;
      q[j] = n < N ? turned(qg, n, p.half, cs) : 0.f;
      k[j] = n < N ? turned(kg, n, p.half, cs) * p.k_scale : 0.f;
    }
    const float v = lane < nc ? ldf(vg + lane) : 0.f;
    float mine = 0.f;
#pragma unroll
    for (int i = 0; i < RS_CH; ++i) {
      const float vi = __shfl_sync(0xffffffffu, v, i);
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < NL; ++j) {
        s[i][j] = a * s[i][j] + k[j] * vi;
        acc += s[i][j] * q[j];
      }
      acc = warp_sum(acc);
      if (lane == i) mine = acc;
    }
    if (lane < nc) y[(size_t)(r - first) * p.H * P + (size_t)h * P + c0 + lane] = mine;
  }
#pragma unroll
  for (int i = 0; i < RS_CH; ++i)
#pragma unroll
    for (int j = 0; j < NL; ++j)
      if (i < nc && lane + 32 * j < N) Sg[(size_t)i * N + lane + 32 * j] = s[i][j];
}

// ------------------------------------------------------------------ portions in blocks
// One CTA (eight warps) per request, head and 64 channels walks the request's blocks of 64 tokens. With t, s = 0 .. n - 1 in the block:
//   o_t = sum_{s <= t} a^(t - s) (q_t . k_s) v_s + a^(t + 1) S^T q_t        warps 0 - 3 the first sum, 4 - 7 the second
//   S  <- a^n S + sum_s a^(n - 1 - s) k_s v_s^T                             all of them, 16 channels and half of the columns each
// v is bf16; the rotated q and k, the weights and S are fp32 and enter a product as the sum of two bf16 numbers (rounding and rest,
// without the product of two rests); accumulation is fp32. An output is divided by its own size afterwards, so what a
// small q . k loses would show.
constexpr int RB_Q = 64, RB_P = 64;

__device__ __forceinline__ void rb_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void rb_mat(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void rb_mat_t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void rb_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  const float2 r = unpack_bf16(hi);
  lo = pack_bf16(a - r.x, b - r.y);
}

template <int NP>
struct RetCfg {
  static constexpr int NROW = NP * 2 + 16, PROW = RB_P * 2 + 16;         // padded rows (bytes)
  static constexpr int MAT = RB_Q * NROW;
  static constexpr int QH_OFF = 0, QL_OFF = MAT, KH_OFF = 2 * MAT, KL_OFF = 3 * MAT, SH_OFF = 4 * MAT, SL_OFF = 5 * MAT, V_OFF = 6 * MAT;
  static constexpr int A_OFF = V_OFF + RB_Q * PROW;                      // a^0 .. a^64
  static constexpr int ZROW = RB_P + 4;                                  // floats; what the state adds to the outputs, over the state's
  static constexpr int Z_OFF = NP >= 64 ? SH_OFF : A_OFF + (RB_Q + 4) * 4;     // own matrices where these are large enough
  static constexpr int SMEM = A_OFF + (RB_Q + 4) * 4 + (NP >= 64 ? 0 : RB_Q * ZROW * 4);
  static_assert(NP < 64 || 2 * MAT >= RB_Q * ZROW * 4, "the sums fit over the state");
};

// NP: N rounded up to 32, 64 or 128 (missing columns are zero).
template <int NP>
__global__ void __launch_bounds__(256, NP == 128 ? 1 : 2)
retention_blocks_kernel(const __nv_bfloat16* __restrict__ z, const float2* __restrict__ rot, const RetArgs p, int e0, float* __restrict__ y) {
  using Cfg = RetCfg<NP>;
  constexpr int NT = NP / 16, KN = NP / 16;                   // tiles of 8 in half of the columns, k-steps of 16 in all
  constexpr int U = NP / 32;                                  // pieces of q and k of a thread when whole heads turn
  extern __shared__ __align__(16) unsigned char sm[];
  const uint32_t sb = smem_u32(sm);
  float* pw = reinterpret_cast<float*>(sm + Cfg::A_OFF);
  const int e = e0 + blockIdx.x, hd = blockIdx.y, p0 = blockIdx.z * RB_P;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const int slot = p.state[e];
  if (slot < 0) return;
  const int N = p.N, P = p.P, r_end = p.cu[e + 1], first = p.cu[e0], np = min(RB_P, P - p0), half = p.half;
  const __nv_bfloat16* qg = z + (size_t)hd * N;
  const __nv_bfloat16* kg = qg + (size_t)p.H * N;
  const __nv_bfloat16* vg = z + (size_t)2 * p.H * N + (size_t)hd * P + p0;
  // this warp's part of the state: rows p = 16 (warp % 4) + gq (+ 8), columns n = n0 + 8 j + 2 tq (+ 1)
  const int wr = warp & 3, n0 = (warp >> 2) * (NP / 2);
  float* Sg = p.S + (((size_t)slot * p.H + hd) * P + p0) * N;
  float st[NT][4];
  const bool fresh = p.start[e] <= 0;
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int c = wr * 16 + gq + 8 * hh, n = n0 + j * 8 + 2 * tq;
      float2 v = make_float2(0.f, 0.f);
      if (!fresh && c < np && n < N) v = *reinterpret_cast<const float2*>(Sg + (size_t)c * N + n);
      st[j][2 * hh] = v.x;
      st[j][2 * hh + 1] = v.y;
    }
  if (tid <= RB_Q) pw[tid] = exp2f(p.log2_decay[hd] * (float)tid);
  const int pairs = half / 4, pieces = pairs + (NP - 2 * half) / 4;       // of a row: four pairs, or four numbers that do not turn
  // A block's rows are on their way while the block before is worked on: U pieces of q and k and two of v per thread.
  uint2 a[U][4];                                          // q, k; q and k half a turn further on, or nothing
  float2 t[U][4];
  uint4 vr[2];
  auto fetch = [&](int r0, int i0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + 256 * u, r = i / pieces, x = i - r * pieces, c = x < pairs ? x * 4 : 2 * half + (x - pairs) * 4;
      const size_t at = (size_t)(r0 + r) * p.ld + c;
      a[u][0] = a[u][1] = a[u][2] = a[u][3] = make_uint2(0u, 0u);
      t[u][0] = t[u][1] = t[u][2] = t[u][3] = make_float2(0.f, 0.f);
      if (r >= RB_Q || r0 + r >= r_end || c >= N) continue;
      a[u][0] = *reinterpret_cast<const uint2*>(qg + at);
      a[u][1] = *reinterpret_cast<const uint2*>(kg + at);
      if (x < pairs) {
        a[u][2] = *reinterpret_cast<const uint2*>(qg + at + half);
        a[u][3] = *reinterpret_cast<const uint2*>(kg + at + half);
        const float2* cs = rot + (size_t)(r0 + r) * p.ldr + c;
#pragma unroll
        for (int w = 0; w < 4; ++w) t[u][w] = cs[w];
      }
    }
  };
  auto fetch_v = [&](int r0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = tid + 256 * u, r = i >> 3, c = (i & 7) * 8;
      vr[u] = make_uint4(0u, 0u, 0u, 0u);
      if (r0 + r < r_end && c < np) vr[u] = *reinterpret_cast<const uint4*>(vg + (size_t)(r0 + r) * p.ld + c);
    }
  };
  auto put = [&](int r, int c, const float (&q)[4], const float (&k)[4]) {
    const int off = r * Cfg::NROW + c * 2;
    uint2 hi, lo;
    rb_split(q[0], q[1], hi.x, lo.x);
    rb_split(q[2], q[3], hi.y, lo.y);
    *reinterpret_cast<uint2*>(sm + Cfg::QH_OFF + off) = hi;
    *reinterpret_cast<uint2*>(sm + Cfg::QL_OFF + off) = lo;
    rb_split(k[0], k[1], hi.x, lo.x);
    rb_split(k[2], k[3], hi.y, lo.y);
    *reinterpret_cast<uint2*>(sm + Cfg::KH_OFF + off) = hi;
    *reinterpret_cast<uint2*>(sm + Cfg::KL_OFF + off) = lo;
  };
  auto store = [&](int i0) {                                 // turned, as two bf16 matrices each
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + 256 * u, r = i / pieces, x = i - r * pieces;
      if (r >= RB_Q) break;
      float q[4], k[4], q2[4], k2[4];
      auto wide = [](const uint2& v, float (&o)[4]) {
        const float2 lo = unpack_bf16(v.x), hi = unpack_bf16(v.y);
        o[0] = lo.x; o[1] = lo.y; o[2] = hi.x; o[3] = hi.y;
      };
      wide(a[u][0], q);
      wide(a[u][1], k);
#pragma unroll
      for (int w = 0; w < 4; ++w) k[w] *= p.k_scale;
      if (x < pairs) {
        wide(a[u][2], q2);
        wide(a[u][3], k2);
#pragma unroll
        for (int w = 0; w < 4; ++w) {
          const float2 cs = t[u][w];
          const float b = q[w], d = q2[w], f = k[w], g = k2[w] * p.k_scale;
          q[w] = b * cs.x - d * cs.y;
          q2[w] = d * cs.x + b * cs.y;
          k[w] = f * cs.x - g * cs.y;
          k2[w] = g * cs.x + f * cs.y;
        }
        put(r, x * 4, q, k);
        put(r, x * 4 + half, q2, k2);
      } else {
        put(r, 2 * half + (x - pairs) * 4, q, k);
      }
    }
  };
  fetch(p.cu[e], tid);
  fetch_v(p.cu[e]);
  for (int r0 = p.cu[e]; r0 < r_end; r0 += RB_Q) {
    const int nr = min(RB_Q, r_end - r0);
    // ---- q, k (turned) and v of the block (rows past the end: zero), the state as two bf16 matrices
    store(tid);
    for (int i0 = tid + 256 * U; i0 < RB_Q * pieces; i0 += 256 * U) {        // heads that hardly turn have more pieces
      fetch(r0, i0);
      store(i0);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = tid + 256 * u;
      *reinterpret_cast<uint4*>(sm + Cfg::V_OFF + (i >> 3) * Cfg::PROW + (i & 7) * 16) = vr[u];
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        uint32_t hi, lo;
        rb_split(st[j][2 * hh], st[j][2 * hh + 1], hi, lo);
        const int off = (wr * 16 + gq + 8 * hh) * Cfg::NROW + (n0 + j * 8 + 2 * tq) * 2;
        *reinterpret_cast<uint32_t*>(sm + Cfg::SH_OFF + off) = hi;
        *reinterpret_cast<uint32_t*>(sm + Cfg::SL_OFF + off) = lo;
      }
    __syncthreads();
    if (r0 + RB_Q < r_end) {
      fetch(r0 + RB_Q, tid);
      fetch_v(r0 + RB_Q);
    }
    const int t0 = wr * 16;                                  // this warp's rows t
    float* zs = reinterpret_cast<float*>(sm + Cfg::Z_OFF);
    if (warp >= 4) {
      // ---- a^(t + 1) q S^T
      float o[RB_P / 8][4];
#pragma unroll
      for (int j = 0; j < RB_P / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
      for (int k = 0; k < KN; ++k) {
        uint32_t qa[4], ql[4];
        rb_mat(sb + Cfg::QH_OFF + (t0 + (mat & 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat >> 1) * 8) * 2, qa);
        rb_mat(sb + Cfg::QL_OFF + (t0 + (mat & 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat >> 1) * 8) * 2, ql);
        uint32_t b[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) rb_mat(sb + Cfg::SH_OFF + (j * 16 + (mat >> 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat & 1) * 8) * 2, b[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          rb_mma(o[2 * j], qa, b[j][0], b[j][1]);
          rb_mma(o[2 * j + 1], qa, b[j][2], b[j][3]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          rb_mma(o[2 * j], ql, b[j][0], b[j][1]);
          rb_mma(o[2 * j + 1], ql, b[j][2], b[j][3]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) rb_mat(sb + Cfg::SL_OFF + (j * 16 + (mat >> 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat & 1) * 8) * 2, b[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          rb_mma(o[2 * j], qa, b[j][0], b[j][1]);
          rb_mma(o[2 * j + 1], qa, b[j][2], b[j][3]);
        }
      }
      if constexpr (NP >= 64) asm volatile("bar.sync 2, 128;" ::: "memory");       // these four have read the state's matrices
      const float w0 = pw[t0 + gq + 1], w1 = pw[t0 + gq + 9];
#pragma unroll
      for (int j = 0; j < RB_P / 8; ++j) {
        float* d = zs + (t0 + gq) * Cfg::ZROW + j * 8 + 2 * tq;
        *reinterpret_cast<float2*>(d) = make_float2(o[j][0] * w0, o[j][1] * w0);
        *reinterpret_cast<float2*>(d + 8 * Cfg::ZROW) = make_float2(o[j][2] * w1, o[j][3] * w1);
      }
      asm volatile("bar.arrive 1, 256;" ::: "memory");
    } else {
      // ---- G = q k^T, then (G weighted) v
      float gm[8][4], o[RB_P / 8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) gm[j][0] = gm[j][1] = gm[j][2] = gm[j][3] = o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
      for (int k = 0; k < KN; ++k) {
        uint32_t qa[4], ql[4];
        rb_mat(sb + Cfg::QH_OFF + (t0 + (mat & 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat >> 1) * 8) * 2, qa);
        rb_mat(sb + Cfg::QL_OFF + (t0 + (mat & 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat >> 1) * 8) * 2, ql);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j > warp) break;                               // rows s of later 16-row groups are all in the future
          const uint32_t off = (j * 16 + (mat >> 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat & 1) * 8) * 2;
          uint32_t b[4], c[4];
          rb_mat(sb + Cfg::KH_OFF + off, b);
          rb_mat(sb + Cfg::KL_OFF + off, c);
          rb_mma(gm[2 * j], qa, b[0], b[1]);
          rb_mma(gm[2 * j + 1], qa, b[2], b[3]);
          rb_mma(gm[2 * j], ql, b[0], b[1]);
          rb_mma(gm[2 * j + 1], ql, b[2], b[3]);
          rb_mma(gm[2 * j], qa, c[0], c[1]);
          rb_mma(gm[2 * j + 1], qa, c[2], c[3]);
        }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {                          // 16 columns s at a time: accumulators of G become the A operand
        if (k > warp) break;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {                        // x: (row half x & 1, column half x >> 1)
          const int d = t0 + gq + (x & 1) * 8 - (k * 16 + (x >> 1) * 8 + 2 * tq);        // t - s of the first of two columns
          const float* gv = &gm[2 * k + (x >> 1)][(x & 1) * 2];
          rb_split(d >= 0 ? gv[0] * pw[max(d, 0)] : 0.f, d >= 1 ? gv[1] * pw[max(d - 1, 0)] : 0.f, hi[x], lo[x]);
        }
#pragma unroll
        for (int j = 0; j < RB_P / 16; ++j) {
          uint32_t b[4];
          rb_mat_t(sb + Cfg::V_OFF + (k * 16 + (mat & 1) * 8 + r8) * Cfg::PROW + (j * 16 + (mat >> 1) * 8) * 2, b);
          rb_mma(o[2 * j], hi, b[0], b[1]);
          rb_mma(o[2 * j + 1], hi, b[2], b[3]);
          rb_mma(o[2 * j], lo, b[0], b[1]);
          rb_mma(o[2 * j + 1], lo, b[2], b[3]);
        }
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");         // the other warps' sums are there
#pragma unroll
      for (int j = 0; j < RB_P / 8; ++j)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int t = t0 + gq + 8 * hh, c = j * 8 + 2 * tq;
          if (t < nr && c < np) {
            const float2 z2 = *reinterpret_cast<const float2*>(zs + t * Cfg::ZROW + c);
            *reinterpret_cast<float2*>(y + (size_t)(r0 - first + t) * p.H * P + (size_t)hd * P + p0 + c) =
                make_float2(o[j][2 * hh] + z2.x, o[j][2 * hh + 1] + z2.y);
          }
        }
    }
    // ---- S <- a^n S + (weighted v)^T k over this warp's part
    const float dec = pw[nr];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      st[j][0] *= dec; st[j][1] *= dec; st[j][2] *= dec; st[j][3] *= dec;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t va[4], hi[4], lo[4];
      // v^T: rows p, columns s; transposed 8 x 8 pieces (s half of the fragment = mat >> 1, p half = mat & 1)
      rb_mat_t(sb + Cfg::V_OFF + (k * 16 + (mat >> 1) * 8 + r8) * Cfg::PROW + (t0 + (mat & 1) * 8) * 2, va);
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = nr - 1 - (k * 16 + (x >> 1) * 8 + 2 * tq);          // rows past the end are zero
        const float2 v = unpack_bf16(va[x]);
        rb_split(v.x * pw[max(d, 0)], v.y * pw[max(d - 1, 0)], hi[x], lo[x]);
      }
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        const uint32_t off = (k * 16 + (mat & 1) * 8 + r8) * Cfg::NROW + (n0 + j * 16 + (mat >> 1) * 8) * 2;
        uint32_t b[4];
        rb_mat_t(sb + Cfg::KH_OFF + off, b);
        rb_mma(st[2 * j], hi, b[0], b[1]);
        rb_mma(st[2 * j + 1], hi, b[2], b[3]);
        rb_mma(st[2 * j], lo, b[0], b[1]);
        rb_mma(st[2 * j + 1], lo, b[2], b[3]);
        rb_mat_t(sb + Cfg::KL_OFF + off, b);
        rb_mma(st[2 * j], hi, b[0], b[1]);
        rb_mma(st[2 * j + 1], hi, b[2], b[3]);
      }
    }
    __syncthreads();                                         // the next block's rows replace these
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int c = wr * 16 + gq + 8 * hh, n = n0 + j * 8 + 2 * tq;
      if (c < np && n < N) *reinterpret_cast<float2*>(Sg + (size_t)c * N + n) = make_float2(st[j][2 * hh], st[j][2 * hh + 1]);
    }
}

// ------------------------------------------------------------------ norm per head, gate
// One CTA per row, a warp per head; y fp32 [R, H * P].
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* __restrict__ y, const T* __restrict__ g, long long ldg, T* __restrict__ out, long long ldo, int H, int P, float eps,
                      float scale) {
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = warp; h < H; h += 8) {
    const float* s = y + ((size_t)row * H + h) * P;
    float ss = 0.f;
    for (int c = lane * V; c < P; c += 32 * V) {
      float v[V];
      ldv<V>(s + c, v);
      for (int e = 0; e < V; ++e) ss += v[e] * v[e];
    }
    const float f = scale / sqrtf(warp_sum(ss) / P + eps);
    for (int c = lane * V; c < P; c += 32 * V) {
      float v[V], w[V];
      ldv<V>(s + c, v);
      ldv<V>(g + row * ldg + (size_t)h * P + c, w);
      for (int e = 0; e < V; ++e) v[e] = v[e] * f * silu_t<sizeof(T) == 2>(w[e]);
      stv<V>(out + row * ldo + (size_t)h * P + c, v);
    }
  }
}

template <int NP>
static int launch_blocks(const __nv_bfloat16* z, const RetArgs& a, int e0, int E, float* y, cudaStream_t s) {
  auto kern = retention_blocks_kernel<NP>;
  static ab2host::DevState st;
  if (ab2host::prepare_launch(kern, RetCfg<NP>::SMEM, st, nullptr)) return 300;
  kern<<<dim3(E - e0, a.H, (a.P + RB_P - 1) / RB_P), 256, RetCfg<NP>::SMEM, s>>>(z, a.rot, a, e0, y);
  return cudaGetLastError() == cudaSuccess ? 0 : 302;
}

template <typename T>
static int launch_rows(const void* z, const RetArgs& a, void* out, long long ldo, int R, float eps, float scale, cudaStream_t s) {
  const size_t smem = (size_t)a.P * 4;
  if (smem > 40 * 1024) return 11;
#define AB2_RD(W, J) launch_pdl(retention_decode_kernel<T, W, J>, dim3(R, a.H), dim3(256), smem, s, (const T*)z, a, (T*)out, ldo, eps, scale)
  if (a.N % 4 == 0 && a.N > 32) {
    if (a.N <= 128) AB2_RD(4, 1); else if (a.N <= 256) AB2_RD(4, 2); else if (a.N <= 512) AB2_RD(4, 4); else return 12;
  } else {
    if (a.N <= 32) AB2_RD(1, 1); else if (a.N <= 64) AB2_RD(1, 2); else if (a.N <= 128) AB2_RD(1, 4); else if (a.N <= 256) AB2_RD(1, 8);
    else if (a.N <= 512) AB2_RD(1, 16); else return 12;
  }
#undef AB2_RD
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

template <typename T>
static int launch_scan(const void* z, const RetArgs& a, int e0, int E, float* y, cudaStream_t s) {
  const dim3 grid(E - e0, a.H, (a.P + 4 * RS_CH - 1) / (4 * RS_CH));
#define AB2_RS(NL) retention_scan_kernel<T, NL><<<grid, 128, 0, s>>>((const T*)z, a, e0, y)
  const int nl = (a.N + 31) / 32;
  if (nl <= 1) AB2_RS(1); else if (nl <= 2) AB2_RS(2); else if (nl <= 4) AB2_RS(4); else if (nl <= 8) AB2_RS(8); else if (nl <= 16) AB2_RS(16);
  else return 12;
#undef AB2_RS
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Rows 0 .. R - 1, row r the only one of entry r (state slot state[r] < 0: padding row, zeros). out [R, H * P], ldo elements from row to row.
int ab2_retention_decode(const void* z, long long ld, const void* rot, int ldr, int half, const float* decay, float k_scale, const int* start,
                         const int* state, float* S, void* out, long long ldo, int R, int H, int N, int P, float eps, float scale, int dt, void* stream) {
  if (R <= 0) return 0;
  if (H < 1 || H > 65535 || half < 0 || 2 * half > N) return 10;
  const RetArgs a{ld, (const float2*)rot, ldr, half, decay, nullptr, k_scale, nullptr, start, state, S, H, N, P};
  return dt == 0 ? launch_rows<__nv_bfloat16>(z, a, out, ldo, R, eps, scale, (cudaStream_t)stream)
                 : launch_rows<float>(z, a, out, ldo, R, eps, scale, (cudaStream_t)stream);
}

// Entries e0 .. E - 1. z and rot from the step's first row on; y [rows of these entries, H * P] fp32 from their first row on.
// blocks: the tensor-core form (bf16; N <= 128, N, P and ld multiples of 8, half a multiple of 4), else token by token.
int ab2_retention_portions(const void* z, long long ld, const void* rot, int ldr, int half, const float* decay, const float* log2_decay, float k_scale,
                           const int* cu, const int* start, const int* state, int e0, int E, float* S, float* y, int H, int N, int P, int blocks, int dt,
                           void* stream) {
  if (E <= e0) return 0;
  if (H < 1 || H > 65535 || half < 0 || 2 * half > N) return 10;
  const RetArgs a{ld, (const float2*)rot, ldr, half, decay, log2_decay, k_scale, cu, start, state, S, H, N, P};
  cudaStream_t s = (cudaStream_t)stream;
  if (!blocks) return dt == 0 ? launch_scan<__nv_bfloat16>(z, a, e0, E, y, s) : launch_scan<float>(z, a, e0, E, y, s);
  if (dt != 0 || N > 128 || (N & 7) || (P & 7) || (ld & 7) || (half & 3) || !aligned_to(z, 16)) return 11;
  const __nv_bfloat16* b = (const __nv_bfloat16*)z;
  if (N <= 32) return launch_blocks<32>(b, a, e0, E, y, s);
  if (N <= 64) return launch_blocks<64>(b, a, e0, E, y, s);
  return launch_blocks<128>(b, a, e0, E, y, s);
}

// out = y / rms(y of a head) * silu(g) * scale
int ab2_head_norm_gate(const float* y, const void* g, long long ldg, void* out, long long ldo, int R, int H, int P, float eps, float scale, int dt,
                       void* stream) {
  if (R <= 0) return 0;
  const bool vec = P % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && aligned_to(g, dt == 0 ? 8 : 16) && aligned_to(out, dt == 0 ? 8 : 16);
  cudaStream_t s = (cudaStream_t)stream;
#define AB2_HG(T, V) head_norm_gate_kernel<T, V><<<R, 256, 0, s>>>(y, (const T*)g, ldg, (T*)out, ldo, H, P, eps, scale)
  if (dt == 0) { if (vec) AB2_HG(__nv_bfloat16, 4); else AB2_HG(__nv_bfloat16, 1); }
  else { if (vec) AB2_HG(float, 4); else AB2_HG(float, 1); }
#undef AB2_HG
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}
}
