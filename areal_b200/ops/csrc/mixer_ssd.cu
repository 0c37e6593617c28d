// Mamba-2 over portions of prompts, in blocks of 64 tokens (state-space duality): inside a block the outputs are a masked
// product (C B^T weighted by the decays) X, across blocks only the head's state is carried, in registers.
//
// One CTA (four warps) per request, head and 64 channels walks the request's blocks. With cum_t the running sum of the
// log decays in the block, L(t, s) = exp(cum_t - cum_s) dt_s:
//   y_t = sum_{s <= t} (C_t . B_s) L(t, s) x_s  +  exp(cum_t) S C_t  +  D x_t
//   S  <- exp(cum_end) S + sum_s exp(cum_end - cum_s) dt_s x_s B_s^T
// x, B and C are bf16 (they come out of the convolution); the decays, weights and S are fp32. Wherever one of those is a
// factor of a tensor-core product it enters as the sum of two bf16 numbers (its rounding and the rest), which keeps
// 16 bits and more of it; accumulation is fp32.
#include "mixer_common.cuh"

namespace ab2 {

constexpr int SD_Q = 64, SD_P = 64;

__device__ __forceinline__ void sd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sd_ldsm(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void sd_ldsm_t(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
// (a, b) as a pair of bf16 plus what the rounding left out, as another pair
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  const float2 r = unpack_bf16(hi);
  lo = pack_bf16(a - r.x, b - r.y);
}

template <int NP>
struct SsdCfg {
  static constexpr int NROW = NP * 2 + 16, PROW = SD_P * 2 + 16;         // padded rows (bytes)
  static constexpr int B_OFF = 0, C_OFF = SD_Q * NROW, X_OFF = 2 * SD_Q * NROW;
  static constexpr int SH_OFF = X_OFF + SD_Q * PROW, SL_OFF = SH_OFF + SD_P * NROW;
  static constexpr int V_OFF = SL_OFF + SD_P * NROW;                     // cum [64], dt [64]
  static constexpr int SMEM = V_OFF + 2 * SD_Q * 4;
};

// NP: state size rounded up to 32, 64 or 128 (missing columns are zero).
template <int NP>
__global__ void __launch_bounds__(128, 2)
mamba2_ssd_kernel(const __nv_bfloat16* __restrict__ xbc, long long ldx, const __nv_bfloat16* __restrict__ dtr, long long ldd,
                  const float* __restrict__ dt_bias, const float* __restrict__ A_log, const float* __restrict__ Dp, const int* __restrict__ cu,
                  const int* __restrict__ start, const int* __restrict__ state, int e0, float* __restrict__ S, float* __restrict__ y, int H, int P,
                  int N, int G) {
  using Cfg = SsdCfg<NP>;
  constexpr int NT = NP / 8, KN = NP / 16;
  extern __shared__ __align__(16) unsigned char sm[];
  const uint32_t sb = smem_u32(sm);
  float* s_cum = reinterpret_cast<float*>(sm + Cfg::V_OFF);
  float* s_dt = s_cum + SD_Q;
  const int e = e0 + blockIdx.x, hd = blockIdx.y, p0 = blockIdx.z * SD_P;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const int slot = state[e];
  if (slot < 0) return;
  const int r_end = cu[e + 1], inner = H * P, g = hd / (H / G), np = min(SD_P, P - p0);
  const float A = -expf(A_log[hd]) * 1.4426950408889634f, bias = dt_bias[hd], Dh = Dp[hd];     // decays as powers of two
  const __nv_bfloat16* xg = xbc + hd * P + p0;
  const __nv_bfloat16* bg = xbc + inner + g * N;
  const __nv_bfloat16* cg = bg + G * N;
  // this warp's 16 channels of the state: rows p = 16 warp + gq (+ 8), columns n = 8 j + 2 tq (+ 1)
  float* Sg = S + (((size_t)slot * H + hd) * P + p0) * N;
  float st[NT][4];
  const bool fresh = start[e] <= 0;
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int p = warp * 16 + gq + 8 * hh, n = j * 8 + 2 * tq;
      float2 v = make_float2(0.f, 0.f);
      if (!fresh && p < np && n < N) v = *reinterpret_cast<const float2*>(Sg + (size_t)p * N + n);
      st[j][2 * hh] = v.x;
      st[j][2 * hh + 1] = v.y;
    }
  for (int r0 = cu[e]; r0 < r_end; r0 += SD_Q) {
    const int nr = min(SD_Q, r_end - r0);
    // ---- stage B, C, x (rows past the end: zero), the state as two bf16 matrices, and the decays
    for (int i = tid; i < SD_Q * (NP / 8); i += 128) {
      const int r = i / (NP / 8), c = (i % (NP / 8)) * 8;
      const bool ok = r < nr && c < N;
      uint4 vb = make_uint4(0u, 0u, 0u, 0u), vc = vb;
      if (ok) {
        vb = *reinterpret_cast<const uint4*>(bg + (size_t)(r0 + r) * ldx + c);
        vc = *reinterpret_cast<const uint4*>(cg + (size_t)(r0 + r) * ldx + c);
      }
      *reinterpret_cast<uint4*>(sm + Cfg::B_OFF + r * Cfg::NROW + c * 2) = vb;
      *reinterpret_cast<uint4*>(sm + Cfg::C_OFF + r * Cfg::NROW + c * 2) = vc;
    }
    for (int i = tid; i < SD_Q * (SD_P / 8); i += 128) {
      const int r = i / (SD_P / 8), c = (i % (SD_P / 8)) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < nr && c < np) v = *reinterpret_cast<const uint4*>(xg + (size_t)(r0 + r) * ldx + c);
      *reinterpret_cast<uint4*>(sm + Cfg::X_OFF + r * Cfg::PROW + c * 2) = v;
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        uint32_t hi, lo;
        split_bf16(st[j][2 * hh], st[j][2 * hh + 1], hi, lo);
        const int off = (warp * 16 + gq + 8 * hh) * Cfg::NROW + (j * 8 + 2 * tq) * 2;
        *reinterpret_cast<uint32_t*>(sm + Cfg::SH_OFF + off) = hi;
        *reinterpret_cast<uint32_t*>(sm + Cfg::SL_OFF + off) = lo;
      }
    if (warp == 0) {
      float d0 = 0.f, d1 = 0.f;                              // rows 2 lane, 2 lane + 1; rows past the end decay nothing
      if (2 * lane < nr) d0 = softplusf(__bfloat162float(dtr[(size_t)(r0 + 2 * lane) * ldd + hd]) + bias);
      if (2 * lane + 1 < nr) d1 = softplusf(__bfloat162float(dtr[(size_t)(r0 + 2 * lane + 1) * ldd + hd]) + bias);
      float c = A * d0 + A * d1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, c, o);
        if (lane >= o) c += v;
      }
      s_dt[2 * lane] = d0;
      s_dt[2 * lane + 1] = d1;
      s_cum[2 * lane] = c - A * d1;
      s_cum[2 * lane + 1] = c;
    }
    __syncthreads();
    // ---- this warp's 16 rows t: C fragments, G = C B^T, z = C S^T
    const int t0 = warp * 16;
    const float cum0 = s_cum[t0 + gq], cum1 = s_cum[t0 + gq + 8];
    float gm[8][4], z[SD_P / 8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) gm[j][0] = gm[j][1] = gm[j][2] = gm[j][3] = z[j][0] = z[j][1] = z[j][2] = z[j][3] = 0.f;
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      uint32_t ca[4];
      sd_ldsm(sb + Cfg::C_OFF + (t0 + (mat & 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat >> 1) * 8) * 2, ca[0], ca[1], ca[2], ca[3]);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const uint32_t off = (j * 16 + (mat >> 1) * 8 + r8) * Cfg::NROW + (k * 16 + (mat & 1) * 8) * 2;
        uint32_t b0, b1, b2, b3;
        if (j <= warp) {                                     // rows s of later 16-row groups are all in the future
          sd_ldsm(sb + Cfg::B_OFF + off, b0, b1, b2, b3);
          sd_mma(gm[2 * j], ca, b0, b1);
          sd_mma(gm[2 * j + 1], ca, b2, b3);
        }
        sd_ldsm(sb + Cfg::SH_OFF + off, b0, b1, b2, b3);
        sd_mma(z[2 * j], ca, b0, b1);
        sd_mma(z[2 * j + 1], ca, b2, b3);
        sd_ldsm(sb + Cfg::SL_OFF + off, b0, b1, b2, b3);
        sd_mma(z[2 * j], ca, b0, b1);
        sd_mma(z[2 * j + 1], ca, b2, b3);
      }
    }
    // ---- y = diag(exp(cum)) z + (G o L) X
    const float e0f = fast_exp2(cum0), e1f = fast_exp2(cum1);
#pragma unroll
    for (int j = 0; j < SD_P / 8; ++j) {
      z[j][0] *= e0f; z[j][1] *= e0f;
      z[j][2] *= e1f; z[j][3] *= e1f;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {                            // 16 columns s at a time: accumulators of G become the A operand
      if (k > warp) break;
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {                          // x: (row half x & 1, column half x >> 1)
        const int s = k * 16 + (x >> 1) * 8 + 2 * tq, t = t0 + gq + (x & 1) * 8;
        const float ct = (x & 1) ? cum1 : cum0;
        const float* gv = &gm[2 * k + (x >> 1)][(x & 1) * 2];
        const float m0 = s <= t ? gv[0] * fast_exp2(ct - s_cum[s]) * s_dt[s] : 0.f;
        const float m1 = s + 1 <= t ? gv[1] * fast_exp2(ct - s_cum[s + 1]) * s_dt[s + 1] : 0.f;
        split_bf16(m0, m1, hi[x], lo[x]);
      }
#pragma unroll
      for (int j = 0; j < SD_P / 16; ++j) {
        uint32_t b0, b1, b2, b3;
        sd_ldsm_t(sb + Cfg::X_OFF + (k * 16 + (mat & 1) * 8 + r8) * Cfg::PROW + (j * 16 + (mat >> 1) * 8) * 2, b0, b1, b2, b3);
        sd_mma(z[2 * j], hi, b0, b1);
        sd_mma(z[2 * j + 1], hi, b2, b3);
        sd_mma(z[2 * j], lo, b0, b1);
        sd_mma(z[2 * j + 1], lo, b2, b3);
      }
    }
#pragma unroll
    for (int j = 0; j < SD_P / 8; ++j)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int t = t0 + gq + 8 * hh, p = j * 8 + 2 * tq;
        if (t < nr && p < np) {
          const float2 xv = unpack_bf16(*reinterpret_cast<const uint32_t*>(sm + Cfg::X_OFF + t * Cfg::PROW + p * 2));
          *reinterpret_cast<float2*>(y + (size_t)(r0 + t) * inner + hd * P + p0 + p) =
              make_float2(z[j][2 * hh] + Dh * xv.x, z[j][2 * hh + 1] + Dh * xv.y);
        }
      }
    // ---- S <- exp(cum_end) S + (w x)^T B over this warp's 16 channels
    const float cend = s_cum[SD_Q - 1], dec = fast_exp2(cend);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      st[j][0] *= dec; st[j][1] *= dec; st[j][2] *= dec; st[j][3] *= dec;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t xa[4], hi[4], lo[4];
      // x^T: rows p, columns s; transposed 8 x 8 pieces (s half of the fragment = mat >> 1, p half = mat & 1)
      sd_ldsm_t(sb + Cfg::X_OFF + (k * 16 + (mat >> 1) * 8 + r8) * Cfg::PROW + (warp * 16 + (mat & 1) * 8) * 2, xa[0], xa[1], xa[2], xa[3]);
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int s = k * 16 + (x >> 1) * 8 + 2 * tq;
        const float2 v = unpack_bf16(xa[x]);
        split_bf16(v.x * fast_exp2(cend - s_cum[s]) * s_dt[s], v.y * fast_exp2(cend - s_cum[s + 1]) * s_dt[s + 1], hi[x], lo[x]);
      }
#pragma unroll
      for (int j = 0; j < NP / 16; ++j) {
        uint32_t b0, b1, b2, b3;
        sd_ldsm_t(sb + Cfg::B_OFF + (k * 16 + (mat & 1) * 8 + r8) * Cfg::NROW + (j * 16 + (mat >> 1) * 8) * 2, b0, b1, b2, b3);
        sd_mma(st[2 * j], hi, b0, b1);
        sd_mma(st[2 * j + 1], hi, b2, b3);
        sd_mma(st[2 * j], lo, b0, b1);
        sd_mma(st[2 * j + 1], lo, b2, b3);
      }
    }
    __syncthreads();                                         // the next block's rows replace these
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int p = warp * 16 + gq + 8 * hh, n = j * 8 + 2 * tq;
      if (p < np && n < N) *reinterpret_cast<float2*>(Sg + (size_t)p * N + n) = make_float2(st[j][2 * hh], st[j][2 * hh + 1]);
    }
}

template <int NP>
static int launch_ssd(const void* xbc, long long ldx, const void* dtr, long long ldd, const float* dtb, const float* Al, const float* D, const int* cu,
                      const int* start, const int* state, int e0, int E, float* S, float* y, int H, int P, int N, int G, cudaStream_t s) {
  auto kern = mamba2_ssd_kernel<NP>;
  static ab2host::DevState st;
  if (ab2host::prepare_launch(kern, SsdCfg<NP>::SMEM, st, nullptr)) return 300;
  kern<<<dim3(E - e0, H, (P + SD_P - 1) / SD_P), 128, SsdCfg<NP>::SMEM, s>>>((const __nv_bfloat16*)xbc, ldx, (const __nv_bfloat16*)dtr, ldd, dtb, Al, D,
                                                                            cu, start, state, e0, S, y, H, P, N, G);
  return cudaGetLastError() == cudaSuccess ? 0 : 302;
}

}  // namespace ab2

// Entries e0 .. E - 1 (arguments as of ab2_mamba2_scan, bf16). P and N multiples of 8, N <= 128, rows of xbc 16-byte aligned.
extern "C" int ab2_mamba2_ssd(const void* xbc, long long ldx, const void* dtr, long long ldd, const float* dt_bias, const float* A_log, const float* D,
                              const int* cu, const int* start, const int* state, int e0, int E, float* S, float* y, int H, int P, int N, int G,
                              void* stream) {
  using namespace ab2;
  if (E <= e0) return 0;
  if (G < 1 || H % G || H > 65535 || (P & 7) || (N & 7) || N > 128 || (ldx & 7) || !aligned_to(xbc, 16)) return 10;
  cudaStream_t s = (cudaStream_t)stream;
  if (N <= 32) return launch_ssd<32>(xbc, ldx, dtr, ldd, dt_bias, A_log, D, cu, start, state, e0, E, S, y, H, P, N, G, s);
  if (N <= 64) return launch_ssd<64>(xbc, ldx, dtr, ldd, dt_bias, A_log, D, cu, start, state, e0, E, S, y, H, P, N, G, s);
  return launch_ssd<128>(xbc, ldx, dtr, ldd, dt_bias, A_log, D, cu, start, state, e0, E, S, y, H, P, N, G, s);
}
