// Attention of single rows over cached latents: one vector c of C numbers per token is key and value of every head (the heads'
// own key part has been applied to the queries, their value part is applied to the result). A row sees its own position and
// the window - 1 before it, or all earlier ones (window = 0).
//
// A CTA takes one row and 16 or 32 of its heads; the CTAs of a cluster share the row's keys in consecutive stretches. Pieces
// of 64 latents are staged by asynchronous copies, once for both products (mma.sync, 32-bit sums):
//   S = Q C^T     every warp its heads and keys, over the whole latent; to shared memory in 32 bits
//   softmax       every warp its heads: running maximum and sum in registers, the weights to shared memory
//   O += P C      every warp its eighth of the latent's columns, for all heads
// Partial results are merged through distributed shared memory.
#include <cooperative_groups.h>

#include "mixer_common.cuh"

namespace ab2 {

constexpr int LD_KEYS = 64, LD_THREADS = 256;

struct LatentArgs {
  const __nv_bfloat16* cache;
  const int *pages, *page_base;
  int max_pages, page_size, H, C;
  float scale;
  int window;
};

// DC: latent size rounded up to 128, 256 or 512 (missing columns are zero-filled); MT: 16-head tiles of a CTA
template <int DC, int MT>
struct LatentCfg {
  static constexpr int ROW = DC * 2 + 16;                          // padded rows: matrix loads touch distinct banks
  static constexpr int STAGE = LD_KEYS * ROW;
  static constexpr int NS = DC == 128 ? 3 : 2;                     // stages
  static constexpr int CTAS = DC == 512 ? 1 : 2;                   // per SM
  static constexpr int HEADS = 16 * MT;
  static constexpr int SROW = LD_KEYS + 4, PROW = LD_KEYS * 2 + 16;
  static constexpr int Q_OFF = NS * STAGE;
  static constexpr int S_OFF = Q_OFF + HEADS * ROW;
  static constexpr int P_OFF = S_OFF + HEADS * SROW * 4;
  static constexpr int A_OFF = P_OFF + HEADS * PROW;               // rescaling factor per head
  static constexpr int ROWS_OFF = A_OFF + HEADS * 4;               // cache row of every key, two pieces
  static constexpr int SMEM = ROWS_OFF + 2 * LD_KEYS * 4;
  static_assert(NS * STAGE >= HEADS * DC * 4, "the merge buffer aliases the stage memory");
};

__device__ __forceinline__ void ld_copy16(uint32_t dst, const void* src, bool ok) {
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ld_mat(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ld_mat_t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ld_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int DC, int MT>
__global__ void __launch_bounds__(LD_THREADS, LatentCfg<DC, MT>::CTAS)
latent_decode_kernel(const __nv_bfloat16* __restrict__ q, const int* __restrict__ pos, const int* __restrict__ slots,
                     const int* __restrict__ row_entry, __nv_bfloat16* __restrict__ out, const LatentArgs p) {
  namespace cg = cooperative_groups;
  using Cfg = LatentCfg<DC, MT>;
  constexpr int KS = DC / 16, RW = Cfg::HEADS / 8;                  // k-steps of a score; softmax rows of a warp
  constexpr int WC = DC / 8, NT = WC / 8;                           // columns of a warp in the second product, in tiles of 8
  extern __shared__ __align__(128) unsigned char dsm[];
  __shared__ float s_ml[2][32];                                     // this CTA's (max, sum) per head
  pdl_wait();
  pdl_trigger();
  const int b = blockIdx.x, h0 = blockIdx.y * Cfg::HEADS, spl = blockIdx.z, nspl = gridDim.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int mat = lane >> 3, r8 = lane & 7;
  const int heads = min(Cfg::HEADS, p.H - h0);
  const int i = pos[b], e = row_entry[b];
  const int lo = p.window > 0 ? max(0, i - p.window + 1) : 0;
  const int len = slots[b] >= 0 ? i + 1 - lo : 0;
  const int per = ((len + nspl - 1) / nspl + LD_KEYS - 1) / LD_KEYS * LD_KEYS;
  const int t0 = lo + spl * per, t1 = min(lo + len, t0 + per);
  const int np = t1 > t0 ? (t1 - t0 + LD_KEYS - 1) / LD_KEYS : 0;
  const int* pt = p.pages + (size_t)e * p.max_pages;
  const int base = p.page_base[e];
  const uint32_t sm = smem_u32(dsm);
  float* s_s = reinterpret_cast<float*>(dsm + Cfg::S_OFF);
  float* s_alpha = reinterpret_cast<float*>(dsm + Cfg::A_OFF);
  int* s_row = reinterpret_cast<int*>(dsm + Cfg::ROWS_OFF);
  auto plan = [&](int c) {
    if (tid < LD_KEYS && c < np) {
      const int t = t0 + c * LD_KEYS + tid;
      s_row[(c & 1) * LD_KEYS + tid] = t < t1 ? pt[t / p.page_size - base] * p.page_size + t % p.page_size : -1;
    }
  };
  auto issue = [&](int c) {                                         // past the last piece: an empty group
    if (c < np) {
      const uint32_t st = sm + (c % Cfg::NS) * Cfg::STAGE;
#pragma unroll 4
      for (int k = 0; k < LD_KEYS * (DC / 8) / LD_THREADS; ++k) {
        const int idx = tid + k * LD_THREADS, r = idx / (DC / 8), piece = idx % (DC / 8);
        const int row = s_row[(c & 1) * LD_KEYS + r];
        const bool ok = row >= 0 && piece * 8 < p.C;
        ld_copy16(st + r * Cfg::ROW + piece * 16, p.cache + (ok ? (size_t)row * p.C + piece * 8 : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int c = 0; c < Cfg::NS - 1; ++c) {
    plan(c);
    __syncthreads();
    issue(c);
  }
  plan(Cfg::NS - 1);
  for (int k = tid; k < Cfg::HEADS * (DC / 8); k += LD_THREADS) {
    const int r = k / (DC / 8), piece = k % (DC / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < heads && piece * 8 < p.C) v = *reinterpret_cast<const uint4*>(q + ((size_t)b * p.H + h0 + r) * p.C + piece * 8);
    *reinterpret_cast<uint4*>(dsm + Cfg::Q_OFF + r * Cfg::ROW + piece * 16) = v;
  }
  const float sc = p.scale * 1.4426950408889634f;                   // scores in base-2 units
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NT; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
  float m_run[RW], l_run[RW];                                       // rows warp * RW ...; sums of this lane's keys only
#pragma unroll
  for (int r = 0; r < RW; ++r) { m_run[r] = -INFINITY; l_run[r] = 0.f; }

  for (int c = 0; c < np; ++c) {
    asm volatile("cp.async.wait_group %0;" ::"n"(Cfg::NS - 2) : "memory");
    __syncthreads();                                                // piece c is here, and nobody reads piece c - 1 any more
    issue(c + Cfg::NS - 1);
    const uint32_t st = sm + (c % Cfg::NS) * Cfg::STAGE;
    // ---- scores
    if constexpr (MT == 2) {
      const int mt = warp & 1, kg = warp >> 1;                      // 16 heads x 16 keys
      const uint32_t qa = sm + Cfg::Q_OFF + (mt * 16 + (mat & 1) * 8 + r8) * Cfg::ROW + (mat >> 1) * 16;
      const uint32_t ka = st + (kg * 16 + (mat >> 1) * 8 + r8) * Cfg::ROW + (mat & 1) * 16;
      float s[2][2][4] = {};                                        // [k-step parity][key half]
#pragma unroll 4
      for (int ks = 0; ks < KS; ks += 2)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t a[4], k[4];
          ld_mat(qa + (ks + x) * 32, a);
          ld_mat(ka + (ks + x) * 32, k);
          ld_mma(s[x][0], a, k[0], k[1]);
          ld_mma(s[x][1], a, k[2], k[3]);
        }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* d = s_s + (mt * 16 + gq) * Cfg::SROW + kg * 16 + n * 8 + 2 * tq;
        *reinterpret_cast<float2*>(d) = make_float2(s[0][n][0] + s[1][n][0], s[0][n][1] + s[1][n][1]);
        *reinterpret_cast<float2*>(d + 8 * Cfg::SROW) = make_float2(s[0][n][2] + s[1][n][2], s[0][n][3] + s[1][n][3]);
      }
    } else {                                                        // 16 heads x 8 keys
      const uint32_t qa = sm + Cfg::Q_OFF + ((mat & 1) * 8 + r8) * Cfg::ROW + (mat >> 1) * 16;
      const uint32_t ka = st + (warp * 8 + r8) * Cfg::ROW + mat * 16;
      float s[2][4] = {};
#pragma unroll 4
      for (int ks = 0; ks < KS; ks += 2) {
        uint32_t k[4];
        ld_mat(ka + ks * 32, k);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t a[4];
          ld_mat(qa + (ks + x) * 32, a);
          ld_mma(s[x], a, k[2 * x], k[2 * x + 1]);
        }
      }
      float* d = s_s + gq * Cfg::SROW + warp * 8 + 2 * tq;
      *reinterpret_cast<float2*>(d) = make_float2(s[0][0] + s[1][0], s[0][1] + s[1][1]);
      *reinterpret_cast<float2*>(d + 8 * Cfg::SROW) = make_float2(s[0][2] + s[1][2], s[0][3] + s[1][3]);
    }
    __syncthreads();
    // ---- softmax: lane has keys 2 lane and 2 lane + 1
    plan(c + Cfg::NS);
#pragma unroll
    for (int r = 0; r < RW; ++r) {
      const int row = warp * RW + r, t = t0 + c * LD_KEYS + 2 * lane;
      const float2 v = *reinterpret_cast<const float2*>(s_s + row * Cfg::SROW + 2 * lane);
      const float a = t < t1 ? v.x * sc : -INFINITY, z = t + 1 < t1 ? v.y * sc : -INFINITY;
      const float mn = fmaxf(m_run[r], warp_max(fmaxf(a, z)));      // finite: every piece has a visible key
      const float alpha = fast_exp2(m_run[r] - mn), pa = fast_exp2(a - mn), pz = fast_exp2(z - mn);
      m_run[r] = mn;
      l_run[r] = l_run[r] * alpha + pa + pz;
      *reinterpret_cast<uint32_t*>(dsm + Cfg::P_OFF + row * Cfg::PROW + 4 * lane) = pack_bf16(pa, pz);
      if (lane == 0) s_alpha[row] = alpha;
    }
    __syncthreads();
    // ---- weighted sum of the latents
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = s_alpha[m * 16 + gq], a1 = s_alpha[m * 16 + gq + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        o[m][j][0] *= a0; o[m][j][1] *= a0;
        o[m][j][2] *= a1; o[m][j][3] *= a1;
      }
    }
    const uint32_t pa0 = sm + Cfg::P_OFF + ((mat & 1) * 8 + r8) * Cfg::PROW + (mat >> 1) * 16;
    const uint32_t va0 = st + ((mat & 1) * 8 + r8) * Cfg::ROW + (warp * WC + (mat >> 1) * 8) * 2;
#pragma unroll
    for (int ks = 0; ks < LD_KEYS / 16; ++ks) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ld_mat(pa0 + m * 16 * Cfg::PROW + ks * 32, pf[m]);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t v[4];
        ld_mat_t(va0 + ks * 16 * Cfg::ROW + j * 16, v);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          ld_mma(o[m][j], pf[m], v[0], v[1]);
          ld_mma(o[m][j + 1], pf[m], v[2], v[3]);
        }
      }
    }
  }
  // ---- this CTA's sums
#pragma unroll
  for (int r = 0; r < RW; ++r) {
    const float l = warp_sum(l_run[r]);
    if (lane == 0) { s_ml[0][warp * RW + r] = m_run[r]; s_ml[1][warp * RW + r] = l; }
  }
  __syncthreads();
  if (nspl == 1) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int row = m * 16 + gq + 8 * hh;
        if (row >= heads) continue;
        const float l = s_ml[1][row], inv = l > 0.f ? 1.f / l : 0.f;
        __nv_bfloat16* dst = out + ((size_t)b * p.H + h0 + row) * p.C;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int col = warp * WC + j * 8 + 2 * tq;
          if (col < p.C) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16(o[m][j][2 * hh] * inv, o[m][j][2 * hh + 1] * inv);
        }
      }
    return;
  }
  // ---- the CTAs of the cluster
  float* mo = reinterpret_cast<float*>(dsm);                        // [HEADS][DC]
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      float* d = mo + (m * 16 + gq) * DC + warp * WC + j * 8 + 2 * tq;
      *reinterpret_cast<float2*>(d) = make_float2(o[m][j][0], o[m][j][1]);
      *reinterpret_cast<float2*>(d + 8 * DC) = make_float2(o[m][j][2], o[m][j][3]);
    }
  cg::cluster_group cl = cg::this_cluster();
  cl.sync();
  for (int k = spl * LD_THREADS + tid; k < heads * (DC / 2); k += LD_THREADS * nspl) {
    const int g = k / (DC / 2), col = (k - g * (DC / 2)) * 2;
    if (col >= p.C) continue;
    float mx = -INFINITY, ll = 0.f, ox = 0.f, oy = 0.f;
    for (int c = 0; c < nspl; ++c) mx = fmaxf(mx, cl.map_shared_rank(&s_ml[0][0], c)[g]);
    for (int c = 0; c < nspl; ++c) {
      const float* ml = cl.map_shared_rank(&s_ml[0][0], c);
      const float wt = ml[g] == -INFINITY ? 0.f : fast_exp2(ml[g] - mx);
      const float2 v = *reinterpret_cast<const float2*>(cl.map_shared_rank(mo, c) + g * DC + col);
      ll += ml[32 + g] * wt;
      ox += v.x * wt;
      oy += v.y * wt;
    }
    const float inv = ll > 0.f ? 1.f / ll : 0.f;
    *reinterpret_cast<uint32_t*>(out + ((size_t)b * p.H + h0 + g) * p.C + col) = pack_bf16(ox * inv, oy * inv);
  }
  cl.sync();                                                        // nobody leaves while its shared memory is being read
}

template <int DC, int MT>
static int launch_latent(const void* q, const int* pos, const int* slots, const int* row_entry, void* out, int R, const LatentArgs& a, cudaStream_t s) {
  using Cfg = LatentCfg<DC, MT>;
  auto kern = latent_decode_kernel<DC, MT>;
  static ab2host::DevState st;
  int sms = 0;
  if (ab2host::prepare_launch(kern, Cfg::SMEM, st, &sms)) return 300;
  const int tiles = (a.H + Cfg::HEADS - 1) / Cfg::HEADS;
  // as many CTAs per row as fit on the GPU at once, and no more than the window has pieces
  const int pieces = a.window > 0 ? (a.window + LD_KEYS - 1) / LD_KEYS : 1 << 20;
  int spl = 1;
  while (spl < 8 && spl < pieces && (long long)R * tiles * spl * 2 <= (long long)sms * Cfg::CTAS) spl *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(R, tiles, spl);
  cfg.blockDim = dim3(LD_THREADS);
  cfg.dynamicSmemBytes = Cfg::SMEM;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = spl;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ab2host::pdl_enabled() ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kern, (const __nv_bfloat16*)q, pos, slots, row_entry, (__nv_bfloat16*)out, a) == cudaSuccess ? 0 : 302;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// q, out [R, H, C] bf16; row r reads the pages of entry row_entry[r] up to position pos[r]; slots[r] < 0: padding row (zeros).
// cache [rows, C] bf16; pages [entries, max_pages] from page number page_base[entry] on. C a multiple of 8 up to 512.
int ab2_latent_decode(const void* q, const int* pos, const int* slots, const int* row_entry, void* out, int R, const void* cache, const int* pages,
                      const int* page_base, int max_pages, int page_size, int H, int C, float scale, int window, void* stream) {
  if (R <= 0) return 0;
  if ((C & 7) || C < 8 || C > 512 || H < 1 || H > 32 * 65535 || page_size < 1) return 10;
  if (!aligned_to(q, 16) || !aligned_to(cache, 16) || !aligned_to(out, 16)) return 11;
  LatentArgs a{(const __nv_bfloat16*)cache, pages, page_base, max_pages, page_size, H, C, scale, window};
  cudaStream_t s = (cudaStream_t)stream;
  if (H <= 16) {
    if (C <= 128) return launch_latent<128, 1>(q, pos, slots, row_entry, out, R, a, s);
    if (C <= 256) return launch_latent<256, 1>(q, pos, slots, row_entry, out, R, a, s);
    return launch_latent<512, 1>(q, pos, slots, row_entry, out, R, a, s);
  }
  if (C <= 128) return launch_latent<128, 2>(q, pos, slots, row_entry, out, R, a, s);
  if (C <= 256) return launch_latent<256, 2>(q, pos, slots, row_entry, out, R, a, s);
  return launch_latent<512, 2>(q, pos, slots, row_entry, out, R, a, s);
}
}
