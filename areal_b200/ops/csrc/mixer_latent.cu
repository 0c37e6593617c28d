// Attention of single rows over cached latents: one vector c of C numbers per token is key and value of every head (the heads'
// own key part has been applied to the queries, their value part is applied to the result). A row sees its own position and
// the window - 1 before it, or all earlier ones (window = 0). Keys and queries may have a second, rotated part of up to 64 numbers
// (stored behind the latent) that adds to the scores; a sink, a gate per head and a factor are those of AttnExtra.
//
// A CTA takes one row and 16 or 32 of its heads; the CTAs of a cluster share the row's keys in consecutive stretches. One warp
// brings pieces of 32 latents from the cache pages by TMA (128-byte swizzle, 64 columns a box); each is used twice. Of the
// eight others every one owns an eighth of the latent's columns, in both products (mma.sync, 32-bit sums):
//   S = Q C^T     every warp its columns' share of all scores; the shares meet in shared memory in 32 bits (of the second
//                 part, every warp takes 16 columns of 16 keys)
//   softmax       a few threads per head: sum of the shares, running maximum and sum, the weights to shared memory
//   O += P C      every warp its columns
// The output of piece c and the softmax of piece c + 1 run side by side. O is rescaled only when a head's maximum has
// grown by more than 2^8 since its reference was set. Partial results of a cluster are merged through distributed shared memory.
#include <cooperative_groups.h>

#include "mixer_common.cuh"

namespace ab2 {

constexpr int LD_KEYS = 32, LD_WARPS = 8, LD_WORK = 32 * LD_WARPS, LD_THREADS = LD_WORK + 32;

struct LatentArgs {
  const int *pages, *page_base;
  int max_pages, page_shift, H, C;
  float scale;
  int window;
  AttnExtra x;
  bool one_box;               // a piece is one box of the tensor map (32 rows, all chunks of 64 columns), else one per chunk (or two)
};

// DC: latent size rounded up to 128, 256 or 512 (missing columns are zero-filled); MT: 16-head tiles of a CTA; DR: 64 with a
// second part, else 0
template <int DC, int MT, int DR>
struct LatentCfg {
  static constexpr int CHUNK = LD_KEYS * 128;                      // 64 columns of a piece
  static constexpr int STAGE = (DC + DR) / 64 * CHUNK;
  static constexpr int NS = (DC == 512 ? 5 : 4) - (DR ? 1 : 0);    // stages: two in use, the others on their way
  static constexpr int CTAS = DC == 512 ? 1 : 2;                   // per SM
  static constexpr int HEADS = 16 * MT;
  static constexpr int SROW = LD_KEYS + 8, PROW = LD_KEYS * 2 + 16;
  static constexpr int S_OFF = NS * STAGE;                         // shares of the scores, [warp][head][key]
  static constexpr int P_OFF = S_OFF + LD_WARPS * HEADS * SROW * 4;
  static constexpr int A_OFF = P_OFF + 2 * HEADS * PROW;           // rescaling factor per head; these and the weights of two pieces
  static constexpr int BAR_OFF = A_OFF + 2 * HEADS * 4;
  static constexpr int SMEM = BAR_OFF + 2 * NS * 8 + 1024;
  static constexpr int MROW = DC + 8;                              // floats of a merge row
  static_assert(NS * STAGE >= HEADS * MROW * 4, "the merge buffer aliases the stage memory");
};

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
__device__ __forceinline__ void ld_sync() { asm volatile("bar.sync 1, %0;" ::"n"(LD_WORK) : "memory"); }     // the working warps

template <int DC, int MT, int DR>
__global__ void __launch_bounds__(LD_THREADS, LatentCfg<DC, MT, DR>::CTAS)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmR, const __nv_bfloat16* __restrict__ q,
                     const int* __restrict__ pos,
                     const int* __restrict__ slots, const int* __restrict__ row_entry, __nv_bfloat16* __restrict__ out, const LatentArgs p, int* err) {
  namespace cg = cooperative_groups;
  using Cfg = LatentCfg<DC, MT, DR>;
  constexpr int NS = Cfg::NS, HEADS = Cfg::HEADS;
  constexpr int WC = DC / LD_WARPS, KS = WC / 16, NT = WC / 8;      // columns of a warp; k-steps and tiles of 8 in them
  constexpr int TPR = LD_WORK / HEADS, KPT = LD_KEYS / TPR;         // softmax: threads per head, keys per thread
  extern __shared__ unsigned char dsm_raw[];
  __shared__ float s_ml[2][32];                                     // this CTA's (max, sum) per head
  __shared__ float s_wt[8][32];                                     // weights of the cluster's partial results
  unsigned char* dsm = dsm_raw + ((1024u - (smem_u32(dsm_raw) & 1023u)) & 1023u);
  const uint32_t sm = smem_u32(dsm), bar = sm + Cfg::BAR_OFF;
  auto full = [&](int s) { return bar + 8u * s; };
  auto empty = [&](int s) { return bar + 8u * (NS + s); };
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    prefetch_tmap(&tmC);
    for (int s = 0; s < NS; ++s) {
      mbar_init(full(s), 1);
      mbar_init(empty(s), LD_WARPS);
    }
    fence_mbar_init();
  }
  __syncthreads();
  pdl_wait();
  pdl_trigger();
  const int b = blockIdx.x, h0 = blockIdx.y * HEADS, spl = blockIdx.z, nspl = gridDim.z;
  const int heads = min(HEADS, p.H - h0);
  const int i = pos[b], e = row_entry[b];
  const int lo = p.window > 0 ? max(0, i - p.window + 1) : 0;
  const int nblk = slots[b] >= 0 ? i / LD_KEYS - lo / LD_KEYS + 1 : 0;      // pieces start at multiples of 32: each lies in one page, or
  const int per = (nblk + nspl - 1) / nspl;                                 // fills two of 16
  const int t0 = (lo / LD_KEYS + spl * per) * LD_KEYS;
  const int np = max(0, min(per, nblk - spl * per));
  float* s_s = reinterpret_cast<float*>(dsm + Cfg::S_OFF);
  float* s_alpha = reinterpret_cast<float*>(dsm + Cfg::A_OFF);
  auto factor = [&](int row) {                                      // of the output of head h0 + row
    const __nv_bfloat16* gate = (const __nv_bfloat16*)p.x.gate;
    return gate ? p.x.out_scale * sigmoid_t<true>(__bfloat162float(gate[b * p.x.ldg + h0 + row])) : p.x.out_scale;
  };

  if (warp == LD_WARPS) {
    if (elect_one() && np > 0) {
      const int* pt = p.pages + (size_t)e * p.max_pages;
      const int base = p.page_base[e], last = p.max_pages - 1, sh = p.page_shift, two = sh == 4 ? 1 : 0;
      auto row_at = [&](int t) {                                    // boxes outside the held pages are masked
        return (pt[min(max((t >> sh) - base, 0), last)] << sh) + (t & ((1 << sh) - 1));
      };
      int row0 = row_at(t0), row1 = two ? row_at(t0 + 16) : 0;
      bool ok = true;
      int s = 0;
      uint32_t ph = 1u;
      for (int c = 0; c < np; ++c) {
        ok = mbar_wait(empty(s), ph, err, ERR_WAIT_EMPTY);
        if (!ok) break;
        const uint32_t dst = sm + s * Cfg::STAGE;
        mbar_expect_tx(full(s), Cfg::STAGE);
        if (p.one_box) {
          tma_load_3d(dst, &tmC, full(s), 0, row0, 0);
        } else {
#pragma unroll 1
          for (int k = 0; k < DC / 64; ++k) {
            tma_load_3d(dst + k * Cfg::CHUNK, &tmC, full(s), k * 64, row0, 0);
            if (two) tma_load_3d(dst + k * Cfg::CHUNK + 16 * 128, &tmC, full(s), k * 64, row1, 0);
          }
        }
        if constexpr (DR > 0) {
          tma_load_3d(dst + DC / 64 * Cfg::CHUNK, &tmR, full(s), 0, row0, 0);
          if (two) tma_load_3d(dst + DC / 64 * Cfg::CHUNK + 16 * 128, &tmR, full(s), 0, row1, 0);
        }
        if (c + 1 < np) {
          row0 = row_at(t0 + (c + 1) * LD_KEYS);
          if (two) row1 = row_at(t0 + (c + 1) * LD_KEYS + 16);
        }
        if (++s == NS) { s = 0; ph ^= 1u; }
      }
      if (!ok) {                                                    // copies in flight get a bounded time to land
        const long long c0 = clock64();
        while (clock64() - c0 < 8000000LL) {}
      }
    }
    __syncwarp();
  } else {
    const int gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
    uint32_t qa[MT][KS][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int ks = 0; ks < KS; ++ks)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int row = m * 16 + gq + (x & 1) * 8, col = warp * WC + ks * 16 + (x >> 1) * 8 + 2 * tq;
          qa[m][ks][x] = row < heads && col < p.C ? *reinterpret_cast<const uint32_t*>(q + ((size_t)b * p.H + h0 + row) * p.C + col) : 0u;
        }
    // of the second part: 16 columns and 16 keys of this warp; these keys come first in its accumulators
    const int ks2 = warp & 3, keys2 = DR ? warp >> 2 : 0;
    uint32_t qr[MT][4];
    if constexpr (DR > 0) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int row = m * 16 + gq + (x & 1) * 8, col = ks2 * 16 + (x >> 1) * 8 + 2 * tq;
          qr[m][x] = row < heads && col < p.x.D2
                         ? *reinterpret_cast<const uint32_t*>((const __nv_bfloat16*)p.x.q2 + b * p.x.ldq2 + (h0 + row) * p.x.hsq2 + col) : 0u;
        }
    }
    const float sc = p.scale * 1.4426950408889634f;                 // scores in base-2 units
    float o[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < NT; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
    const int srow = tid / TPR, skey = tid % TPR * KPT;
    float m_run = -INFINITY, l_run = 0.f;                           // of head srow; the sum over this thread's keys only
    bool ok = true;                                                 // after a wait that gave up: no more waits, same barriers
    // this warp's columns inside a stage: chunk and first 16-byte piece of its rows (pieces are swizzled by the row)
    const uint32_t mine = (warp * WC / 64) * Cfg::CHUNK;
    constexpr int PIECES = WC / 8;
    const int c0 = warp * PIECES % 8;

    auto scores = [&](int stage) {
      const uint32_t st = sm + stage * Cfg::STAGE + mine + ((mat >> 1) * 8 + r8) * 128;
      float s[MT][LD_KEYS / 8][4] = {};
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const uint32_t a = st + (((c0 + ks * 2 + (mat & 1)) ^ r8) << 4);
#pragma unroll
        for (int n = 0; n < LD_KEYS / 8; n += 2) {
          uint32_t k[4];
          ld_mat(a + (n ^ (2 * keys2)) * 8 * 128, k);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            ld_mma(s[m][n], qa[m][ks], k[0], k[1]);
            ld_mma(s[m][n + 1], qa[m][ks], k[2], k[3]);
          }
        }
      }
      if constexpr (DR > 0) {
        uint32_t k[4];
        ld_mat(sm + stage * Cfg::STAGE + DC / 64 * Cfg::CHUNK + (keys2 * 16 + (mat >> 1) * 8 + r8) * 128 + (((ks2 * 2 + (mat & 1)) ^ r8) << 4), k);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          ld_mma(s[m][0], qr[m], k[0], k[1]);
          ld_mma(s[m][1], qr[m], k[2], k[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < LD_KEYS / 8; ++n) {
          float* d = s_s + (warp * HEADS + m * 16 + gq) * Cfg::SROW + (n ^ (2 * keys2)) * 8 + 2 * tq;
          *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(d + 8 * Cfg::SROW) = make_float2(s[m][n][2], s[m][n][3]);
        }
    };
    auto sums = [&](float (&v)[KPT]) {
#pragma unroll
      for (int k = 0; k < KPT; ++k) v[k] = 0.f;
#pragma unroll
      for (int w = 0; w < LD_WARPS; ++w) {
        const float* d = s_s + (w * HEADS + srow) * Cfg::SROW + skey;
        if constexpr (KPT == 4) {
          const float4 x = *reinterpret_cast<const float4*>(d);
          v[0] += x.x; v[1] += x.y; v[2] += x.z; v[3] += x.w;
        } else {
          const float2 x = *reinterpret_cast<const float2*>(d);
          v[0] += x.x; v[1] += x.y;
        }
      }
    };
    auto softmax = [&](int c, float (&v)[KPT]) {
      const int t = t0 + c * LD_KEYS + skey;
      float mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = t + k >= lo && t + k <= i ? v[k] * sc : -INFINITY;
        mx = fmaxf(mx, v[k]);
      }
#pragma unroll
      for (int x = TPR / 2; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));    // finite: every piece has a visible key
      float alpha = 1.f;
      if (mx > m_run + 8.f || m_run == -INFINITY) {
        alpha = fast_exp2(m_run - mx);
        m_run = mx;
      }
      float sum = 0.f;
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = fast_exp2(v[k] - m_run);
        sum += v[k];
      }
      l_run = l_run * alpha + sum;
      uint32_t* d = reinterpret_cast<uint32_t*>(dsm + Cfg::P_OFF + ((c & 1) * HEADS + srow) * Cfg::PROW + skey * 2);
#pragma unroll
      for (int k = 0; k < KPT / 2; ++k) d[k] = pack_bf16(v[2 * k], v[2 * k + 1]);
      if (skey == 0) s_alpha[(c & 1) * HEADS + srow] = alpha;
    };
    auto arrived = [&](int stage, uint32_t ph) {
      ok = ok && mbar_wait(full(stage), ph, err, ERR_WAIT_FULL);
      __syncwarp();
    };
    const uint32_t pa = sm + Cfg::P_OFF + ((mat & 1) * 8 + r8) * Cfg::PROW + (mat >> 1) * 16;
    if (np > 0) {
      arrived(0, 0u);
      scores(0);
      ld_sync();
      float v[KPT];
      sums(v);
      softmax(0, v);
    }
    int cur = 0, nxt = 1;                                           // stages of pieces c and c + 1
    uint32_t ph = 0u;                                               // of piece c + 1
    for (int c = 0; c < np; ++c) {
      ld_sync();                                                    // weights of piece c are there, shares of the scores free
      if (c + 1 < np) {
        arrived(nxt, ph);
        scores(nxt);
      }
      ld_sync();                                                    // shares of piece c + 1 are there
      float v[KPT];
      if (c + 1 < np) sums(v);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float* al = s_alpha + (c & 1) * HEADS + m * 16 + gq;
        const float a0 = al[0], a1 = al[8];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            o[m][j][0] *= a0; o[m][j][1] *= a0;
            o[m][j][2] *= a1; o[m][j][3] *= a1;
          }
        }
      }
      const uint32_t st = sm + cur * Cfg::STAGE + mine + ((mat & 1) * 8 + r8) * 128;
#pragma unroll
      for (int ks = 0; ks < LD_KEYS / 16; ++ks) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ld_mat(pa + ((c & 1) * HEADS + m * 16) * Cfg::PROW + ks * 32, pf[m]);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t cf[4];
          ld_mat_t(st + ks * 16 * 128 + (((c0 + j + (mat >> 1)) ^ r8) << 4), cf);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            ld_mma(o[m][j], pf[m], cf[0], cf[1]);
            ld_mma(o[m][j + 1], pf[m], cf[2], cf[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty(cur));
      cur = nxt;
      if (++nxt == NS) { nxt = 0; ph ^= 1u; }
      if (c + 1 < np) softmax(c + 1, v);
    }
    // ---- this CTA's sums
#pragma unroll
    for (int x = TPR / 2; x > 0; x >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
    if (skey == 0) { s_ml[0][srow] = m_run; s_ml[1][srow] = l_run; }
    ld_sync();
    if (nspl == 1) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int row = m * 16 + gq + 8 * hh;
          if (row >= heads) continue;
          const float sink = p.x.sink_of(h0 + row) * 1.4426950408889634f, mx = fmaxf(s_ml[0][row], sink);
          const float w = s_ml[0][row] == -INFINITY ? 0.f : fast_exp2(s_ml[0][row] - mx);
          const float l = s_ml[1][row] * w + (sink > -INFINITY ? fast_exp2(sink - mx) : 0.f), inv = l > 0.f ? w / l * factor(row) : 0.f;
          __nv_bfloat16* dst = out + ((size_t)b * p.H + h0 + row) * p.C;
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            const int col = warp * WC + j * 8 + 2 * tq;
            if (col < p.C) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16(o[m][j][2 * hh] * inv, o[m][j][2 * hh + 1] * inv);
          }
        }
    } else {
      float* mo = reinterpret_cast<float*>(dsm);                    // [HEADS][MROW], over the stages: every piece has been used
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          float* d = mo + (m * 16 + gq) * Cfg::MROW + warp * WC + j * 8 + 2 * tq;
          *reinterpret_cast<float2*>(d) = make_float2(o[m][j][0], o[m][j][1]);
          *reinterpret_cast<float2*>(d + 8 * Cfg::MROW) = make_float2(o[m][j][2], o[m][j][3]);
        }
    }
  }
  if (nspl == 1) return;
  // ---- the CTAs of the cluster
  cg::cluster_group cl = cg::this_cluster();
  cl.sync();
  if (tid < heads) {
    const float sink = p.x.sink_of(h0 + tid) * 1.4426950408889634f, f = factor(tid);
    float m[8], l[8], mx = sink, ll = 0.f;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      const float* ml = cl.map_shared_rank(&s_ml[0][0], min(c, nspl - 1));
      m[c] = c < nspl ? ml[tid] : -INFINITY;
      l[c] = ml[32 + tid];
      mx = fmaxf(mx, m[c]);
    }
    if (sink > -INFINITY) ll = fast_exp2(sink - mx);
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      m[c] = m[c] == -INFINITY ? 0.f : fast_exp2(m[c] - mx);
      ll += l[c] * m[c];
    }
#pragma unroll
    for (int c = 0; c < 8; ++c) s_wt[c][tid] = ll > 0.f ? m[c] / ll * f : 0.f;
  }
  __syncthreads();
  const float* mo = reinterpret_cast<const float*>(dsm);
  for (int k = spl * LD_THREADS + tid; k < heads * (DC / 4); k += LD_THREADS * nspl) {
    const int g = k / (DC / 4), col = (k - g * (DC / 4)) * 4;
    if (col >= p.C) continue;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = 0; c < nspl; ++c) {
      const float w = s_wt[c][g];
      const float4 v = *reinterpret_cast<const float4*>(cl.map_shared_rank(mo, c) + g * Cfg::MROW + col);
      s.x += v.x * w; s.y += v.y * w; s.z += v.z * w; s.w += v.w * w;
    }
    *reinterpret_cast<uint2*>(out + ((size_t)b * p.H + h0 + g) * p.C + col) = make_uint2(pack_bf16(s.x, s.y), pack_bf16(s.z, s.w));
  }
  cl.sync();                                                        // nobody leaves while its shared memory is being read
}

template <int DC, int MT, int DR>
static int launch_latent(const void* q, const int* pos, const int* slots, const int* row_entry, void* out, int R, const void* cache, int cache_rows,
                         LatentArgs a, cudaStream_t s) {
  using Cfg = LatentCfg<DC, MT, DR>;
  auto kern = latent_decode_kernel<DC, MT, DR>;
  static ab2host::DevState st;
  int sms = 0;
  if (ab2host::prepare_launch(kern, Cfg::SMEM, st, &sms)) return 300;
  CUtensorMap tc, tr;
  a.one_box = a.C % 64 == 0 && a.page_shift > 4;
  const uint64_t ld = (uint64_t)a.x.ldk * 2;
  const uint32_t box = a.page_shift > 4 ? LD_KEYS : 16;
  if (a.one_box) {             // (column of the chunk, row, chunk)
    if (ab2host::encode_tmap_3d(&tc, cache, 2, 64, cache_rows, a.C / 64, ld, 128, 64, LD_KEYS, DC / 64, true, 0)) return 100;
  } else if (ab2host::encode_tmap_3d(&tc, cache, 2, a.C, cache_rows, 1, ld, ld, 64, box, 1, true, 0)) {
    return 101;
  }
  tr = tc;
  if (DR && ab2host::encode_tmap_3d(&tr, a.x.k2, 2, a.x.D2, cache_rows, 1, (uint64_t)a.x.ldk2 * 2, (uint64_t)a.x.ldk2 * 2, 64, box, 1, true, 0)) return 102;
  int* err = ab2host::error_flag();
  if (!err) return 301;
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
  return cudaLaunchKernelEx(&cfg, kern, tc, tr, (const __nv_bfloat16*)q, pos, slots, row_entry, (__nv_bfloat16*)out, a, err) == cudaSuccess ? 0 : 302;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// q, out [R, H, C] bf16; row r reads the pages of entry row_entry[r] up to position pos[r]; slots[r] < 0: padding row (zeros).
// cache [cache_rows, C] bf16 (x->ldk elements from row to row); pages [entries, max_pages] from page number page_base[entry] on. C a
// multiple of 8 up to 512, page_size a power of two from 16 on. x: null, or second part (up to 64 numbers), sink, gate per head, factor.
int ab2_latent_decode(const void* q, const int* pos, const int* slots, const int* row_entry, void* out, int R, const void* cache, int cache_rows,
                      const int* pages, const int* page_base, int max_pages, int page_size, int H, int C, float scale, int window, const AttnExtra* x,
                      void* stream) {
  if (R <= 0) return 0;
  if ((C & 7) || C < 8 || C > 512 || H < 1 || H > 16 * 65535 || page_size < 16 || (page_size & (page_size - 1))) return 10;
  if (!aligned_to(q, 16) || !aligned_to(cache, 16) || !aligned_to(out, 16)) return 11;
  LatentArgs a{pages, page_base, max_pages, __builtin_ctz(page_size), H, C, scale, window, x ? *x : AttnExtra(), false};
  if (!a.x.ldk) a.x.ldk = C;
  if (!a.x.q2) a.x.D2 = 0;
  if ((a.x.ldk & 7) || (a.x.gate && !a.x.gate_per_head)) return 12;
  if (a.x.D2 && ((a.x.D2 & 7) || a.x.D2 > 64 || ((a.x.ldq2 | a.x.hsq2 | a.x.ldk2) & 7) || !aligned_to(a.x.q2, 16) || !aligned_to(a.x.k2, 16))) return 13;
#define AB2_LATENT(DC, MT)                                                                                                                    \
  return a.x.D2 ? launch_latent<DC, MT, 64>(q, pos, slots, row_entry, out, R, cache, cache_rows, a, (cudaStream_t)stream)                     \
                : launch_latent<DC, MT, 0>(q, pos, slots, row_entry, out, R, cache, cache_rows, a, (cudaStream_t)stream)
  if (H <= 16) {
    if (C <= 128) AB2_LATENT(128, 1);
    if (C <= 256) AB2_LATENT(256, 1);
    AB2_LATENT(512, 1);
  }
  if (C <= 128) AB2_LATENT(128, 2);
  if (C <= 256) AB2_LATENT(256, 2);
  AB2_LATENT(512, 2);
#undef AB2_LATENT
}
}
