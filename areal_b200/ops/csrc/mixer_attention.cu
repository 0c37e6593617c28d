// Attention of mixer stacks over the paged cache: scores capped by softcap * tanh(s / softcap), a logarithmic distance
// bias r1[h] * ln(1 + r2[h] * distance) taken off (both optional), and only the earlier keys of the query's own chunk of
// positions visible (chunks counted from position 0 of the sequence), or those of a sliding window (the query's position
// and the window - 1 before it), or all of them (chunk = window = 0). Query / key and value sizes may differ.
// Optional, all in AttnExtra: a second part of queries and keys that all heads share a key of (rotated parts beside latents),
// a sink (a score that only enters the denominator), a sigmoid gate on the output (per head or per channel), a factor of the
// output, a factor per key, row strides. Keys may be the values as well (vc = kc): then single-token rows read them once.
//
//   chunk_attn_plain_kernel   any sizes, bf16 or 32-bit: a warp per (row, head)
//   chunk_decode_kernel       single-token rows, bf16: a cluster of CTAs splits a request's chunk, mma.sync products,
//                             partial results merged through distributed shared memory
//   chunk_prefill_kernel      portions, bf16: tcgen05 products with accumulators in TMEM (second half of this file)
//
// Keys and values of the step's own tokens have been appended to the cache before. A query at position i needs rows
// of pages[entry][j / page_size - page_base[entry]] for the positions j that it sees.
#include <cooperative_groups.h>

#include "mixer_common.cuh"

namespace ab2 {

struct ChunkArgs {
  const void *kc, *vc;
  const int *pages, *page_base;
  int max_pages, page_size, Hq, Hkv, D, Dv;
  float scale, softcap;
  const float *r1, *r2;
  int chunk, window;          // at most one of them set
  AttnExtra x;

  __host__ void defaults() {  // strides that were left open: contiguous
    if (!x.ldq) { x.ldq = (long long)Hq * D; x.hsq = D; }
    if (!x.ldo) x.ldo = (long long)Hq * Dv;
    if (!x.ldk) x.ldk = (long long)Hkv * D;
    if (!x.ldv) x.ldv = (long long)Hkv * Dv;
    if (!x.q2) x.D2 = 0;
  }

  // first position that a query at i sees (never decreases with i)
  __device__ __forceinline__ int first_key(int i) const {
    if (window > 0) return max(0, i - window + 1);
    return chunk > 0 ? i / chunk * chunk : 0;
  }
};

// Score in base-2 units: log2(e) * (cap(s * scale) - r1 ln(1 + r2 d)). u_scale and s_out are set up by score_consts().
struct ScoreConsts {
  float u_scale, s_out;     // with a cap: tanh argument * 2 log2(e), cap * log2(e); without: scale * log2(e), -
};
__device__ __forceinline__ ScoreConsts score_consts(float scale, float softcap) {
  constexpr float L2E = 1.4426950408889634f;
  if (softcap > 0.f) return {2.f * L2E * scale / softcap, softcap * L2E};
  return {scale * L2E, 0.f};
}
template <bool CAP>
__device__ __forceinline__ float capped(float s, const ScoreConsts& c) {
  if constexpr (CAP) {
    // tanh(u) = 1 - 2 / (1 + e^{2u}); e^{2u} may overflow to infinity (tanh = 1)
    return c.s_out - __fdividef(2.f * c.s_out, 1.f + fast_exp2(fminf(s * c.u_scale, 80.f)));
  }
  return s * c.u_scale;
}

// ------------------------------------------------------------------ plain form
constexpr int PLAIN_MAX_DV = 512;

template <typename T>
__global__ void __launch_bounds__(128)
chunk_attn_plain_kernel(const T* __restrict__ q, const int* __restrict__ pos, const int* __restrict__ slots, const int* __restrict__ row_entry,
                        T* __restrict__ out, ChunkArgs p) {
  extern __shared__ float sq_all[];
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * 4 + warp;
  if (h >= p.Hq) return;
  // values wider than one CTA's registers: blockIdx.z takes its stretch of them
  const int v0 = blockIdx.z * PLAIN_MAX_DV, nv = min(p.Dv - v0, PLAIN_MAX_DV);
  T* o = out + row * p.x.ldo + (size_t)h * p.Dv + v0;
  if (slots[row] < 0) {
    for (int d = lane; d < nv; d += 32) stf(o + d, 0.f);
    return;
  }
  float* sq = sq_all + warp * (p.D + p.x.D2);
  float* sq2 = sq + p.D;
  for (int d = lane; d < p.D; d += 32) sq[d] = ldf(q + row * p.x.ldq + h * p.x.hsq + d) * p.scale;
  for (int d = lane; d < p.x.D2; d += 32) sq2[d] = ldf((const T*)p.x.q2 + row * p.x.ldq2 + h * p.x.hsq2 + d) * p.scale;
  __syncwarp();
  const bool vec = p.D % 4 == 0 && p.x.ldk % 4 == 0;
  const int e = row_entry[row], i = pos[row], kvh = h / (p.Hq / p.Hkv);
  const int lo = p.first_key(i);
  const int* pt = p.pages + (size_t)e * p.max_pages;
  const int base = p.page_base[e];
  const float r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
  float m = p.x.sink_of(h), l = m > -INFINITY ? 1.f : 0.f, acc[PLAIN_MAX_DV / 32];
#pragma unroll
  for (int k = 0; k < PLAIN_MAX_DV / 32; ++k) acc[k] = 0.f;
  for (int j0 = lo; j0 <= i; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    long long kv = 0;
    if (j <= i) {
      kv = (long long)pt[j / p.page_size - base] * p.page_size + j % p.page_size;
      const T* kr = (const T*)p.kc + kv * p.x.ldk + (size_t)kvh * p.D;
      float dot = 0.f;
      if (vec) {
        for (int d = 0; d < p.D; d += 4) {
          float v[4];
          ldv<4>(kr + d, v);
          dot += v[0] * sq[d] + v[1] * sq[d + 1] + v[2] * sq[d + 2] + v[3] * sq[d + 3];
        }
      } else {
        for (int d = 0; d < p.D; ++d) dot += ldf(kr + d) * sq[d];
      }
      const T* k2 = (const T*)p.x.k2 + kv * p.x.ldk2;
      for (int d = 0; d < p.x.D2; ++d) dot += ldf(k2 + d) * sq2[d];
      if (p.x.kf) dot *= p.x.kf[kv * p.Hkv + kvh];
      s = p.softcap > 0.f ? p.softcap * tanhf(dot / p.softcap) : dot;
      if (p.r1) s -= r1 * log1pf(r2 * (float)(i - j));
    }
    const float mn = fmaxf(m, warp_max(s));
    const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
    const float w = expf(s - mn);
    l = l * alpha + warp_sum(w);
    m = mn;
#pragma unroll
    for (int k = 0; k < PLAIN_MAX_DV / 32; ++k) acc[k] *= alpha;
    const int nj = min(32, i - j0 + 1);
    for (int t = 0; t < nj; ++t) {
      const float wt = __shfl_sync(0xffffffffu, w, t);
      const T* vr = (const T*)p.vc + __shfl_sync(0xffffffffu, kv, t) * p.x.ldv + (size_t)kvh * p.Dv + v0;
#pragma unroll
      for (int k = 0; k < PLAIN_MAX_DV / 32; ++k) {
        if (k * 32 >= nv) break;
        if (k * 32 + lane < nv) acc[k] += wt * ldf(vr + k * 32 + lane);
      }
    }
  }
  const T* gate = (const T*)p.x.gate;
  const float f = p.x.out_scale * (gate && p.x.gate_per_head ? sigmoid_t<false>(ldf(gate + row * p.x.ldg + h)) : 1.f);
  const bool each = gate && !p.x.gate_per_head;
#pragma unroll
  for (int k = 0; k < PLAIN_MAX_DV / 32; ++k) {
    const int d = k * 32 + lane;
    if (d < nv) stf(o + d, acc[k] / l * f * (each ? sigmoid_t<false>(ldf(gate + row * p.x.ldg + (size_t)h * p.Dv + v0 + d)) : 1.f));
  }
}

// ------------------------------------------------------------------ single-token rows
// As the paged decode kernel of infer.cu: 64-key pieces staged by asynchronous copies, one warp per 16 keys, the query
// heads of the group as rows of a 16-row tile. DK / DV are the sizes rounded up to 64 or 128 (missing columns are
// zero-filled in shared memory). The SPL CTAs of a cluster take consecutive stretches of the chunk.
constexpr int CD_KEYS = 64;

__device__ __forceinline__ void cd_copy16(uint32_t dst, const void* src, bool ok) {
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cd_ldsm(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void cd_ldsm_t(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void cd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int DK, int DV>
struct ChunkDecodeCfg {
  static constexpr int KROW = DK * 2 + 16, VROW = DV * 2 + 16;     // padded rows: matrix loads touch distinct banks
  static constexpr int STAGE = CD_KEYS * (KROW + VROW);
  static constexpr int Q_OFF = 2 * STAGE;
  static constexpr int ROWS_OFF = Q_OFF + 16 * KROW;               // cache row of every key, four pieces
  static constexpr int SMEM = ROWS_OFF + 4 * CD_KEYS * 4;
};

template <int DK, int DV, int SPL, bool CAP>
__device__ __forceinline__ void chunk_decode_body(const __nv_bfloat16* __restrict__ q, const int* __restrict__ pos, const int* __restrict__ slots,
                                                  __nv_bfloat16* __restrict__ out, const ChunkArgs& p) {
  namespace cg = cooperative_groups;
  using Cfg = ChunkDecodeCfg<DK, DV>;
  constexpr int KS = DK / 16;
  extern __shared__ __align__(128) unsigned char dsm[];
  __shared__ float s_ml[2][16];                                     // this CTA's merged (max, sum) per head
  __shared__ float s_kf[4][CD_KEYS];                                // factors of the keys of four pieces
  pdl_wait();
  pdl_trigger();
  const int b = blockIdx.x, h = blockIdx.y, spl = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int G = p.Hq / p.Hkv;
  const int i = pos[b];
  const bool live = slots[b] >= 0;
  const int lo = p.first_key(i);
  const int len = live ? i + 1 - lo : 0;
  const int per = ((len + SPL - 1) / SPL + CD_KEYS - 1) / CD_KEYS * CD_KEYS;
  const int t0 = lo + spl * per, t1 = min(lo + len, t0 + per);
  const int np = t1 > t0 ? (t1 - t0 + CD_KEYS - 1) / CD_KEYS : 0;
  const int* pt = p.pages + (size_t)b * p.max_pages;
  const int base = p.page_base[b];
  const uint32_t sm = smem_u32(dsm);
  int* s_row = reinterpret_cast<int*>(dsm + Cfg::ROWS_OFF);
  // keys that are the values: one copy of a piece serves both products, and twice as many pieces are on their way
  const bool same = DK == DV && p.vc == p.kc;
  const int ahead = same ? 3 : 1, stage = same ? CD_KEYS * Cfg::KROW : Cfg::STAGE;
  auto row_of = [&](int c) {                                        // cache row of this thread's key of piece c
    const int t = t0 + c * CD_KEYS + tid;
    return tid < CD_KEYS && t < t1 ? pt[t / p.page_size - base] * p.page_size + t % p.page_size : -1;
  };
  auto plan = [&](int c, int row) {
    if (tid < CD_KEYS) s_row[(c & 3) * CD_KEYS + tid] = row;
  };
  auto issue = [&](int c) {
    const uint32_t st = sm + (c & ahead) * stage;
#pragma unroll
    for (int k = 0; k < CD_KEYS * (DK / 8) / 128; ++k) {
      const int idx = tid + k * 128, r = idx / (DK / 8), piece = idx % (DK / 8);
      const int row = s_row[(c & 3) * CD_KEYS + r];
      const bool ok = row >= 0 && piece * 8 < p.D;
      cd_copy16(st + r * Cfg::KROW + piece * 16, (const __nv_bfloat16*)p.kc + (ok ? row * p.x.ldk + h * p.D + piece * 8 : 0), ok);
    }
    if (!same) {
#pragma unroll
      for (int k = 0; k < CD_KEYS * (DV / 8) / 128; ++k) {
        const int idx = tid + k * 128, r = idx / (DV / 8), piece = idx % (DV / 8);
        const int row = s_row[(c & 3) * CD_KEYS + r];
        const bool ok = row >= 0 && piece * 8 < p.Dv;
        cd_copy16(st + CD_KEYS * Cfg::KROW + r * Cfg::VROW + piece * 16, (const __nv_bfloat16*)p.vc + (ok ? row * p.x.ldv + h * p.Dv + piece * 8 : 0), ok);
      }
    }
    if (p.x.kf && tid < CD_KEYS) {
      const int row = s_row[(c & 3) * CD_KEYS + tid];
      const float* f = p.x.kf + (row >= 0 ? (long long)row * p.Hkv + h : 0);
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(&s_kf[c & 3][tid])), "l"(f), "r"(row >= 0 ? 4 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int c = 0; c < 4; ++c)
    if (c < np && c <= ahead) plan(c, row_of(c));
  __syncthreads();
  for (int c = 0; c < min(np, ahead); ++c) issue(c);
  for (int k = tid; k < 16 * (DK / 8); k += 128) {
    const int r = k / (DK / 8), piece = k % (DK / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < G && piece * 8 < p.D) v = *reinterpret_cast<const uint4*>(q + b * p.x.ldq + (h * G + r) * p.x.hsq + piece * 8);
    *reinterpret_cast<uint4*>(dsm + Cfg::Q_OFF + r * Cfg::KROW + piece * 16) = v;
  }
  __syncthreads();
  const int mat = lane >> 3, r8 = lane & 7;
  uint32_t qa[KS][4];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks)
    cd_ldsm(sm + Cfg::Q_OFF + ((mat & 1) * 8 + r8) * Cfg::KROW + (ks * 16 + (mat >> 1) * 8) * 2, qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
  float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
  if (p.r1) {
#pragma unroll
    for (int hh = 0; hh < 2; ++hh)
      if (gq + 8 * hh < G) { r1[hh] = p.r1[h * G + gq + 8 * hh]; r2[hh] = p.r2[h * G + gq + 8 * hh]; }
  }
  const ScoreConsts sc = score_consts(p.scale, p.softcap);
  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  for (int c = 0; c < np; ++c) {
    if (c + ahead < np) issue(c + ahead);
    const int later = min(np - 1 - c, ahead);         // pieces that need not be there yet
    if (later == 0) asm volatile("cp.async.wait_group 0;" ::: "memory");
    else if (later == 1) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else if (later == 2) asm volatile("cp.async.wait_group 2;" ::: "memory");
    else asm volatile("cp.async.wait_group 3;" ::: "memory");
    __syncthreads();
    const int next = c + ahead + 1 < np ? row_of(c + ahead + 1) : -1;      // looked up while this piece is worked on
    const uint32_t ka = sm + (c & ahead) * stage + warp * 16 * Cfg::KROW;
    const uint32_t va = same ? ka : sm + (c & 1) * Cfg::STAGE + CD_KEYS * Cfg::KROW + warp * 16 * Cfg::VROW;
    float s[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t b0, b1, b2, b3;
      cd_ldsm(ka + ((mat >> 1) * 8 + r8) * Cfg::KROW + (ks * 16 + (mat & 1) * 8) * 2, b0, b1, b2, b3);
      cd_mma(s[0], qa[ks], b0, b1);
      cd_mma(s[1], qa[ks], b2, b3);
    }
    const int tok = t0 + c * CD_KEYS + warp * 16 + 2 * tq;
    if (p.x.kf) {
      const float* f = &s_kf[c & 3][warp * 16 + 2 * tq];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float v = f[(k >> 1) * 8 + (k & 1)];
        s[k >> 1][k & 1] *= v;
        s[k >> 1][2 + (k & 1)] *= v;
      }
    }
    uint32_t pa[4];
    float alpha[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      if (hh * 8 >= G) {                                // a group of up to 8 heads leaves the lower half of the tile empty
        pa[hh] = pa[2 + hh] = 0u;
        alpha[hh] = 1.f;
        continue;
      }
      float v[4];
      float mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int t = tok + (k >> 1) * 8 + (k & 1);
        v[k] = -INFINITY;
        if (t < t1) v[k] = capped<CAP>(s[k >> 1][2 * hh + (k & 1)], sc) - r1[hh] * __log2f(1.f + r2[hh] * (float)(i - t));
        mx = fmaxf(mx, v[k]);
      }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m_run[hh], mx), mref = mn == -INFINITY ? 0.f : mn;
      alpha[hh] = fast_exp2(m_run[hh] - mref);
      m_run[hh] = mn;
#pragma unroll
      for (int k = 0; k < 4; ++k) v[k] = fast_exp2(v[k] - mref);
      l_run[hh] = l_run[hh] * alpha[hh] + (v[0] + v[1] + v[2] + v[3]);
      pa[hh] = pack_bf16(v[0], v[1]);
      pa[2 + hh] = pack_bf16(v[2], v[3]);
    }
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) {
      o[j][0] *= alpha[0]; o[j][1] *= alpha[0];
      o[j][2] *= alpha[1]; o[j][3] *= alpha[1];
    }
#pragma unroll
    for (int jj = 0; jj < DV / 16; ++jj) {
      uint32_t b0, b1, b2, b3;
      cd_ldsm_t(va + ((mat & 1) * 8 + r8) * Cfg::VROW + (jj * 16 + (mat >> 1) * 8) * 2, b0, b1, b2, b3);
      cd_mma(o[2 * jj], pa, b0, b1);
      cd_mma(o[2 * jj + 1], pa, b2, b3);
    }
    if (c + ahead + 1 < np) plan(c + ahead + 1, next);                     // that part of the table is free: its piece has been issued
    __syncthreads();
  }
  // ---- the four warps, then the CTAs of the cluster
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
  }
  float* mo = reinterpret_cast<float*>(dsm);          // [4][16][DV], later the merged [16][DV] in its first part
  float* mm = mo + 4 * 16 * DV;
  float* ml = mm + 4 * 16;
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) {
    const int col = j * 8 + 2 * tq;
    *reinterpret_cast<float2*>(mo + (warp * 16 + gq) * DV + col) = make_float2(o[j][0], o[j][1]);
    *reinterpret_cast<float2*>(mo + (warp * 16 + gq + 8) * DV + col) = make_float2(o[j][2], o[j][3]);
  }
  if (tq == 0) {
    mm[warp * 16 + gq] = m_run[0]; mm[warp * 16 + gq + 8] = m_run[1];
    ml[warp * 16 + gq] = l_run[0]; ml[warp * 16 + gq + 8] = l_run[1];
  }
  __syncthreads();
  // the sink joins the denominator where the last sums are made; then gate and factor
  auto store = [&](int g, int d, float ll, float oo) {
    if (d >= p.Dv) return;
    const int head = h * G + g;
    float f = ll > 0.f ? p.x.out_scale / ll : 0.f;
    const __nv_bfloat16* gate = (const __nv_bfloat16*)p.x.gate;
    if (gate) f *= sigmoid_t<true>(__bfloat162float(gate[b * p.x.ldg + (p.x.gate_per_head ? head : head * p.Dv + d)]));
    out[b * p.x.ldo + (size_t)head * p.Dv + d] = __float2bfloat16(oo * f);
  };
  for (int k = tid; k < G * DV; k += 128) {
    const int g = k / DV, d = k - g * DV;
    float mx = -INFINITY, ll = 0.f, oo = 0.f;
    if constexpr (SPL == 1) mx = p.x.sink_of(h * G + g) * 1.4426950408889634f;
    const float sink = mx;
#pragma unroll
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, mm[w * 16 + g]);
    if (sink > -INFINITY) ll = fast_exp2(sink - mx);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = mm[w * 16 + g];
      const float wt = mw == -INFINITY ? 0.f : fast_exp2(mw - mx);
      ll += ml[w * 16 + g] * wt;
      oo += mo[(w * 16 + g) * DV + d] * wt;
    }
    if constexpr (SPL == 1) {
      store(g, d, ll, oo);
    } else {
      mo[g * DV + d] = oo;                             // only this thread reads (w, g, d) and writes (0, g, d)
      if (d == 0) { s_ml[0][g] = mx; s_ml[1][g] = ll; }
    }
  }
  if constexpr (SPL > 1) {
    cg::cluster_group cl = cg::this_cluster();
    cl.sync();
    for (int k = spl * 128 + tid; k < G * DV; k += 128 * SPL) {
      const int g = k / DV, d = k - g * DV;
      const float sink = p.x.sink_of(h * G + g) * 1.4426950408889634f;
      float mx = sink, ll = 0.f, oo = 0.f;
#pragma unroll
      for (int c = 0; c < SPL; ++c) mx = fmaxf(mx, cl.map_shared_rank(&s_ml[0][0], c)[g]);
      if (sink > -INFINITY) ll = fast_exp2(sink - mx);
#pragma unroll
      for (int c = 0; c < SPL; ++c) {
        const float mc = cl.map_shared_rank(&s_ml[0][0], c)[g];
        const float wt = mc == -INFINITY ? 0.f : fast_exp2(mc - mx);
        ll += cl.map_shared_rank(&s_ml[0][0], c)[16 + g] * wt;
        oo += cl.map_shared_rank(mo, c)[g * DV + d] * wt;
      }
      store(g, d, ll, oo);
    }
    cl.sync();                                         // nobody leaves while its shared memory is being read
  }
}

template <int DK, int DV, bool CAP>
__global__ void __launch_bounds__(128, 3)
chunk_decode_kernel(const __nv_bfloat16* __restrict__ q, const int* __restrict__ pos, const int* __restrict__ slots, __nv_bfloat16* __restrict__ out,
                    const ChunkArgs p) {
  chunk_decode_body<DK, DV, 1, CAP>(q, pos, slots, out, p);
}
template <int DK, int DV, int SPL, bool CAP>
__global__ void __cluster_dims__(1, 1, SPL) __launch_bounds__(128, 3)
chunk_decode_split_kernel(const __nv_bfloat16* __restrict__ q, const int* __restrict__ pos, const int* __restrict__ slots,
                          __nv_bfloat16* __restrict__ out, const ChunkArgs p) {
  chunk_decode_body<DK, DV, SPL, CAP>(q, pos, slots, out, p);
}

// ------------------------------------------------------------------ portions: tcgen05
// One CTA: up to 256 query rows of one request (two 128-row tiles) of one head; the tiles share every K / V block of 64
// keys, and while one tile's softmax runs the other's products do. K and V come straight from the cache pages by TMA
// (box: one page, or 64 keys of it). Per tile and key block
//   S = Q K^T        tcgen05.mma, both operands from swizzled shared memory, S in TMEM (two buffers per tile)
//   softmax          four warps, one query row per thread: cap, distance bias (one value per diagonal of a warp's
//                    part of the block, worked out once in shared memory), mask, running maximum; P (bf16) over S in TMEM
//   O += P V         tcgen05.mma, P from TMEM, V from shared memory
// O is rescaled only when a row's maximum has grown by more than 2^8 since its reference was set.
// 384 threads: warp 0 TMA, warp 1 MMA issue and TMEM, warps 4-7 and 8-11 the softmax of the two tiles.
constexpr int CP_Q = 128, CP_K = 64;

// DR: 64 when queries and keys have a second part (up to 64 numbers, keys without heads), else 0; it is one more chunk of 64 columns.
template <int DK, int DV, int DR>
struct ChunkPrefillCfg {
  static constexpr int QC = (DK + DR) / 64, VC = DV / 64;    // 64-column chunks
  static constexpr int CP_ST = DK + DR > 128 ? 3 : 4;        // stages of K and V
  static constexpr int Q_BYTES = QC * CP_Q * 128;            // one tile
  static constexpr int K_BYTES = QC * CP_K * 128, V_BYTES = VC * CP_K * 128;
  static constexpr int BAR_OFF = 2 * Q_BYTES + CP_ST * (K_BYTES + V_BYTES);
  static constexpr int BIAS_OFF = BAR_OFF + 256;             // [softmax warp][buffer][96]
  static constexpr int SMEM = BIAS_OFF + 16 * 96 * 4 + 1024;
};

// ADJ: what else a score gets, from shared memory.
constexpr int ADJ_NONE = 0, ADJ_DISTANCE = 1, ADJ_KEY = 2;
template <int DK, int DV, int DR, bool CAP, int ADJ>
__global__ void __launch_bounds__(384, 1)
chunk_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                     const __grid_constant__ CUtensorMap tmQ2, const __grid_constant__ CUtensorMap tmK2, const int* __restrict__ cu,
                     const int* __restrict__ start, const int* __restrict__ tiles, __nv_bfloat16* __restrict__ out, const ChunkArgs p, int* err) {
  using Cfg = ChunkPrefillCfg<DK, DV, DR>;
  constexpr int CP_ST = Cfg::CP_ST, HC = DK / 64;             // chunks of the heads' own part
  const int e = tiles[2 * blockIdx.x], row0 = tiles[2 * blockIdx.x + 1], head = blockIdx.y;
  const int kvh = head / (p.Hq / p.Hkv);
  const int rows = min(2 * CP_Q, cu[e + 1] - row0);
  const int q0 = start[e] + row0 - cu[e];                     // position of the first query row
  const int ntile = rows > CP_Q ? 2 : 1;
  const int lo0 = p.first_key(q0);
  const int k0 = lo0 & ~(CP_K - 1);                           // first key block, on a 64-position boundary
  int nb[2];
  nb[0] = (q0 + min(rows, CP_Q) - 1 - k0) / CP_K + 1;
  nb[1] = ntile == 2 ? (q0 + rows - 1 - k0) / CP_K + 1 : 0;
  const int nmax = max(nb[0], nb[1]);

  extern __shared__ uint8_t smem_raw[];
  const uint32_t sb = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sQ = sb, sK = sb + 2 * Cfg::Q_BYTES, sV = sK + CP_ST * Cfg::K_BYTES, bar = sb + Cfg::BAR_OFF;
  float* bias = reinterpret_cast<float*>(smem_raw + (sb - smem_u32(smem_raw)) + Cfg::BIAS_OFF);
  const uint32_t q_full = bar;
  auto k_full = [&](int s) { return bar + 8u * (1 + s); };
  auto k_empty = [&](int s) { return bar + 8u * (5 + s); };
  auto v_full = [&](int s) { return bar + 8u * (9 + s); };
  auto v_empty = [&](int s) { return bar + 8u * (13 + s); };
  auto s_full = [&](int t, int b) { return bar + 8u * (17 + 2 * t + b); };
  auto p_ready = [&](int t) { return bar + 8u * (21 + t); };
  auto o_done = [&](int t) { return bar + 8u * (23 + t); };
  const uint32_t tmem_slot = bar + 8u * 25;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
    mbar_init(q_full, 1);
    for (int s = 0; s < CP_ST; ++s) {
      mbar_init(k_full(s), 1);
      mbar_init(k_empty(s), 1);
      mbar_init(v_full(s), 1);
      mbar_init(v_empty(s), 1);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(s_full(t, 0), 1);
      mbar_init(s_full(t, 1), 1);
      mbar_init(p_ready(t), 128);
      mbar_init(o_done(t), 1);
    }
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  uint32_t tm;
  asm volatile("ld.shared.b32 %0, [%1];" : "=r"(tm) : "r"(tmem_slot));
  auto s_col = [&](int t, int b) { return tm + t * 128 + b * 64; };      // S buffers, P over their first 32 columns
  auto o_col = [&](int t) { return tm + 256 + t * 128; };

  if (warp == 0) {
    if (elect_one()) {
      const int box = min(p.page_size, CP_K), per = CP_K / box;
      const int* pt = p.pages + (size_t)e * p.max_pages;
      const int base = p.page_base[e];
      bool ok = true;
      mbar_expect_tx(q_full, ntile * Cfg::Q_BYTES);
      for (int t = 0; t < ntile; ++t)
        for (int c = 0; c < Cfg::QC; ++c)
          tma_load_3d(sQ + t * Cfg::Q_BYTES + c * CP_Q * 128, c < HC ? &tmQ : &tmQ2, q_full, c < HC ? c * 64 : 0, head, row0 + t * CP_Q);
      for (int j = 0; j < nmax; ++j) {
        const int s = j % CP_ST;
        const uint32_t ph = (uint32_t)(j / CP_ST) & 1u;
        int crow[4];                                          // cache row of every box of the block
        for (int x = 0; x < per; ++x) {
          const int pos = k0 + j * CP_K + x * box;
          const int pg = min(max(pos / p.page_size - base, 0), p.max_pages - 1);   // boxes outside the held pages are masked
          crow[x] = pt[pg] * p.page_size + pos % p.page_size;
        }
        if (!mbar_wait(k_empty(s), ph ^ 1u, err, ERR_WAIT_EMPTY)) { ok = false; break; }
        mbar_expect_tx(k_full(s), Cfg::K_BYTES);
        for (int c = 0; c < Cfg::QC; ++c)
          for (int x = 0; x < per; ++x)
            tma_load_3d(sK + s * Cfg::K_BYTES + c * CP_K * 128 + x * box * 128, c < HC ? &tmK : &tmK2, k_full(s), c < HC ? c * 64 : 0, c < HC ? kvh : 0,
                        crow[x]);
        if (!mbar_wait(v_empty(s), ph ^ 1u, err, ERR_WAIT_EMPTY)) { ok = false; break; }
        mbar_expect_tx(v_full(s), Cfg::V_BYTES);
        for (int c = 0; c < Cfg::VC; ++c)
          for (int x = 0; x < per; ++x)
            tma_load_3d(sV + s * Cfg::V_BYTES + c * CP_K * 128 + x * box * 128, &tmV, v_full(s), c * 64, kvh, crow[x]);
      }
      if (!ok) {                                              // copies in flight get a bounded time to land
        const long long t0 = clock64();
        while (clock64() - t0 < 8000000LL) {}
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc(CP_Q, CP_K, 1, 1, 0, 0);
      constexpr uint32_t idesc_o = make_idesc(CP_Q, DV, 1, 1, 0, 1);
      bool ok = mbar_wait(q_full, 0, err, ERR_WAIT_FULL);
      auto issue_s = [&](int t, int j) {
        const int s = j % CP_ST;
#pragma unroll
        for (int kk = 0; kk < (DK + DR) / 16; ++kk) {
          if (DR && kk >= DK / 16 && (kk - DK / 16) * 16 >= p.x.D2) break;     // only zeros from here on
          const uint64_t ad = make_smem_desc_sw128(sQ + t * Cfg::Q_BYTES + (kk >> 2) * CP_Q * 128, 16, 1024) + (uint64_t)((kk & 3) * 2);
          const uint64_t bd = make_smem_desc_sw128(sK + s * Cfg::K_BYTES + (kk >> 2) * CP_K * 128, 16, 1024) + (uint64_t)((kk & 3) * 2);
          umma_f16(s_col(t, j & 1), ad, bd, idesc_s, kk != 0 ? 1u : 0u);
        }
        umma_commit(s_full(t, j & 1));
        if (t == ntile - 1) umma_commit(k_empty(s));
      };
      for (int j = 0; j < 2 && j < nmax && ok; ++j) {
        if (!mbar_wait(k_full(j), 0, err, ERR_WAIT_FULL)) { ok = false; break; }
        tc_fence_after();
        for (int t = 0; t < ntile; ++t)
          if (j < nb[t]) issue_s(t, j);
      }
      for (int j = 0; j < nmax && ok; ++j) {
        const int s = j % CP_ST;
        const uint32_t ph = (uint32_t)(j / CP_ST) & 1u;
        if (!mbar_wait(v_full(s), ph, err, ERR_WAIT_FULL)) { ok = false; break; }
        for (int t = 0; t < ntile && ok; ++t) {
          if (j >= nb[t]) continue;
          if (!mbar_wait(p_ready(t), (uint32_t)j & 1u, err, ERR_WAIT_MISC)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < CP_K / 16; ++kk) {
            const uint64_t bd = make_smem_desc_sw128(sV + s * Cfg::V_BYTES, CP_K * 128, 1024) + (uint64_t)(kk * (16 * 128 >> 4));
            umma_f16_ts(o_col(t), s_col(t, j & 1) + kk * 8, bd, idesc_o, (j | kk) != 0 ? 1u : 0u);
          }
          umma_commit(o_done(t));
        }
        if (!ok) break;
        umma_commit(v_empty(s));
        if (j + 2 < nmax) {
          const int s2 = (j + 2) % CP_ST;
          if (!mbar_wait(k_full(s2), (uint32_t)((j + 2) / CP_ST) & 1u, err, ERR_WAIT_FULL)) { ok = false; break; }
          for (int t = 0; t < ntile && ok; ++t) {
            if (j + 2 >= nb[t]) continue;
            // the buffer of S(j + 2) holds P(j): its product must be through
            if (!mbar_wait(o_done(t), (uint32_t)j & 1u, err, ERR_WAIT_MISC)) { ok = false; break; }
            tc_fence_after();
            issue_s(t, j + 2);
          }
        }
      }
    }
  } else if (warp >= 4) {
    const int t = (warp - 4) >> 2;
    const int qd = warp & 3, row = qd * 32 + lane;            // TMEM lane == row of the tile
    const uint32_t lane_off = (uint32_t)(qd * 32) << 16;
    const int nbt = t == 0 ? nb[0] : nb[1];
    const int first = q0 + t * CP_Q;                           // position of the tile's first row
    const int i = first + row;
    const int lo = p.first_key(i);
    const int last = min(rows - t * CP_Q, CP_Q) - 1;
    const int lo_last = p.first_key(first + max(last, 0));
    const ScoreConsts sc = score_consts(p.scale, p.softcap);
    const float r1 = p.r1 ? p.r1[head] : 0.f, r2 = p.r1 ? p.r2[head] : 0.f;
    float m_run = p.x.sink_of(head) * 1.4426950408889634f, l_run = m_run > -INFINITY ? 1.f : 0.f;
    bool ok = true;
    // factors of a block's keys, fetched a block ahead: this lane's are those of its keys lane and lane + 32
    float kf[2] = {0.f, 0.f};
    auto fetch_factors = [&](int j) {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int pos = k0 + j * CP_K + lane + 32 * x, pg = min(max(pos / p.page_size - p.page_base[e], 0), p.max_pages - 1);
        kf[x] = p.x.kf[((long long)p.pages[(size_t)e * p.max_pages + pg] * p.page_size + pos % p.page_size) * p.Hkv + kvh] * sc.u_scale;
      }
    };
    if constexpr (ADJ == ADJ_KEY)
      if (nbt > 0) fetch_factors(0);
    for (int j = 0; j < nbt && ok; ++j) {
      const int kb = k0 + j * CP_K;
      float* bs = bias + ((warp - 4) * 2 + (j & 1)) * 96;
      // diagonal x of this warp's 32 rows: distance first + 32 qd - kb + x - 63
      if constexpr (ADJ == ADJ_KEY) {
        bs[lane] = kf[0];
        bs[lane + 32] = kf[1];
        __syncwarp();
        if (j + 1 < nbt) fetch_factors(j + 1);
      }
      if constexpr (ADJ == ADJ_DISTANCE) {
        for (int x = lane; x < 95; x += 32) bs[x] = r1 * __log2f(1.f + r2 * (float)max(first + qd * 32 - kb + x - 63, 0));
        __syncwarp();
      }
      ok = __all_sync(0xffffffffu, mbar_wait(s_full(t, j & 1), (uint32_t)(j >> 1) & 1u, err, ERR_WAIT_TMEM_FULL));
      if (!ok) break;                                          // a warp gives up as a whole
      tc_fence_after();
      uint32_t u[64];
      tmem_ld32(s_col(t, j & 1) + lane_off, u);
      tmem_ld32(s_col(t, j & 1) + lane_off + 32, u + 32);
      tmem_ld_wait();
      const bool edge = kb < lo_last || kb + CP_K - 1 > first;
      float mx = -INFINITY;
      if constexpr (ADJ == ADJ_KEY) {
#pragma unroll
        for (int c = 0; c < 64; c += 4) {
          const float4 f = *reinterpret_cast<const float4*>(bs + c);
          u[c] = __float_as_uint(__uint_as_float(u[c]) * f.x);
          u[c + 1] = __float_as_uint(__uint_as_float(u[c + 1]) * f.y);
          u[c + 2] = __float_as_uint(__uint_as_float(u[c + 2]) * f.z);
          u[c + 3] = __float_as_uint(__uint_as_float(u[c + 3]) * f.w);
        }
      }
#pragma unroll
      for (int c = 0; c < 64; ++c) {
        float v = ADJ == ADJ_KEY ? __uint_as_float(u[c]) : capped<CAP>(__uint_as_float(u[c]), sc);
        if constexpr (ADJ == ADJ_DISTANCE) v -= bs[lane - c + 63];
        if (edge && (kb + c > i || kb + c < lo)) v = -INFINITY;
        u[c] = __float_as_uint(v);
        mx = fmaxf(mx, v);
      }
      float alpha = 1.f;
      const bool grow = mx > m_run + 8.f || (m_run == -INFINITY && mx > -INFINITY);
      const bool any_grow = __any_sync(0xffffffffu, grow);
      if (grow) {
        alpha = m_run == -INFINITY ? 0.f : fast_exp2(m_run - mx);
        m_run = mx;
      }
      const float mref = m_run == -INFINITY ? 0.f : m_run;
      float sum = 0.f;
      uint32_t pk[32];
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        const float a = fast_exp2(__uint_as_float(u[2 * c]) - mref), b = fast_exp2(__uint_as_float(u[2 * c + 1]) - mref);
        sum += a + b;
        pk[c] = pack_bf16(a, b);
      }
      l_run = l_run * alpha + sum;
      tmem_st32(s_col(t, j & 1) + lane_off, pk);
      if (j > 0) {
        ok = __all_sync(0xffffffffu, mbar_wait(o_done(t), (uint32_t)(j - 1) & 1u, err, ERR_WAIT_MISC));
        if (!ok) break;
        tc_fence_after();
        if (any_grow) {
#pragma unroll 1
          for (int c = 0; c < DV / 32; ++c) {
            uint32_t r[32];
            tmem_ld32(o_col(t) + lane_off + c * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int x = 0; x < 32; ++x) r[x] = __float_as_uint(__uint_as_float(r[x]) * alpha);
            tmem_st32(o_col(t) + lane_off + c * 32, r);
          }
        }
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(p_ready(t));
    }
    if (ok && nbt > 0) ok = __all_sync(0xffffffffu, mbar_wait(o_done(t), (uint32_t)(nbt - 1) & 1u, err, ERR_WAIT_MISC));
    if (ok && nbt > 0) {
      tc_fence_after();
      float inv = l_run > 0.f ? p.x.out_scale / l_run : 0.f;
      const size_t grow_ = row0 + t * CP_Q + min(row, max(last, 0));
      __nv_bfloat16* dst = out + grow_ * p.x.ldo + (size_t)head * p.Dv;
      const __nv_bfloat16* gate = (const __nv_bfloat16*)p.x.gate;
      const __nv_bfloat16* each = gate && !p.x.gate_per_head ? gate + grow_ * p.x.ldg + (size_t)head * p.Dv : nullptr;
      if (gate && p.x.gate_per_head) inv *= sigmoid_t<true>(__bfloat162float(gate[grow_ * p.x.ldg + head]));
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t r[32];
        tmem_ld32(o_col(t) + lane_off + c * 32, r);
        tmem_ld_wait();
        if (row <= last) {
#pragma unroll
          for (int x = 0; x < 4; ++x)
            if (c * 32 + x * 8 < p.Dv) {
              float v[8], g[8];
#pragma unroll
              for (int k = 0; k < 8; ++k) v[k] = __uint_as_float(r[8 * x + k]) * inv;
              if (each) {
                ldv<8>(each + c * 32 + x * 8, g);
#pragma unroll
                for (int k = 0; k < 8; ++k) v[k] *= sigmoid_t<true>(g[k]);
              }
              stv<8>(dst + c * 32 + x * 8, v);
            }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tm, 512);
  }
}

template <int DK, int DV, int, bool CAP, int>
static int launch_decode(const void* q, const int* pos, const int* slots, void* out, int R, const ChunkArgs& a, cudaStream_t s) {
  constexpr int SMEM = ChunkDecodeCfg<DK, DV>::SMEM;
  static_assert(2 * ChunkDecodeCfg<DK, DV>::STAGE >= (4 * 16 * DV + 8 * 16) * 4, "the merge buffers alias the stage memory");
  // as many pieces of a request as still run at once (three CTAs per SM); halves where whole requests leave a short second wave
  const long long pairs = (long long)R * a.Hkv, room = 3 * 148;
  const int spl = pairs * 8 <= room ? 8 : (pairs * 4 <= room ? 4 : (pairs * 2 <= room || (pairs > room && pairs < 2 * room) ? 2 : 1));
  auto go = [&](auto kern, ab2host::DevState& st) -> int {
    if (ab2host::prepare_launch(kern, SMEM, st, nullptr)) return 300;
    launch_pdl(kern, dim3(R, a.Hkv, spl), dim3(128), (size_t)SMEM, s, (const __nv_bfloat16*)q, pos, slots, (__nv_bfloat16*)out, a);
    return cudaGetLastError() == cudaSuccess ? 0 : 302;
  };
  static ab2host::DevState st1, st2, st4, st8;
  if (spl == 1) return go(chunk_decode_kernel<DK, DV, CAP>, st1);
  if (spl == 2) return go(chunk_decode_split_kernel<DK, DV, 2, CAP>, st2);
  if (spl == 4) return go(chunk_decode_split_kernel<DK, DV, 4, CAP>, st4);
  return go(chunk_decode_split_kernel<DK, DV, 8, CAP>, st8);
}

template <int DK, int DV, int DR, bool CAP, int ADJ>
static int launch_prefill(const void* q, const int* cu, const int* start, const int* tiles, int nt, void* out, int R, int cache_rows, const ChunkArgs& a,
                          cudaStream_t s) {
  using Cfg = ChunkPrefillCfg<DK, DV, DR>;
  CUtensorMap tq, tk, tv, tq2, tk2;
  const uint32_t box = a.page_size < CP_K ? a.page_size : CP_K;
  auto map = [&](CUtensorMap* m, const void* base, int cols, int heads, int rows, long long head_stride, long long row_stride, uint32_t box_rows) {
    return ab2host::encode_tmap_3d(m, base, 2, cols, heads, rows, (uint64_t)head_stride * 2, (uint64_t)row_stride * 2, 64, 1, box_rows, true, 0);
  };
  if (map(&tq, q, a.D, a.Hq, R, a.x.hsq, a.x.ldq, CP_Q)) return 100;
  if (map(&tk, a.kc, a.D, a.Hkv, cache_rows, a.D, a.x.ldk, box)) return 101;
  if (map(&tv, a.vc, a.Dv, a.Hkv, cache_rows, a.Dv, a.x.ldv, box)) return 102;
  tq2 = tq;
  tk2 = tk;
  if (DR && map(&tq2, a.x.q2, a.x.D2, a.Hq, R, a.x.hsq2, a.x.ldq2, CP_Q)) return 103;
  if (DR && map(&tk2, a.x.k2, a.x.D2, 1, cache_rows, a.x.ldk2, a.x.ldk2, box)) return 104;
  auto kern = chunk_prefill_kernel<DK, DV, DR, CAP, ADJ>;
  static ab2host::DevState st;
  if (ab2host::prepare_launch(kern, Cfg::SMEM, st, nullptr)) return 300;
  int* err = ab2host::error_flag();
  if (!err) return 301;
  kern<<<dim3(nt, a.Hq), 384, Cfg::SMEM, s>>>(tq, tk, tv, tq2, tk2, cu, start, tiles, (__nv_bfloat16*)out, a, err);
  return cudaGetLastError() == cudaSuccess ? 0 : 302;
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// q [R, Hq, D], out [R, Hq, Dv], one row per (pos, slot, entry); slot < 0: padding row (zeros). Cache: kc [rows, Hkv, D],
// vc [rows, Hkv, Dv]; pages [entries, max_pages] from page number page_base[entry] on. r1 / r2 [Hq] or null. x: null, or what
// AttnExtra says. dt 0 bf16, 1 fp32.
int ab2_chunk_attn_plain(const void* q, const int* pos, const int* slots, const int* row_entry, void* out, int R, const void* kc, const void* vc,
                         const int* pages, const int* page_base, int max_pages, int page_size, int Hq, int Hkv, int D, int Dv, float scale,
                         float softcap, const float* r1, const float* r2, int chunk, int window, const AttnExtra* x, int dt, void* stream) {
  if (R <= 0) return 0;
  ChunkArgs a{kc, vc, pages, page_base, max_pages, page_size, Hq, Hkv, D, Dv, scale, softcap, r1, r2, chunk, window, x ? *x : AttnExtra()};
  a.defaults();
  const int smem = 16 * (D + a.x.D2);
  if (Hq % Hkv || Dv > 65535 || smem > 48 * 1024) return 10;
  const dim3 grid(R, (Hq + 3) / 4, (Dv + PLAIN_MAX_DV - 1) / PLAIN_MAX_DV);
  if (dt == 0)
    chunk_attn_plain_kernel<__nv_bfloat16><<<grid, 128, smem, (cudaStream_t)stream>>>((const __nv_bfloat16*)q, pos, slots, row_entry,
                                                                                     (__nv_bfloat16*)out, a);
  else
    chunk_attn_plain_kernel<float><<<grid, 128, smem, (cudaStream_t)stream>>>((const float*)q, pos, slots, row_entry, (float*)out, a);
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

#define AB2_BY_SIZE2(FN, DR, CAP, ADJ, ...)                                                                               \
  if (D <= 64) return Dv <= 64 ? FN<64, 64, DR, CAP, ADJ>(__VA_ARGS__) : FN<64, 128, DR, CAP, ADJ>(__VA_ARGS__);          \
  return Dv <= 64 ? FN<128, 64, DR, CAP, ADJ>(__VA_ARGS__) : FN<128, 128, DR, CAP, ADJ>(__VA_ARGS__)

// Row r is the only row of entry r. bf16; D, Dv multiples of 8 up to 128, at most 16 query heads per key head; no second part.
int ab2_chunk_decode(const void* q, const int* pos, const int* slots, void* out, int R, const void* kc, const void* vc, const int* pages,
                     const int* page_base, int max_pages, int page_size, int Hq, int Hkv, int D, int Dv, float scale, float softcap,
                     const float* r1, const float* r2, int chunk, int window, const AttnExtra* x, void* stream) {
  if (R <= 0) return 0;
  ChunkArgs a{kc, vc, pages, page_base, max_pages, page_size, Hq, Hkv, D, Dv, scale, softcap, r1, r2, chunk, window, x ? *x : AttnExtra()};
  a.defaults();
  if (Hq % Hkv || Hq / Hkv > 16 || (D & 7) || (Dv & 7) || D > 128 || Dv > 128 || Hkv > 65535 || a.x.D2) return 10;
  if (!aligned_to(q, 16) || !aligned_to(kc, 16) || !aligned_to(vc, 16) || ((a.x.ldq | a.x.hsq | a.x.ldk | a.x.ldv) & 7)) return 11;
  cudaStream_t s = (cudaStream_t)stream;
  if (softcap > 0.f) { AB2_BY_SIZE2(launch_decode, 0, true, 0, q, pos, slots, out, R, a, s); }
  AB2_BY_SIZE2(launch_decode, 0, false, 0, q, pos, slots, out, R, a, s);
}

// tiles [nt, 2] = (entry, first row); q / out hold all R rows of the step. bf16; D, Dv multiples of 8 up to 128; a second part up to 64;
// factors of the keys only without a second part, a cap and a distance bias;
// page_size 16, 32 or a multiple of 64. ldk / ldv: elements from one cache row to the next.
int ab2_chunk_prefill(const void* q, const int* cu, const int* start, const int* tiles, int nt, void* out, int R, int cache_rows, long long ldk,
                      long long ldv, const void* kc, const void* vc, const int* pages, const int* page_base, int max_pages, int page_size, int Hq, int Hkv, int D, int Dv,
                      float scale, float softcap, const float* r1, const float* r2, int chunk, int window, const AttnExtra* x, void* stream) {
  if (nt <= 0) return 0;
  ChunkArgs a{kc, vc, pages, page_base, max_pages, page_size, Hq, Hkv, D, Dv, scale, softcap, r1, r2, chunk, window, x ? *x : AttnExtra()};
  a.x.ldk = ldk;
  a.x.ldv = ldv;
  a.defaults();
  const AttnExtra& e = a.x;
  if (Hq % Hkv || (D & 7) || (Dv & 7) || D > 128 || Dv > 128 || Hq > 65535) return 10;
  if (!aligned_to(q, 16) || !aligned_to(kc, 16) || !aligned_to(vc, 16) || !aligned_to(out, 16)) return 11;
  if (!(page_size == 16 || page_size == 32 || (page_size > 0 && page_size % 64 == 0))) return 12;
  if ((e.ldk | e.ldv | e.ldq | e.hsq | e.ldo) & 7) return 13;
  if (e.gate && !e.gate_per_head && (!aligned_to(e.gate, 16) || (e.ldg & 7))) return 14;
  if (e.D2 && ((e.D2 & 7) || e.D2 > 64 || ((e.ldq2 | e.hsq2 | e.ldk2) & 7) || !aligned_to(e.q2, 16) || !aligned_to(e.k2, 16) || softcap > 0.f || r1)) return 15;
  cudaStream_t s = (cudaStream_t)stream;
  if (e.kf && (e.D2 || r1 || softcap > 0.f)) return 16;
  if (e.D2) { AB2_BY_SIZE2(launch_prefill, 64, false, ADJ_NONE, q, cu, start, tiles, nt, out, R, cache_rows, a, s); }
  if (e.kf) { AB2_BY_SIZE2(launch_prefill, 0, false, ADJ_KEY, q, cu, start, tiles, nt, out, R, cache_rows, a, s); }
  if (r1 && softcap > 0.f) { AB2_BY_SIZE2(launch_prefill, 0, true, ADJ_DISTANCE, q, cu, start, tiles, nt, out, R, cache_rows, a, s); }
  if (softcap > 0.f) { AB2_BY_SIZE2(launch_prefill, 0, true, ADJ_NONE, q, cu, start, tiles, nt, out, R, cache_rows, a, s); }
  if (r1) { AB2_BY_SIZE2(launch_prefill, 0, false, ADJ_DISTANCE, q, cu, start, tiles, nt, out, R, cache_rows, a, s); }
  AB2_BY_SIZE2(launch_prefill, 0, false, ADJ_NONE, q, cu, start, tiles, nt, out, R, cache_rows, a, s);
}
}
