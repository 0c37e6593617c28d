// Elementwise, norm, convolution and small-product kernels of mixer stacks (bf16 or fp32 activations, fp32 residual
// stream, norm weights and states): grouped sandwich norms, norms behind a sublayer and residual sums before a norm (both
// fused with the expert sum), whole-projection q / k norms fused with the cache append, causal convolutions with carried
// tails, xIELU, GELU, SiLU gate, clamped gated units, token side gate, expert combine, capped logits, and a plain grouped
// product for 32-bit experts and odd sizes.
#include "mixer_common.cuh"

namespace ab2 {

// ------------------------------------------------------------------ grouped norms
// How a CTA shares `groups` equal parts of a row: with no more groups than warps every group gets wpg warps (its
// elements interleaved over their lanes), otherwise a warp walks several groups. Sums have a fixed order.
struct GroupMap {
  int groups, part, wpg, warp, lane, nw;
  __device__ GroupMap(int groups_, int H) : groups(groups_), part(H / groups_) {
    warp = threadIdx.x >> 5;
    lane = threadIdx.x & 31;
    nw = blockDim.x >> 5;
    wpg = groups <= nw ? nw / groups : 1;
  }
  __device__ int first() const { return groups <= nw ? warp / wpg : warp; }
  __device__ int step() const { return groups <= nw ? groups : nw; }       // one group per warp, or every nw-th
  __device__ int offset() const { return groups <= nw ? (warp % wpg) * 32 + lane : lane; }
  __device__ int stride() const { return wpg * 32; }
  __device__ int sub() const { return groups <= nw ? warp % wpg : 0; }
  __device__ float total(const float* sums, int g) const {
    float s = 0.f;
    for (int i = 0; i < wpg; ++i) s += sums[g * wpg + i];
    return s;
  }
};

// Row by row: v = h (or the fp32 residual taken from an embedding row); with w_post: resid += norm(h) * w_post;
// then x = norm(resid) * w_next. The row stays in shared memory between the passes.
template <typename T, int V>
__global__ void sandwich_norm_kernel(const int* __restrict__ ids, const T* __restrict__ table, int vocab, const T* __restrict__ h,
                                     long long ldh, const float* __restrict__ w_post, float* __restrict__ resid,
                                     const float* __restrict__ w_next, T* __restrict__ x, int H, int groups, float eps) {
  extern __shared__ __align__(16) float srow[];       // [H] values, then the partial sums
  pdl_wait();
  pdl_trigger();
  const GroupMap gm(groups, H);
  float* sums = srow + ((H + 3) & ~3);
  float* sums2 = sums + groups * gm.wpg;
  const int row = blockIdx.x;
  float* rr = resid + (size_t)row * H;
  const int pv = gm.part / V;
  if (h != nullptr) {
    const T* hr = h + (size_t)row * ldh;
    for (int g = gm.first(); g < groups; g += gm.step()) {
      float ss = 0.f;
      for (int i = gm.offset(); i < pv; i += gm.stride()) {
        float v[V];
        ldv<V>(hr + g * gm.part + i * V, v);
        for (int e = 0; e < V; ++e) ss += v[e] * v[e];
        stv<V>(srow + g * gm.part + i * V, v);
      }
      ss = warp_sum(ss);
      if (gm.lane == 0) sums[g * gm.wpg + gm.sub()] = ss;
    }
    __syncthreads();
  }
  int id = 0;
  if (h == nullptr) {
    id = ids[row];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  }
  for (int g = gm.first(); g < groups; g += gm.step()) {
    const float rstd = h != nullptr ? 1.f / sqrtf(gm.total(sums, g) / gm.part + eps) : 0.f;
    float ss = 0.f;
    for (int i = gm.offset(); i < pv; i += gm.stride()) {
      const int c = g * gm.part + i * V;
      float v[V];
      if (h != nullptr) {
        float r[V], w[V];
        ldv<V>(srow + c, v);
        ldv<V>(rr + c, r);
        ldv<V>(w_post + c, w);
        for (int e = 0; e < V; ++e) v[e] = r[e] + v[e] * rstd * w[e];
      } else {
        ldv<V>(table + (size_t)id * H + c, v);
      }
      stv<V>(rr + c, v);
      stv<V>(srow + c, v);
      for (int e = 0; e < V; ++e) ss += v[e] * v[e];
    }
    ss = warp_sum(ss);
    if (gm.lane == 0) sums2[g * gm.wpg + gm.sub()] = ss;
  }
  __syncthreads();
  for (int g = gm.first(); g < groups; g += gm.step()) {
    const float rstd = 1.f / sqrtf(gm.total(sums2, g) / gm.part + eps);
    for (int i = gm.offset(); i < pv; i += gm.stride()) {
      const int c = g * gm.part + i * V;
      float v[V], w[V];
      ldv<V>(srow + c, v);
      ldv<V>(w_next + c, w);
      for (int e = 0; e < V; ++e) v[e] = v[e] * rstd * w[e];
      stv<V>(x + (size_t)row * H + c, v);
    }
  }
}

// out = norm(y * silu(z)) * w in groups; y fp32.
template <typename T, int V>
__global__ void gated_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long long ldz, const float* __restrict__ w,
                                  T* __restrict__ out, int C, int groups, float eps) {
  extern __shared__ __align__(16) float srow[];
  pdl_wait();
  pdl_trigger();
  const GroupMap gm(groups, C);
  float* sums = srow + ((C + 3) & ~3);
  const int row = blockIdx.x;
  const int pv = gm.part / V;
  for (int g = gm.first(); g < groups; g += gm.step()) {
    float ss = 0.f;
    for (int i = gm.offset(); i < pv; i += gm.stride()) {
      const int c = g * gm.part + i * V;
      float a[V], b[V];
      ldv<V>(y + (size_t)row * C + c, a);
      ldv<V>(z + (size_t)row * ldz + c, b);
      for (int e = 0; e < V; ++e) {
        a[e] *= silu_t<sizeof(T) == 2>(b[e]);
        ss += a[e] * a[e];
      }
      stv<V>(srow + c, a);
    }
    ss = warp_sum(ss);
    if (gm.lane == 0) sums[g * gm.wpg + gm.sub()] = ss;
  }
  __syncthreads();
  for (int g = gm.first(); g < groups; g += gm.step()) {
    const float rstd = 1.f / sqrtf(gm.total(sums, g) / gm.part + eps);
    for (int i = gm.offset(); i < pv; i += gm.stride()) {
      const int c = g * gm.part + i * V;
      float a[V], b[V];
      ldv<V>(srow + c, a);
      ldv<V>(w + c, b);
      for (int e = 0; e < V; ++e) a[e] = a[e] * rstd * b[e];
      stv<V>(out + (size_t)row * C + c, a);
    }
  }
}

// ------------------------------------------------------------------ norms behind a sublayer
// h = base row + the sum of the token's k expert rows (either may be missing); resid += mult * norm(h) * (off + w);
// x = resid, or norm(resid) * (off_next + w_next) when there is a next norm. One CTA per row, the row in shared memory.
template <typename T, int V, bool EXPERTS>
__global__ void post_norm_kernel(const T* __restrict__ base, long long ldb, const T* __restrict__ y, const int* __restrict__ inv, int k, int n_rows,
                                 const float* __restrict__ w, float off, float mult, float* __restrict__ resid, const float* __restrict__ w_next,
                                 float off_next, T* __restrict__ x, int H, float eps) {
  extern __shared__ __align__(16) float srow[];       // [H] values, then two rows of partial sums
  pdl_wait();
  pdl_trigger();
  float* sums = srow + ((H + 3) & ~3);
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  auto total = [&](const float* part) {
    float s = 0.f;
    for (int i = 0; i < nw; ++i) s += part[i];
    return s;
  };
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float h[V];
    if (base != nullptr) ldv<V>(base + (size_t)row * ldb + c, h);
    else
      for (int e = 0; e < V; ++e) h[e] = 0.f;
    for (int s0 = 0; EXPERTS && s0 < k; s0 += 4) {     // four rows on their way at a time
      float v[4][V];
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const int r = s0 + s < k ? inv[(size_t)row * k + s0 + s] : -1;
        if (r >= 0 && r < n_rows) ldv<V>(y + (size_t)r * H + c, v[s]);
        else
          for (int e = 0; e < V; ++e) v[s][e] = 0.f;
      }
#pragma unroll
      for (int s = 0; s < 4; ++s)
        for (int e = 0; e < V; ++e) h[e] += v[s][e];
    }
    for (int e = 0; e < V; ++e) ss += h[e] * h[e];
    stv<V>(srow + c, h);
  }
  ss = warp_sum(ss);
  if (lane == 0) sums[warp] = ss;
  __syncthreads();
  const float rstd = mult / sqrtf(total(sums) / H + eps);
  float* rr = resid + (size_t)row * H;
  ss = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float h[V], r[V], g[V];
    ldv<V>(srow + c, h);
    ldv<V>(rr + c, r);
    ldv<V>(w + c, g);
    for (int e = 0; e < V; ++e) r[e] += h[e] * rstd * (off + g[e]);
    stv<V>(rr + c, r);
    if (w_next == nullptr) {
      stv<V>(x + (size_t)row * H + c, r);
    } else {
      stv<V>(srow + c, r);
      for (int e = 0; e < V; ++e) ss += r[e] * r[e];
    }
  }
  if (w_next == nullptr) return;
  ss = warp_sum(ss);
  if (lane == 0) sums[nw + warp] = ss;
  __syncthreads();
  const float rn = 1.f / sqrtf(total(sums + nw) / H + eps);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float r[V], g[V];
    ldv<V>(srow + c, r);
    ldv<V>(w_next + c, g);
    for (int e = 0; e < V; ++e) r[e] = r[e] * rn * (off_next + g[e]);
    stv<V>(x + (size_t)row * H + c, r);
  }
}

// ------------------------------------------------------------------ residual sum, then the next norm
// h = base row (times sigmoid(logit), if there is one) + the token's k expert rows times their weights + vec, each optional;
// resid += h; x = norm(resid) * w_next * mult, or resid when there is no norm. One CTA per row, the row in shared memory.
template <typename T, int V, bool EXPERTS>
__global__ void residual_norm_kernel(const T* __restrict__ base, long long ldb, const float* __restrict__ logit, long long ldl, const T* __restrict__ y,
                                     const int* __restrict__ inv, const float* __restrict__ topw, int k, int n_rows, const float* __restrict__ vec,
                                     float* __restrict__ resid, const float* __restrict__ w_next, float mult, T* __restrict__ x, long long ldx, int H,
                                     float eps) {
  extern __shared__ __align__(16) float srow[];       // [H] values, then the partial sums
  pdl_wait();
  pdl_trigger();
  float* sums = srow + ((H + 3) & ~3);
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const float f = logit != nullptr ? sigmoid_t<false>(logit[row * ldl]) : 1.f;
  float* rr = resid + (size_t)row * H;
  T* xr = x + row * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float r[V];
    ldv<V>(rr + c, r);
    if (base != nullptr) {
      float b[V];
      ldv<V>(base + row * ldb + c, b);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] += f * b[e];
    }
    if (vec != nullptr) {
      float b[V];
      ldv<V>(vec + c, b);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] += b[e];
    }
    for (int s0 = 0; EXPERTS && s0 < k; s0 += 4) {     // four rows on their way at a time
      float v[4][V], w[4];
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const int i = s0 + s < k ? inv[(size_t)row * k + s0 + s] : -1;
        w[s] = 0.f;
        if (i >= 0 && i < n_rows) {
          w[s] = topw[(size_t)row * k + s0 + s];
          ldv<V>(y + (size_t)i * H + c, v[s]);
        } else {
          for (int e = 0; e < V; ++e) v[s][e] = 0.f;
        }
      }
#pragma unroll
      for (int s = 0; s < 4; ++s)
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += w[s] * v[s][e];
    }
    stv<V>(rr + c, r);
    if (w_next == nullptr) {
      stv<V>(xr + c, r);
    } else {
      stv<V>(srow + c, r);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += r[e] * r[e];
    }
  }
  if (w_next == nullptr) return;
  ss = warp_sum(ss);
  if (lane == 0) sums[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < nw; ++i) ss += sums[i];
  const float rstd = mult / sqrtf(ss / H + eps);
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float r[V], g[V];
    ldv<V>(srow + c, r);
    ldv<V>(w_next + c, g);
#pragma unroll
    for (int e = 0; e < V; ++e) r[e] = r[e] * rstd * g[e];
    stv<V>(xr + c, r);
  }
}

// resid = table[ids] (+ pos_table[pos]) in fp32, x the same in T (and once more at x2, if that is given).
template <typename T, int V>
__global__ void embed_rows_kernel(const int* __restrict__ ids, const T* __restrict__ table, int vocab, const int* __restrict__ pos,
                                  const T* __restrict__ pos_table, int n_pos, float* __restrict__ resid, T* __restrict__ x, T* __restrict__ x2,
                                  long long ldx, long long total, int H) {
  pdl_wait();
  pdl_trigger();
  const int hv = H / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / hv;
    const int c = (int)(i - r * hv) * V;
    const int id = min(max(ids[r], 0), vocab - 1);
    float v[V];
    ldv<V>(table + (size_t)id * H + c, v);
    if (pos_table != nullptr) {
      float p[V];
      ldv<V>(pos_table + (size_t)min(max(pos[r], 0), n_pos - 1) * H + c, p);
      for (int e = 0; e < V; ++e) v[e] += p[e];
    }
    stv<V>(resid + r * H + c, v);
    stv<V>(x + r * ldx + c, v);
    if (x2 != nullptr) stv<V>(x2 + r * ldx + c, v);
  }
}

static inline int norm_threads(int H) { return H <= 1024 ? 128 : (H <= 4096 ? 256 : 512); }
static inline size_t norm_smem(int H, int groups, int threads) {
  const int nw = threads / 32;
  const int per = groups <= nw ? groups * (nw / groups) : groups;
  return (size_t)(((H + 3) & ~3) + 2 * per) * 4;
}

// ------------------------------------------------------------------ q / k norm + cache append
template <typename T, int V>
__global__ void qk_norm_append_kernel(const T* __restrict__ qkv, long long ld, const float* __restrict__ wq, const float* __restrict__ wk,
                                      const int* __restrict__ slots, T* __restrict__ q, T* __restrict__ kc, T* __restrict__ vc, int nq, int nk,
                                      int nv, float eps) {
  __shared__ float red[2][32];
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  const T* src = qkv + (size_t)row * ld;
  float sq = 0.f, sk = 0.f;
  for (int i = tid * V; i < nq + nk; i += blockDim.x * V) {
    float v[V];
    ldv<V>(src + i, v);
    float s = 0.f;
    for (int e = 0; e < V; ++e) s += v[e] * v[e];
    if (i < nq) sq += s; else sk += s;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < nw; ++w) { sq += red[0][w]; sk += red[1][w]; }
  const float rq = 1.f / sqrtf(sq / nq + eps), rk = 1.f / sqrtf(sk / nk + eps);
  const int slot = slots[row];
  for (int i = tid * V; i < nq + nk + nv; i += blockDim.x * V) {
    float v[V], w[V];
    ldv<V>(src + i, v);
    if (i < nq) {
      ldv<V>(wq + i, w);
      for (int e = 0; e < V; ++e) v[e] = v[e] * rq * w[e];
      stv<V>(q + (size_t)row * nq + i, v);
    } else if (slot >= 0) {
      if (i < nq + nk) {
        ldv<V>(wk + i - nq, w);
        for (int e = 0; e < V; ++e) v[e] = v[e] * rk * w[e];
        stv<V>(kc + (size_t)slot * nk + i - nq, v);
      } else {
        stv<V>(vc + (size_t)slot * nv + i - nq - nk, v);
      }
    }
  }
}

// ------------------------------------------------------------------ causal convolution
// Single-token rows: the window is the slot's tail plus the row; the tail moves on by one.
template <typename T>
__global__ void conv_decode_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ bin, const float* __restrict__ w,
                                   const float* __restrict__ bias, int silu, const int* __restrict__ start, const int* __restrict__ state,
                                   float* __restrict__ tail, T* __restrict__ out, int C, int K) {
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int slot = state[row];
  if (slot < 0) { stf(out + (size_t)row * C + c, 0.f); return; }
  const bool fresh = start[row] <= 0;
  float* tl = tail + ((size_t)slot * C + c) * (K - 1);
  const float cur = ldf(x + (size_t)row * ld + c) + (bin ? bin[c] : 0.f);
  float acc = bias[c] + w[(size_t)c * K + K - 1] * cur;
  for (int m = 0; m < K - 1; ++m) acc += w[(size_t)c * K + m] * (fresh ? 0.f : tl[m]);
  for (int m = 0; m + 1 < K - 1; ++m) tl[m] = fresh ? 0.f : tl[m + 1];
  if (K > 1) tl[K - 2] = cur;
  stf(out + (size_t)row * C + c, silu ? silu_t<sizeof(T) == 2>(acc) : acc);
}

// Portions: a CTA walks the rows of one block (64 rows of one entry), every thread V neighbouring channels with their
// last inputs in registers. KT = taps (1..4), 0: any number, inputs re-read.
template <typename T, int KT, int V>
__global__ void __launch_bounds__(128)
conv_prefill_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ bin, const float* __restrict__ w, const float* __restrict__ bias,
                    int silu, const int* __restrict__ cu, const int* __restrict__ start, const int* __restrict__ state,
                    const int4* __restrict__ blocks, const float* __restrict__ tail, T* __restrict__ out, int C, int Kdyn) {
  const int K = KT > 0 ? KT : Kdyn;
  const int4 blk = blocks[blockIdx.y];
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int e = blk.x, r0 = blk.y, n = blk.z, first = cu[e];
  const int slot = state[e];
  const bool fresh = start[e] <= 0;
  float bi[V], b0[V];
  for (int v = 0; v < V; ++v) {
    bi[v] = bin ? bin[c + v] : 0.f;
    b0[v] = bias[c + v];
  }
  const float* tl = tail + ((size_t)slot * C + c) * (K - 1);
  auto at = [&](int r, float (&o)[V]) {                 // inputs at row r of this entry (before its first row: the tail)
    if (r >= first) {
      ldv<V>(x + (size_t)r * ld + c, o);
      for (int v = 0; v < V; ++v) o[v] += bi[v];
    } else {
      const int m = K - 1 + (r - first);
      for (int v = 0; v < V; ++v) o[v] = (fresh || m < 0) ? 0.f : tl[v * (K - 1) + m];
    }
  };
  if constexpr (KT > 0) {
    float wv[KT][V], win[KT][V];
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
      for (int v = 0; v < V; ++v) wv[j][v] = w[(size_t)(c + v) * KT + j];
#pragma unroll
    for (int j = 0; j < KT - 1; ++j) at(r0 - (KT - 1) + j, win[j + 1]);
    float nxt[V];
    ldv<V>(x + (size_t)r0 * ld + c, nxt);
    for (int i = 0; i < n; ++i) {
#pragma unroll
      for (int j = 0; j < KT - 1; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) win[j][v] = win[j + 1][v];
#pragma unroll
      for (int v = 0; v < V; ++v) win[KT - 1][v] = nxt[v] + bi[v];
      if (i + 1 < n) ldv<V>(x + (size_t)(r0 + i + 1) * ld + c, nxt);
      float acc[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        acc[v] = b0[v];
#pragma unroll
        for (int j = 0; j < KT; ++j) acc[v] += wv[j][v] * win[j][v];
        if (silu) acc[v] = silu_t<sizeof(T) == 2>(acc[v]);
      }
      stv<V>(out + (size_t)(r0 + i) * C + c, acc);
    }
  } else {
    for (int i = 0; i < n; ++i) {
      float acc[V], o[V];
      for (int v = 0; v < V; ++v) acc[v] = b0[v];
      for (int j = 0; j < K; ++j) {
        at(r0 + i - (K - 1) + j, o);
        for (int v = 0; v < V; ++v) acc[v] += w[(size_t)(c + v) * K + j] * o[v];
      }
      for (int v = 0; v < V; ++v)
        if (silu) acc[v] = silu_t<sizeof(T) == 2>(acc[v]);
      stv<V>(out + (size_t)(r0 + i) * C + c, acc);
    }
  }
}

// After the convolution: the last K - 1 inputs of every portion become its slot's tail.
template <typename T>
__global__ void conv_tail_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ bin, const int* __restrict__ cu,
                                 const int* __restrict__ start, const int* __restrict__ state, int n_dec, float* __restrict__ tail, int C, int K) {
  const int e = n_dec + blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int slot = state[e];
  if (slot < 0) return;
  const int r0 = cu[e], L = cu[e + 1] - r0;
  const bool fresh = start[e] <= 0;
  float* tl = tail + ((size_t)slot * C + c) * (K - 1);
  for (int m = 0; m < K - 1; ++m) {                     // ascending: a slot entry is read before it is overwritten
    const int r = L - (K - 1) + m;
    tl[m] = r >= 0 ? ldf(x + (size_t)(r0 + r) * ld + c) + (bin ? bin[c] : 0.f) : (fresh ? 0.f : tl[m + L]);
  }
}

// ------------------------------------------------------------------ activations, combine, cap
template <typename T, int V>
__global__ void xielu_kernel(const T* __restrict__ x, long long ld, const float* __restrict__ pq, T* __restrict__ out, long long total, int C) {
  pdl_wait();
  pdl_trigger();
  const float sp = softplusf(pq[0]), sq = 0.5f + softplusf(pq[1]);
  const int cv = C / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cv;
    const int c = (int)(i - r * cv) * V;
    float v[V];
    ldv<V>(x + r * ld + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float n = fminf(v[e], 0.f), q = v[e] > 0.f ? sp * v[e] * v[e] : sq * (expm1_neg<sizeof(T) == 2>(n) - n);
      v[e] = 0.5f * v[e] + q;
    }
    stv<V>(out + r * C + c, v);
  }
}

template <typename T, int V>
__global__ void glu_silu_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, long long total, int I) {
  pdl_wait();
  pdl_trigger();
  const int cv = I / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cv;
    const int c = (int)(i - r * cv) * V;
    float g[V], u[V];
    ldv<V>(gu + r * ld + c, g);
    ldv<V>(gu + r * ld + I + c, u);
    for (int e = 0; e < V; ++e) g[e] = silu_t<sizeof(T) == 2>(g[e]) * u[e];
    stv<V>(out + r * I + c, g);
  }
}

template <typename T, int V>
__global__ void gelu_erf_kernel(const T* __restrict__ x, long long ld, T* __restrict__ out, long long total, int C) {
  pdl_wait();
  pdl_trigger();
  const int cv = C / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cv;
    const int c = (int)(i - r * cv) * V;
    float v[V];
    ldv<V>(x + r * ld + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = 0.5f * v[e] * (1.f + erff(v[e] * 0.7071067811865476f));
    stv<V>(out + r * C + c, v);
  }
}

// Clamped gated units: rows g | u, both first multiplied by the row's weight when there are weights (topw by entry, order:
// the entry of a row).
template <typename T, int V>
__global__ void glu_clamped_kernel(const T* __restrict__ gu, long long ld, const int* __restrict__ order, const float* __restrict__ topw,
                                   T* __restrict__ out, long long total, int I, float limit, float alpha) {
  pdl_wait();
  pdl_trigger();
  const int cv = I / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cv;
    const int c = (int)(i - r * cv) * V;
    float w = 1.f;
    if (topw != nullptr) {
      const int n = order[r];
      w = n >= 0 && n < total / cv ? topw[n] : 0.f;
    }
    float g[V], u[V];
    ldv<V>(gu + r * ld + c, g);
    ldv<V>(gu + r * ld + I + c, u);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float a = fminf(w * g[e], limit), b = fminf(fmaxf(w * u[e], -limit), limit);
      g[e] = a * sigmoid_t<sizeof(T) == 2>(alpha * a) * (b + 1.f);
    }
    stv<V>(out + r * I + c, g);
  }
}

// out = gelu_tanh(g) * table[ids, col:col + D]
template <typename T, int V>
__global__ void side_gate_kernel(const T* __restrict__ g, long long ld, const int* __restrict__ ids, const T* __restrict__ table, int vocab,
                                 long long ldt, int col, T* __restrict__ out, long long total, int D) {
  pdl_wait();
  pdl_trigger();
  const int dv = D / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / dv;
    const int c = (int)(i - r * dv) * V;
    const int id = min(max(ids[r], 0), vocab - 1);
    float v[V], t[V];
    ldv<V>(g + r * ld + c, v);
    ldv<V>(table + id * ldt + col + c, t);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = gelu_tanh_t<sizeof(T) == 2>(v[e]) * t[e];
    stv<V>(out + r * D + c, v);
  }
}

template <typename T, int V>
__global__ void expert_combine_kernel(const T* __restrict__ y, const int* __restrict__ inv, const float* __restrict__ topw, T* __restrict__ out,
                                      long long total, int k, int H, int n_rows) {
  pdl_wait();
  pdl_trigger();
  const int hv = H / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / hv;
    const int c = (int)(i - t * hv) * V;
    float acc[V];
    for (int e = 0; e < V; ++e) acc[e] = 0.f;
    for (int s = 0; s < k; ++s) {
      const int r = inv[t * k + s];
      if (r < 0 || r >= n_rows) continue;
      const float w = topw[t * k + s];
      float v[V];
      ldv<V>(y + (size_t)r * H + c, v);
      for (int e = 0; e < V; ++e) acc[e] += w * v[e];
    }
    stv<V>(out + t * H + c, acc);
  }
}

__global__ void softcap_kernel(float* __restrict__ z, long long ld, int R, int C, float cap, float inv_cap) {
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.y;
  for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < C; c += gridDim.x * blockDim.x) {
    float* p = z + (size_t)r * ld + c;
    *p = cap * tanhf(*p * inv_cap);
  }
}

// ------------------------------------------------------------------ plain grouped product
// 128 x 64 output tile per CTA, fp32 FMA; rows of `tiles` are (expert, first row, valid rows, -).
template <typename T>
__global__ void __launch_bounds__(256)
grouped_plain_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ out, const int4* __restrict__ tiles,
                     const int* __restrict__ n_tiles, int N, int K) {
  if ((int)blockIdx.x >= *n_tiles) return;
  __shared__ float sa[16][132], sb[16][68];
  const int4 t = tiles[blockIdx.x];
  const int n0 = blockIdx.y * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* we = w + (size_t)t.x * N * K;
  float acc[8][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 128 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      sa[k][r] = (r < t.z && k0 + k < K) ? ldf(x + (size_t)(t.y + r) * K + k0 + k) : 0.f;
    }
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int n = i >> 4, k = i & 15;
      sb[k][n] = (n0 + n < N && k0 + k < K) ? ldf(we + (size_t)(n0 + n) * K + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[8], b[4];
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = sa[k][ty * 8 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = sb[k][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
  for (int i = 0; i < 8; ++i)
    for (int j = 0; j < 4; ++j)
      if (ty * 8 + i < t.z && n0 + tx * 4 + j < N) stf(out + (size_t)(t.y + ty * 8 + i) * N + n0 + tx * 4 + j, acc[i][j]);
}

static inline int flat_grid(long long n) {
  const long long g = (n + 255) / 256;
  return (int)(g < 148 * 16 ? g : 148 * 16);
}

}  // namespace ab2

// T = __nv_bfloat16 (dt 0) or float (dt 1); V = 4 when every row start and length allows it.
#define AB2_TYPED(dt, vec, ...)                                                                              \
  do {                                                                                                       \
    if ((dt) == 0) {                                                                                         \
      using T = __nv_bfloat16;                                                                               \
      if (vec) { constexpr int V = 4; __VA_ARGS__; } else { constexpr int V = 1; __VA_ARGS__; }                 \
    } else {                                                                                                 \
      using T = float;                                                                                       \
      if (vec) { constexpr int V = 4; __VA_ARGS__; } else { constexpr int V = 1; __VA_ARGS__; }                 \
    }                                                                                                        \
  } while (0)
// as AB2_TYPED with a third width: V = 8 when `vec8`
#define AB2_TYPED8(dt, vec8, vec, ...)                                                                       \
  do {                                                                                                       \
    if ((dt) == 0 && (vec8)) { using T = __nv_bfloat16; constexpr int V = 8; __VA_ARGS__; }                  \
    else AB2_TYPED(dt, vec, __VA_ARGS__);                                                                    \
  } while (0)
#define AB2_DONE return cudaGetLastError() == cudaSuccess ? 0 : 1

extern "C" {
using namespace ab2;

// resid [R, H] fp32, x [R, H]. With h: resid += norm(h) * w_post first; without: resid = table[ids].
int ab2_sandwich_norm(const int* ids, const void* table, int vocab, const void* h, long long ldh, const float* w_post, float* resid,
                      const float* w_next, void* x, int R, int H, int groups, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  if (groups < 1 || H % groups) return 10;
  const int th = norm_threads(H);
  const size_t smem = norm_smem(H, groups, th);
  if (smem > 200 * 1024) return 11;
  const int eb = dt == 0 ? 2 : 4;
  const bool vec = (H / groups) % 4 == 0 && ldh % 4 == 0 && aligned_to(h ? h : table, 4 * eb) && aligned_to(x, 4 * eb);
  AB2_TYPED(dt, vec, {
    auto kern = sandwich_norm_kernel<T, V>;
    static ab2host::DevState st;
    if (ab2host::prepare_launch(kern, 200 * 1024, st, nullptr)) return 12;
    launch_pdl(kern, dim3(R), dim3(th), smem, (cudaStream_t)stream, ids, (const T*)table, vocab, (const T*)h, ldh, w_post, resid, w_next, (T*)x, H,
               groups, eps);
  });
  AB2_DONE;
}

// x and resid [R, H]; base [R, H] (ldb) and / or y [n_rows, H] with inv [R, k]. w_next may be null.
int ab2_post_norm(const void* base, long long ldb, const void* y, const int* inv, int k, int n_rows, const float* w, float off, float mult,
                  float* resid, const float* w_next, float off_next, void* x, int R, int H, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  if (H < 1 || (base == nullptr && y == nullptr)) return 10;
  const int th = norm_threads(H);
  const size_t smem = (size_t)(((H + 3) & ~3) + 2 * (th / 32)) * 4;
  if (smem > 200 * 1024) return 11;
  const int eb = dt == 0 ? 2 : 4;
  if (y == nullptr) k = 0;
  auto fits = [&](int v) {
    return H % v == 0 && ldb % v == 0 && aligned_to(base, v * eb) && aligned_to(y, v * eb) && aligned_to(x, v * eb) && aligned_to(resid, 16) &&
           aligned_to(w, 16) && aligned_to(w_next, 16);
  };
  AB2_TYPED8(dt, fits(8), fits(4), {
    auto kern = k > 0 ? post_norm_kernel<T, V, true> : post_norm_kernel<T, V, false>;
    static ab2host::DevState st[2];
    if (ab2host::prepare_launch(kern, 200 * 1024, st[k > 0], nullptr)) return 12;
    launch_pdl(kern, dim3(R), dim3(th), smem, (cudaStream_t)stream, (const T*)base, ldb, (const T*)y, inv, k, n_rows, w, off, mult, resid, w_next,
               off_next, (T*)x, H, eps);
  });
  AB2_DONE;
}

// resid [R, H], x and x2 (or null) [R, H] with ldx elements from row to row; base [R, H] (ldb) with logit [R] (ldl), y [n_rows, H] with inv
// and topw [R, k], vec [H]: each may be null, like w_next.
int ab2_residual_norm(const void* base, long long ldb, const float* logit, long long ldl, const void* y, const int* inv, const float* topw, int k,
                      int n_rows, const float* vec, float* resid, const float* w_next, float mult, void* x, long long ldx, int R, int H, float eps, int dt,
                      void* stream) {
  if (R <= 0) return 0;
  if (H < 1 || (y != nullptr && (inv == nullptr || topw == nullptr))) return 10;
  const int th = norm_threads(H);
  const size_t smem = (size_t)(((H + 3) & ~3) + th / 32) * 4;
  if (smem > 200 * 1024) return 11;
  const int eb = dt == 0 ? 2 : 4;
  if (y == nullptr) k = 0;
  auto fits = [&](int v) {
    return H % v == 0 && ldb % v == 0 && ldx % v == 0 && aligned_to(base, v * eb) && aligned_to(y, v * eb) && aligned_to(x, v * eb) &&
           aligned_to(resid, 16) && aligned_to(vec, 16) && aligned_to(w_next, 16);
  };
  AB2_TYPED8(dt, fits(8), fits(4), {
    auto kern = k > 0 ? residual_norm_kernel<T, V, true> : residual_norm_kernel<T, V, false>;
    static ab2host::DevState st[2];
    if (ab2host::prepare_launch(kern, 200 * 1024, st[k > 0], nullptr)) return 12;
    launch_pdl(kern, dim3(R), dim3(th), smem, (cudaStream_t)stream, (const T*)base, ldb, logit, ldl, (const T*)y, inv, topw, k, n_rows, vec, resid,
               w_next, mult, (T*)x, ldx, H, eps);
  });
  AB2_DONE;
}

int ab2_embed_rows(const int* ids, const void* table, int vocab, const int* pos, const void* pos_table, int n_pos, float* resid, void* x, void* x2,
                   long long ldx, int R, int H, int dt, void* stream) {
  if (R <= 0) return 0;
  if (vocab < 1 || (pos_table != nullptr && n_pos < 1)) return 10;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) {
    return H % v == 0 && ldx % v == 0 && aligned_to(table, v * eb) && aligned_to(pos_table, v * eb) && aligned_to(x, v * eb) &&
           aligned_to(x2, v * eb) && aligned_to(resid, 16);
  };
  AB2_TYPED8(dt, fits(8), fits(4), {
    const long long n = (long long)R * (H / V);
    launch_pdl(embed_rows_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, ids, (const T*)table, vocab, pos, (const T*)pos_table,
               n_pos, resid, (T*)x, (T*)x2, ldx, n, H);
  });
  AB2_DONE;
}

int ab2_gated_group_norm(const float* y, const void* z, long long ldz, const float* w, void* out, int R, int C, int groups, float eps, int dt,
                         void* stream) {
  if (R <= 0) return 0;
  if (groups < 1 || C % groups) return 10;
  const int th = norm_threads(C);
  const size_t smem = norm_smem(C, groups, th);
  if (smem > 200 * 1024) return 11;
  const int eb = dt == 0 ? 2 : 4;
  const bool vec = (C / groups) % 4 == 0 && ldz % 4 == 0 && aligned_to(z, 4 * eb);
  AB2_TYPED(dt, vec, {
    auto kern = gated_norm_kernel<T, V>;
    static ab2host::DevState st;
    if (ab2host::prepare_launch(kern, 200 * 1024, st, nullptr)) return 12;
    launch_pdl(kern, dim3(R), dim3(th), smem, (cudaStream_t)stream, y, (const T*)z, ldz, w, (T*)out, C, groups, eps);
  });
  AB2_DONE;
}

int ab2_qk_norm_append(const void* qkv, long long ld, const float* wq, const float* wk, const int* slots, void* q, void* kc, void* vc, int R,
                       int nq, int nk, int nv, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  const int eb = dt == 0 ? 2 : 4;
  const bool vec = nq % 4 == 0 && nk % 4 == 0 && nv % 4 == 0 && ld % 4 == 0 && aligned_to(qkv, 4 * eb);
  AB2_TYPED8(dt, nq % 8 == 0 && nk % 8 == 0 && nv % 8 == 0 && ld % 8 == 0 && aligned_to(qkv, 16), vec, {
    launch_pdl(qk_norm_append_kernel<T, V>, dim3(R), dim3(256), 0, (cudaStream_t)stream, (const T*)qkv, ld, wq, wk, slots, (T*)q, (T*)kc, (T*)vc, nq,
               nk, nv, eps);
  });
  AB2_DONE;
}

// Rows of the first n_dec entries are single tokens; `blocks` lists the 64-row blocks of the other entries.
int ab2_causal_conv(const void* x, long long ld, const float* bin, const float* w, const float* bias, int silu, const int* cu, const int* start,
                    const int* state, const void* blocks, int nb, int n_dec, int n_entries, float* tail, void* out, int C, int K, int dt,
                    void* stream) {
  if (C <= 0 || K < 1) return 10;
  cudaStream_t s = (cudaStream_t)stream;
  const int gx = (C + 127) / 128;
  if (n_dec > 0) {
    if (n_dec > 65535) return 11;
    if (dt == 0)
      launch_pdl(conv_decode_kernel<__nv_bfloat16>, dim3(gx, n_dec), dim3(128), 0, s, (const __nv_bfloat16*)x, ld, bin, w, bias, silu, start, state,
                 tail, (__nv_bfloat16*)out, C, K);
    else
      launch_pdl(conv_decode_kernel<float>, dim3(gx, n_dec), dim3(128), 0, s, (const float*)x, ld, bin, w, bias, silu, start, state, tail,
                 (float*)out, C, K);
  }
  if (nb > 0) {
    if (nb > 65535 || n_entries - n_dec > 65535) return 11;
    const bool vec = C % 4 == 0 && ld % 4 == 0 && aligned_to(x, dt == 0 ? 8 : 16);
#define AB2_CONV(KK)                                                                                                                       \
  AB2_TYPED(dt, vec, conv_prefill_kernel<T, KK, V><<<dim3((C / V + 127) / 128, nb), 128, 0, s>>>((const T*)x, ld, bin, w, bias, silu, cu, start, \
                                                                                                 state, (const int4*)blocks, tail, (T*)out, C, K))
    switch (K) {
      case 1: AB2_CONV(1); break;
      case 2: AB2_CONV(2); break;
      case 3: AB2_CONV(3); break;
      case 4: AB2_CONV(4); break;
      default: AB2_CONV(0);
    }
#undef AB2_CONV
    if (K > 1) {
      if (dt == 0)
        conv_tail_kernel<__nv_bfloat16><<<dim3(gx, n_entries - n_dec), 128, 0, s>>>((const __nv_bfloat16*)x, ld, bin, cu, start, state, n_dec, tail, C, K);
      else
        conv_tail_kernel<float><<<dim3(gx, n_entries - n_dec), 128, 0, s>>>((const float*)x, ld, bin, cu, start, state, n_dec, tail, C, K);
    }
  }
  AB2_DONE;
}

int ab2_xielu(const void* x, long long ld, const float* pq, void* out, int R, int C, int dt, void* stream) {
  if (R <= 0) return 0;
  const int eb = dt == 0 ? 2 : 4;
  const bool vec = C % 4 == 0 && ld % 4 == 0 && aligned_to(x, 4 * eb);
  AB2_TYPED8(dt, C % 8 == 0 && ld % 8 == 0 && aligned_to(x, 16), vec, {
    const long long n = (long long)R * (C / V);
    launch_pdl(xielu_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)x, ld, pq, (T*)out, n, C);
  });
  AB2_DONE;
}

int ab2_glu_silu(const void* gu, long long ld, void* out, int R, int I, int dt, void* stream) {
  if (R <= 0) return 0;
  const int eb = dt == 0 ? 2 : 4;
  const bool vec = I % 4 == 0 && ld % 4 == 0 && aligned_to(gu, 4 * eb);
  AB2_TYPED8(dt, I % 8 == 0 && ld % 8 == 0 && aligned_to(gu, 16), vec, {
    const long long n = (long long)R * (I / V);
    launch_pdl(glu_silu_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)gu, ld, (T*)out, n, I);
  });
  AB2_DONE;
}

int ab2_gelu_erf(const void* x, long long ld, void* out, int R, int C, int dt, void* stream) {
  if (R <= 0) return 0;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) { return C % v == 0 && ld % v == 0 && aligned_to(x, v * eb) && aligned_to(out, v * eb); };
  AB2_TYPED8(dt, fits(8), fits(4), {
    const long long n = (long long)R * (C / V);
    launch_pdl(gelu_erf_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)x, ld, (T*)out, n, C);
  });
  AB2_DONE;
}

// order [R] and topw [R] together or not at all
int ab2_glu_clamped(const void* gu, long long ld, const int* order, const float* topw, void* out, int R, int I, float limit, float alpha, int dt,
                    void* stream) {
  if (R <= 0) return 0;
  if ((order == nullptr) != (topw == nullptr)) return 10;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) { return I % v == 0 && ld % v == 0 && aligned_to(gu, v * eb) && aligned_to(out, v * eb); };
  AB2_TYPED8(dt, fits(8), fits(4), {
    const long long n = (long long)R * (I / V);
    launch_pdl(glu_clamped_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)gu, ld, order, topw, (T*)out, n, I, limit,
               alpha);
  });
  AB2_DONE;
}

int ab2_side_gate(const void* g, long long ld, const int* ids, const void* table, int vocab, long long ldt, int col, void* out, int R, int D, int dt,
                  void* stream) {
  if (R <= 0) return 0;
  if (vocab < 1 || col < 0 || col + D > ldt) return 10;
  const int eb = dt == 0 ? 2 : 4;
  auto fits = [&](int v) { return D % v == 0 && ld % v == 0 && ldt % v == 0 && col % v == 0 && aligned_to(g, v * eb) && aligned_to(table, v * eb); };
  AB2_TYPED8(dt, fits(8), fits(4), {
    const long long n = (long long)R * (D / V);
    launch_pdl(side_gate_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)g, ld, ids, (const T*)table, vocab, ldt, col,
               (T*)out, n, D);
  });
  AB2_DONE;
}

int ab2_expert_combine(const void* y, const int* inv, const float* topw, void* out, int T_, int k, int H, int dt, void* stream) {
  if (T_ <= 0) return 0;
  AB2_TYPED8(dt, H % 8 == 0, H % 4 == 0, {
    const long long n = (long long)T_ * (H / V);
    launch_pdl(expert_combine_kernel<T, V>, dim3(flat_grid(n)), dim3(256), 0, (cudaStream_t)stream, (const T*)y, inv, topw, (T*)out, n, k, H, T_ * k);
  });
  AB2_DONE;
}

int ab2_softcap(float* z, long long ld, int R, int C, float cap, void* stream) {
  if (R <= 0) return 0;
  if (R > 65535 || cap <= 0.f) return 10;
  const int gx = (C + 1023) / 1024;
  launch_pdl(softcap_kernel, dim3(gx < 64 ? gx : 64, R), dim3(256), 0, (cudaStream_t)stream, z, ld, R, C, cap, 1.f / cap);
  AB2_DONE;
}

int ab2_grouped_plain(const void* x, const void* w, void* out, const void* tiles, const int* n_tiles, int max_tiles, int N, int K, int dt,
                      void* stream) {
  if (max_tiles <= 0) return 0;
  if ((N + 63) / 64 > 65535) return 10;
  const dim3 grid(max_tiles, (N + 63) / 64);
  if (dt == 0)
    grouped_plain_kernel<__nv_bfloat16><<<grid, 256, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)x, (const __nv_bfloat16*)w, (__nv_bfloat16*)out,
                                                                                (const int4*)tiles, n_tiles, N, K);
  else
    grouped_plain_kernel<float><<<grid, 256, 0, (cudaStream_t)stream>>>((const float*)x, (const float*)w, (float*)out, (const int4*)tiles, n_tiles, N, K);
  AB2_DONE;
}
}
