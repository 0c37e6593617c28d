// The 32-bit stream of a mixer stack on its way into a sublayer: what the last sublayer gave (a row, two normed branches, or a scaled
// embedding row at the very start) is added, the sum is normed, and the token shift blends every normed row with the one before it:
//   s = s' + add;   h = norm(s) * w;   x = h + (h_prev - h) * share
// A sequence's last h (32-bit) is kept in its slot for the rows of its next step.
//
// With a shift the stream goes from one buffer to another, and a CTA takes a stretch of rows of one entry, the row before them
// normed once more (its inputs are still there: nobody writes over them). The first row of an entry is done by the CTA of
// the entry's last stretch, so that one CTA alone reads the slot and writes it. Every thread keeps its own columns of every row.
//
//   stream_norm_rows_kernel   rows whose width a CTA holds in registers, several rows per round: one trip to memory and one barrier
//                             per sum for all of them
//   stream_norm_kernel        any width: row by row, in shared memory
#include "mixer_common.cuh"

namespace ab2 {

// V elements as they are
template <int V, typename T>
__device__ __forceinline__ void copy_regs(T (&o)[V], const T* src) {
  if constexpr (V * sizeof(T) == 16) *reinterpret_cast<uint4*>(o) = *reinterpret_cast<const uint4*>(src);
  else if constexpr (V * sizeof(T) == 8) *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(src);
  else
    for (int v = 0; v < V; ++v) o[v] = src[v];
}

enum StreamSource { SRC_NONE = 0, SRC_ROW = 1, SRC_PAIR = 2, SRC_EMBED = 3 };

template <typename T>
struct StreamArgs {
  const int* ids;                         // SRC_EMBED: scale * table[ids]
  const T* table;
  int vocab;
  float scale;
  const T *a, *b;                         // SRC_ROW: a; SRC_PAIR: scale * (norm(a) * wa + norm(b) * wb)
  long long lda, ldb;
  const float *wa, *wb;
  const float* vec;                       // [H] added to every row, or null
  const float* resid_in;
  float* resid_out;                       // without a shift it may be resid_in
  const float *w, *share;
  float mult;                             // of the normed row (before the shift)
  T* x;
  long long ldx;
  const int *cu, *start, *state;
  const int4* blocks;
  float* S;                               // [slots, H] last normed row of every sequence
  int R, H, n_dec, stretch;
  float eps;
};

// The rows of a CTA: its own, r0 .. r1 - 1, and in front of them (with a shift) the entry's first row, if this is its last stretch,
// and the row before r0, of which only the normed form is wanted. r1 < r0: nothing to do.
struct Stretch {
  int r0, r1, first = 0, lead = 0, slot = -1;
  bool at_last = false, fresh = true;

  template <typename T>
  __device__ static Stretch plain(const StreamArgs<T>& p) {
    Stretch s;
    s.r0 = blockIdx.x * p.stretch;
    s.r1 = min(s.r0 + p.stretch, p.R);
    return s;
  }
  template <typename T>
  __device__ static Stretch shifted(const StreamArgs<T>& p) {
    Stretch s;
    int e;
    if ((int)blockIdx.x < p.n_dec) {
      e = s.r0 = blockIdx.x;
      s.r1 = s.r0 + 1;
    } else {
      const int per = (64 + p.stretch - 1) / p.stretch, k = blockIdx.x - p.n_dec;
      const int4 b = p.blocks[k / per];
      const int o = k % per * p.stretch;
      e = b.x;
      s.r0 = b.y + o;
      s.r1 = min(s.r0 + p.stretch, b.y + b.z);
      if (o >= b.z) {
        s.r1 = s.r0 - 1;
        return s;
      }
    }
    s.first = p.cu[e];
    s.slot = p.state[e];
    s.at_last = s.r1 == p.cu[e + 1];
    s.fresh = s.slot < 0 || p.start[e] <= 0;
    const bool at_first = s.r0 == s.first;
    s.lead = (s.at_last && !at_first) + !(at_first && s.at_last);
    if (at_first && !s.at_last) ++s.r0;
    return s;
  }
  __device__ __forceinline__ int count() const { return lead + r1 - r0; }
  __device__ __forceinline__ int row(int i) const { return i >= lead ? r0 + i - lead : (i == lead - 1 ? r0 - 1 : first); }
  __device__ __forceinline__ bool own(int i) const { return i >= lead || (lead == 2 && i == 0); }
};

template <typename T, int SRC>
__device__ __forceinline__ const T* source_row(const StreamArgs<T>& p, int row) {
  if constexpr (SRC == SRC_EMBED) return p.table + (size_t)min(max(p.ids[row], 0), p.vocab - 1) * p.H;
  return p.a + row * p.lda;
}

// Sums over the CTA (up to 16 warps) of N numbers; `part` holds two sets of [N][16], which take turns, so one barrier is enough.
template <int N>
__device__ __forceinline__ void totals(float (&s)[N], float* part, int& turn) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  float* q = part + turn * N * 16;
  turn ^= 1;
#pragma unroll
  for (int j = 0; j < N; ++j) {
    s[j] = warp_sum(s[j]);
    if (lane == 0) q[j * 16 + warp] = s[j];
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < N; ++j) s[j] = warp_sum(lane < nw ? q[j * 16 + lane] : 0.f);
}

// ------------------------------------------------------------------ rows in registers
// A thread has K pieces of V columns, a round NR rows.
template <typename T, int V, int K, int NR, int SRC, bool SHIFT>
__global__ void __launch_bounds__(512, sizeof(T) == 2 && K == 1 ? 2 : 1)
stream_norm_rows_kernel(const StreamArgs<T> p) {
  constexpr bool PAIR = SRC == SRC_PAIR;
  __shared__ float part[2 * NR * 16], part2[PAIR ? 4 * NR * 16 : 1];
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, H = p.H;
  Stretch st;
  if constexpr (SHIFT) st = Stretch::shifted(p);
  else st = Stretch::plain(p);
  if (st.r1 < st.r0) return;
  const int n = st.count();
  int turn = 0, turn2 = 0;
  auto col = [&](int k) { return (tid + k * (int)blockDim.x) * V; };
  float prev[SHIFT ? K : 1][V];
  if constexpr (SHIFT)
    if (st.at_last) {
#pragma unroll
      for (int k = 0; k < K; ++k) {
#pragma unroll
        for (int v = 0; v < V; ++v) prev[k][v] = 0.f;
        if (!st.fresh && col(k) < H) ldv<V>(p.S + (size_t)st.slot * H + col(k), prev[k]);
      }
    }
  for (int i0 = 0; i0 < n; i0 += NR) {                // rows behind the last one count as zeros
    float cur[NR][K][V];
    if constexpr (PAIR) {
      T a[NR][K][V], b[NR][K][V];
      float sums[2 * NR];
#pragma unroll
      for (int j = 0; j < NR; ++j)
#pragma unroll
        for (int k = 0; k < K; ++k) {
          const bool in = i0 + j < n && col(k) < H;
          if (in) {
            const int row = st.row(i0 + j), c = col(k);
            copy_regs<V>(a[j][k], p.a + row * p.lda + c);
            copy_regs<V>(b[j][k], p.b + row * p.ldb + c);
            ldv<V>(p.resid_in + (size_t)row * H + c, cur[j][k]);
          } else {
#pragma unroll
            for (int v = 0; v < V; ++v) {
              a[j][k][v] = b[j][k][v] = T(0.f);
              cur[j][k][v] = 0.f;
            }
          }
        }
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        sums[2 * j] = sums[2 * j + 1] = 0.f;
#pragma unroll
        for (int k = 0; k < K; ++k)
#pragma unroll
          for (int v = 0; v < V; ++v) {
            const float x = (float)a[j][k][v], y = (float)b[j][k][v];
            sums[2 * j] += x * x;
            sums[2 * j + 1] += y * y;
          }
      }
      totals<2 * NR>(sums, part2, turn2);
#pragma unroll
      for (int k = 0; k < K; ++k) {
        if (col(k) >= H) break;
        float wa[V], wb[V];
        ldv<V>(p.wa + col(k), wa);
        ldv<V>(p.wb + col(k), wb);
#pragma unroll
        for (int j = 0; j < NR; ++j) {
          const float ra = p.scale / sqrtf(sums[2 * j] / H + p.eps), rb = p.scale / sqrtf(sums[2 * j + 1] / H + p.eps);
#pragma unroll
          for (int v = 0; v < V; ++v) cur[j][k][v] += (float)a[j][k][v] * ra * wa[v] + (float)b[j][k][v] * rb * wb[v];
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const bool on = i0 + j < n;
        const int row = on ? st.row(i0 + j) : 0;
        const T* src = SRC == SRC_NONE || !on ? nullptr : source_row<T, SRC>(p, row);
#pragma unroll
        for (int k = 0; k < K; ++k) {
          float r[V], a[V];
#pragma unroll
          for (int v = 0; v < V; ++v) r[v] = a[v] = 0.f;
          if (on && col(k) < H) {
            if constexpr (SRC != SRC_EMBED) ldv<V>(p.resid_in + (size_t)row * H + col(k), r);
            if constexpr (SRC != SRC_NONE) ldv<V>(src + col(k), a);
          }
#pragma unroll
          for (int v = 0; v < V; ++v) cur[j][k][v] = SRC == SRC_EMBED ? a[v] * p.scale : r[v] + a[v];
        }
      }
    }
    if (p.vec != nullptr)
#pragma unroll
      for (int k = 0; k < K; ++k) {
        if (col(k) >= H) break;
        float x[V];
        ldv<V>(p.vec + col(k), x);
#pragma unroll
        for (int j = 0; j < NR; ++j)
#pragma unroll
          for (int v = 0; v < V; ++v) cur[j][k][v] += x[v];
      }
    float ss[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      ss[j] = 0.f;
#pragma unroll
      for (int k = 0; k < K; ++k) {
#pragma unroll
        for (int v = 0; v < V; ++v) ss[j] += cur[j][k][v] * cur[j][k][v];
        if (i0 + j < n && st.own(i0 + j) && col(k) < H) stv<V>(p.resid_out + (size_t)st.row(i0 + j) * H + col(k), cur[j][k]);
      }
    }
    totals<NR>(ss, part, turn);
#pragma unroll
    for (int j = 0; j < NR; ++j) ss[j] = p.mult / sqrtf(ss[j] / H + p.eps);
#pragma unroll
    for (int k = 0; k < K; ++k) {
      if (col(k) >= H) break;
      const int c = col(k);
      float w[V], m[V];
      ldv<V>(p.w + c, w);
      if constexpr (SHIFT) ldv<V>(p.share + c, m);
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        if (i0 + j >= n) break;
        const int row = st.row(i0 + j);
#pragma unroll
        for (int v = 0; v < V; ++v) cur[j][k][v] *= ss[j] * w[v];
        if constexpr (SHIFT) {
          if (st.own(i0 + j)) {
            float x[V];
#pragma unroll
            for (int v = 0; v < V; ++v) x[v] = cur[j][k][v] + (prev[k][v] - cur[j][k][v]) * m[v];
            stv<V>(p.x + row * p.ldx + c, x);
          }
#pragma unroll
          for (int v = 0; v < V; ++v) prev[k][v] = cur[j][k][v];
        } else {
          stv<V>(p.x + row * p.ldx + c, cur[j][k]);
        }
      }
    }
  }
  if constexpr (SHIFT)
    if (st.at_last && st.slot >= 0)
#pragma unroll
      for (int k = 0; k < K; ++k)
        if (col(k) < H) stv<V>(p.S + (size_t)st.slot * H + col(k), prev[k]);
}

// ------------------------------------------------------------------ any width
// Shared memory: the row, [SHIFT: the normed row before], [SRC_PAIR: the other branch].
template <typename T, int V, int SRC, bool SHIFT>
__global__ void __launch_bounds__(512)
stream_norm_kernel(const StreamArgs<T> p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float part[2 * 16], part2[2 * 2 * 16];
  const int H = p.H, HP = (H + 3) & ~3, step = blockDim.x * V, c0 = threadIdx.x * V;
  float* cur = sm;
  float* prev = sm + HP;
  float* other = sm + (SHIFT ? 2 : 1) * HP;
  pdl_wait();
  pdl_trigger();
  Stretch st;
  if constexpr (SHIFT) st = Stretch::shifted(p);
  else st = Stretch::plain(p);
  if (st.r1 < st.r0) return;
  const int n = st.count();
  int turn = 0, turn2 = 0;
  if constexpr (SHIFT)
    if (st.at_last)
      for (int c = c0; c < H; c += step) {
        float v[V];
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = 0.f;
        if (!st.fresh) ldv<V>(p.S + (size_t)st.slot * H + c, v);
        stv<V>(prev + c, v);
      }
  for (int i = 0; i < n; ++i) {
    const int row = st.row(i);
    const bool write = st.own(i);
    float rs[2] = {0.f, 0.f};
    if constexpr (SRC == SRC_PAIR) {
      for (int c = c0; c < H; c += step) {
        float a[V], b[V];
        ldv<V>(p.a + row * p.lda + c, a);
        ldv<V>(p.b + row * p.ldb + c, b);
#pragma unroll
        for (int e = 0; e < V; ++e) { rs[0] += a[e] * a[e]; rs[1] += b[e] * b[e]; }
        stv<V>(cur + c, a);
        stv<V>(other + c, b);
      }
      totals<2>(rs, part2, turn2);
      rs[0] = p.scale / sqrtf(rs[0] / H + p.eps);
      rs[1] = p.scale / sqrtf(rs[1] / H + p.eps);
    }
    const T* src = SRC == SRC_ROW || SRC == SRC_EMBED ? source_row<T, SRC>(p, row) : nullptr;
    float ss[1] = {0.f};
    for (int c = c0; c < H; c += step) {
      float r[V], v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] = 0.f;
      if constexpr (SRC != SRC_EMBED) ldv<V>(p.resid_in + (size_t)row * H + c, r);
      if constexpr (SRC == SRC_ROW || SRC == SRC_EMBED) {
        ldv<V>(src + c, v);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += SRC == SRC_EMBED ? v[e] * p.scale : v[e];
      }
      if constexpr (SRC == SRC_PAIR) {
        float g[V], o[V], k[V];
        ldv<V>(cur + c, v);
        ldv<V>(p.wa + c, g);
        ldv<V>(other + c, o);
        ldv<V>(p.wb + c, k);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += v[e] * rs[0] * g[e] + o[e] * rs[1] * k[e];
      }
      if (p.vec != nullptr) {
        ldv<V>(p.vec + c, v);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += v[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) ss[0] += r[e] * r[e];
      stv<V>(cur + c, r);
      if (write) stv<V>(p.resid_out + (size_t)row * H + c, r);
    }
    totals<1>(ss, part, turn);
    const float rstd = p.mult / sqrtf(ss[0] / H + p.eps);
    for (int c = c0; c < H; c += step) {
      float r[V], g[V];
      ldv<V>(cur + c, r);
      ldv<V>(p.w + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] *= rstd * g[e];
      if constexpr (SHIFT) {
        if (write) {
          float q[V], m[V];
          ldv<V>(prev + c, q);
          ldv<V>(p.share + c, m);
#pragma unroll
          for (int e = 0; e < V; ++e) q[e] = r[e] + (q[e] - r[e]) * m[e];
          stv<V>(p.x + row * p.ldx + c, q);
        }
        stv<V>(prev + c, r);
        if (st.at_last && st.slot >= 0 && i == n - 1) stv<V>(p.S + (size_t)st.slot * H + c, r);
      } else {
        stv<V>(p.x + row * p.ldx + c, r);
      }
    }
  }
}

template <typename T, int V, int SRC, bool SHIFT>
static int launch_stream(const StreamArgs<T>& p, int grid, cudaStream_t s) {
  if constexpr (V > 1) {
    constexpr int ONE = SRC == SRC_PAIR ? 2 : 4, TWO = SRC == SRC_PAIR ? 1 : 2;      // rows of a round
    const int pieces = (p.H + V - 1) / V;
    if (pieces <= 1024) {
      if (pieces <= 512) launch_pdl(stream_norm_rows_kernel<T, V, 1, ONE, SRC, SHIFT>, dim3(grid), dim3((pieces + 31) / 32 * 32), 0, s, p);
      else launch_pdl(stream_norm_rows_kernel<T, V, 2, TWO, SRC, SHIFT>, dim3(grid), dim3((pieces + 63) / 64 * 32), 0, s, p);
      return cudaGetLastError() == cudaSuccess ? 0 : 1;
    }
  }
  constexpr int MAX = 200 * 1024;
  const int th = p.H <= 1024 ? 128 : (p.H <= 4096 ? 256 : 512);
  const size_t smem = (size_t)(1 + (SHIFT ? 1 : 0) + (SRC == SRC_PAIR ? 1 : 0)) * ((p.H + 3) & ~3) * 4;
  if (smem > MAX) return 11;
  auto kern = stream_norm_kernel<T, V, SRC, SHIFT>;
  static ab2host::DevState st;
  if (ab2host::prepare_launch(kern, MAX, st, nullptr)) return 12;
  launch_pdl(kern, dim3(grid), dim3(th), smem, s, p);
  return cudaGetLastError() == cudaSuccess ? 0 : 1;
}

template <typename T, int V, int SRC>
static int launch_stream_source(const StreamArgs<T>& p, int grid, cudaStream_t s) {
  return p.share ? launch_stream<T, V, SRC, true>(p, grid, s) : launch_stream<T, V, SRC, false>(p, grid, s);
}

template <typename T, int V>
static int launch_stream_size(const StreamArgs<T>& p, int grid, cudaStream_t s) {
  if (p.table) return launch_stream_source<T, V, SRC_EMBED>(p, grid, s);
  if (p.b) return launch_stream_source<T, V, SRC_PAIR>(p, grid, s);
  if (p.a) return launch_stream_source<T, V, SRC_ROW>(p, grid, s);
  return launch_stream_source<T, V, SRC_NONE>(p, grid, s);
}

template <typename T>
static int launch_stream_typed(const StreamArgs<T>& p, int grid, cudaStream_t s) {
  auto fits = [&](int v) {
    const int eb = v * (int)sizeof(T);
    return p.H % v == 0 && p.lda % v == 0 && p.ldb % v == 0 && p.ldx % v == 0 && aligned_to(p.table, eb) && aligned_to(p.a, eb) && aligned_to(p.b, eb) &&
           aligned_to(p.x, eb) && aligned_to(p.wa, 16) && aligned_to(p.wb, 16) && aligned_to(p.vec, 16) && aligned_to(p.resid_in, 16) &&
           aligned_to(p.resid_out, 16) && aligned_to(p.w, 16) && aligned_to(p.share, 16) && aligned_to(p.S, 16);
  };
  if constexpr (sizeof(T) == 2)
    if (fits(8)) return launch_stream_size<T, 8>(p, grid, s);
  return fits(4) ? launch_stream_size<T, 4>(p, grid, s) : launch_stream_size<T, 1>(p, grid, s);
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Sources: table (ids [R], scale), or a [R, H] (lda), or a and b with their weights (times scale), or none of them; vec or null. x [R, H]
// (ldx). stretch: rows that a CTA walks (up to 64). share null: no shift, nothing below is used; else the first n_dec entries have one row
// each, `blocks` lists the 64-row blocks of the others (nb of them), S [slots, H], and resid_in is not resid_out.
int ab2_stream_norm(const int* ids, const void* table, int vocab, const void* a, long long lda, const void* b, long long ldb, const float* wa,
                    const float* wb, float scale, const float* vec, const float* resid_in, float* resid_out, const float* w, float mult,
                    const float* share, void* x, long long ldx, const int* cu, const int* start, const int* state, const void* blocks, int nb,
                    int n_dec, int stretch, float* S, int R, int H, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  if (H < 1 || (table ? (ids == nullptr || vocab < 1) : resid_in == nullptr) || (b && (!a || !wa || !wb))) return 10;
  if (stretch < 1 || stretch > 64) return 15;
  if (share && (!cu || !start || !state || !S || (nb > 0 && !blocks) || (!table && resid_in == resid_out))) return 13;
  const long long grid = share ? n_dec + (long long)nb * ((64 + stretch - 1) / stretch) : (R + stretch - 1) / stretch;
  if (grid <= 0 || grid > 0x7fffffffLL) return 14;
  auto go = [&](auto t) {
    using T = decltype(t);
    const StreamArgs<T> p{ids, (const T*)table, vocab, scale, (const T*)a, (const T*)b, lda, ldb, wa, wb, vec, resid_in, resid_out, w, share, mult,
                          (T*)x, ldx, cu, start, state, (const int4*)blocks, S, R, H, n_dec, stretch, eps};
    return launch_stream_typed<T>(p, (int)grid, (cudaStream_t)stream);
  };
  return dt == 0 ? go(__nv_bfloat16()) : go(0.f);
}
}
