// The 32-bit stream of a mixer stack on its way into a sublayer: what the last sublayer gave (a row, two normed branches, or a scaled
// embedding row at the very start) is added, the sum is normed, and the token shift blends every normed row with the one before it:
//   s = s' + add;   h = norm(s) * w;   x = h + (h_prev - h) * share
// A sequence's last h (32-bit) is kept in its slot for the rows of its next step.
//
// With a shift the stream goes from one buffer to another, and a CTA takes a stretch of rows of one entry, the row before them
// normed once more (its inputs are still there: nobody writes over them). The first row of an entry is done by the CTA of
// the entry's last stretch, so that one CTA alone reads the slot and writes it. Every thread keeps its own columns, so rows
// follow one another with one barrier per sum.
#include "mixer_common.cuh"

namespace ab2 {

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
  int H, n_dec, stretch;
  float eps;
};

template <typename T, int V, int SRC, bool SHIFT>
__global__ void __launch_bounds__(512)
stream_norm_kernel(const StreamArgs<T> p) {
  extern __shared__ __align__(16) float sm[];      // the row, [SHIFT: the normed row before it], [SRC_PAIR: the other branch], partial sums
  const int HP = (p.H + 3) & ~3;
  float* cur = sm;
  float* prev = sm + HP;
  float* other = sm + (SHIFT ? 2 : 1) * HP;
  float2* part = reinterpret_cast<float2*>(sm + (1 + (SHIFT ? 1 : 0) + (SRC == SRC_PAIR ? 1 : 0)) * HP);
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5, H = p.H, step = blockDim.x * V;
  int turn = 0;
  auto total = [&](float s, float t) {             // sums over the CTA; two sets of partial sums take turns, so one barrier is enough
    s = warp_sum(s);
    if constexpr (SRC == SRC_PAIR) t = warp_sum(t);
    float2* q = part + (turn & 1) * nw;
    ++turn;
    if (lane == 0) q[warp] = make_float2(s, t);
    __syncthreads();
    float2 r = make_float2(0.f, 0.f);
    for (int i = 0; i < nw; ++i) { r.x += q[i].x; r.y += q[i].y; }
    return r;
  };
  // `write`: the row is this CTA's own; otherwise only its normed form is wanted (in prev)
  auto do_row = [&](int row, bool write) {
    float ra = 0.f, rb = 0.f;
    if constexpr (SRC == SRC_PAIR) {
      float sa = 0.f, sb = 0.f;
      for (int c = tid * V; c < H; c += step) {
        float a[V], b[V];
        ldv<V>(p.a + row * p.lda + c, a);
        ldv<V>(p.b + row * p.ldb + c, b);
#pragma unroll
        for (int e = 0; e < V; ++e) { sa += a[e] * a[e]; sb += b[e] * b[e]; }
        stv<V>(cur + c, a);
        stv<V>(other + c, b);
      }
      const float2 s = total(sa, sb);
      ra = p.scale / sqrtf(s.x / H + p.eps);
      rb = p.scale / sqrtf(s.y / H + p.eps);
    }
    const T* src = nullptr;
    if constexpr (SRC == SRC_ROW) src = p.a + row * p.lda;
    if constexpr (SRC == SRC_EMBED) src = p.table + (size_t)min(max(p.ids[row], 0), p.vocab - 1) * H;
    float ss = 0.f;
    for (int c = tid * V; c < H; c += step) {
      float r[V], v[V];
      if constexpr (SRC == SRC_EMBED) {
        ldv<V>(src + c, r);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] *= p.scale;
      } else {
        ldv<V>(p.resid_in + (size_t)row * H + c, r);
      }
      if constexpr (SRC == SRC_ROW) {
        ldv<V>(src + c, v);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += v[e];
      }
      if constexpr (SRC == SRC_PAIR) {
        float g[V], o[V], k[V];
        ldv<V>(cur + c, v);
        ldv<V>(p.wa + c, g);
        ldv<V>(other + c, o);
        ldv<V>(p.wb + c, k);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += v[e] * ra * g[e] + o[e] * rb * k[e];
      }
      if (p.vec != nullptr) {
        ldv<V>(p.vec + c, v);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] += v[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) ss += r[e] * r[e];
      stv<V>(cur + c, r);
      if (write) stv<V>(p.resid_out + (size_t)row * H + c, r);
    }
    const float rstd = p.mult / sqrtf(total(ss, 0.f).x / H + p.eps);
    for (int c = tid * V; c < H; c += step) {
      float r[V], g[V];
      ldv<V>(cur + c, r);
      ldv<V>(p.w + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) r[e] = r[e] * rstd * g[e];
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
      } else {
        stv<V>(p.x + row * p.ldx + c, r);
      }
    }
  };
  if constexpr (!SHIFT) {
    do_row(blockIdx.x, true);
  } else {
    int e, r0, r1;
    if ((int)blockIdx.x < p.n_dec) {
      e = r0 = blockIdx.x;
      r1 = r0 + 1;
    } else {
      const int per = (64 + p.stretch - 1) / p.stretch, k = blockIdx.x - p.n_dec;
      const int4 b = p.blocks[k / per];
      const int o = k % per * p.stretch;
      if (o >= b.z) return;
      e = b.x;
      r0 = b.y + o;
      r1 = min(r0 + p.stretch, b.y + b.z);
    }
    const int first = p.cu[e], slot = p.state[e];
    const bool at_first = r0 == first, at_last = r1 == p.cu[e + 1];
    float* st = p.S + (size_t)max(slot, 0) * H;
    if (at_last) {
      const bool fresh = slot < 0 || p.start[e] <= 0;
      for (int c = tid * V; c < H; c += step) {
        float v[V];
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = 0.f;
        if (!fresh) ldv<V>(st + c, v);
        stv<V>(prev + c, v);
      }
      if (!at_first) do_row(first, true);
    }
    if (!(at_first && at_last)) do_row(at_first ? first : r0 - 1, false);
    for (int r = at_first && !at_last ? r0 + 1 : r0; r < r1; ++r) do_row(r, true);
    if (at_last && slot >= 0)
      for (int c = tid * V; c < H; c += step) {
        float v[V];
        ldv<V>(prev + c, v);
        stv<V>(st + c, v);
      }
  }
}

template <typename T, int V, int SRC, bool SHIFT>
static int launch_stream(const StreamArgs<T>& p, int grid, cudaStream_t s) {
  constexpr int MAX = 220 * 1024;
  const int th = p.H <= 1024 ? 128 : (p.H <= 4096 ? 256 : 512);
  const size_t smem = ((size_t)(1 + (SHIFT ? 1 : 0) + (SRC == SRC_PAIR ? 1 : 0)) * ((p.H + 3) & ~3) + 4 * (th / 32)) * 4;
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
  if (sizeof(T) == 2 && fits(8)) return launch_stream_size<T, 8>(p, grid, s);
  return fits(4) ? launch_stream_size<T, 4>(p, grid, s) : launch_stream_size<T, 1>(p, grid, s);
}

}  // namespace ab2

extern "C" {
using namespace ab2;

// Sources: table (ids [R], scale), or a [R, H] (lda), or a and b with their weights (times scale), or none of them; vec or null. x [R, H]
// (ldx). share null: no shift, a row each, nothing below is used; else the first n_dec entries have one row each, `blocks` lists the 64-row
// blocks of the others (nb of them, in stretches of `stretch` rows), S [slots, H], and resid_in is not resid_out.
int ab2_stream_norm(const int* ids, const void* table, int vocab, const void* a, long long lda, const void* b, long long ldb, const float* wa,
                    const float* wb, float scale, const float* vec, const float* resid_in, float* resid_out, const float* w, float mult,
                    const float* share, void* x, long long ldx, const int* cu, const int* start, const int* state, const void* blocks, int nb,
                    int n_dec, int stretch, float* S, int R, int H, float eps, int dt, void* stream) {
  if (R <= 0) return 0;
  if (H < 1 || (table ? (ids == nullptr || vocab < 1) : resid_in == nullptr) || (b && (!a || !wa || !wb))) return 10;
  if (share && (!cu || !start || !state || !S || stretch < 1 || stretch > 64 || (nb > 0 && !blocks) || (!table && resid_in == resid_out))) return 13;
  const long long grid = share ? n_dec + (long long)nb * ((64 + stretch - 1) / stretch) : R;
  if (grid <= 0 || grid > 0x7fffffffLL) return 14;
  auto go = [&](auto t) {
    using T = decltype(t);
    const StreamArgs<T> p{ids, (const T*)table, vocab, scale, (const T*)a, (const T*)b, lda, ldb, wa, wb, vec, resid_in, resid_out, w, share, mult,
                          (T*)x, ldx, cu, start, state, (const int4*)blocks, S, H, n_dec, stretch, eps};
    return launch_stream_typed<T>(p, (int)grid, (cudaStream_t)stream);
  };
  return dt == 0 ? go(__nv_bfloat16()) : go(0.f);
}
}
