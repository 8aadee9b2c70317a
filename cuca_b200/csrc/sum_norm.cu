// The residual stream of blocks that norm the sum: x <- N(alpha x + s * y) * w with y a sublayer's output (a weighted sum
// of terms), s a factor per channel and N the RMS norm; the sublayers read x itself. A mixer may read its input mixed with
// the previous token's, h_t = x_t + (x_(t-1) - x_t) * mix, where x_(t-1) of a request's first row of a step is what the
// request's slot keeps (zeros for a new one), and its last row is kept for the next step.
//   sum_norm         x in place, and the new rows in the compute dtype, which the next sublayer reads
//   sum_norm_shift   x out of place, and the new rows mixed with their predecessors
//   shift_rows       the mixing alone
// All arithmetic is 32-bit. Rows that an earlier kernel of the stream wrote are read past L1 (a dependent launch may find it
// holding what was there before).
#include "terms.cuh"
#include <math.h>

namespace {

struct SumNorm {
  const float* x;
  CucaTerms terms;
  const float* s;   // [E] or null: ones
  const float* w;   // [E]
  float alpha, eps;
  int E;
};

template <int V, int AHEAD = 4>
__device__ __forceinline__ Pack<V> summed(const SumNorm& p, size_t row, int i) {
  const Pack<V> x = ld_cg<V>(p.x + row * p.E + i);
  Pack<V> s;
  if (p.s) s = ld<V>(p.s + i);
  Pack<V> z = term_sum<V, AHEAD>(p.terms, row * p.E + i);
  if (p.s) {
#pragma unroll
    for (int k = 0; k < V; ++k) z.v[k] *= s.v[k];
  }
#pragma unroll
  for (int k = 0; k < V; ++k) z.v[k] = fmaf(p.alpha, x.v[k], z.v[k]);
  return z;
}

// sums of N values over the block; `red` holds 32 N floats
template <int N>
__device__ __forceinline__ void block_sums(float (&s)[N], float* red) {
#pragma unroll
  for (int j = 0; j < N; ++j) s[j] = warp_sum(s[j]);
  __syncthreads();  // earlier readers of `red` are done
  if ((threadIdx.x & 31) == 0) {
#pragma unroll
    for (int j = 0; j < N; ++j) red[j * 32 + (threadIdx.x >> 5)] = s[j];
  }
  __syncthreads();
  const int nw = blockDim.x >> 5;
#pragma unroll
  for (int j = 0; j < N; ++j) {
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += red[j * 32 + i];
    s[j] = t;
  }
}

// One block per row. R > 0: a thread holds R packs of V values (blockDim R V >= E); R = 0: the sum stays in x between the
// passes (rows wider than a block can hold). AHEAD: slices asked for at once (many: few rows, whose time is latency; one:
// many rows, whose terms are whole tensors, so that more blocks fit an SM).
template <typename TO, int V, int R, int AHEAD>
__global__ void __launch_bounds__(1024, AHEAD == 1 ? 2 : 1)
sum_norm_kernel(const SumNorm p, float* __restrict__ x, TO* __restrict__ out) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int step = blockDim.x * V;
  constexpr int HELD = R > 0 ? R : 1;
  Pack<V> z[HELD];
  float q[1] = {0.f};
  auto finish = [&](int i, Pack<V> v, const Pack<V> w, float inv) {
#pragma unroll
    for (int k = 0; k < V; ++k) v.v[k] = v.v[k] * inv * w.v[k];
    st<V>(x + row * p.E + i, v);
    if (out) st<V>(out + row * p.E + i, v);
  };
  Pack<V> wv[HELD];  // (asked for before the reduction)
  if (R > 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
      if (i >= p.E) continue;
      wv[r] = ld<V>(p.w + i);
      z[r] = summed<V, AHEAD>(p, row, i);
#pragma unroll
      for (int k = 0; k < V; ++k) q[0] = fmaf(z[r].v[k], z[r].v[k], q[0]);
    }
  } else {
    for (int i = threadIdx.x * V; i < p.E; i += step) {
      const Pack<V> v = summed<V, AHEAD>(p, row, i);
      st<V>(x + row * p.E + i, v);
#pragma unroll
      for (int k = 0; k < V; ++k) q[0] = fmaf(v.v[k], v.v[k], q[0]);
    }
  }
  block_sums<1>(q, red);
  const float inv = 1.f / sqrtf(q[0] / (float)p.E + p.eps);
  if (R > 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
      if (i < p.E) finish(i, z[r], wv[r], inv);
    }
  } else {
    for (int i = threadIdx.x * V; i < p.E; i += step) finish(i, ld<V>(x + row * p.E + i), ld<V>(p.w + i), inv);
  }
}

struct Shift {
  const float* mix;   // [E]
  float* kept;        // [slots, E]
  const int* seq_of_row;
  const int* req_row0;
  const int* req_count;
  int n_rows, n_seqs;
};

// ROWS consecutive rows per block, all held in registers at once together with the row before them (worked out anew when
// it belongs to the same request): one reduction for all. A request's kept row is read by the block that has the request's
// first row of the step and written by the same block after that, be the last row its own or not (then it is worked out
// here once more), so no two blocks touch it.
template <typename TO, int V, int R, int ROWS>
__global__ void __launch_bounds__(1024, 1)
sum_norm_shift_kernel(const SumNorm p, const Shift sh, float* __restrict__ x_out, TO* __restrict__ out) {
  __shared__ float red[32 * (ROWS + 1)];
  __shared__ int s_last;
  pdl_trigger();
  pdl_wait();
  const int r0 = blockIdx.x * ROWS, step = blockDim.x * V;
  if (threadIdx.x == 0) s_last = r0;
  int seq[ROWS + 1];   // of rows r0 - 1 .. r0 + ROWS - 1 (-1: none, or padding)
#pragma unroll
  for (int j = 0; j <= ROWS; ++j) {
    const int row = r0 - 1 + j;
    seq[j] = row >= 0 && row < sh.n_rows ? sh.seq_of_row[row] : -1;
  }
  if (seq[0] != seq[1]) seq[0] = -1;  // the row before belongs to another request
  Pack<V> z[ROWS + 1][R];
  float q[ROWS + 1];
  // one row a block (single tokens, mostly): what the rest of the row needs is asked for before the reduction
  constexpr bool EARLY = ROWS == 1 && R == 1;
  constexpr int AHEAD = EARLY ? 6 : ROWS > 1 ? 1 : 2;
  Pack<V> wv, mixv, keptv;
  const int i0 = threadIdx.x * V;
  if (EARLY && i0 < p.E && seq[1] >= 0) {
    wv = ld<V>(p.w + i0);
    mixv = ld<V>(sh.mix + i0);
    if (seq[0] < 0) keptv = ld_cg<V>(sh.kept + (size_t)seq[1] * p.E + i0);
  }
#pragma unroll
  for (int j = 0; j <= ROWS; ++j) {
    q[j] = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
#pragma unroll
      for (int k = 0; k < V; ++k) z[j][r].v[k] = 0.f;
      if (seq[j] < 0 || i >= p.E) continue;
      z[j][r] = summed<V, AHEAD>(p, r0 - 1 + j, i);
#pragma unroll
      for (int k = 0; k < V; ++k) q[j] = fmaf(z[j][r].v[k], z[j][r].v[k], q[j]);
    }
  }
  block_sums<ROWS + 1>(q, red);
#pragma unroll
  for (int j = 0; j <= ROWS; ++j) {
    const float inv = 1.f / sqrtf(q[j] / (float)p.E + p.eps);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
      if (i >= p.E || seq[j] < 0) continue;
      const Pack<V> w = EARLY ? wv : ld<V>(p.w + i);
#pragma unroll
      for (int k = 0; k < V; ++k) z[j][r].v[k] = z[j][r].v[k] * inv * w.v[k];
    }
  }
  int open = -1;  // the request whose first row is here and whose last row is not
#pragma unroll
  for (int j = 1; j <= ROWS; ++j) {
    const int row = r0 - 1 + j;
    if (row >= sh.n_rows) break;
    const bool first = seq[j] >= 0 && seq[j - 1] != seq[j];
    if (first) open = seq[j];
    const bool last = row + 1 >= sh.n_rows || sh.seq_of_row[row + 1] != seq[j];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
      if (i >= p.E) continue;
      Pack<V> h = z[j][r];
      if (seq[j] >= 0) {
        float* keep = sh.kept + (size_t)seq[j] * p.E + i;
        const Pack<V> before = first ? (EARLY ? keptv : ld_cg<V>(keep)) : z[j - 1][r], mix = EARLY ? mixv : ld<V>(sh.mix + i);
#pragma unroll
        for (int k = 0; k < V; ++k) h.v[k] = fmaf(before.v[k] - h.v[k], mix.v[k], h.v[k]);
        if (last && open == seq[j]) st<V>(keep, z[j][r]);
      }
      st<V>(x_out + (size_t)row * p.E + i, z[j][r]);
      st<V>(out + (size_t)row * p.E + i, h);
    }
    if (last) open = -1;
  }
  if (open < 0) return;  // (the same in every thread)
  for (int i = threadIdx.x; i < sh.n_seqs; i += blockDim.x) {
    const int a = sh.req_row0[i], n = sh.req_count[i];
    if (n > 0 && a >= r0 && a < r0 + ROWS && a + n > r0 + ROWS) s_last = a + n - 1;  // one request spans the block's end
  }
  __syncthreads();
  const int row = min(s_last, sh.n_rows - 1);
  float t[1] = {0.f};
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = threadIdx.x * V + r * step;
    if (i >= p.E) continue;
    z[0][r] = summed<V, AHEAD>(p, row, i);
#pragma unroll
    for (int k = 0; k < V; ++k) t[0] = fmaf(z[0][r].v[k], z[0][r].v[k], t[0]);
  }
  block_sums<1>(t, red);
  const float inv = 1.f / sqrtf(t[0] / (float)p.E + p.eps);
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = threadIdx.x * V + r * step;
    if (i >= p.E) continue;
    const Pack<V> w = ld<V>(p.w + i);
#pragma unroll
    for (int k = 0; k < V; ++k) z[0][r].v[k] = z[0][r].v[k] * inv * w.v[k];
    st<V>(sh.kept + (size_t)open * p.E + i, z[0][r]);
  }
}

// Row b of the step for b < n_rows unless it is its request's first; block n_rows + i has request i's first row and then
// keeps its last.
template <typename TO, int V>
__global__ void __launch_bounds__(256)
shift_rows_kernel(const float* __restrict__ x, const Shift sh, TO* __restrict__ out, const int* __restrict__ slots, int E) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x;
  int row, last = -1, seq;
  if (b < sh.n_rows) {
    row = b;
    seq = sh.seq_of_row[b];
    if (seq >= 0 && (b == 0 || sh.seq_of_row[b - 1] != seq)) return;
    if (seq < 0) {
      for (int i = threadIdx.x * V; i < E; i += blockDim.x * V) st<V>(out + (size_t)row * E + i, Pack<V>{});
      return;
    }
  } else {
    const int q = b - sh.n_rows;
    seq = slots[q];
    row = sh.req_row0[q];
    if (seq < 0 || sh.req_count[q] <= 0) return;
    last = row + sh.req_count[q] - 1;
  }
  for (int i = threadIdx.x * V; i < E; i += blockDim.x * V) {
    Pack<V> h = ld_cg<V>(x + (size_t)row * E + i);
    const Pack<V> before = last < 0 ? ld_cg<V>(x + (size_t)(row - 1) * E + i) : ld_cg<V>(sh.kept + (size_t)seq * E + i);
    const Pack<V> mix = ld<V>(sh.mix + i);
#pragma unroll
    for (int k = 0; k < V; ++k) h.v[k] = fmaf(before.v[k] - h.v[k], mix.v[k], h.v[k]);
    st<V>(out + (size_t)row * E + i, h);
    if (last >= 0) st<V>(sh.kept + (size_t)seq * E + i, ld_cg<V>(x + (size_t)last * E + i));
  }
}

constexpr int FUSED_MAX_PACKS = 4096;  // a block of 1,024 threads with four packs each

// packs a thread holds (1, 2 or 4; 0: too wide) and threads of a block for rows of `packs` packs
void shape_for(int packs, int* threads, int* held) {
  int r = 1;
  while (r < 4 && (packs + r - 1) / r > 1024) r *= 2;
  *held = (packs + r - 1) / r > 1024 ? 0 : r;
  *threads = *held ? ((packs + r - 1) / r + 31) / 32 * 32 : 1024;
}

template <typename TO, int V>
void launch_sum_norm(const SumNorm& p, float* x, TO* out, int n_rows, cudaStream_t stream) {
  int threads, held;
  shape_for(p.E / V, &threads, &held);
  const bool many = n_rows > 512;  // (beyond what leaves K slices)
#define SN(R, AHEAD)                                                                                                    \
  do {                                                                                                                  \
    if (many) cuca_launch(sum_norm_kernel<TO, V, R, 1>, dim3(n_rows), dim3(threads), 0, stream, true, p, x, out);       \
    else cuca_launch(sum_norm_kernel<TO, V, R, AHEAD>, dim3(n_rows), dim3(threads), 0, stream, true, p, x, out);        \
  } while (0)
  if (held == 1) SN(1, 8);
  else if (held == 2) SN(2, 4);
  else if (held == 4) SN(4, 2);
  else SN(0, 4);
#undef SN
}

template <typename TO, int V>
void launch_sum_norm_shift(const SumNorm& p, const Shift& sh, float* x_out, TO* out, cudaStream_t stream) {
  int threads, held;
  shape_for(p.E / V, &threads, &held);
#define SNS(R, ROWS)                                                                                              \
  cuca_launch(sum_norm_shift_kernel<TO, V, R, ROWS>, dim3((sh.n_rows + ROWS - 1) / ROWS), dim3(threads), 0, stream, \
              true, p, sh, x_out, out)
  const bool many = sh.n_rows > 256;  // several rows a block, so that fewer rows are worked out twice
  if (held == 1) { if (many) SNS(1, 4); else SNS(1, 1); }
  else if (held == 2) { if (many) SNS(2, 2); else SNS(2, 1); }
  else SNS(4, 1);
#undef SNS
}

}  // namespace

// x <- N(alpha x + s * y) * w in place, y the weighted sum of the terms; out (or null): the new x in out_dtype.
CUCA_API int cuca_sum_norm(float* x, const CucaTerms* terms, const float* s, const float* w, float alpha, float eps, void* out,
                           int out_dtype, int n_rows, int E, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && terms && terms->n >= 0 && terms->n <= CUCA_MAX_TERMS, "sum_norm: bad sizes (E=%d)", E);
  const SumNorm p{x, *terms, s, w, alpha, eps, E};
  const bool wide = E % 4 == 0 && terms_wide(*terms) && aligned_to(x, 16) && aligned_to(s, 16) && aligned_to(w, 16) && aligned_to(out, 16);
#define SN(TO)                                                                      \
  do {                                                                              \
    if (wide) launch_sum_norm<TO, 4>(p, x, (TO*)out, n_rows, stream);               \
    else launch_sum_norm<TO, 1>(p, x, (TO*)out, n_rows, stream);                    \
  } while (0)
  if (out == nullptr || out_dtype == CUCA_F32) SN(float);
  else if (out_dtype == CUCA_BF16) SN(__nv_bfloat16);
  else CUCA_REQUIRE(false, "sum_norm: unknown dtype %d", out_dtype);
#undef SN
  CUCA_CHECK_LAUNCH("sum_norm");
  return 0;
}

// 1 if cuca_sum_norm_shift takes rows of this width (else: cuca_sum_norm, then cuca_shift_rows).
CUCA_API int cuca_sum_norm_shift_supported(int E) { return E > 0 && (E % 4 == 0 ? E / 4 : E) <= FUSED_MAX_PACKS; }

// The same out of place (x_out must not overlap x), and out[r] = x_out[r] + (x_out[r - 1] - x_out[r]) * mix, where the row
// before a request's first row of the step is kept[slot], which then becomes the request's last row. Padding rows (slot
// < 0) become zeros.
CUCA_API int cuca_sum_norm_shift(const float* x, const CucaTerms* terms, const float* s, const float* w, float alpha, float eps,
                                 float* x_out, const float* mix, float* kept, void* out, int out_dtype,
                                 const int* seq_of_row, const int* req_row0, const int* req_count, int n_rows, int n_seqs,
                                 int E, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(terms && terms->n >= 0 && terms->n <= CUCA_MAX_TERMS && n_seqs > 0, "sum_norm_shift: bad sizes (E=%d)", E);
  const bool wide = E % 4 == 0 && terms_wide(*terms) && aligned_to(x, 16) && aligned_to(s, 16) && aligned_to(w, 16) &&
                    aligned_to(x_out, 16) && aligned_to(mix, 16) && aligned_to(kept, 16) && aligned_to(out, 16);
  CUCA_REQUIRE(E > 0 && (wide ? E / 4 : E) <= FUSED_MAX_PACKS, "sum_norm_shift: rows of %d values are too wide", E);
  const SumNorm p{x, *terms, s, w, alpha, eps, E};
  const Shift sh{mix, kept, seq_of_row, req_row0, req_count, n_rows, n_seqs};
#define SNS(TO)                                                                           \
  do {                                                                                    \
    if (wide) launch_sum_norm_shift<TO, 4>(p, sh, x_out, (TO*)out, stream);               \
    else launch_sum_norm_shift<TO, 1>(p, sh, x_out, (TO*)out, stream);                    \
  } while (0)
  if (out_dtype == CUCA_F32) SNS(float);
  else if (out_dtype == CUCA_BF16) SNS(__nv_bfloat16);
  else CUCA_REQUIRE(false, "sum_norm_shift: unknown dtype %d", out_dtype);
#undef SNS
  CUCA_CHECK_LAUNCH("sum_norm_shift");
  return 0;
}

// out[r] = x[r] + (x[r - 1] - x[r]) * mix with the kept rows as above.
CUCA_API int cuca_shift_rows(const float* x, const float* mix, float* kept, void* out, int out_dtype, const int* seq_of_row,
                             const int* req_row0, const int* req_count, const int* slots, int n_rows, int n_seqs, int E,
                             cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && n_seqs > 0, "shift_rows: bad sizes E=%d requests=%d", E, n_seqs);
  const bool wide = E % 4 == 0 && aligned_to(x, 16) && aligned_to(mix, 16) && aligned_to(kept, 16) && aligned_to(out, 16);
  const Shift sh{mix, kept, seq_of_row, req_row0, req_count, n_rows, n_seqs};
  const dim3 grid(n_rows + n_seqs);
#define SR(TO)                                                                                                            \
  do {                                                                                                                    \
    if (wide) cuca_launch(shift_rows_kernel<TO, 4>, grid, dim3(256), 0, stream, true, x, sh, (TO*)out, slots, E);         \
    else cuca_launch(shift_rows_kernel<TO, 1>, grid, dim3(256), 0, stream, true, x, sh, (TO*)out, slots, E);              \
  } while (0)
  if (out_dtype == CUCA_F32) SR(float);
  else if (out_dtype == CUCA_BF16) SR(__nv_bfloat16);
  else CUCA_REQUIRE(false, "shift_rows: unknown dtype %d", out_dtype);
#undef SR
  CUCA_CHECK_LAUNCH("shift_rows");
  return 0;
}
