// What becomes of a sublayer's output before it reaches the residual stream. An output arrives as up to eight terms,
// each a 32-bit tensor [rows, E] or the unadded K slices of a contraction over few tokens, with a factor of its own:
//   y = sum_i scale_i * (sum of term i's slices)
//   norm_add        x += N(y) * w, and in the same pass the new x rounded to the compute dtype, which is what the next
//                   sublayer reads where the norm stands on the outputs only; N is the layer norm
//                   (y - mean) / sqrt(mean((y - mean)^2) + eps), or without the mean the RMS norm
//   layer_norm      out = N(x[rows]) * w
//   add_terms       x (+)= y
//   round_rows      out = x in the compute dtype
//   row_norm_gate   out = o / rms(o) * w * sigmoid(gate), over whole rows
// All arithmetic is 32-bit. Terms and slices are added in their order; a row's reduction order depends on the width
// and on how many values a thread holds, which follows the number of rows.
#include "terms.cuh"
#include <math.h>

namespace {

__device__ __forceinline__ float block_sum(float s, float* red) {
  s = warp_sum(s);
  __syncthreads();  // earlier readers of `red` are done
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = s;
  __syncthreads();
  float tot = 0.f;
  const int nw = blockDim.x >> 5;
  for (int i = 0; i < nw; ++i) tot += red[i];
  return tot;
}

// One block per row. R > 0: a thread holds R packs of V values from the first pass to the last (blockDim R V >= E);
// R = 0: the values are worked out anew in every pass (rows wider than a block can hold).
// ADD: y is the terms' sum; x += N(y) w and, with out, out = the new x. Else y is row rows[r] of x and out = N(y) w.
template <typename TO, bool ADD, int V, int R>
__global__ void __launch_bounds__(1024)
norm_kernel(float* __restrict__ x, const CucaTerms terms, const float* __restrict__ w, TO* __restrict__ out,
            const int* __restrict__ rows, int E, float eps, int center) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int irow = rows ? rows[blockIdx.x] : (int)blockIdx.x;
  if (irow < 0) return;
  const size_t at = (size_t)irow * E;
  auto value = [&](int i) { return ADD ? term_sum<V>(terms, at + i) : ld<V>(x + at + i); };
  constexpr int HELD = R > 0 ? R : 1;
  Pack<V> y[HELD];
  const int step = blockDim.x * V;
  float mean = 0.f;
  if (R > 0) {
    float s = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
#pragma unroll
      for (int k = 0; k < V; ++k) y[r].v[k] = 0.f;
      if (i < E) y[r] = value(i);
#pragma unroll
      for (int k = 0; k < V; ++k) s += y[r].v[k];
    }
    if (center) mean = block_sum(s, red) / (float)E;
    float q = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (threadIdx.x * V + r * step < E) {
#pragma unroll
        for (int k = 0; k < V; ++k) { const float d = y[r].v[k] - mean; q = fmaf(d, d, q); }
      }
    }
    const float inv = 1.f / sqrtf(block_sum(q, red) / (float)E + eps);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x * V + r * step;
      if (i >= E) break;
      const Pack<V> wv = ld<V>(w + i);
      Pack<V> o;
#pragma unroll
      for (int k = 0; k < V; ++k) o.v[k] = (y[r].v[k] - mean) * inv * wv.v[k];
      if (ADD) {
        const Pack<V> xv = ld<V>(x + at + i);
#pragma unroll
        for (int k = 0; k < V; ++k) o.v[k] += xv.v[k];
        st<V>(x + at + i, o);
        if (out) st<V>(out + at + i, o);
      } else {
        st<V>(out + (size_t)blockIdx.x * E + i, o);
      }
    }
    return;
  }
  if (center) {
    float s = 0.f;
    for (int i = threadIdx.x * V; i < E; i += step) {
      const Pack<V> v = value(i);
#pragma unroll
      for (int k = 0; k < V; ++k) s += v.v[k];
    }
    mean = block_sum(s, red) / (float)E;
  }
  float q = 0.f;
  for (int i = threadIdx.x * V; i < E; i += step) {
    const Pack<V> v = value(i);
#pragma unroll
    for (int k = 0; k < V; ++k) { const float d = v.v[k] - mean; q = fmaf(d, d, q); }
  }
  const float inv = 1.f / sqrtf(block_sum(q, red) / (float)E + eps);
  for (int i = threadIdx.x * V; i < E; i += step) {
    Pack<V> o = value(i);
    const Pack<V> wv = ld<V>(w + i);
#pragma unroll
    for (int k = 0; k < V; ++k) o.v[k] = (o.v[k] - mean) * inv * wv.v[k];
    if (ADD) {
      const Pack<V> xv = ld<V>(x + at + i);
#pragma unroll
      for (int k = 0; k < V; ++k) o.v[k] += xv.v[k];
      st<V>(x + at + i, o);
      if (out) st<V>(out + at + i, o);
    } else {
      st<V>(out + (size_t)blockIdx.x * E + i, o);
    }
  }
}

template <int V>
__global__ void __launch_bounds__(256)
add_terms_kernel(float* __restrict__ x, const CucaTerms terms, int store, size_t n) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V) {
    Pack<V> y = term_sum<V>(terms, i);
    if (!store) {
      const Pack<V> xv = ld<V>(x + i);
#pragma unroll
      for (int k = 0; k < V; ++k) y.v[k] += xv.v[k];
    }
    st<V>(x + i, y);
  }
}

template <typename TO, int V>
__global__ void __launch_bounds__(256)
round_rows_kernel(const float* __restrict__ x, TO* __restrict__ out, size_t n) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V)
    st<V>(out + i, ld<V>(x + i));
}

template <int V> __device__ __forceinline__ Pack<V> ld_as_f32(const float* p) { return ld<V>(p); }
template <int V> __device__ __forceinline__ Pack<V> ld_as_f32(const __nv_bfloat16* p) {
  Pack<V> r;
  if (V == 4) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
    r.v[0] = a.x;
    if (V > 1) r.v[V > 1 ? 1 : 0] = a.y;
    if (V > 2) r.v[V > 2 ? 2 : 0] = b.x;
    if (V > 3) r.v[V > 3 ? 3 : 0] = b.y;
  } else {
    r.v[0] = __bfloat162float(p[0]);
  }
  return r;
}

// o: [rows, n] 32-bit; gate: rows of stride ldg. One block per row.
template <typename TG, typename TO, int V>
__global__ void __launch_bounds__(512)
row_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const TG* __restrict__ gate, int ldg,
                     TO* __restrict__ out, int n, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  const float* orow = o + row * n;
  const TG* grow = gate + row * ldg;
  TO* dst = out + row * n;
  float q = 0.f;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    const Pack<V> v = ld<V>(orow + i);
#pragma unroll
    for (int k = 0; k < V; ++k) q = fmaf(v.v[k], v.v[k], q);
  }
  const float inv = 1.f / sqrtf(block_sum(q, red) / (float)n + eps);
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    Pack<V> v = ld<V>(orow + i);
    const Pack<V> g = ld_as_f32<V>(grow + i), wv = ld<V>(w + i);
#pragma unroll
    for (int k = 0; k < V; ++k) v.v[k] = v.v[k] * inv * wv.v[k] / (1.f + expf(-g.v[k]));
    st<V>(dst + i, v);
  }
}

// threads and held packs for rows of `packs` packs: few rows get as many threads as a row has packs, many rows a
// quarter of that with four packs each
void norm_shape(int packs, int n_rows, int* threads, int* held) {
  int r = n_rows >= 512 && packs > 1024 ? 2 : 1;
  while (r < 8 && (packs + r - 1) / r > 1024) r *= 2;
  if ((packs + r - 1) / r > 1024) { *threads = 1024; *held = 0; return; }
  *threads = ((packs + r - 1) / r + 31) / 32 * 32;
  *held = r;
}

template <typename TO, bool ADD, int V>
void launch_norm(float* x, const CucaTerms& t, const float* w, TO* out, const int* rows, int n_rows, int E, float eps,
                 int center, cudaStream_t stream) {
  int threads, held;
  norm_shape(E / V, n_rows, &threads, &held);
#define NK(R) cuca_launch(norm_kernel<TO, ADD, V, R>, dim3(n_rows), dim3(threads), 0, stream, true, x, t, w, out, rows, E, eps, center)
  if (held == 1) NK(1);
  else if (held == 2) NK(2);
  else if (held == 4) NK(4);
  else if (held == 8) NK(8);
  else NK(0);
#undef NK
}

}  // namespace

CUCA_API int cuca_max_terms() { return CUCA_MAX_TERMS; }

// x[r] += N(y[r]) * w with y the weighted sum of the terms; out (or null) = the new x in out_dtype. center 1: layer
// norm; 0: RMS norm.
CUCA_API int cuca_norm_add(float* x, const CucaTerms* terms, const float* w, void* out, int out_dtype, int n_rows, int E,
                           float eps, int center, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && terms && terms->n >= 0 && terms->n <= CUCA_MAX_TERMS, "norm_add: bad sizes (E=%d)", E);
  const bool wide = E % 4 == 0 && terms_wide(*terms) && aligned_to(x, 16) && aligned_to(w, 16) && aligned_to(out, 16);
#define NA(TO)                                                                                                         \
  do {                                                                                                                 \
    if (wide) launch_norm<TO, true, 4>(x, *terms, w, (TO*)out, nullptr, n_rows, E, eps, center, stream);               \
    else launch_norm<TO, true, 1>(x, *terms, w, (TO*)out, nullptr, n_rows, E, eps, center, stream);                    \
  } while (0)
  if (out == nullptr || out_dtype == CUCA_F32) NA(float);
  else if (out_dtype == CUCA_BF16) NA(__nv_bfloat16);
  else CUCA_REQUIRE(false, "norm_add: unknown dtype %d", out_dtype);
#undef NA
  CUCA_CHECK_LAUNCH("norm_add");
  return 0;
}

// out[r] = N(x[rows ? rows[r] : r]) * w, the layer norm (rows[r] < 0: padding, skipped)
CUCA_API int cuca_layer_norm(const float* x, const float* w, void* out, int out_dtype, const int* rows, int n_rows, int E,
                             float eps, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0, "layer_norm: bad width %d", E);
  CucaTerms none = {};
  float* xm = const_cast<float*>(x);  // not written
  const bool wide = E % 4 == 0 && aligned_to(x, 16) && aligned_to(w, 16) && aligned_to(out, 16);
#define LN(TO)                                                                                                         \
  do {                                                                                                                 \
    if (wide) launch_norm<TO, false, 4>(xm, none, w, (TO*)out, rows, n_rows, E, eps, 1, stream);                       \
    else launch_norm<TO, false, 1>(xm, none, w, (TO*)out, rows, n_rows, E, eps, 1, stream);                            \
  } while (0)
  if (out_dtype == CUCA_F32) LN(float);
  else if (out_dtype == CUCA_BF16) LN(__nv_bfloat16);
  else CUCA_REQUIRE(false, "layer_norm: unknown dtype %d", out_dtype);
#undef LN
  CUCA_CHECK_LAUNCH("layer_norm");
  return 0;
}

static unsigned grid_for(size_t work) {
  const size_t b = (work + 255) / 256;
  return (unsigned)(b < 1 ? 1 : (b > 8192 ? 8192 : b));
}

CUCA_API int cuca_add_terms(float* x, const CucaTerms* terms, int store, size_t n, cudaStream_t stream) {
  if (n == 0) return 0;
  CUCA_REQUIRE(terms && terms->n >= 0 && terms->n <= CUCA_MAX_TERMS, "add_terms: bad terms");
  if (n % 4 == 0 && terms_wide(*terms) && aligned_to(x, 16))
    cuca_launch(add_terms_kernel<4>, dim3(grid_for(n / 4)), dim3(256), 0, stream, true, x, *terms, store, n);
  else
    cuca_launch(add_terms_kernel<1>, dim3(grid_for(n)), dim3(256), 0, stream, true, x, *terms, store, n);
  CUCA_CHECK_LAUNCH("add_terms");
  return 0;
}

CUCA_API int cuca_round_rows(const float* x, void* out, int out_dtype, size_t n, cudaStream_t stream) {
  if (n == 0) return 0;
  const bool wide = n % 4 == 0 && aligned_to(x, 16) && aligned_to(out, 16);
#define RR(TO)                                                                                                         \
  do {                                                                                                                 \
    if (wide) cuca_launch(round_rows_kernel<TO, 4>, dim3(grid_for(n / 4)), dim3(256), 0, stream, true, x, (TO*)out, n); \
    else cuca_launch(round_rows_kernel<TO, 1>, dim3(grid_for(n)), dim3(256), 0, stream, true, x, (TO*)out, n);          \
  } while (0)
  if (out_dtype == CUCA_F32) RR(float);
  else if (out_dtype == CUCA_BF16) RR(__nv_bfloat16);
  else CUCA_REQUIRE(false, "round_rows: unknown dtype %d", out_dtype);
#undef RR
  CUCA_CHECK_LAUNCH("round_rows");
  return 0;
}

// out[r] = o[r] / sqrt(mean(o[r]^2) + eps) * w * sigmoid(gate[r]); o: [n_rows, n] 32-bit, gate: rows of stride ldg
CUCA_API int cuca_row_norm_gate(const float* o, const float* w, const void* gate, int gate_dtype, int ldg, void* out,
                                int out_dtype, int n_rows, int n, float eps, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(n > 0, "row_norm_gate: bad width %d", n);
  const bool wide = n % 4 == 0 && ldg % 4 == 0 && aligned_to(o, 16) && aligned_to(w, 16) && aligned_to(gate, gate_dtype == CUCA_F32 ? 16 : 8) &&
                    aligned_to(out, 16);
  const int packs = wide ? n / 4 : n;
  int threads = (packs + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  if (n_rows >= 512 && threads > 256) threads = 256;
#define RNG(TG, TO)                                                                                                    \
  do {                                                                                                                 \
    if (wide) cuca_launch(row_norm_gate_kernel<TG, TO, 4>, dim3(n_rows), dim3(threads), 0, stream, true, o, w,          \
                          (const TG*)gate, ldg, (TO*)out, n, eps);                                                     \
    else cuca_launch(row_norm_gate_kernel<TG, TO, 1>, dim3(n_rows), dim3(threads), 0, stream, true, o, w,               \
                     (const TG*)gate, ldg, (TO*)out, n, eps);                                                          \
  } while (0)
  if (gate_dtype == CUCA_F32 && out_dtype == CUCA_F32) RNG(float, float);
  else if (gate_dtype == CUCA_F32 && out_dtype == CUCA_BF16) RNG(float, __nv_bfloat16);
  else if (gate_dtype == CUCA_BF16 && out_dtype == CUCA_BF16) RNG(__nv_bfloat16, __nv_bfloat16);
  else CUCA_REQUIRE(false, "row_norm_gate: unsupported dtypes %d/%d", gate_dtype, out_dtype);
#undef RNG
  CUCA_CHECK_LAUNCH("row_norm_gate");
  return 0;
}
