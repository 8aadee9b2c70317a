// Memory-bound kernels of the step: embedding gather, RMSNorm (with optional
// row gather), rotary encoding fused with the paged key/value write, SwiGLU.
// All arithmetic is 32-bit; the residual stream is 32-bit in every mode.
#include "common.cuh"
#include <stdarg.h>
#include <string>

static thread_local std::string g_last_error;
void cuca_set_error(const char* fmt, ...) {
  char buf[1024];
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(buf, sizeof(buf), fmt, ap);
  va_end(ap);
  g_last_error = buf;
}
CUCA_API const char* cuca_last_error() { return g_last_error.c_str(); }
CUCA_API int cuca_abi_version() { return 4; }

#include <stdlib.h>
static int g_pdl = -1;
bool cuca_pdl_enabled() {
  if (g_pdl < 0) {
    const char* e = getenv("CUCA_PDL");
    g_pdl = (e && e[0] == '0') ? 0 : 1;
  }
  return g_pdl != 0;
}
// 1: kernels are launched as programmatic dependents of their predecessors (default); 0: plain stream order.
CUCA_API int cuca_set_pdl(int on) { g_pdl = on ? 1 : 0; return 0; }

// ---------------------------------------------------------------- embedding
template <typename T>
__global__ void embed_kernel(const T* __restrict__ table, const int* __restrict__ tokens,
                             float* __restrict__ x, int E, int V, int* err, float scale) {
  pdl_trigger();
  pdl_wait();
  int row = blockIdx.x;
  int tok = tokens[row];
  if (tok < 0 || tok >= V) {
    if (threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
    for (int i = threadIdx.x; i < E; i += blockDim.x) x[(size_t)row * E + i] = 0.f;
    return;
  }
  const T* src = table + (size_t)tok * E;
  float* dst = x + (size_t)row * E;
  // 16 bytes per thread and round where the row allows it (a 4096-wide row in two rounds instead of sixteen rounds
  // of one value each: at eight rows the kernel is all latency)
  if (sizeof(T) == 2 && (E & 7) == 0 && (((size_t)src) & 15) == 0 && (((size_t)dst) & 15) == 0) {
    for (int i = threadIdx.x; i < (E >> 3); i += blockDim.x) {
      const uint4 w = reinterpret_cast<const uint4*>(src)[i];
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&w);
      const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]), c = __bfloat1622float2(h[2]),
                   d = __bfloat1622float2(h[3]);
      reinterpret_cast<float4*>(dst)[2 * i] = make_float4(a.x * scale, a.y * scale, b.x * scale, b.y * scale);
      reinterpret_cast<float4*>(dst)[2 * i + 1] = make_float4(c.x * scale, c.y * scale, d.x * scale, d.y * scale);
    }
    return;
  }
  if (sizeof(T) == 4 && (E & 3) == 0 && (((size_t)src) & 15) == 0 && (((size_t)dst) & 15) == 0) {
    for (int i = threadIdx.x; i < (E >> 2); i += blockDim.x) {
      const float4 v = reinterpret_cast<const float4*>(src)[i];
      reinterpret_cast<float4*>(dst)[i] = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
    }
    return;
  }
  for (int i = threadIdx.x; i < E; i += blockDim.x) dst[i] = to_f32(src[i]) * scale;
}

// Embedding rows of `tokens[n_rows]`, times `scale`, into the 32-bit stream x[n_rows, E].
CUCA_API int cuca_embed_scaled(const void* table, int table_dtype, const int* tokens, float* x,
                               int n_rows, int E, int V, float scale, int* err, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && V > 0, "embed: bad sizes E=%d V=%d", E, V);
  if (table_dtype == CUCA_F32)
    embed_kernel<float><<<n_rows, 256, 0, stream>>>((const float*)table, tokens, x, E, V, err, scale);
  else if (table_dtype == CUCA_BF16)
    embed_kernel<__nv_bfloat16><<<n_rows, 256, 0, stream>>>((const __nv_bfloat16*)table, tokens, x, E, V, err, scale);
  else
    CUCA_REQUIRE(false, "embed: unknown dtype %d", table_dtype);
  CUCA_CHECK_LAUNCH("embed");
  return 0;
}

CUCA_API int cuca_embed(const void* table, int table_dtype, const int* tokens, float* x,
                        int n_rows, int E, int V, int* err, cudaStream_t stream) {
  return cuca_embed_scaled(table, table_dtype, tokens, x, n_rows, E, V, 1.f, err, stream);
}

// ---------------------------------------------------------------- embedding plus a learned position vector
// x[r] = table[tokens[r]] * scale + pos_table[positions[r]] into the 32-bit stream. A token or position outside its table
// is recorded and contributes nothing.
template <typename T>
__global__ void __launch_bounds__(256)
embed_pos_kernel(const T* __restrict__ table, const T* __restrict__ pos_table, const int* __restrict__ tokens,
                 const int* __restrict__ positions, float* __restrict__ x, int E, int V, int n_pos, float scale, int* err) {
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.y;
  const int tok = tokens[row], pos = positions[row];
  const bool tok_ok = tok >= 0 && tok < V, pos_ok = pos >= 0 && pos < n_pos;
  if (!(tok_ok && pos_ok) && blockIdx.x == 0 && threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
  const T* a = table + (size_t)(tok_ok ? tok : 0) * E;
  const T* b = pos_table + (size_t)(pos_ok ? pos : 0) * E;
  const float fa = tok_ok ? scale : 0.f, fb = pos_ok ? 1.f : 0.f;
  float* dst = x + row * E;
  const int first = blockIdx.x * blockDim.x + threadIdx.x, step = gridDim.x * blockDim.x;
  // four values a thread and round where the rows allow it
  constexpr int A = 4 * sizeof(T) - 1;
  if ((E & 3) == 0 && (((size_t)table | (size_t)pos_table) & A) == 0 && (((size_t)x) & 15) == 0) {
    for (int i = first; i < (E >> 2); i += step) {
      float va[4], vb[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) { va[k] = to_f32(a[4 * i + k]); vb[k] = to_f32(b[4 * i + k]); }
      reinterpret_cast<float4*>(dst)[i] = make_float4(va[0] * fa + vb[0] * fb, va[1] * fa + vb[1] * fb, va[2] * fa + vb[2] * fb, va[3] * fa + vb[3] * fb);
    }
    return;
  }
  for (int i = first; i < E; i += step) dst[i] = to_f32(a[i]) * fa + to_f32(b[i]) * fb;
}

CUCA_API int cuca_embed_pos(const void* table, const void* pos_table, int table_dtype, const int* tokens, const int* positions,
                            float* x, int n_rows, int E, int V, int n_pos, float scale, int* err, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && V > 0 && n_pos > 0, "embed_pos: bad sizes E=%d V=%d positions=%d", E, V, n_pos);
  CUCA_REQUIRE(n_rows <= 65535, "embed_pos: %d rows in one step exceed the launch limit 65535", n_rows);
  const dim3 grid((E + 1023) / 1024, n_rows);
  if (table_dtype == CUCA_F32)
    cuca_launch(embed_pos_kernel<float>, grid, dim3(256), 0, stream, true, (const float*)table, (const float*)pos_table,
                tokens, positions, x, E, V, n_pos, scale, err);
  else if (table_dtype == CUCA_BF16)
    cuca_launch(embed_pos_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, true, (const __nv_bfloat16*)table,
                (const __nv_bfloat16*)pos_table, tokens, positions, x, E, V, n_pos, scale, err);
  else
    CUCA_REQUIRE(false, "embed_pos: unknown dtype %d", table_dtype);
  CUCA_CHECK_LAUNCH("embed_pos");
  return 0;
}

// ---------------------------------------------------------------- embedding followed by an RMS norm
// x[r] = e / sqrt(mean(e^2) + eps) * w with e = table[tokens[r]] * scale: the stream starts as the normed embedding
// row. One block per row, two passes over the row (the second one hits the cache); the sum's order depends on E alone.
template <typename T>
__global__ void __launch_bounds__(256)
embed_norm_kernel(const T* __restrict__ table, const int* __restrict__ tokens, float* __restrict__ x, int E, int V,
                  float scale, const float* __restrict__ w, float eps, int* err) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const int tok = tokens[row];
  float* dst = x + (size_t)row * E;
  if (tok < 0 || tok >= V) {
    if (threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
    for (int i = threadIdx.x; i < E; i += blockDim.x) dst[i] = 0.f;
    return;
  }
  const T* src = table + (size_t)tok * E;
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += blockDim.x) { const float v = to_f32(src[i]) * scale; ss = fmaf(v, v, ss); }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / (float)E + eps);
  for (int i = threadIdx.x; i < E; i += blockDim.x) dst[i] = to_f32(src[i]) * scale * inv * w[i];
}

CUCA_API int cuca_embed_norm(const void* table, int table_dtype, const int* tokens, float* x, int n_rows, int E, int V,
                             float scale, const float* w, float eps, int* err, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && V > 0 && w != nullptr, "embed_norm: bad sizes E=%d V=%d", E, V);
  if (table_dtype == CUCA_F32)
    cuca_launch(embed_norm_kernel<float>, dim3(n_rows), dim3(256), 0, stream, true, (const float*)table, tokens, x, E, V,
                scale, w, eps, err);
  else if (table_dtype == CUCA_BF16)
    cuca_launch(embed_norm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(256), 0, stream, true, (const __nv_bfloat16*)table,
                tokens, x, E, V, scale, w, eps, err);
  else
    CUCA_REQUIRE(false, "embed_norm: unknown dtype %d", table_dtype);
  CUCA_CHECK_LAUNCH("embed_norm");
  return 0;
}

// ---------------------------------------------------------------- RMSNorm
// One block per output row. Every thread takes four consecutive values at a time and the block is as wide as
// the row needs (up to 1024 threads), so all loads of a row are in flight together. The reduction order depends
// only on E, so a row's result does not depend on what else is in the batch.
static inline int norm_block(int E) {
  int t = ((E + 3) / 4 + 31) / 32 * 32;
  return t < 32 ? 32 : (t > 1024 ? 1024 : t);
}

__device__ __forceinline__ float block_sum_1024(float s, float* red) {
  s = warp_sum(s);
  const int nw = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = s;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  return tot;
}

// four consecutive outputs with one store where the address allows it
__device__ __forceinline__ void store4(float* o, float a, float b, float c, float d) {
  if ((((size_t)o) & 15) == 0) *reinterpret_cast<float4*>(o) = make_float4(a, b, c, d);
  else { o[0] = a; o[1] = b; o[2] = c; o[3] = d; }
}
__device__ __forceinline__ void store4(__nv_bfloat16* o, float a, float b, float c, float d) {
  if ((((size_t)o) & 7) == 0) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(o) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  } else {
    o[0] = __float2bfloat16_rn(a); o[1] = __float2bfloat16_rn(b); o[2] = __float2bfloat16_rn(c); o[3] = __float2bfloat16_rn(d);
  }
}

// PARTIAL: x[row] += sum over slices first (written back), see below.
// VL: value groups per thread and round. A block of B threads with VL groups each does exactly the arithmetic
// of a block of B * VL threads with one group each (thread t plays the lanes t, t + B, ...: the same warp
// shuffles, the same order across warps), so many-row launches can use narrow blocks with bit-equal results.
template <typename TW, typename TO, bool PARTIAL, int VL>
__global__ void rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ partial, int n_slices,
                               size_t slice_stride, const TW* __restrict__ w, TO* __restrict__ out,
                               const int* __restrict__ rows, int E, float eps, int groups) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  // `groups` equal consecutive parts of a row are normed apart: a block takes one part of E values (the row is
  // groups * E wide), so a part's arithmetic is that of a whole row of its width
  int orow = blockIdx.x, part = 0;
  if (groups > 1) { part = orow % groups; orow /= groups; }
  int irow = rows ? rows[orow] : orow;
  if (irow < 0) return;
  const size_t ld = (size_t)E * groups;
  float* xr = x + (size_t)irow * ld + (size_t)part * E;
  const float* pr = PARTIAL ? partial + (size_t)irow * ld + (size_t)part * E : nullptr;
  TO* o = out + (size_t)orow * ld + (size_t)part * E;
  w += (size_t)part * E;
  float s = 0.f;
  const bool vec = (E & 3) == 0 && (((size_t)xr) & 15) == 0 && (!PARTIAL || ((((size_t)pr) | (slice_stride * 4)) & 15) == 0);
  if (vec) {
    const int nvec = E >> 2;
    // One value group (four floats) per thread and round. The first two rounds (rows up to 8192 wide) stay in
    // registers between the two passes; wider rows are read again.
    auto take = [&](int i) {
      float4 v = reinterpret_cast<const float4*>(xr)[i];
      if (PARTIAL) {
        for (int k0 = 0; k0 < n_slices; k0 += 4) {  // four slices' loads in flight at once, added in slice order
          float4 q[4];
#pragma unroll
          for (int u = 0; u < 4; ++u)
            q[u] = k0 + u < n_slices ? __ldcg(reinterpret_cast<const float4*>(pr + (k0 + u) * slice_stride) + i)
                                     : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int u = 0; u < 4; ++u) { v.x += q[u].x; v.y += q[u].y; v.z += q[u].z; v.w += q[u].w; }
        }
        reinterpret_cast<float4*>(xr)[i] = v;
      }
      s = fmaf(v.x, v.x, s); s = fmaf(v.y, v.y, s); s = fmaf(v.z, v.z, s); s = fmaf(v.w, v.w, s);
      return v;
    };
    auto put = [&](int i, float4 v, float r) {
      const int e = i << 2;
      const float w0 = to_f32(w[e]), w1 = to_f32(w[e + 1]), w2 = to_f32(w[e + 2]), w3 = to_f32(w[e + 3]);
      store4(o + e, v.x * r * w0, v.y * r * w1, v.z * r * w2, v.w * r * w3);
    };
    const int VB = blockDim.x * VL;  // virtual block width
    float4 v0[VL], v1[VL];
    float sk[VL];
#pragma unroll
    for (int k = 0; k < VL; ++k) {
      const int i0 = threadIdx.x + blockDim.x * k, i1 = i0 + VB;
      s = 0.f;
      v0[k] = v1[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i0 < nvec) v0[k] = take(i0);
      if (i1 < nvec) v1[k] = take(i1);
      for (int i = i1 + VB; i < nvec; i += VB) take(i);
      sk[k] = s;
    }
    // reduction in the order of the virtual block: warp sums, then the warps in ascending order
    const int real_warps = blockDim.x >> 5;
#pragma unroll
    for (int k = 0; k < VL; ++k) {
      float wsum = warp_sum(sk[k]);
      if ((threadIdx.x & 31) == 0) red[(threadIdx.x >> 5) + real_warps * k] = wsum;
    }
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < real_warps * VL; ++i) tot += red[i];
    const float r = rsqrtf(tot / (float)E + eps);
#pragma unroll
    for (int k = 0; k < VL; ++k) {
      const int i0 = threadIdx.x + blockDim.x * k, i1 = i0 + VB;
      if (i0 < nvec) put(i0, v0[k], r);
      if (i1 < nvec) put(i1, v1[k], r);
      for (int i = i1 + VB; i < nvec; i += VB) put(i, reinterpret_cast<const float4*>(xr)[i], r);
    }
  } else {
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
      float v = xr[i];
      if (PARTIAL) {
        for (int k = 0; k < n_slices; ++k) v += __ldcg(pr + k * slice_stride + i);
        xr[i] = v;
      }
      s = fmaf(v, v, s);
    }
    float r = rsqrtf(block_sum_1024(s, red) / (float)E + eps);
    for (int i = threadIdx.x; i < E; i += blockDim.x) o[i] = from_f32<TO>(xr[i] * r * to_f32(w[i]));
  }
}

// out[r] = x[rows ? rows[r] : r] * rsqrt(mean(x^2) + eps) * w; with groups > 1 every one of `groups` equal consecutive
// parts of a row is divided by its own root mean square.
CUCA_API int cuca_rmsnorm_groups(const float* x, const void* w, int w_dtype, void* out, int out_dtype,
                                 const int* rows, int n_rows, int E, float eps, int groups, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && groups >= 1 && E % groups == 0, "rmsnorm: %d parts do not divide the width %d", groups, E);
  CUCA_REQUIRE((long long)n_rows * groups < (1ll << 31), "rmsnorm: %d rows of %d parts exceed the launch limit", n_rows, groups);
  E /= groups;
  n_rows *= groups;
  float* xm = const_cast<float*>(x);  // not written without PARTIAL
  // many rows: a quarter of the threads per block, four value groups each (bit-equal to the wide block)
  const bool narrow = norm_block(E) == 1024 && n_rows >= 64 && (E & 3) == 0;
#define LAUNCH(TW, TO)                                                                                          \
  do {                                                                                                          \
    if (narrow)                                                                                                 \
      cuca_launch(rmsnorm_kernel<TW, TO, false, 4>, dim3(n_rows), dim3(256), 0, stream, true, xm,               \
                  (const float*)nullptr, 0, (size_t)0, (const TW*)w, (TO*)out, rows, E, eps, groups);           \
    else                                                                                                        \
      cuca_launch(rmsnorm_kernel<TW, TO, false, 1>, dim3(n_rows), dim3(norm_block(E)), 0, stream, true, xm,     \
                  (const float*)nullptr, 0, (size_t)0, (const TW*)w, (TO*)out, rows, E, eps, groups);           \
  } while (0)
  if (w_dtype == CUCA_F32 && out_dtype == CUCA_F32) LAUNCH(float, float);
  else if (w_dtype == CUCA_F32 && out_dtype == CUCA_BF16) LAUNCH(float, __nv_bfloat16);
  else if (w_dtype == CUCA_BF16 && out_dtype == CUCA_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (w_dtype == CUCA_BF16 && out_dtype == CUCA_F32) LAUNCH(__nv_bfloat16, float);
  else CUCA_REQUIRE(false, "rmsnorm: unknown dtypes %d %d", w_dtype, out_dtype);
#undef LAUNCH
  CUCA_CHECK_LAUNCH("rmsnorm");
  return 0;
}

CUCA_API int cuca_rmsnorm(const float* x, const void* w, int w_dtype, void* out, int out_dtype,
                          const int* rows, int n_rows, int E, float eps, cudaStream_t stream) {
  return cuca_rmsnorm_groups(x, w, w_dtype, out, out_dtype, rows, n_rows, E, eps, 1, stream);
}

// ---------------------------------------------------------------- rotary + paged K/V write
// qkv: [T, (nh + 2 nkv) d]. q and k heads are rotated (first `rot` values of a
// head, pairs (i, i + rot/2)); q in place, k and v go to their page (nkv = 0:
// the layer owns no keys, only q is rotated):
// pool[block][kv head][row in block][d], block = table[seq][pos / bs].
template <typename T>
__global__ void __launch_bounds__(256)
rope_store_kernel(T* __restrict__ qkv, const int* __restrict__ positions,
                  const int* __restrict__ seq_of_row, const int* __restrict__ tables,
                  int table_stride, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                  int table_rows, int rot, T* __restrict__ kpool, T* __restrict__ vpool,
                  int n_blocks, int bs, int nh, int nkv, int d, int* err) {
  // one block per row; its threads walk all heads of the row: rotated pairs, pass-through values, v copies
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const int seq = seq_of_row[row];
  if (seq < 0) return;
  const int pos = positions[row];
  const int half = rot / 2;
  T* base = qkv + (size_t)row * (nh + 2 * nkv) * d;
  long long page_off = -1;  // offset of this position's row in a pool, per kv head add kvh * bs * d
  if (nkv > 0) {
    int blk = pos >= 0 ? tables[(size_t)seq * table_stride + pos / bs] : -1;
    if (blk < 0 || blk >= n_blocks) {
      if (threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_BLOCK_RANGE);
    } else {
      page_off = ((long long)blk * nkv * bs + (pos % bs)) * d;
    }
  }
  const bool in_table = pos >= 0 && pos < table_rows;
  if (!in_table && half > 0 && threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
  const float* cr = cos_t + (size_t)(in_table ? pos : 0) * half;
  const float* sr = sin_t + (size_t)(in_table ? pos : 0) * half;
  // q and k heads: `half` rotated pairs + (d - rot) values that pass through
  const int per_head = half + (d - rot);
  const int qk_items = (nh + nkv) * per_head;
  for (int idx = threadIdx.x; idx < qk_items; idx += blockDim.x) {
    const int head = idx / per_head, i = idx % per_head;
    T* src = base + (size_t)head * d;
    T* dst = nullptr;  // k heads go to their page; q heads are rotated in place
    const bool is_k = head >= nh;
    if (is_k) {
      if (page_off < 0) continue;
      dst = kpool + page_off + (size_t)(head - nh) * bs * d;
    }
    if (i < half) {
      float c = in_table ? cr[i] : 1.f, sn = in_table ? sr[i] : 0.f;
      float a = to_f32(src[i]), b = to_f32(src[i + half]);
      T ra = from_f32<T>(a * c - b * sn), rb = from_f32<T>(a * sn + b * c);
      if (is_k) { dst[i] = ra; dst[i + half] = rb; }
      else { src[i] = ra; src[i + half] = rb; }
    } else if (is_k) {
      const int e = rot + (i - half);
      dst[e] = src[e];
    }
  }
  if (nkv > 0 && page_off >= 0) {
    const T* vsrc = base + (size_t)(nh + nkv) * d;
    for (int idx = threadIdx.x; idx < nkv * d; idx += blockDim.x) {
      const int kvh = idx / d, e = idx % d;
      vpool[page_off + (size_t)kvh * bs * d + e] = vsrc[idx];
    }
  }
}

// The same for bf16 rows whose heads are rotated whole (rot = d) with d a multiple of 16: a thread takes eight
// pairs (16 bytes of each half of a head, eight cosines and sines) or 16 bytes of v at a time. Same arithmetic,
// element by element, as the kernel above.
__global__ void __launch_bounds__(256)
rope_store_vec_kernel(__nv_bfloat16* __restrict__ qkv, const int* __restrict__ positions,
                      const int* __restrict__ seq_of_row, const int* __restrict__ tables, int table_stride,
                      const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_rows,
                      __nv_bfloat16* __restrict__ kpool, __nv_bfloat16* __restrict__ vpool, int n_blocks, int bs,
                      int nh, int nkv, int d, int* err) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const int seq = seq_of_row[row];
  if (seq < 0) return;
  const int pos = positions[row];
  const int half = d / 2;
  __nv_bfloat16* base = qkv + (size_t)row * (nh + 2 * nkv) * d;
  long long page_off = -1;
  if (nkv > 0) {
    int blk = pos >= 0 ? tables[(size_t)seq * table_stride + pos / bs] : -1;
    if (blk < 0 || blk >= n_blocks) {
      if (threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_BLOCK_RANGE);
    } else {
      page_off = ((long long)blk * nkv * bs + (pos % bs)) * d;
    }
  }
  const bool in_table = pos >= 0 && pos < table_rows;
  if (!in_table && threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
  const float* cr = cos_t + (size_t)(in_table ? pos : 0) * half;
  const float* sr = sin_t + (size_t)(in_table ? pos : 0) * half;
  const int per_head = half / 8;  // items of eight pairs
  const int qk_items = (nh + nkv) * per_head;
  const int v_items = (nkv > 0 && page_off >= 0) ? nkv * d / 8 : 0;
  for (int idx = threadIdx.x; idx < qk_items + v_items; idx += blockDim.x) {
    if (idx >= qk_items) {
      const int e = (idx - qk_items) * 8, kvh = e / d;
      const uint4 v = *reinterpret_cast<const uint4*>(base + (size_t)(nh + nkv) * d + e);
      *reinterpret_cast<uint4*>(vpool + page_off + (size_t)kvh * bs * d + (e - kvh * d)) = v;
      continue;
    }
    const int head = idx / per_head, i = (idx - head * per_head) * 8;
    __nv_bfloat16* src = base + (size_t)head * d;
    const bool is_k = head >= nh;
    if (is_k && page_off < 0) continue;
    __nv_bfloat16* dst = is_k ? kpool + page_off + (size_t)(head - nh) * bs * d : src;
    uint4 ua = *reinterpret_cast<const uint4*>(src + i), ub = *reinterpret_cast<const uint4*>(src + i + half);
    float c[8], sn[8];
    if (in_table) {
      *reinterpret_cast<float4*>(c) = *reinterpret_cast<const float4*>(cr + i);
      *reinterpret_cast<float4*>(c + 4) = *reinterpret_cast<const float4*>(cr + i + 4);
      *reinterpret_cast<float4*>(sn) = *reinterpret_cast<const float4*>(sr + i);
      *reinterpret_cast<float4*>(sn + 4) = *reinterpret_cast<const float4*>(sr + i + 4);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) { c[j] = 1.f; sn[j] = 0.f; }
    }
    const __nv_bfloat16* pa = reinterpret_cast<const __nv_bfloat16*>(&ua);
    const __nv_bfloat16* pb = reinterpret_cast<const __nv_bfloat16*>(&ub);
    uint4 oa, ob;
    __nv_bfloat16* qa = reinterpret_cast<__nv_bfloat16*>(&oa);
    __nv_bfloat16* qb = reinterpret_cast<__nv_bfloat16*>(&ob);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float a = __bfloat162float(pa[j]), b = __bfloat162float(pb[j]);
      qa[j] = __float2bfloat16_rn(a * c[j] - b * sn[j]);
      qb[j] = __float2bfloat16_rn(a * sn[j] + b * c[j]);
    }
    *reinterpret_cast<uint4*>(dst + i) = oa;
    *reinterpret_cast<uint4*>(dst + i + half) = ob;
  }
}

CUCA_API int cuca_rope_store(void* qkv, int dtype, const int* positions, const int* seq_of_row,
                             const int* tables, int table_stride, const float* cos_t, const float* sin_t,
                             int table_rows, int rot, void* kpool, void* vpool, int n_blocks, int bs,
                             int n_rows, int nh, int nkv, int d, int* err, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0, "rope_store: rotary size %d does not fit head size %d", rot, d);
  CUCA_REQUIRE(bs > 0 && nh > 0 && nkv >= 0 && d > 0, "rope_store: bad sizes");
  dim3 grid(n_rows);
  int threads = 256;
  const bool aligned = (((uintptr_t)qkv | (uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)cos_t | (uintptr_t)sin_t) & 15) == 0;
  if (dtype == CUCA_BF16 && rot == d && d % 16 == 0 && aligned)
    cuca_launch(rope_store_vec_kernel, grid, dim3(threads), 0, stream, true, (__nv_bfloat16*)qkv, positions, seq_of_row,
                tables, table_stride, cos_t, sin_t, table_rows, (__nv_bfloat16*)kpool, (__nv_bfloat16*)vpool, n_blocks,
                bs, nh, nkv, d, err);
  else if (dtype == CUCA_F32)
    cuca_launch(rope_store_kernel<float>, grid, dim3(threads), 0, stream, true, (float*)qkv, positions, seq_of_row,
                tables, table_stride, cos_t, sin_t, table_rows, rot, (float*)kpool, (float*)vpool, n_blocks, bs, nh,
                nkv, d, err);
  else if (dtype == CUCA_BF16)
    cuca_launch(rope_store_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, true, (__nv_bfloat16*)qkv,
                positions, seq_of_row, tables, table_stride, cos_t, sin_t, table_rows, rot, (__nv_bfloat16*)kpool,
                (__nv_bfloat16*)vpool, n_blocks, bs, nh, nkv, d, err);
  else
    CUCA_REQUIRE(false, "rope_store: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("rope_store");
  return 0;
}

// ---------------------------------------------------------------- SwiGLU (unfused form)
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, T* __restrict__ out, int ff, size_t total) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  size_t r = i / ff;
  int j = (int)(i % ff);
  float g = to_f32(gu[r * 2 * ff + j]);
  float u = to_f32(gu[r * 2 * ff + ff + j]);
  out[i] = from_f32<T>(g / (1.f + expf(-g)) * u);
}

// out[r, j] = silu(gu[r, j]) * gu[r, ff + j]
CUCA_API int cuca_swiglu(const void* gu, void* out, int dtype, int n_rows, int ff, cudaStream_t stream) {
  size_t total = (size_t)n_rows * ff;
  if (total == 0) return 0;
  unsigned blocks = (unsigned)((total + 255) / 256);
  if (dtype == CUCA_F32) swiglu_kernel<float><<<blocks, 256, 0, stream>>>((const float*)gu, (float*)out, ff, total);
  else if (dtype == CUCA_BF16)
    swiglu_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, ff, total);
  else CUCA_REQUIRE(false, "swiglu: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("swiglu");
  return 0;
}

// ---------------------------------------------------------------- a gated unit with capped inputs
// out[r, j] = g sigmoid(alpha g) (u + 1) with g = min(gu[r, j], limit), u = clamp(gu[r, ff + j], -limit, limit)
template <typename T>
__global__ void glu_capped_kernel(const T* __restrict__ gu, T* __restrict__ out, int ff, size_t total, float limit,
                                  float alpha) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / ff;
    const int j = (int)(i % ff);
    const float g = fminf(to_f32(gu[r * 2 * ff + j]), limit);
    const float u = fminf(fmaxf(to_f32(gu[r * 2 * ff + ff + j]), -limit), limit);
    out[i] = from_f32<T>(g / (1.f + expf(-alpha * g)) * (u + 1.f));
  }
}

CUCA_API int cuca_glu_capped(const void* gu, void* out, int dtype, int n_rows, int ff, float limit, float alpha,
                             cudaStream_t stream) {
  const size_t total = (size_t)n_rows * ff;
  if (total == 0) return 0;
  CUCA_REQUIRE(limit > 0.f, "glu_capped: the cap %g must be positive", (double)limit);
  size_t blocks = (total + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
  if (dtype == CUCA_F32)
    cuca_launch(glu_capped_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const float*)gu,
                (float*)out, ff, total, limit, alpha);
  else if (dtype == CUCA_BF16)
    cuca_launch(glu_capped_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, ff, total, limit, alpha);
  else
    CUCA_REQUIRE(false, "glu_capped: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("glu_capped");
  return 0;
}

// ---------------------------------------------------------------- a gated unit with a chosen activation
// out[r, j] = act(gu[r, j]) * gu[r, ff + j]; act 0: silu, 1: the tanh form of gelu,
// 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))).
__device__ __forceinline__ float glu_activation(float z, int act) {
  if (act == 1) return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  return z / (1.f + expf(-z));
}

template <typename T>
__global__ void glu_act_kernel(const T* __restrict__ gu, T* __restrict__ out, int ff, size_t total, int act) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / ff;
    const int j = (int)(i % ff);
    out[i] = from_f32<T>(glu_activation(to_f32(gu[r * 2 * ff + j]), act) * to_f32(gu[r * 2 * ff + ff + j]));
  }
}

CUCA_API int cuca_glu_act(const void* gu, void* out, int dtype, int n_rows, int ff, int act, cudaStream_t stream) {
  const size_t total = (size_t)n_rows * ff;
  if (total == 0) return 0;
  CUCA_REQUIRE(act == 0 || act == 1, "glu_act: unknown activation %d", act);
  size_t blocks = (total + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
  if (dtype == CUCA_F32)
    cuca_launch(glu_act_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const float*)gu, (float*)out,
                ff, total, act);
  else if (dtype == CUCA_BF16)
    cuca_launch(glu_act_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, ff, total, act);
  else
    CUCA_REQUIRE(false, "glu_act: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("glu_act");
  return 0;
}

// ---------------------------------------------------------------- one gate per head
// a[r, h dv + j] *= sigmoid(gate[r, h]) for every head h of dv values; a: rows of stride lda, gate: rows of stride ldg.
// VEC values (16 bytes of bfloat16, or one 32-bit value) a thread at a time; a run of VEC values lies within one head.
template <typename T, int VEC>
__global__ void head_gate_kernel(T* __restrict__ a, int lda, const T* __restrict__ gate, int ldg, int n_rows, int H,
                                 int dv) {
  pdl_trigger();
  pdl_wait();
  const int per_row = H * dv / VEC;
  const size_t total = (size_t)n_rows * per_row;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / per_row;
    const int c = (int)(i % per_row) * VEC;
    const float g = 1.f / (1.f + expf(-to_f32(gate[r * ldg + c / dv])));
    T* at = a + r * lda + c;
    if (VEC == 8) {
      uint4 w = *reinterpret_cast<const uint4*>(at);
      __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&w);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h2[e]);
        h2[e] = __floats2bfloat162_rn(f.x * g, f.y * g);
      }
      *reinterpret_cast<uint4*>(at) = w;
    } else {
      *at = from_f32<T>(to_f32(*at) * g);
    }
  }
}

CUCA_API int cuca_head_gate(void* a, int lda, const void* gate, int ldg, int dtype, int n_rows, int H, int dv,
                            cudaStream_t stream) {
  const size_t total = (size_t)n_rows * H * dv;
  if (total == 0) return 0;
  const bool wide = dtype == CUCA_BF16 && dv % 8 == 0 && lda % 8 == 0 && ((uintptr_t)a & 15) == 0;
  size_t blocks = (total / (wide ? 8 : 1) + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
  if (dtype == CUCA_F32)
    cuca_launch(head_gate_kernel<float, 1>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (float*)a, lda,
                (const float*)gate, ldg, n_rows, H, dv);
  else if (dtype == CUCA_BF16 && wide)
    cuca_launch(head_gate_kernel<__nv_bfloat16, 8>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (__nv_bfloat16*)a, lda, (const __nv_bfloat16*)gate, ldg, n_rows, H, dv);
  else if (dtype == CUCA_BF16)
    cuca_launch(head_gate_kernel<__nv_bfloat16, 1>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (__nv_bfloat16*)a, lda, (const __nv_bfloat16*)gate, ldg, n_rows, H, dv);
  else
    CUCA_REQUIRE(false, "head_gate: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("head_gate");
  return 0;
}

// ---------------------------------------------------------------- a smooth cap: a <- c tanh(a / c), 32-bit, in place
__global__ void softcap_kernel(float* __restrict__ a, size_t n, float cap) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    a[i] = cap * tanhf(a[i] / cap);
}

CUCA_API int cuca_softcap(float* a, size_t n, float cap, cudaStream_t stream) {
  if (n == 0) return 0;
  CUCA_REQUIRE(cap > 0.f, "softcap: the cap %g must be positive", (double)cap);
  size_t blocks = (n + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
  cuca_launch(softcap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, true, a, n, cap);
  CUCA_CHECK_LAUNCH("softcap");
  return 0;
}

// ---------------------------------------------------------------- stream += delta
template <typename T>
__global__ void add_kernel(float* __restrict__ x, const T* __restrict__ delta, size_t total) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < total) x[i] += to_f32(delta[i]);
}

CUCA_API int cuca_add_to_stream(float* x, const void* delta, int dtype, size_t total, cudaStream_t stream) {
  if (total == 0) return 0;
  unsigned blocks = (unsigned)((total + 255) / 256);
  if (dtype == CUCA_F32) add_kernel<float><<<blocks, 256, 0, stream>>>(x, (const float*)delta, total);
  else if (dtype == CUCA_BF16) add_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>(x, (const __nv_bfloat16*)delta, total);
  else CUCA_REQUIRE(false, "add_to_stream: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("add_to_stream");
  return 0;
}

// ---------------------------------------------------------------- table updates
__global__ void scatter_int_kernel(int* __restrict__ dst, const int* __restrict__ idx, const int* __restrict__ val,
                                   int n, long long limit) {
  int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n && idx[i] >= 0 && (long long)idx[i] < limit) dst[idx[i]] = val[i];
}

// dst[idx[i]] = val[i] for i < n; entries outside 0..limit-1 are skipped
CUCA_API int cuca_scatter_int(int* dst, const int* idx, const int* val, int n, long long limit, cudaStream_t stream) {
  if (n == 0) return 0;
  scatter_int_kernel<<<(n + 255) / 256, 256, 0, stream>>>(dst, idx, val, n, limit);
  CUCA_CHECK_LAUNCH("scatter_int");
  return 0;
}

// ---------------------------------------------------------------- consumers of partial sums (decode)
// A contraction over few tokens is cut along K over several CTAs. Instead of adding the slices up itself (a
// second pass through global memory at the end of a short kernel), it leaves them as [slice][row][feature]
// 32-bit sums, and the next kernel, which reads every value anyway, adds them in slice order.

// x[row] += sum over slices; out[orow] = RMSNorm(x[row]) * w (the RMSNorm kernel above with PARTIAL).
CUCA_API int cuca_add_partials_rmsnorm_groups(float* x, const float* partial, int n_slices, size_t slice_stride,
                                              const float* w, void* out, int out_dtype, const int* rows, int n_rows,
                                              int E, float eps, int groups, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(E > 0 && n_slices >= 1 && groups >= 1 && E % groups == 0, "add_partials_rmsnorm: bad sizes");
  E /= groups;
  n_rows *= groups;
  if (out_dtype == CUCA_BF16)
    cuca_launch(rmsnorm_kernel<float, __nv_bfloat16, true, 1>, dim3(n_rows), dim3(norm_block(E)), 0, stream, true, x,
                partial, n_slices, slice_stride, w, (__nv_bfloat16*)out, rows, E, eps, groups);
  else if (out_dtype == CUCA_F32)
    cuca_launch(rmsnorm_kernel<float, float, true, 1>, dim3(n_rows), dim3(norm_block(E)), 0, stream, true, x, partial,
                n_slices, slice_stride, w, (float*)out, rows, E, eps, groups);
  else
    CUCA_REQUIRE(false, "add_partials_rmsnorm: unknown dtype %d", out_dtype);
  CUCA_CHECK_LAUNCH("add_partials_rmsnorm");
  return 0;
}

CUCA_API int cuca_add_partials_rmsnorm(float* x, const float* partial, int n_slices, size_t slice_stride,
                                       const float* w, void* out, int out_dtype, const int* rows, int n_rows, int E,
                                       float eps, cudaStream_t stream) {
  return cuca_add_partials_rmsnorm_groups(x, partial, n_slices, slice_stride, w, out, out_dtype, rows, n_rows, E, eps, 1,
                                          stream);
}

// x += sum over slices: for a reader of the stream that does not add the slices itself.
__global__ void add_partials_kernel(float* __restrict__ x, const float* __restrict__ partial, int n_slices,
                                    size_t slice_stride, size_t total) {
  pdl_trigger();
  pdl_wait();
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  float v = x[i];
  for (int k = 0; k < n_slices; ++k) v += __ldcg(partial + k * slice_stride + i);
  x[i] = v;
}

CUCA_API int cuca_add_partials(float* x, const float* partial, int n_slices, size_t slice_stride, size_t total,
                               cudaStream_t stream) {
  if (total == 0) return 0;
  cuca_launch(add_partials_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, true, x, partial,
              n_slices, slice_stride, total);
  CUCA_CHECK_LAUNCH("add_partials");
  return 0;
}

// The q/k/v projection arrives as partial sums [slice][row][(nh + 2 nkv) d]: add them (and the bias), rotate q
// and k in 32-bit, write q as bf16 to q_out[row][nh d] and k, v to their pages.
__global__ void rope_store_partial_kernel(const float* __restrict__ partial, int n_slices, size_t slice_stride,
                                          const __nv_bfloat16* __restrict__ bias, __nv_bfloat16* __restrict__ q_out,
                                          const int* __restrict__ positions, const int* __restrict__ seq_of_row,
                                          const int* __restrict__ tables, int table_stride,
                                          const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                          int table_rows, int rot, __nv_bfloat16* __restrict__ kpool,
                                          __nv_bfloat16* __restrict__ vpool, int n_blocks, int bs, int nh, int nkv,
                                          int d, int* err) {
  pdl_trigger();
  pdl_wait();
  int row = blockIdx.x;
  int head = blockIdx.y;
  int seq = seq_of_row[row];
  if (seq < 0) return;
  int pos = positions[row];
  const size_t width = (size_t)(nh + 2 * nkv) * d;
  const float* src = partial + (size_t)row * width + (size_t)head * d;
  const __nv_bfloat16* b = bias ? bias + (size_t)head * d : nullptr;
  auto value = [&](int i) {
    float v = b ? __bfloat162float(b[i]) : 0.f;
    for (int k0 = 0; k0 < n_slices; k0 += 4) {  // four slices' loads in flight at once, added in slice order
      float q[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) q[u] = k0 + u < n_slices ? __ldcg(src + (k0 + u) * slice_stride + i) : 0.f;
#pragma unroll
      for (int u = 0; u < 4; ++u) v += q[u];
    }
    return v;
  };
  bool is_v = head >= nh + nkv;
  bool is_k = !is_v && head >= nh;
  __nv_bfloat16* dst;
  if (is_k || is_v) {
    int blk = pos >= 0 ? tables[(size_t)seq * table_stride + pos / bs] : -1;
    if (blk < 0 || blk >= n_blocks) {
      if (threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_BLOCK_RANGE);
      return;
    }
    int kvh = is_k ? head - nh : head - nh - nkv;
    dst = (is_k ? kpool : vpool) + (((size_t)blk * nkv + kvh) * bs + (pos % bs)) * d;
  } else {
    dst = q_out + (size_t)row * nh * d + (size_t)head * d;
  }
  if (is_v) {
    for (int i = threadIdx.x; i < d; i += blockDim.x) dst[i] = __float2bfloat16_rn(value(i));
    return;
  }
  int half = rot / 2;
  bool in_table = pos >= 0 && pos < table_rows;
  if (!in_table && half > 0 && threadIdx.x == 0 && err) atomicExch(err, CUCA_ERR_TOKEN_RANGE);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float c = in_table ? cos_t[(size_t)pos * half + i] : 1.f;
    float s = in_table ? sin_t[(size_t)pos * half + i] : 0.f;
    float a = value(i), bb = value(i + half);
    dst[i] = __float2bfloat16_rn(a * c - bb * s);
    dst[i + half] = __float2bfloat16_rn(a * s + bb * c);
  }
  for (int i = rot + threadIdx.x; i < d; i += blockDim.x) dst[i] = __float2bfloat16_rn(value(i));
}

CUCA_API int cuca_rope_store_partial(const float* partial, int n_slices, size_t slice_stride, const void* bias,
                                     void* q_out, const int* positions, const int* seq_of_row, const int* tables,
                                     int table_stride, const float* cos_t, const float* sin_t, int table_rows,
                                     int rot, void* kpool, void* vpool, int n_blocks, int bs, int n_rows, int nh,
                                     int nkv, int d, int* err, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CUCA_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0, "rope_store_partial: rotary size %d does not fit head size %d", rot, d);
  CUCA_REQUIRE(bs > 0 && nh > 0 && nkv >= 0 && d > 0 && n_slices >= 1, "rope_store_partial: bad sizes");
  dim3 grid(n_rows, nh + 2 * nkv);
  int threads = d / 2 >= 64 ? 64 : 32;
  cuca_launch(rope_store_partial_kernel, grid, dim3(threads), 0, stream, true, partial, n_slices, slice_stride,
              (const __nv_bfloat16*)bias, (__nv_bfloat16*)q_out, positions, seq_of_row, tables, table_stride, cos_t,
              sin_t, table_rows, rot, (__nv_bfloat16*)kpool, (__nv_bfloat16*)vpool, n_blocks, bs, nh, nkv, d, err);
  CUCA_CHECK_LAUNCH("rope_store_partial");
  return 0;
}

// ---------------------------------------------------------------- random weights
// Element i of a tensor is a function of (key, i) alone, so the same values come out on the host and on the
// device, whole or in pieces: outputs 3i, 3i+1, 3i+2 of a SplitMix64 stream that starts at `key` give twelve
// 16-bit fields whose sum is near-normal (Irwin-Hall); v = (2 sum - 12 * 65535) * scale, then mean + v, each a
// single 32-bit rounding (no fused multiply-add, so the host restates it exactly).
__device__ __forceinline__ unsigned long long splitmix_out(unsigned long long state) {
  unsigned long long z = state;
  z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
  z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
  return z ^ (z >> 31);
}

template <typename T>
__global__ void random_normal_kernel(T* __restrict__ out, size_t n, size_t first, unsigned long long key, float mean,
                                     float scale) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const unsigned long long e = first + i;
  int sum = 0;
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    unsigned long long h = splitmix_out(key + (3ull * e + (unsigned long long)j + 1ull) * 0x9E3779B97F4A7C15ull);
    sum += (int)(h & 0xFFFF) + (int)((h >> 16) & 0xFFFF) + (int)((h >> 32) & 0xFFFF) + (int)(h >> 48);
  }
  float v = __fadd_rn(mean, __fmul_rn((float)(2 * sum - 12 * 65535), scale));
  out[i] = from_f32<T>(v);
}

// out[i] = mean + normal(first + i) * std for i < n (`first`: the element number out[0] has in its tensor).
CUCA_API int cuca_random_normal(void* out, int dtype, size_t n, size_t first, unsigned long long key, float mean,
                                float scale, cudaStream_t stream) {
  if (n == 0) return 0;
  CUCA_REQUIRE(n < ((size_t)1 << 40), "random_normal: %zu elements in one call", n);
  unsigned blocks = (unsigned)((n + 255) / 256);
  if (dtype == CUCA_F32)
    random_normal_kernel<float><<<blocks, 256, 0, stream>>>((float*)out, n, first, key, mean, scale);
  else if (dtype == CUCA_BF16)
    random_normal_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)out, n, first, key, mean, scale);
  else
    CUCA_REQUIRE(false, "random_normal: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("random_normal");
  return 0;
}
