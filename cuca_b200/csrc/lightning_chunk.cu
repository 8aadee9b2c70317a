// Lightning attention over prompt portions, chunk by chunk on the tensor cores (bfloat16 projections, 32-bit state):
//   S_t = a S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t   with q, k, v = silu of the projection's columns and one decay a a head.
// A request's rows of the step are cut into chunks of 64 tokens. With S the state before a chunk and i, j counted
// within it,
//   o_i = a^(i+1) S^T q_i + sum_(j<=i) a^(i-j) (q_i . k_j) v_j,      S <- a^n S + sum_j a^(n-1-j) k_j v_j^T:
//   chunk_state   per (chunk, head): the chunk's own sum  sum_j a^(n-1-j) k_j v_j^T
//   chunk_carry   per (request, head): the state before every chunk, in place of those sums, and the state after the last
//   chunk_output  per (chunk, head): o from the state before the chunk and the chunk's own tokens
// Decays enter as non-negative powers only, so nothing is divided by a small number. The projections are bfloat16 (their
// silu is taken in 32-bit and rounded); everything behind them keeps 32-bit precision: products accumulate in 32-bit,
// and a 32-bit factor (the state, decayed keys, decayed scores) goes into a product as the sum of two bfloat16 numbers,
// x = hi + lo, one product each.
#include "common.cuh"
#include <math.h>

namespace {

constexpr int C = 64;        // tokens of a chunk
constexpr int CW = 64;       // value columns (and, for the chunk's sum, key channels) of a block
constexpr int PITCH = CW + 8;  // values of a staged row of CW values: 16 bytes apart modulo 128, so that ldmatrix hits all banks
constexpr int MAX_DIM = 256;

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
// d += a b for a 16 x 16 tile of a and a 16 x 8 tile of b
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&t);
}
__device__ __forceinline__ float rounded(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
// (rounded to bfloat16 right after: the fast quotient and exponential are exact enough)
__device__ __forceinline__ float silu_(float v) { return __fdividef(v, 1.f + __expf(-v)); }

// Which chunk of which request the gid-th chunk of the step is, worked out by one warp.
struct Where { int req, chunk; };
__device__ Where find_chunk(int gid, const int* __restrict__ req_count, int n_seqs) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int r0 = 0; r0 < n_seqs; r0 += 32) {
    const int mine = r0 + lane < n_seqs ? (req_count[r0 + lane] + C - 1) / C : 0;
    int upto = mine;  // chunks of this request and those before it in the group
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto += v;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, before + upto > gid);
    if (hit) {
      const int l = __ffs(hit) - 1;
      const int start = before + __shfl_sync(0xffffffffu, upto - mine, l);
      return {r0 + l, gid - start};
    }
    before += __shfl_sync(0xffffffffu, upto, 31);
  }
  return {-1, 0};
}

// silu of a chunk's rows: n_cols columns from `src` (rows of stride ld) into rows of `pitch` values, zeros beyond the
// chunk's `n` rows and beyond n_cols up to `pad` columns. weight(j), if given, multiplies row j before the value is split
// into hi + lo; without `lo` the value is rounded.
template <typename W>
__device__ __forceinline__ void stage_silu(const __nv_bfloat16* __restrict__ src, int ld, int n, int n_cols, int pad,
                                           __nv_bfloat16* hi, __nv_bfloat16* lo, int pitch, bool wide, W weight) {
  const int groups = pad / 8, total = C * groups;
  constexpr int U = 4;  // pieces a thread asks for before it works on the first
  for (int e0 = threadIdx.x; e0 < total; e0 += U * blockDim.x) {
    uint4 raw[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int e = e0 + u * blockDim.x, j = e / groups, c = (e % groups) * 8;
      raw[u] = make_uint4(0u, 0u, 0u, 0u);
      if (e >= total || j >= n) continue;
      const __nv_bfloat16* at = src + (size_t)j * ld + c;
      if (wide && c + 8 <= n_cols) {
        raw[u] = *reinterpret_cast<const uint4*>(at);
      } else {
        uint32_t q[4] = {0u, 0u, 0u, 0u};
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (c + k < n_cols) q[k >> 1] |= (uint32_t)__bfloat16_as_ushort(at[k]) << (16 * (k & 1));
        raw[u] = make_uint4(q[0], q[1], q[2], q[3]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int e = e0 + u * blockDim.x, j = e / groups, c = (e % groups) * 8;
      if (e >= total) break;
      const __nv_bfloat162* v2 = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
      const float wt = weight(j);
      uint4 h4, l4;
      uint32_t* hp = reinterpret_cast<uint32_t*>(&h4);
      uint32_t* lp = reinterpret_cast<uint32_t*>(&l4);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 f = __bfloat1622float2(v2[k]);
        float a = rounded(silu_(f.x)), b = rounded(silu_(f.y));
        if (lo) {
          a *= wt; b *= wt;
          const float ah = rounded(a), bh = rounded(b);
          lp[k] = pack2(a - ah, b - bh);
          a = ah; b = bh;
        }
        hp[k] = pack2(a, b);
      }
      *reinterpret_cast<uint4*>(hi + (size_t)j * pitch + c) = h4;
      if (lo) *reinterpret_cast<uint4*>(lo + (size_t)j * pitch + c) = l4;
    }
  }
}

// powers decay^0 .. decay^C by repeated multiplication, as the recurrence itself would
__device__ __forceinline__ void stage_powers(float* pw, float decay) {
  for (int t = threadIdx.x; t <= C; t += blockDim.x) {
    float p = 1.f;
    for (int i = 0; i < t; ++i) p *= decay;
    pw[t] = p;
  }
}

struct Args {
  const __nv_bfloat16* proj;  // rows of stride ld: q heads at q_col (H of d), k heads at k_col, v heads at v_col (H of dv)
  int ld, q_col, k_col, v_col;
  const float* decay;
  float* state;    // [slots, H, dv, d]
  float* chunks;   // [chunks of the step, H, dv, d]
  float* out;      // [rows, H dv]
  const int *req_row0, *req_count, *slots;
  int n_seqs, H, d, dv, wide;
};

// chunks[gid, h, c, r] = sum_j decay^(n-1-j) v_j[c] k_j[r] over the chunk's n tokens. Four warps of 16 value columns
// each; a block takes CW columns and CW key channels.
__global__ void __launch_bounds__(128)
chunk_state_kernel(const Args p) {
  __shared__ __align__(16) __nv_bfloat16 sv[C * PITCH], sk_hi[C * PITCH], sk_lo[C * PITCH];
  __shared__ float pw[C + 1];
  pdl_trigger();
  pdl_wait();
  const int gid = blockIdx.x, h = blockIdx.y, c_tiles = (p.dv + CW - 1) / CW;
  const int c0 = (blockIdx.z % c_tiles) * CW, r0 = (blockIdx.z / c_tiles) * CW;
  const Where w = find_chunk(gid, p.req_count, p.n_seqs);
  if (w.req < 0) return;
  const int left = p.req_count[w.req] - w.chunk * C, n = left < C ? left : C;
  const size_t row0 = (size_t)p.req_row0[w.req] + (size_t)w.chunk * C;
  stage_powers(pw, p.decay[h]);
  __syncthreads();
  const int nc = p.dv - c0 < CW ? p.dv - c0 : CW, nr = p.d - r0 < CW ? p.d - r0 : CW;
  stage_silu(p.proj + row0 * p.ld + p.v_col + (size_t)h * p.dv + c0, p.ld, n, nc, CW, sv, (__nv_bfloat16*)nullptr, PITCH, p.wide,
             [](int) { return 1.f; });
  stage_silu(p.proj + row0 * p.ld + p.k_col + (size_t)h * p.d + r0, p.ld, n, nr, CW, sk_hi, sk_lo, PITCH, p.wide,
             [&](int j) { return j < n ? pw[n - 1 - j] : 0.f; });
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, li = lane & 7;
  float acc[8][4];
#pragma unroll
  for (int t = 0; t < 8; ++t)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[t][k] = 0.f;
#pragma unroll
  for (int kk = 0; kk < C / 16; ++kk) {
    uint32_t a[4];
    ldsm4_t(a, sv + (kk * 16 + (mi >> 1) * 8 + li) * PITCH + warp * 16 + (mi & 1) * 8);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      uint32_t bh[4], bl[4];
      const int at = (kk * 16 + (mi & 1) * 8 + li) * PITCH + np * 16 + (mi >> 1) * 8;
      ldsm4_t(bh, sk_hi + at);
      ldsm4_t(bl, sk_lo + at);
      mma16816(acc[2 * np], a, bh[0], bh[1]);
      mma16816(acc[2 * np + 1], a, bh[2], bh[3]);
      mma16816(acc[2 * np], a, bl[0], bl[1]);
      mma16816(acc[2 * np + 1], a, bl[2], bl[3]);
    }
  }
  float* dst = p.chunks + ((size_t)gid * p.H + h) * p.dv * p.d;
  const bool pairs = (p.d & 1) == 0;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int c = c0 + warp * 16 + (lane >> 2) + half * 8;
    if (c >= p.dv) continue;
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const int r = r0 + t * 8 + (lane & 3) * 2;
      float* o = dst + (size_t)c * p.d + r;
      if (pairs && r + 1 < p.d) *reinterpret_cast<float2*>(o) = make_float2(acc[t][2 * half], acc[t][2 * half + 1]);
      else {
        if (r < p.d) o[0] = acc[t][2 * half];
        if (r + 1 < p.d) o[1] = acc[t][2 * half + 1];
      }
    }
  }
}

// Per (request, head) and element of the state: chunks[.] becomes the state before each chunk, state the one behind the
// last. V elements a thread.
template <int V>
__global__ void __launch_bounds__(128)
chunk_carry_kernel(const Args p) {
  struct alignas(4 * V) Pack { float v[V]; };
  pdl_trigger();
  pdl_wait();
  const int rq = blockIdx.z, h = blockIdx.y;
  const int slot = p.slots[rq], count = p.req_count[rq];
  if (slot < 0 || count <= 0) return;
  const int per = p.dv * p.d;
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  int first = 0;  // chunks of the requests before this one
  for (int r = threadIdx.x & 31; r < rq; r += 32) first += (p.req_count[r] + C - 1) / C;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) first += __shfl_xor_sync(0xffffffffu, first, o);
  if (e >= per) return;
  const int nc = (count + C - 1) / C;
  const float a = p.decay[h];
  float full = 1.f, last = 1.f;
  for (int i = 0; i < C; ++i) full *= a;
  for (int i = 0; i < count - (nc - 1) * C; ++i) last *= a;
  float* st = p.state + ((size_t)slot * p.H + h) * per + e;
  float* ch = p.chunks + ((size_t)first * p.H + h) * per + e;
  const size_t step = (size_t)p.H * per;
  Pack s = *reinterpret_cast<const Pack*>(st);
  constexpr int AHEAD = 16;  // chunks whose sums are asked for together
  for (int c0 = 0; c0 < nc; c0 += AHEAD) {
    Pack kv[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < nc) kv[u] = *reinterpret_cast<const Pack*>(ch + (size_t)(c0 + u) * step);
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      if (c0 + u >= nc) break;
      *reinterpret_cast<Pack*>(ch + (size_t)(c0 + u) * step) = s;
      const float f = c0 + u + 1 < nc ? full : last;
#pragma unroll
      for (int k = 0; k < V; ++k) s.v[k] = fmaf(f, s.v[k], kv[u].v[k]);
    }
  }
  *reinterpret_cast<Pack*>(st) = s;
}

// out rows of the chunk, CW value columns of head h. Eight warps: 16 tokens and half of the columns each (both halves work
// the scores of their tokens out: the blocks are bound by latency, not by products). dp: d rounded up to 16.
__global__ void __launch_bounds__(256)
chunk_output_kernel(const Args p, int dp) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float pw[C + 1];
  const int pitch = dp + 8;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(raw);
  __nv_bfloat16* sk = sq + C * pitch;
  __nv_bfloat16* sv = sk + C * pitch;
  __nv_bfloat16* ss_hi = sv + C * PITCH;
  __nv_bfloat16* ss_lo = ss_hi + CW * pitch;
  pdl_trigger();
  pdl_wait();
  const int gid = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CW;
  const Where w = find_chunk(gid, p.req_count, p.n_seqs);
  if (w.req < 0) return;
  const int left = p.req_count[w.req] - w.chunk * C, n = left < C ? left : C;
  const size_t row0 = (size_t)p.req_row0[w.req] + (size_t)w.chunk * C;
  const int nc = p.dv - c0 < CW ? p.dv - c0 : CW;
  auto one = [](int) { return 1.f; };
  stage_silu(p.proj + row0 * p.ld + p.q_col + (size_t)h * p.d, p.ld, n, p.d, dp, sq, (__nv_bfloat16*)nullptr, pitch, p.wide, one);
  stage_silu(p.proj + row0 * p.ld + p.k_col + (size_t)h * p.d, p.ld, n, p.d, dp, sk, (__nv_bfloat16*)nullptr, pitch, p.wide, one);
  stage_silu(p.proj + row0 * p.ld + p.v_col + (size_t)h * p.dv + c0, p.ld, n, nc, CW, sv, (__nv_bfloat16*)nullptr, PITCH, p.wide, one);
  {  // the state before the chunk, columns c0.., split in two
    const float* st = p.chunks + (((size_t)gid * p.H + h) * p.dv + c0) * p.d;
    const int groups = dp / 4;
    const bool wide = (p.d & 3) == 0;
    constexpr int U = 8;  // pieces a thread asks for before it splits the first
    for (int e0 = threadIdx.x; e0 < CW * groups; e0 += U * blockDim.x) {
      float4 v4[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int e = e0 + u * blockDim.x, c = e / groups, r = (e % groups) * 4;
        v4[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= nc) continue;
        const float* at = st + (size_t)c * p.d + r;
        if (wide && r + 4 <= p.d) v4[u] = *reinterpret_cast<const float4*>(at);
        else {
          if (r < p.d) v4[u].x = at[0];
          if (r + 1 < p.d) v4[u].y = at[1];
          if (r + 2 < p.d) v4[u].z = at[2];
          if (r + 3 < p.d) v4[u].w = at[3];
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int e = e0 + u * blockDim.x, c = e / groups, r = (e % groups) * 4;
        if (c >= CW) break;
        const float4 v = v4[u];
        const float h0 = rounded(v.x), h1 = rounded(v.y), h2 = rounded(v.z), h3 = rounded(v.w);
        *reinterpret_cast<uint2*>(ss_hi + (size_t)c * pitch + r) = make_uint2(pack2(h0, h1), pack2(h2, h3));
        *reinterpret_cast<uint2*>(ss_lo + (size_t)c * pitch + r) = make_uint2(pack2(v.x - h0, v.y - h1), pack2(v.z - h2, v.w - h3));
      }
    }
  }
  stage_powers(pw, p.decay[h]);
  __syncthreads();
  const int warp = (threadIdx.x >> 5) & 3, half_no = threadIdx.x >> 7, lane = threadIdx.x & 31, mi = lane >> 3, li = lane & 7;
  const int i0 = warp * 16 + (lane >> 2);  // this thread's rows: i0 and i0 + 8
  if (warp * 16 >= n) return;
  float o[4][4], s[8][4];
#pragma unroll
  for (int t = 0; t < 8; ++t)
#pragma unroll
    for (int k = 0; k < 4; ++k) { o[t & 3][k] = 0.f; s[t][k] = 0.f; }
  for (int kk = 0; kk < dp / 16; ++kk) {
    uint32_t a[4];
    ldsm4(a, sq + (warp * 16 + (mi & 1) * 8 + li) * pitch + kk * 16 + (mi >> 1) * 8);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      uint32_t b[4];
      const int at = (np * 16 + (mi >> 1) * 8 + li) * pitch + kk * 16 + (mi & 1) * 8;
      if (np < 2) {
        const int col = at + half_no * 32 * pitch;
        ldsm4(b, ss_hi + col);
        mma16816(o[(2 * np) & 3], a, b[0], b[1]);
        mma16816(o[(2 * np + 1) & 3], a, b[2], b[3]);
        ldsm4(b, ss_lo + col);
        mma16816(o[(2 * np) & 3], a, b[0], b[1]);
        mma16816(o[(2 * np + 1) & 3], a, b[2], b[3]);
      }
      if (np <= warp) {  // keys of this warp's own tokens and those before them
        ldsm4(b, sk + at);
        mma16816(s[2 * np], a, b[0], b[1]);
        mma16816(s[2 * np + 1], a, b[2], b[3]);
      }
    }
  }
  const float f0 = pw[i0 + 1], f1 = pw[i0 + 9];
#pragma unroll
  for (int t = 0; t < 4; ++t) { o[t][0] *= f0; o[t][1] *= f0; o[t][2] *= f1; o[t][3] *= f1; }
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {  // 16 keys at a time
    if (kk > warp) break;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int q = 0; q < 4; ++q) {  // the A operand's four pieces: rows i0 / i0 + 8, keys of the lower / upper eight
      const int t = 2 * kk + (q >> 1), i = i0 + (q & 1) * 8, j = t * 8 + (lane & 3) * 2;
      const float x = i >= j ? s[t][2 * (q & 1)] * pw[i - j] : 0.f;
      const float y = i >= j + 1 ? s[t][2 * (q & 1) + 1] * pw[i - j - 1] : 0.f;
      const float xh = rounded(x), yh = rounded(y);
      hi[q] = pack2(xh, yh);
      lo[q] = pack2(x - xh, y - yh);
    }
#pragma unroll
    for (int np = 0; np < 2; ++np) {
      uint32_t b[4];
      ldsm4_t(b, sv + (kk * 16 + (mi & 1) * 8 + li) * PITCH + half_no * 32 + np * 16 + (mi >> 1) * 8);
      mma16816(o[2 * np], hi, b[0], b[1]);
      mma16816(o[2 * np + 1], hi, b[2], b[3]);
      mma16816(o[2 * np], lo, b[0], b[1]);
      mma16816(o[2 * np + 1], lo, b[2], b[3]);
    }
  }
  const bool pairs = (p.dv & 1) == 0;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = i0 + half * 8;
    if (i >= n) continue;
    float* dst = p.out + (row0 + i) * p.H * p.dv + (size_t)h * p.dv;
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      const int c = c0 + half_no * 32 + t * 8 + (lane & 3) * 2;
      if (pairs && c + 1 < p.dv) *reinterpret_cast<float2*>(dst + c) = make_float2(o[t][2 * half], o[t][2 * half + 1]);
      else {
        if (c < p.dv) dst[c] = o[t][2 * half];
        if (c + 1 < p.dv) dst[c + 1] = o[t][2 * half + 1];
      }
    }
  }
}

size_t output_smem(int dp) { return ((size_t)2 * C * (dp + 8) + (size_t)C * PITCH + (size_t)2 * CW * (dp + 8)) * 2; }

}  // namespace

// Tokens of a chunk: a step needs scratch for sum over its requests of ceil(count / this) chunks of H dv d floats.
CUCA_API int cuca_lightning_chunk_tokens() { return C; }
CUCA_API int cuca_lightning_chunk_max_dim() { return MAX_DIM; }

// proj: bfloat16 rows of stride ld holding q, k, v before their activation, contiguous from col0 on (H heads of d, H
// heads of d, H heads of dv). chunks: scratch [n_chunks, H, dv, d]; n_chunks: of all requests of the step.
CUCA_API int cuca_lightning_chunked(const void* proj, int ld, int col0, const float* decay, float* state, float* chunks,
                                    float* out, const int* req_row0, const int* req_count, const int* slots, int n_seqs,
                                    int n_chunks, int H, int d, int dv, cudaStream_t stream) {
  if (n_seqs == 0 || n_chunks == 0) return 0;
  CUCA_REQUIRE(H > 0 && d > 0 && dv > 0 && d <= MAX_DIM, "lightning_chunked: bad sizes heads=%d dim=%d vdim=%d (dim <= %d)", H,
               d, dv, MAX_DIM);
  CUCA_REQUIRE(n_seqs <= 65535 && H <= 65535, "lightning_chunked: %d requests or %d heads exceed the launch limit", n_seqs, H);
  Args p;
  p.proj = (const __nv_bfloat16*)proj; p.ld = ld; p.q_col = col0; p.k_col = col0 + H * d; p.v_col = col0 + 2 * H * d;
  p.decay = decay; p.state = state; p.chunks = chunks; p.out = out;
  p.req_row0 = req_row0; p.req_count = req_count; p.slots = slots; p.n_seqs = n_seqs; p.H = H; p.d = d; p.dv = dv;
  // 16-byte loads where every head starts at a 16-byte boundary
  p.wide = ((uintptr_t)proj & 15) == 0 && ld % 8 == 0 && col0 % 8 == 0 && d % 8 == 0 && dv % 8 == 0;
  const int c_tiles = (dv + CW - 1) / CW, r_tiles = (d + CW - 1) / CW;
  cuca_launch(chunk_state_kernel, dim3(n_chunks, H, c_tiles * r_tiles), dim3(128), 0, stream, true, p);
  CUCA_CHECK_LAUNCH("lightning_chunk_state");
  const int per = dv * d;
  if (per % 4 == 0 && ((uintptr_t)chunks & 15) == 0 && ((uintptr_t)state & 15) == 0)
    cuca_launch(chunk_carry_kernel<4>, dim3((per / 4 + 127) / 128, H, n_seqs), dim3(128), 0, stream, true, p);
  else
    cuca_launch(chunk_carry_kernel<1>, dim3((per + 127) / 128, H, n_seqs), dim3(128), 0, stream, true, p);
  CUCA_CHECK_LAUNCH("lightning_chunk_carry");
  const int dp = (d + 15) / 16 * 16;
  const size_t smem = output_smem(dp);
  static size_t allowed = 0;
  if (smem > 48 * 1024 && smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(chunk_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    CUCA_REQUIRE(e == cudaSuccess, "lightning_chunked: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
    allowed = smem;
  }
  cuca_launch(chunk_output_kernel, dim3(n_chunks, H, c_tiles), dim3(256), smem, stream, true, p, dp);
  CUCA_CHECK_LAUNCH("lightning_chunk_output");
  return 0;
}
