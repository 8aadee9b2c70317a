// A routed feed-forward: every token goes to the `top` experts with the largest router logits.
//   moe_route        per token: the chosen experts (largest logit first, the lower number on a tie), their weights
//                    (a softmax of just those logits) and, optionally, the weights spread over all experts
//   moe_act_dense    a[t, e, f] = relu(u[t, e, f])^2 * weight[t, e]: all experts' up-projections at once, the ones a
//                    token did not choose weighted 0, so that one contraction over (e, f) is the weighted sum
//   moe_up_sparse / moe_down_sparse   few tokens: only the chosen experts' weights are read, a warp per output
//   moe_up_shared / moe_down_shared   the same by expert on the tensor cores, for bfloat16 tokens that share experts:
//                    each weight row is read once
//   moe_route_scored scores are a softmax over ALL router outputs; the choice goes by score + a correction per output,
//                    the weights are the chosen scores over their sum; the last outputs may stand for experts that
//                    return their input (their weights are summed per token for `moe_identity_add`)
//   moe_route_grouped  scores are sigmoids; experts form equal groups of neighbours, only those of the best groups (by
//                    the sum of a group's two largest scores) can be chosen; the weights are the chosen scores times a
//                    constant. A shared expert rides along as one more entry, weighted by the sigmoid of its own logit
//   moe_glu_dense    a[t, c] = silu(g[t, c]) u[t, c] * weight[t, expert of c]: gated experts, and behind them the
//                    columns of a shared expert that every token uses with weight 1
//   moe_glu_capped_dense  the same for capped gated units (see `capped_unit`); the shared columns have a cap and a
//                    weight per token of their own
// Routing arithmetic is 32-bit. A token's experts are summed in a fixed order, whatever else is in the batch.
#include "common.cuh"
#include <math.h>

namespace {

constexpr int MAX_TOP = 32;
constexpr int MAX_EXPERTS = 1024;

__global__ void __launch_bounds__(128)
moe_route_kernel(const float* __restrict__ logits, int T, int E, int top, int* __restrict__ idx,
                 float* __restrict__ wts, float* __restrict__ dense) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* z = logits + (size_t)t * E;
  unsigned taken = 0;  // bit j: this lane's expert lane + 32 j is chosen already
  float my_z = 0.f;    // lane j keeps the j-th chosen logit
  int my_e = 0;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int k = 0; lane + 32 * k < E; ++k) {
      const int e = lane + 32 * k;
      float v = z[e];
      v = v == v ? v : -INFINITY;  // a row of padding may hold anything: every lane must still see one order
      if (!((taken >> k) & 1u) && (v > best || (v == best && e < be) || be == 0x7fffffff)) { best = v; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > best || (ov == best && oe < be))) { best = ov; be = oe; }
    }
    if (be < E && (be & 31) == lane) taken |= 1u << (be >> 5);
    if (lane == j) { my_z = best; my_e = be < E ? be : 0; }
  }
  const float zmax = __shfl_sync(0xffffffffu, my_z, 0);
  const float p = lane < top ? expf(my_z - zmax) : 0.f;
  const float w = p / warp_sum(p);
  if (dense)
    for (int e = lane; e < E; e += 32) dense[(size_t)t * E + e] = 0.f;
  __syncwarp();
  if (lane < top) {
    idx[(size_t)t * top + lane] = my_e;
    wts[(size_t)t * top + lane] = w;
    if (dense) dense[(size_t)t * E + my_e] = w;
  }
}

template <typename T>
__global__ void moe_act_dense_kernel(const T* __restrict__ u, const float* __restrict__ dense, T* __restrict__ a,
                                     size_t n, int E, int F) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / ((size_t)E * F);
    const int e = (int)((i / F) % E);
    const float w = dense[t * E + e];
    const float v = fmaxf(to_f32(u[i]), 0.f);
    a[i] = from_f32<T>(w == 0.f ? 0.f : v * v * w);
  }
}

// Scores over all E router outputs; `top` chosen by score + correction (the lower number on a tie); weights
// s / (sum of the chosen s + 1e-20). Outputs from n_real on are identity experts: their chosen weights are summed in
// ident[t]. A warp per token; lane l holds outputs l, l + 32, ...
__global__ void __launch_bounds__(128)
moe_route_scored_kernel(const float* __restrict__ logits, const float* __restrict__ correction, int T, int E, int n_real,
                        int top, int* __restrict__ idx, float* __restrict__ wts, float* __restrict__ dense,
                        float* __restrict__ ident) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* z = logits + (size_t)t * E;
  float zmax = -INFINITY;
  for (int e = lane; e < E; e += 32) {
    const float v = z[e];
    zmax = fmaxf(zmax, v == v ? v : -INFINITY);
  }
  zmax = warp_max(zmax);
  if (zmax == -INFINITY) zmax = 0.f;  // a row of padding may hold anything
  float total = 0.f;
  for (int e = lane; e < E; e += 32) {
    const float v = z[e];
    total += v == v ? expf(v - zmax) : 0.f;
  }
  total = warp_sum(total);
  const float inv_total = total > 0.f ? 1.f / total : 0.f;
  unsigned taken = 0;
  float my_s = 0.f;
  int my_e = 0;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY, best_s = 0.f;
    int be = 0x7fffffff;
    for (int k = 0; lane + 32 * k < E; ++k) {
      const int e = lane + 32 * k;
      const float v = z[e];
      const float sc = v == v ? expf(v - zmax) * inv_total : 0.f;
      float c = sc + (correction ? correction[e] : 0.f);
      c = c == c ? c : -INFINITY;
      if (!((taken >> k) & 1u) && (c > best || (c == best && e < be) || be == 0x7fffffff)) { best = c; be = e; best_s = sc; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const float os = __shfl_xor_sync(0xffffffffu, best_s, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > best || (ov == best && oe < be))) { best = ov; be = oe; best_s = os; }
    }
    if (be < E && (be & 31) == lane) taken |= 1u << (be >> 5);
    if (lane == j) { my_s = best_s; my_e = be < E ? be : 0; }
  }
  const float chosen = warp_sum(lane < top ? my_s : 0.f);
  const float w = my_s / (chosen + 1e-20f);
  const float iw = warp_sum(lane < top && my_e >= n_real ? w : 0.f);
  if (dense)
    for (int e = lane; e < E; e += 32) dense[(size_t)t * E + e] = 0.f;
  __syncwarp();
  if (lane < top) {
    idx[(size_t)t * top + lane] = my_e;
    wts[(size_t)t * top + lane] = w;
    if (dense) dense[(size_t)t * E + my_e] = w;
  }
  if (ident && lane == 0) ident[t] = iw;
}

// The capped gated unit: g = min(gate, limit), u = clamp(up, -limit, limit), g sigmoid(alpha g) (u + 1).
__device__ __forceinline__ float capped_unit(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

// Scores s = sigmoid(z) of E experts in `groups` equal groups of neighbours. A group's score is the sum of its two
// largest (of its one, where it has one); the `keep` best groups' experts can be chosen, the `top` largest of them are
// (the lower number on a tie), with weights s * scale. Column E of a row of logits, where has_shared, belongs to a shared
// expert that every token uses, with weight sigmoid(z): it becomes entry `top` of idx / wts (number E) and column E of
// dense. One warp; lane l holds experts l, l + 32, ...; z: the token's logits, gs: shared memory for a score per group.
__device__ void route_grouped(const float* z, float* gs, int t, int lane, int E, int groups, int keep, int top, float scale,
                              int has_shared, int* __restrict__ idx, float* __restrict__ wts, float* __restrict__ dense) {
  const int n_out = E + (has_shared ? 1 : 0), entries = top + (has_shared ? 1 : 0);
  auto score = [&](int e) {  // (a row of padding may hold anything: every lane must still see one order)
    const float v = z[e];
    return v == v ? 1.f / (1.f + expf(-v)) : -1.f;
  };
  unsigned open = 0xffffffffu;  // bit k: this lane's expert lane + 32 k can be chosen
  if (groups > 1 && keep < groups) {
    const int size = E / groups;
    if (size <= 32) {  // a lane per group
      for (int g = lane; g < groups; g += 32) {
        float a = -INFINITY, b = -INFINITY;
        for (int i = 0; i < size; ++i) {
          const float v = score(g * size + i);
          if (v > a) { b = a; a = v; } else if (v > b) b = v;
        }
        gs[g] = size > 1 ? a + b : a;
      }
    } else {  // few large groups: the warp's lanes share each
      for (int g = 0; g < groups; ++g) {
        float a = -INFINITY, b = -INFINITY;
        for (int i = lane; i < size; i += 32) {
          const float v = score(g * size + i);
          if (v > a) { b = a; a = v; } else if (v > b) b = v;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
          const float hi = fmaxf(a, oa), lo = fminf(a, oa);
          b = fmaxf(lo, fmaxf(b, ob));
          a = hi;
        }
        if (lane == 0) gs[g] = a + b;
      }
    }
    __syncwarp();
    open = 0;
    for (int k = 0; lane + 32 * k < E; ++k) {  // an expert is open if fewer than `keep` groups come before its own
      const int g = (lane + 32 * k) / size;
      const float mine = gs[g];
      int before = 0;
      for (int i = 0; i < groups; ++i) before += (gs[i] > mine || (gs[i] == mine && i < g)) ? 1 : 0;
      if (before < keep) open |= 1u << k;
    }
  }
  float my_s = 0.f;
  int my_e = 0;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int k = 0; lane + 32 * k < E; ++k) {
      if (!((open >> k) & 1u)) continue;
      const int e = lane + 32 * k;
      const float v = score(e);
      if (v > best || be == 0x7fffffff) { best = v; be = e; }  // (ascending numbers: the first of equals stays)
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > best || (ov == best && oe < be))) { best = ov; be = oe; }
    }
    if (be < E && (be & 31) == lane) open &= ~(1u << (be >> 5));
    if (lane == j) { my_s = best; my_e = be < E ? be : 0; }
  }
  const float w = my_s * scale;
  if (dense)
    for (int e = lane; e < n_out; e += 32) dense[(size_t)t * n_out + e] = 0.f;
  __syncwarp();
  if (lane < top) {
    idx[(size_t)t * entries + lane] = my_e;
    wts[(size_t)t * entries + lane] = w;
    if (dense) dense[(size_t)t * n_out + my_e] = w;
  }
  if (has_shared && lane == 0) {
    const float sw = 1.f / (1.f + expf(-z[E]));
    idx[(size_t)t * entries + top] = E;
    wts[(size_t)t * entries + top] = sw;
    if (dense) dense[(size_t)t * n_out + E] = sw;
  }
}

__global__ void __launch_bounds__(128)
moe_route_grouped_kernel(const float* __restrict__ logits, int T, int E, int groups, int keep, int top, float scale,
                         int has_shared, int* __restrict__ idx, float* __restrict__ wts, float* __restrict__ dense) {
  __shared__ float group_score[4][MAX_EXPERTS];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, t = blockIdx.x * 4 + warp;
  if (t >= T) return;
  route_grouped(logits + (size_t)t * (E + (has_shared ? 1 : 0)), group_score[warp], t, threadIdx.x & 31, E, groups, keep, top,
                scale, has_shared, idx, wts, dense);
}

// gu: [T, 2 C] (gates, then ups); a[t, c] = capped_unit(g, u) w; c < EF: expert c / F's columns, w = dense[t, c / F] and
// cap `limit`; behind: the shared expert's, w = dense[t, EF / F] and cap `limit_s`. V values a thread (16 bytes), or 1.
template <typename T, int V>
__global__ void __launch_bounds__(256)
moe_glu_capped_dense_kernel(const T* __restrict__ gu, const float* __restrict__ dense, int ld_dense, T* __restrict__ a,
                            size_t n_vec, int C, int EF, int F, float limit, float limit_s, float alpha) {
  pdl_trigger();
  pdl_wait();
  const int cv = C / V;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n_vec; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / cv;
    const int c = (int)(i % cv) * V;
    const bool shared = c >= EF;
    const float w = dense[t * ld_dense + (shared ? EF / F : c / F)];
    const float lim = shared ? limit_s : limit;
    const T* gp = gu + t * 2 * C + c;
    if (V == 1) {
      a[t * C + c] = from_f32<T>(w == 0.f ? 0.f : capped_unit(to_f32(gp[0]), to_f32(gp[C]), lim, alpha) * w);
      continue;
    }
    uint4 out4 = make_uint4(0u, 0u, 0u, 0u);
    if (w != 0.f) {  // (an expert the token did not choose: its rows are not read)
      const uint4 g4 = *reinterpret_cast<const uint4*>(gp), u4 = *reinterpret_cast<const uint4*>(gp + C);
      const T* g = reinterpret_cast<const T*>(&g4);
      const T* u = reinterpret_cast<const T*>(&u4);
      T* o = reinterpret_cast<T*>(&out4);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = from_f32<T>(capped_unit(to_f32(g[e]), to_f32(u[e]), lim, alpha) * w);
    }
    *reinterpret_cast<uint4*>(a + t * C + c) = out4;
  }
}

// gu: [T, 2 C] (gates, then ups); a[t, c] = silu(g) u w with w = dense[t, c / F] for c < EF (ld_dense outputs a row),
// 1 for the columns behind (a shared expert).
template <typename T>
__global__ void moe_glu_dense_kernel(const T* __restrict__ gu, const float* __restrict__ dense, int ld_dense,
                                     T* __restrict__ a, size_t n, int C, int EF, int F) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / C;
    const int c = (int)(i % C);
    const float w = c < EF ? dense[t * ld_dense + c / F] : 1.f;
    const float g = to_f32(gu[t * 2 * C + c]), u = to_f32(gu[t * 2 * C + C + c]);
    a[i] = from_f32<T>(w == 0.f ? 0.f : g / (1.f + expf(-g)) * u * w);
  }
}

// The same, 16 bytes a thread (V values of one expert: F, EF and C are multiples of V).
template <typename T, int V>
__global__ void moe_glu_dense_vec_kernel(const T* __restrict__ gu, const float* __restrict__ dense, int ld_dense,
                                         T* __restrict__ a, size_t n_vec, int C, int EF, int F) {
  pdl_trigger();
  pdl_wait();
  const int cv = C / V;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n_vec; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / cv;
    const int c = (int)(i % cv) * V;
    const float w = c < EF ? dense[t * ld_dense + c / F] : 1.f;
    uint4 out4 = make_uint4(0u, 0u, 0u, 0u);
    if (w != 0.f) {  // (an expert the token did not choose: its rows are not read)
      const uint4 g4 = *reinterpret_cast<const uint4*>(gu + t * 2 * C + c);
      const uint4 u4 = *reinterpret_cast<const uint4*>(gu + t * 2 * C + C + c);
      const T* g = reinterpret_cast<const T*>(&g4);
      const T* u = reinterpret_cast<const T*>(&u4);
      T* o = reinterpret_cast<T*>(&out4);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float gv = to_f32(g[e]);
        o[e] = from_f32<T>(gv / (1.f + expf(-gv)) * to_f32(u[e]) * w);
      }
    }
    *reinterpret_cast<uint4*>(a + t * C + c) = out4;
  }
}

// y[t] (+)= ident[t] * h[t]: the experts that return their input.
template <typename T>
__global__ void moe_identity_add_kernel(float* __restrict__ y, const T* __restrict__ h, const float* __restrict__ ident,
                                        int store, size_t n, int N) {
  pdl_trigger();
  pdl_wait();
  if ((N & 3) == 0 && ((uintptr_t)y & 15) == 0) {  // four values a thread
    const size_t n4 = n / 4;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (size_t)gridDim.x * blockDim.x) {
      const float w = ident[(i * 4) / N];
      float4 v = store ? make_float4(0.f, 0.f, 0.f, 0.f) : reinterpret_cast<const float4*>(y)[i];
      const T* hv = h + i * 4;
      v.x += w * to_f32(hv[0]); v.y += w * to_f32(hv[1]); v.z += w * to_f32(hv[2]); v.w += w * to_f32(hv[3]);
      reinterpret_cast<float4*>(y)[i] = v;
    }
    return;
  }
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const float v = ident[i / N] * to_f32(h[i]);
    y[i] = store ? v : y[i] + v;
  }
}

// A warp's dot product of two rows of n values: 16 bytes a lane at a time where the rows allow it.
__device__ __forceinline__ float warp_dot(const float* w, const float* x, int n, int lane) {
  float acc = 0.f;
  for (int i = lane; i < n; i += 32) acc = fmaf(w[i], x[i], acc);
  return warp_sum(acc);
}
__device__ __forceinline__ float warp_dot(const __nv_bfloat16* w, const __nv_bfloat16* x, int n, int lane) {
  float acc = 0.f;
  if (n % 8 == 0 && ((((uintptr_t)w) | ((uintptr_t)x)) & 15) == 0) {
    for (int i = lane * 8; i < n; i += 256) {
      const uint4 a = *reinterpret_cast<const uint4*>(w + i), b = *reinterpret_cast<const uint4*>(x + i);
      const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&a);
      const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&b);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 fa = __bfloat1622float2(pa[k]), fb = __bfloat1622float2(pb[k]);
        acc = fmaf(fa.x, fb.x, acc);
        acc = fmaf(fa.y, fb.y, acc);
      }
    }
  } else {
    for (int i = lane; i < n; i += 32) acc = fmaf(__bfloat162float(w[i]), __bfloat162float(x[i]), acc);
  }
  return warp_sum(acc);
}

// What a sparse launch's experts compute. ACT 0: relu(up)^2; 1: silu(gate) up; 2: `capped_unit`.
struct SparseUnit {
  float limit, limit_s, alpha;  // ACT 2: the caps of the experts and of the shared expert
};

// Few tokens and few experts: the router's logits (32-bit sums) and the choice in one launch, a block per token.
constexpr int ROUTER_MAX_OUTPUTS = 64;
template <typename T>
__global__ void __launch_bounds__(512)
moe_router_grouped_kernel(const T* __restrict__ h, const T* __restrict__ w, int K, int E, int groups, int keep, int top,
                          float scale, int has_shared, int* __restrict__ idx, float* __restrict__ wts) {
  __shared__ float z[ROUTER_MAX_OUTPUTS], group_score[ROUTER_MAX_OUTPUTS];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_out = E + (has_shared ? 1 : 0);
  for (int e = warp; e < n_out; e += 16) {
    const float v = warp_dot(w + (size_t)e * K, h + (size_t)t * K, K, lane);
    if (lane == 0) z[e] = v;
  }
  __syncthreads();
  if (warp == 0) route_grouped(z, group_score, t, lane, E, groups, keep, top, scale, has_shared, idx, wts, nullptr);
}

// a[pair, f] = act(W[e(pair)] . h[t]) * weight(pair); pair = t * entries + j. ACT 0: W_up [E F, K]. ACT 1 and 2: w_up
// holds every expert's gate rows and, `up_rows` rows further on, its up rows. Entry number n_real is the shared expert
// where Fs > 0: its Fs rows follow the experts'. Any other number from n_real on has no weights (such an expert
// returns its input): nothing is written for it. Rows of a are lda values.
template <typename T, int ACT>
__global__ void __launch_bounds__(256)
moe_up_sparse_kernel(const T* __restrict__ h, const T* __restrict__ w_up, const int* __restrict__ idx,
                     const float* __restrict__ wts, T* __restrict__ a, int lda, int entries, int F, int Fs, int K,
                     int n_real, size_t up_rows, const SparseUnit unit) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.y, f = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int e = idx[pair];
  if (f >= (e < n_real ? F : (e == n_real ? Fs : 0))) return;
  const T* wr = w_up + ((size_t)e * F + f) * K;
  const T* hr = h + (size_t)(pair / entries) * K;
  float v;
  if (ACT == 0) {
    v = fmaxf(warp_dot(wr, hr, K, lane), 0.f);
    v = v * v;
  } else {
    const float g = warp_dot(wr, hr, K, lane), u = warp_dot(wr + up_rows * K, hr, K, lane);
    v = ACT == 1 ? g / (1.f + expf(-g)) * u : capped_unit(g, u, e == n_real ? unit.limit_s : unit.limit, unit.alpha);
  }
  if (lane == 0) a[(size_t)pair * lda + f] = from_f32<T>(v * wts[pair]);
}

// y[t, o] (+)= sum_j W_down[o, e(t, j) F ..] . a[t * entries + j]; W_down: [N, ld] (ld columns a row)
template <typename T>
__global__ void __launch_bounds__(256)
moe_down_sparse_kernel(const T* __restrict__ a, int lda, const T* __restrict__ w_down, const int* __restrict__ idx,
                       float* __restrict__ y, int store, int entries, int F, int Fs, int ld, int N, int n_real) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.y, o = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (o >= N) return;
  float acc = 0.f;
  for (int j = 0; j < entries; ++j) {
    const int e = idx[(size_t)t * entries + j];
    const int n = e < n_real ? F : (e == n_real ? Fs : 0);
    if (n == 0) continue;
    const T* wr = w_down + (size_t)o * ld + (size_t)e * F;
    const T* ar = a + ((size_t)t * entries + j) * lda;
    acc += warp_dot(wr, ar, n, lane);
  }
  if (lane == 0) y[(size_t)t * N + o] = store ? acc : y[(size_t)t * N + o] + acc;
}

// ---- the same for a few bfloat16 tokens that share experts: an expert's rows are read once, straight into tensor-core
// operands, for up to sixteen tokens that chose it. The order of k within a product is free as long as both operands
// agree: a lane takes eight consecutive values (16 bytes) of its weight row and of its token, and they serve as its
// operands of two 16-wide steps.
constexpr int SHARED_MAX_TOKENS = 32, SHARED_MAX_EXPERTS = 64, SHARED_TILE = 16, SHARED_K = 32;

__device__ __forceinline__ void mma_tokens(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                           uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// d[token, row] += 32 values of tokens (lo: tokens 0..7, hi: 8..15) times 32 values of weight rows
__device__ __forceinline__ void mma_k32(float (&d)[4], const uint4& lo, const uint4& hi, const uint4& w) {
  mma_tokens(d, lo.x, hi.x, lo.y, hi.y, w.x, w.y);
  mma_tokens(d, lo.z, hi.z, lo.w, hi.w, w.z, w.w);
}
__device__ __forceinline__ uint4 load16(const __nv_bfloat16* p, bool on) {
  return on ? *reinterpret_cast<const uint4*>(p) : make_uint4(0u, 0u, 0u, 0u);
}

// Block (x, e, z): eight rows f of expert e for the sixteen of its tokens from number 16 z on; the eight warps take K's runs
// of 32 in turn and their sums are added in order. Arguments as in `moe_up_sparse_kernel`; K, F and Fs are multiples of
// 32. (Tokens of a batch may all choose the same two experts: what is in flight must not hang on their number.)
template <int ACT>
__global__ void __launch_bounds__(256)
moe_up_shared_kernel(const __nv_bfloat16* __restrict__ h, const __nv_bfloat16* __restrict__ w_up, const int* __restrict__ idx,
                     const float* __restrict__ wts, __nv_bfloat16* __restrict__ a, int lda, int n_tokens, int entries, int F,
                     int Fs, int K, int n_real, size_t up_rows, const SparseUnit unit) {
  __shared__ int pair_of[SHARED_MAX_TOKENS];
  __shared__ int members[SHARED_MAX_TOKENS];
  __shared__ int n_members;
  __shared__ float sums[ACT == 0 ? 1 : 2][8][SHARED_TILE * 8];
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < SHARED_MAX_TOKENS) pair_of[threadIdx.x] = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < n_tokens * entries; i += blockDim.x)
    if (idx[i] == e) pair_of[i / entries] = i;
  __syncthreads();
  if (warp == 0) {
    const int mine = pair_of[lane];
    const unsigned who = __ballot_sync(0xffffffffu, mine >= 0);
    if (mine >= 0) members[__popc(who & ((1u << lane) - 1u))] = mine;
    if (lane == 0) n_members = __popc(who);
  }
  __syncthreads();
  const int count = n_members - (int)blockIdx.z * SHARED_TILE, f0 = blockIdx.x * 8;
  if (count <= 0 || f0 >= (e < n_real ? F : Fs)) return;
  const int* mem = members + blockIdx.z * SHARED_TILE;
  const int g = lane >> 2, q = lane & 3;
  const __nv_bfloat16* wg = w_up + ((size_t)e * F + f0 + g) * K + q * 8;
  const __nv_bfloat16* wu = wg + up_rows * K;
  const bool on0 = g < count, on1 = g + 8 < count;
  const __nv_bfloat16* h0 = h + (size_t)(on0 ? mem[g] / entries : 0) * K + q * 8;
  const __nv_bfloat16* h1 = h + (size_t)(on1 ? mem[g + 8] / entries : 0) * K + q * 8;
  float dg[4] = {0.f, 0.f, 0.f, 0.f}, du[4] = {0.f, 0.f, 0.f, 0.f};
  constexpr int U = 4;  // runs asked for together
  for (int k0 = warp * SHARED_K; k0 < K; k0 += U * 8 * SHARED_K) {
    uint4 xg[U], xu[U], lo[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = k0 + u * 8 * SHARED_K;
      xg[u] = load16(wg + k, k < K);
      if (ACT != 0) xu[u] = load16(wu + k, k < K);
      lo[u] = load16(h0 + k, k < K && on0);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = k0 + u * 8 * SHARED_K;
      const uint4 hi = load16(h1 + k, k < K && on1);
      mma_k32(dg, lo[u], hi, xg[u]);
      if (ACT != 0) mma_k32(du, lo[u], hi, xu[u]);
    }
  }
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    const int at = (g + (c >> 1) * 8) * 8 + q * 2 + (c & 1);
    sums[0][warp][at] = dg[c];
    if (ACT != 0) sums[ACT == 0 ? 0 : 1][warp][at] = du[c];
  }
  __syncthreads();
  const int m = threadIdx.x >> 3;
  if (m >= SHARED_TILE || m >= count) return;
  float x = 0.f, y = 0.f;
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    x += sums[0][k][threadIdx.x];
    if (ACT != 0) y += sums[ACT == 0 ? 0 : 1][k][threadIdx.x];
  }
  float v;
  if (ACT == 0) { v = fmaxf(x, 0.f); v = v * v; }
  else if (ACT == 1) v = x / (1.f + expf(-x)) * y;
  else v = capped_unit(x, y, e == n_real ? unit.limit_s : unit.limit, unit.alpha);
  const int pair = mem[m];
  a[(size_t)pair * lda + f0 + (threadIdx.x & 7)] = __float2bfloat16_rn(v * wts[pair]);
}

// Block (x, y): eight output columns for the sixteen tokens from 16 y on. W_down's columns are dealt to the eight warps in
// runs of 32 by their place in the row (so a token's sum does not depend on which experts others chose); a chosen
// expert's columns are read once. The warps' sums are added in order.
__global__ void __launch_bounds__(256)
moe_down_shared_kernel(const __nv_bfloat16* __restrict__ a, int lda, const __nv_bfloat16* __restrict__ w_down,
                       const int* __restrict__ idx, float* __restrict__ y, int store, int n_tokens, int entries, int F, int Fs,
                       int ld, int N, int n_real) {
  __shared__ short pair_of[SHARED_MAX_EXPERTS][SHARED_TILE];
  __shared__ int chosen[SHARED_MAX_EXPERTS];
  __shared__ float sums[8][SHARED_TILE * 8];
  pdl_trigger();
  pdl_wait();
  const int t0 = blockIdx.y * SHARED_TILE, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nt = n_tokens - t0 < SHARED_TILE ? n_tokens - t0 : SHARED_TILE;
  const int n_experts = n_real + (Fs > 0 ? 1 : 0);
  for (int i = threadIdx.x; i < n_experts * SHARED_TILE; i += blockDim.x) pair_of[i / SHARED_TILE][i % SHARED_TILE] = -1;
  for (int i = threadIdx.x; i < n_experts; i += blockDim.x) chosen[i] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < nt * entries; i += blockDim.x) {
    const int e = idx[t0 * entries + i];
    if (e < n_experts) { pair_of[e][i / entries] = (short)(t0 * entries + i); chosen[e] = 1; }
  }
  __syncthreads();
  const int g = lane >> 2, q = lane & 3, o0 = blockIdx.x * 8;
  const int row = o0 + g < N ? o0 + g : N - 1;  // (rows past the last are not stored)
  float d[4] = {0.f, 0.f, 0.f, 0.f};
  for (int e = 0; e < n_experts; ++e) {
    if (!chosen[e]) continue;
    const int n = e < n_real ? F : Fs, first = (e * F / SHARED_K) & 7;  // the warp that has the expert's first run
    const __nv_bfloat16* wr = w_down + (size_t)row * ld + (size_t)e * F + q * 8;
    const int p0 = pair_of[e][g], p1 = pair_of[e][g + 8];
    const __nv_bfloat16* a0 = a + (size_t)(p0 < 0 ? 0 : p0) * lda + q * 8;
    const __nv_bfloat16* a1 = a + (size_t)(p1 < 0 ? 0 : p1) * lda + q * 8;
    constexpr int U = 8;  // runs asked for together
    for (int k0 = ((warp - first) & 7) * SHARED_K; k0 < n; k0 += U * 8 * SHARED_K) {
      uint4 x[U], lo[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = k0 + u * 8 * SHARED_K;
        x[u] = load16(wr + k, k < n);
        lo[u] = load16(a0 + k, k < n && p0 >= 0);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = k0 + u * 8 * SHARED_K;
        mma_k32(d, lo[u], load16(a1 + k, k < n && p1 >= 0), x[u]);
      }
    }
  }
#pragma unroll
  for (int c = 0; c < 4; ++c) sums[warp][(g + (c >> 1) * 8) * 8 + q * 2 + (c & 1)] = d[c];
  __syncthreads();
  if (threadIdx.x < SHARED_TILE * 8) {
    const int t = threadIdx.x >> 3, o = o0 + (threadIdx.x & 7);
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) v += sums[k][threadIdx.x];
    if (t < nt && o < N) {
      float* at = y + (size_t)(t0 + t) * N + o;
      *at = store ? v : *at + v;
    }
  }
}

}  // namespace

CUCA_API int cuca_moe_max_experts() { return MAX_EXPERTS; }

CUCA_API int cuca_moe_route(const float* logits, int T, int E, int top, int* idx, float* wts, float* dense,
                            cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(E >= 1 && E <= MAX_EXPERTS && top >= 1 && top <= E && top <= MAX_TOP,
               "moe_route: %d of %d experts is outside what the kernel takes (experts <= %d, chosen <= %d)", top, E,
               MAX_EXPERTS, MAX_TOP);
  cuca_launch(moe_route_kernel, dim3((T + 3) / 4), dim3(128), 0, stream, true, logits, T, E, top, idx, wts, dense);
  CUCA_CHECK_LAUNCH("moe_route");
  return 0;
}

CUCA_API int cuca_moe_act_dense(const void* u, const float* dense, void* a, int dtype, int T, int E, int F,
                                cudaStream_t stream) {
  if (T == 0) return 0;
  const size_t n = (size_t)T * E * F;
  size_t blocks = (n + 255) / 256;
  blocks = blocks > 8192 ? 8192 : blocks;
  if (dtype == CUCA_F32)
    cuca_launch(moe_act_dense_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const float*)u, dense,
                (float*)a, n, E, F);
  else if (dtype == CUCA_BF16)
    cuca_launch(moe_act_dense_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (const __nv_bfloat16*)u, dense, (__nv_bfloat16*)a, n, E, F);
  else
    CUCA_REQUIRE(false, "moe_act_dense: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("moe_act_dense");
  return 0;
}

// act 0: relu(up)^2 experts, w_up [E F, K], w_down [N, E F]. act 1 (silu-gated) and 2 (capped units): w_up [2 C, K] (every
// expert's gate rows, then C rows on every expert's up rows), w_down [N, C]; C >= E F. `entries` idx / wts a token. Fs > 0:
// number E is a shared expert of Fs rows behind the experts' (with cap limit_s); numbers beyond (with Fs = 0: from E
// on) are skipped. a: [T * entries, lda], lda >= max(F, Fs).
CUCA_API int cuca_moe_sparse_act(const void* h, const void* w_up, const void* w_down, const int* idx, const float* wts,
                                 void* a, int lda, float* y, int store, int dtype, int T, int entries, int E, int F,
                                 int Fs, int K, int N, int act, int C, float limit, float limit_s, float alpha,
                                 cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(T * entries <= 65535 && T <= 65535, "moe_sparse: %d tokens exceed the launch limit", T);
  const int ld = act ? C : E * F, wide = F > Fs ? F : Fs;
  CUCA_REQUIRE(ld >= E * F + Fs, "moe_sparse: %d columns do not hold %d experts of %d and a shared one of %d", ld, E, F, Fs);
  CUCA_REQUIRE(lda >= wide, "moe_sparse: rows of %d values do not hold %d", lda, wide);
  CUCA_REQUIRE(act >= 0 && act <= 2, "moe_sparse: unknown activation %d", act);
  const SparseUnit unit = {limit, limit_s, alpha};
  const int n_experts = E + (Fs > 0 ? 1 : 0);
  // bfloat16 tokens that may share experts, and sizes the tensor cores take: by expert, each weight row read once
  auto even = [&](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (dtype == CUCA_BF16 && T >= 2 && T <= SHARED_MAX_TOKENS && n_experts <= SHARED_MAX_EXPERTS && even(h) && even(w_up) &&
      even(w_down) && even(a) && K % SHARED_K == 0 && F % SHARED_K == 0 && Fs % SHARED_K == 0 && lda % 8 == 0 && ld % 8 == 0) {
    const int tiles = (T + SHARED_TILE - 1) / SHARED_TILE;
    const dim3 grid(wide / 8, n_experts, tiles);
#define UPS(ACT)                                                                                                    \
  cuca_launch(moe_up_shared_kernel<ACT>, grid, dim3(256), 0, stream, true, (const __nv_bfloat16*)h,                 \
              (const __nv_bfloat16*)w_up, idx, wts, (__nv_bfloat16*)a, lda, T, entries, F, Fs, K, E, (size_t)C, unit)
    if (act == 0) UPS(0);
    else if (act == 1) UPS(1);
    else UPS(2);
#undef UPS
    CUCA_CHECK_LAUNCH("moe_up_shared");
    cuca_launch(moe_down_shared_kernel, dim3((N + 7) / 8, tiles), dim3(256), 0, stream, true, (const __nv_bfloat16*)a, lda,
                (const __nv_bfloat16*)w_down, idx, y, store, T, entries, F, Fs, ld, N, E);
    CUCA_CHECK_LAUNCH("moe_down_shared");
    return 0;
  }
#define UP(TT, ACT)                                                                                                 \
  cuca_launch(moe_up_sparse_kernel<TT, ACT>, dim3((wide + 7) / 8, T * entries), dim3(256), 0, stream, true,         \
              (const TT*)h, (const TT*)w_up, idx, wts, (TT*)a, lda, entries, F, Fs, K, E, (size_t)C, unit)
#define SPARSE(TT)                                                                                                  \
  do {                                                                                                              \
    if (act == 0) UP(TT, 0);                                                                                        \
    else if (act == 1) UP(TT, 1);                                                                                   \
    else UP(TT, 2);                                                                                                 \
    CUCA_CHECK_LAUNCH("moe_up_sparse");                                                                             \
    cuca_launch(moe_down_sparse_kernel<TT>, dim3((N + 7) / 8, T), dim3(256), 0, stream, true, (const TT*)a, lda,    \
                (const TT*)w_down, idx, y, store, entries, F, Fs, ld, N, E);                                        \
  } while (0)
  if (dtype == CUCA_F32) SPARSE(float);
  else if (dtype == CUCA_BF16) SPARSE(__nv_bfloat16);
  else CUCA_REQUIRE(false, "moe_sparse: unknown dtype %d", dtype);
#undef SPARSE
#undef UP
  CUCA_CHECK_LAUNCH("moe_down_sparse");
  return 0;
}

// The same without a shared expert: glu 0: relu(up)^2 experts, 1: silu-gated ones.
CUCA_API int cuca_moe_sparse(const void* h, const void* w_up, const void* w_down, const int* idx, const float* wts,
                             void* a, float* y, int store, int dtype, int T, int top, int E, int F, int K, int N,
                             int glu, int C, cudaStream_t stream) {
  return cuca_moe_sparse_act(h, w_up, w_down, idx, wts, a, F, y, store, dtype, T, top, E, F, 0, K, N, glu ? 1 : 0, C, 0.f,
                             0.f, 0.f, stream);
}

// logits: [T, E + 1] with has_shared (the last column the shared expert's), else [T, E]; idx, wts: [T, top + 1] or
// [T, top]; dense (or null): as wide as the logits.
CUCA_API int cuca_moe_route_grouped(const float* logits, int T, int E, int groups, int keep, int top, float scale,
                                    int has_shared, int* idx, float* wts, float* dense, cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(E >= 1 && E <= MAX_EXPERTS && top >= 1 && top <= MAX_TOP,
               "moe_route: %d of %d experts is outside what the kernel takes (experts <= %d, chosen <= %d)", top, E,
               MAX_EXPERTS, MAX_TOP);
  CUCA_REQUIRE(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && top <= keep * (E / groups),
               "moe_route: %d of the %d experts in %d of %d groups cannot be chosen", top, E, keep, groups);
  cuca_launch(moe_route_grouped_kernel, dim3((T + 3) / 4), dim3(128), 0, stream, true, logits, T, E, groups, keep, top,
              scale, has_shared, idx, wts, dense);
  CUCA_CHECK_LAUNCH("moe_route_grouped");
  return 0;
}

// The same from the activations: h [T, K], router weights w [E (+ 1), K] of one dtype; up to 64 outputs.
CUCA_API int cuca_moe_router_grouped(const void* h, const void* w, int dtype, int T, int K, int E, int groups, int keep,
                                     int top, float scale, int has_shared, int* idx, float* wts, cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(E >= 1 && E + (has_shared ? 1 : 0) <= ROUTER_MAX_OUTPUTS && top >= 1 && top <= MAX_TOP,
               "moe_router: %d of %d experts is outside what the kernel takes (outputs <= %d, chosen <= %d)", top, E,
               ROUTER_MAX_OUTPUTS, MAX_TOP);
  CUCA_REQUIRE(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && top <= keep * (E / groups),
               "moe_router: %d of the %d experts in %d of %d groups cannot be chosen", top, E, keep, groups);
  if (dtype == CUCA_F32)
    cuca_launch(moe_router_grouped_kernel<float>, dim3(T), dim3(512), 0, stream, true, (const float*)h, (const float*)w, K, E,
                groups, keep, top, scale, has_shared, idx, wts);
  else if (dtype == CUCA_BF16)
    cuca_launch(moe_router_grouped_kernel<__nv_bfloat16>, dim3(T), dim3(512), 0, stream, true, (const __nv_bfloat16*)h,
                (const __nv_bfloat16*)w, K, E, groups, keep, top, scale, has_shared, idx, wts);
  else
    CUCA_REQUIRE(false, "moe_router: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("moe_router_grouped");
  return 0;
}

CUCA_API int cuca_moe_glu_capped_dense(const void* gu, const float* dense, int ld_dense, void* a, int dtype, int T, int C,
                                       int EF, int F, float limit, float limit_s, float alpha, cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(F >= 1 && EF % F == 0 && EF <= C && EF / F + (C > EF ? 1 : 0) <= ld_dense,
               "moe_glu_capped_dense: bad sizes C=%d EF=%d F=%d", C, EF, F);
  const int V = dtype == CUCA_BF16 ? 8 : 4;
  const bool vec = F % V == 0 && C % V == 0 && ((uintptr_t)gu & 15) == 0 && ((uintptr_t)a & 15) == 0;
  const size_t work = (size_t)T * C / (vec ? V : 1);
  size_t blocks = (work + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
#define CD(TT, VV)                                                                                                     \
  cuca_launch(moe_glu_capped_dense_kernel<TT, VV>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const TT*)gu,  \
              dense, ld_dense, (TT*)a, work, C, EF, F, limit, limit_s, alpha)
  if (dtype == CUCA_F32) { if (vec) CD(float, 4); else CD(float, 1); }
  else if (dtype == CUCA_BF16) { if (vec) CD(__nv_bfloat16, 8); else CD(__nv_bfloat16, 1); }
  else CUCA_REQUIRE(false, "moe_glu_capped_dense: unknown dtype %d", dtype);
#undef CD
  CUCA_CHECK_LAUNCH("moe_glu_capped_dense");
  return 0;
}

CUCA_API int cuca_moe_route_scored(const float* logits, const float* correction, int T, int E, int n_real, int top,
                                   int* idx, float* wts, float* dense, float* ident, cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(E >= 1 && E <= MAX_EXPERTS && top >= 1 && top <= E && top <= MAX_TOP && n_real >= 0 && n_real <= E,
               "moe_route: %d of %d experts (%d with weights) is outside what the kernel takes (experts <= %d, "
               "chosen <= %d)", top, E, n_real, MAX_EXPERTS, MAX_TOP);
  cuca_launch(moe_route_scored_kernel, dim3((T + 3) / 4), dim3(128), 0, stream, true, logits, correction, T, E, n_real,
              top, idx, wts, dense, ident);
  CUCA_CHECK_LAUNCH("moe_route_scored");
  return 0;
}

CUCA_API int cuca_moe_glu_dense(const void* gu, const float* dense, int ld_dense, void* a, int dtype, int T, int C,
                                int EF, int F, cudaStream_t stream) {
  if (T == 0) return 0;
  CUCA_REQUIRE(F >= 1 && EF % F == 0 && EF <= C && EF / F <= ld_dense, "moe_glu_dense: bad sizes C=%d EF=%d F=%d", C, EF, F);
  const size_t n = (size_t)T * C;
  const int V = dtype == CUCA_BF16 ? 8 : 4;
  const bool vec = F % V == 0 && EF % V == 0 && C % V == 0 && ((uintptr_t)gu & 15) == 0 && ((uintptr_t)a & 15) == 0;
  const size_t work = vec ? n / V : n;
  size_t blocks = (work + 255) / 256;
  blocks = blocks > 16384 ? 16384 : blocks;
  if (dtype == CUCA_F32 && vec)
    cuca_launch(moe_glu_dense_vec_kernel<float, 4>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const float*)gu,
                dense, ld_dense, (float*)a, work, C, EF, F);
  else if (dtype == CUCA_BF16 && vec)
    cuca_launch(moe_glu_dense_vec_kernel<__nv_bfloat16, 8>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (const __nv_bfloat16*)gu, dense, ld_dense, (__nv_bfloat16*)a, work, C, EF, F);
  else if (dtype == CUCA_F32)
    cuca_launch(moe_glu_dense_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, true, (const float*)gu, dense,
                ld_dense, (float*)a, n, C, EF, F);
  else if (dtype == CUCA_BF16)
    cuca_launch(moe_glu_dense_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, true,
                (const __nv_bfloat16*)gu, dense, ld_dense, (__nv_bfloat16*)a, n, C, EF, F);
  else
    CUCA_REQUIRE(false, "moe_glu_dense: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("moe_glu_dense");
  return 0;
}

CUCA_API int cuca_moe_identity_add(float* y, const void* h, int dtype, const float* ident, int store, int T, int N,
                                   cudaStream_t stream) {
  if (T == 0) return 0;
  const size_t n = (size_t)T * N;
  size_t blocks = (n + 255) / 256;
  blocks = blocks > 8192 ? 8192 : blocks;
  if (dtype == CUCA_F32)
    cuca_launch(moe_identity_add_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, true, y, (const float*)h,
                ident, store, n, N);
  else if (dtype == CUCA_BF16)
    cuca_launch(moe_identity_add_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, true, y,
                (const __nv_bfloat16*)h, ident, store, n, N);
  else
    CUCA_REQUIRE(false, "moe_identity_add: unknown dtype %d", dtype);
  CUCA_CHECK_LAUNCH("moe_identity_add");
  return 0;
}
