// Routed experts, the plain kernels: a router that picks the `top` largest of E logits per token
// and weighs them by a softmax over the chosen ones, each token's gate/up products against the
// weights of its chosen experts, and the weighted sum of the experts' down products added into the
// residual stream (an id beyond the experts names one that returns its input, or nothing). 32-bit arithmetic; every output is a sum in a fixed order (over k within a
// product, then over a token's choices in the router's order), so a token's result does not depend
// on the rest of the batch.
#include "common.cuh"

namespace {

constexpr int MAX_EXPERTS = 512;
constexpr int MAX_TOP = 32;

// One block per token: its warps share out the experts (z_e = h . W[e] + b[e] in 32-bit, the bias
// 32-bit, each logit one warp's sum in a fixed order), then warp 0 picks the `top` largest in
// descending order (the lower index first among equals); weights = softmax over the chosen logits
// (mode 0), or each chosen expert's own sigmoid(z_e), not renormalized (mode 1), or its share of a
// softmax over all E logits, not renormalized either (mode 2).
// logits [T, E] (or null): h . W is in there already, the block is one warp.
// correction [E] (or null; modes 1 and 2): the choice is by score + correction, the weights are the scores
// without it. groups > 0: the experts form so many equal groups of neighbours, a group's score is its best
// expert's, and only experts of the `keep` best groups (the lower index first among equals) can be chosen.
template <typename HT, typename WT>
__global__ void __launch_bounds__(1024)
route_topk_kernel(const HT* __restrict__ h, const WT* __restrict__ w, const float* __restrict__ logits,
                  const float* __restrict__ bias, int T, int E, int K, int top, int mode, const float* __restrict__ correction, int groups, int keep,
                  int32_t* __restrict__ ids, float* __restrict__ weights) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  extern __shared__ __align__(16) float sm[];        // h[K], z[E] (what the choice goes by), score[E], best of each group[E]
  float* h_s = sm;
  float* z = sm + (logits != nullptr ? 0 : K);
  float* score = z + E;
  float* best_of = score + E;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int t = blockIdx.x;
  const HT* hr = h + (size_t)t * K;
  if (logits != nullptr) {
    for (int e = threadIdx.x; e < E; e += blockDim.x) z[e] = logits[(size_t)t * E + e] + (bias ? bias[e] : 0.f);
  } else {
    for (int k = threadIdx.x; k < K; k += blockDim.x) h_s[k] = gb::to_float<HT>(hr[k]);
  }
  __syncthreads();
  for (int e = warp; e < (logits != nullptr ? 0 : E); e += warps) {
    const WT* wr = w + (size_t)e * K;
    float acc = 0.f;
    if (sizeof(WT) == 2 && K % 8 == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0) {        // eight neighbouring weights in one load (rows start on 16 bytes)
#pragma unroll 8
      for (int k = lane * 8; k < K; k += 256) {
        const uint4 v = *reinterpret_cast<const uint4*>(wr + k);
        const uint32_t pairs[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          acc = fmaf(h_s[k + 2 * i], __uint_as_float(pairs[i] << 16), acc);
          acc = fmaf(h_s[k + 2 * i + 1], __uint_as_float(pairs[i] & 0xffff0000u), acc);
        }
      }
    } else {
      for (int k = lane; k < K; k += 32) acc = fmaf(h_s[k], gb::to_float<WT>(wr[k]), acc);
    }
    acc = gb::warp_sum(acc);
    if (lane == 0) z[e] = acc + (bias ? bias[e] : 0.f);
  }
  __syncthreads();
  if (warp != 0) return;
  // the softmax over every expert needs the largest logit and the sum before logits are struck out
  float all_max = -INFINITY, all_sum = 0.f;
  if (mode == 2) {
    for (int e = lane; e < E; e += 32) all_max = fmaxf(all_max, z[e]);
    all_max = gb::warp_max(all_max);
    for (int e = lane; e < E; e += 32) all_sum += expf(z[e] - all_max);
    all_sum = gb::warp_sum(all_sum);
  }
  if (correction != nullptr) {
    for (int e = lane; e < E; e += 32) {
      score[e] = mode == 2 ? expf(z[e] - all_max) / all_sum : 1.0f / (1.0f + expf(-z[e]));
      z[e] = score[e] + correction[e];
    }
    __syncwarp();
  }
  // the largest of n values, the first of equals, every lane the same
  auto largest_of = [&](const float* v, int n, float& best, int& at) {
    best = -INFINITY;
    at = 0x7fffffff;
    for (int e = lane; e < n; e += 32)
      if (v[e] > best) { best = v[e]; at = e; }      // the first of equals within a lane
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
    }
  };
  if (groups > 0) {
    const int size = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float m = -INFINITY;
      for (int e = 0; e < size; ++e) m = fmaxf(m, z[g * size + e]);
      best_of[g] = m;
    }
    __syncwarp();
    for (int j = 0; j < keep; ++j) {               // a kept group's best becomes a mark no score can have
      float best;
      int at;
      largest_of(best_of, groups, best, at);
      if (lane == 0 && at < groups) best_of[at] = -INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (best_of[e / size] != -INFINITY) z[e] = -INFINITY;
    __syncwarp();
  }
  // `top` rounds of a warp-wide arg-max; a chosen expert's logit is replaced by -inf
  float chosen[MAX_TOP];
  for (int j = 0; j < top; ++j) {
    float best;
    int at;
    largest_of(z, E, best, at);
    chosen[j] = correction != nullptr && at < E ? score[at] : best;
    if (lane == 0) {
      ids[(size_t)t * top + j] = at < E ? at : 0;
      if (at < E) z[at] = -INFINITY;
    }
    __syncwarp();
  }
  if (lane == 0 && correction != nullptr) {
    for (int j = 0; j < top; ++j) weights[(size_t)t * top + j] = chosen[j];
  } else if (lane == 0 && mode == 1) {
    for (int j = 0; j < top; ++j) weights[(size_t)t * top + j] = 1.0f / (1.0f + expf(-chosen[j]));
  } else if (lane == 0 && mode == 2) {
    for (int j = 0; j < top; ++j) weights[(size_t)t * top + j] = expf(chosen[j] - all_max) / all_sum;
  } else if (lane == 0) {
    const float largest = chosen[0];
    float sum = 0.f;
    for (int j = 0; j < top; ++j) {
      chosen[j] = expf(chosen[j] - largest);
      sum += chosen[j];
    }
    for (int j = 0; j < top; ++j) weights[(size_t)t * top + j] = chosen[j] / sum;
  }
}

__device__ __forceinline__ float gate_act(int kind, float limit, float g, float u) {
  if (kind == 1) return g / (1.0f + expf(-1.5957691216057308f * (g + 0.044715f * g * g * g))) * u;      // (1 + tanh v) / 2 is the sigmoid of 2 v
  if (kind == 2) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return (g / (1.0f + expf(-1.702f * g))) * (u + 1.0f);
  }
  return (g / (1.0f + expf(-g))) * u;
}

// an activation of one value, for experts without a gate
__device__ __forceinline__ float plain_act(int kind, float z) {
  switch (kind) {
    case 0: return 1.0f / (1.0f + expf(-z));
    case 1: return z / (1.0f + expf(-z));
    case 2: return fmaxf(z, 0.f) * fmaxf(z, 0.f);
    case 3: return tanhf(z);
    default: return 0.5f * z * erfcf(z * -0.7071067811865476f);
  }
}

// grid (T, top). act[(t * top + j)][f] = act(up_e[f] . h_t), e = ids[t][j], the expert's weights [F, K]; a warp
// per feature, lanes over k. in_scale as below.
template <typename HT, typename WT, typename OT>
__global__ void __launch_bounds__(128)
moe_up_kernel(const HT* __restrict__ h, const WT* __restrict__ w, const int32_t* __restrict__ ids, OT* __restrict__ act,
              int top, int E, int F, int K, int kind, const float* __restrict__ in_scale) {
  extern __shared__ float h_s[];
  const int t = blockIdx.x, j = blockIdx.y;
  if ((unsigned)ids[(size_t)t * top + j] >= (unsigned)E) return;
  for (int k = threadIdx.x; k < K; k += blockDim.x) h_s[k] = gb::to_float<HT>(h[(size_t)t * K + k]);
  __syncthreads();
  const float s_in = in_scale ? in_scale[(size_t)t * top + j] : 1.0f;
  const WT* we = w + (size_t)ids[(size_t)t * top + j] * F * K;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int f = warp; f < F; f += 4) {
    const WT* ur = we + (size_t)f * K;
    float u = 0.f;
    for (int k = lane; k < K; k += 32) u = fmaf(h_s[k], gb::to_float<WT>(ur[k]), u);
    u = gb::warp_sum(u) * s_in;
    if (lane == 0) act[((size_t)t * top + j) * F + f] = gb::from_float<OT>(plain_act(kind, u));
  }
}

// grid (T, top). act[(t * top + j)][f] = act(gate_e[f] . h_t, up_e[f] . h_t), e = ids[t][j]; the
// expert's weights are [2F, K]: F gate rows, then F up rows. A warp per feature, lanes over k.
// in_scale [T, top] (or null): the pair's factor on the expert's input, expert(s h): both products
// are linear in h, so they are multiplied by s before the activation.
template <typename HT, typename WT, typename OT>
__global__ void __launch_bounds__(128)
moe_gate_up_kernel(const HT* __restrict__ h, const WT* __restrict__ w, const int32_t* __restrict__ ids,
                   OT* __restrict__ act, int top, int E, int F, int K, int kind, float limit,
                   const float* __restrict__ in_scale) {
  extern __shared__ float h_s[];
  const int t = blockIdx.x, j = blockIdx.y;
  if ((unsigned)ids[(size_t)t * top + j] >= (unsigned)E) return;
  for (int k = threadIdx.x; k < K; k += blockDim.x) h_s[k] = gb::to_float<HT>(h[(size_t)t * K + k]);
  __syncthreads();
  const int e = ids[(size_t)t * top + j];
  const float s_in = in_scale ? in_scale[(size_t)t * top + j] : 1.0f;
  const WT* we = w + (size_t)e * 2 * F * K;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int f = warp; f < F; f += 4) {
    const WT* gr = we + (size_t)f * K;
    const WT* ur = we + (size_t)(F + f) * K;
    float g = 0.f, u = 0.f;
    for (int k = lane; k < K; k += 32) {
      g = fmaf(h_s[k], gb::to_float<WT>(gr[k]), g);
      u = fmaf(h_s[k], gb::to_float<WT>(ur[k]), u);
    }
    g = gb::warp_sum(g) * s_in;
    u = gb::warp_sum(u) * s_in;
    if (lane == 0) act[((size_t)t * top + j) * F + f] = gb::from_float<OT>(gate_act(kind, limit, g, u));
  }
}

// One block per token. x[t][n] += alpha * sum_j weights[t][j] * (down_e(j)[n] . act[t][j]); weights null: all one.
// An id beyond the E experts: identity[t][n] in place of the product (null: nothing).
template <typename AT, typename WT>
__global__ void __launch_bounds__(256)
moe_down_kernel(const AT* __restrict__ act, const WT* __restrict__ w, const int32_t* __restrict__ ids,
                const float* __restrict__ weights, float* __restrict__ x, int top, int E, int F, int N, float alpha,
                const AT* __restrict__ identity) {
  extern __shared__ float a_s[];        // [top][F]
  const int t = blockIdx.x;
  for (int e = threadIdx.x; e < top * F; e += blockDim.x)
    a_s[e] = (unsigned)ids[(size_t)t * top + e / F] < (unsigned)E ? gb::to_float<AT>(act[(size_t)t * top * F + e]) : 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int n = warp; n < N; n += 8) {
    float total = 0.f;
    for (int j = 0; j < top; ++j) {
      const int e = ids[(size_t)t * top + j];
      if ((unsigned)e >= (unsigned)E) {
        if (identity != nullptr)
          total = fmaf(weights ? weights[(size_t)t * top + j] : 1.0f, gb::to_float<AT>(identity[(size_t)t * N + n]), total);
        continue;
      }
      const WT* wr = w + ((size_t)e * N + n) * F;
      float acc = 0.f;
      for (int f = lane; f < F; f += 32) acc = fmaf(a_s[j * F + f], gb::to_float<WT>(wr[f]), acc);
      total = fmaf(weights ? weights[(size_t)t * top + j] : 1.0f, gb::warp_sum(acc), total);
    }
    if (lane == 0) x[(size_t)t * N + n] = fmaf(alpha, total, x[(size_t)t * N + n]);
  }
}

}  // namespace

// logits [T, E] 32-bit (or null): the products h . W, made by the caller.
GB_EXPORT int gb_route_topk(const void* h, int h_dtype, const void* w, const float* logits, const float* bias, int w_dtype, int T, int E,
                            int K, int top, int mode, const float* correction, int groups, int keep, int32_t* ids,
                            float* weights, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if (mode < 0 || mode > 2) return gb::fail(GB_BAD_ARGUMENT, "route_topk: mode %d", mode);
  if (E < 1 || E > MAX_EXPERTS || top < 1 || top > MAX_TOP || top > E)
    return gb::fail(GB_UNSUPPORTED, "route_topk: %d of %d experts (at most %d of %d)", top, E, MAX_TOP, MAX_EXPERTS);
  if (correction != nullptr && mode == 0) return gb::fail(GB_BAD_ARGUMENT, "route_topk: a correction goes with scores of their own");
  if (groups < 0 || (groups > 0 && (E % groups || keep < 1 || keep > groups || top > E / groups * keep)))
    return gb::fail(GB_BAD_ARGUMENT, "route_topk: %d of %d groups of %d experts, %d chosen", keep, groups, E, top);
  const size_t smem = (size_t)(3 * E + (logits != nullptr ? 0 : K)) * sizeof(float);
  if (smem > 200 * 1024) return gb::fail(GB_UNSUPPORTED, "route_topk: width %d", K);
  // few tokens: a warp for every expert, up to a block's 32
  const int threads = logits != nullptr ? 32 : (T < 148 && E > 8 ? (E < 32 ? E * 32 : 1024) : 256);
  return GB_DISPATCH_DTYPE(h_dtype, HT, [&]() -> int {
    return GB_DISPATCH_DTYPE(w_dtype, WT, [&]() -> int {
      if (smem > 48 * 1024) {     // rare (rows beyond 12,000 values): asked for at every such launch
        cudaError_t e = cudaFuncSetAttribute(route_topk_kernel<HT, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return gb::fail(GB_CUDA_ERROR, "route_topk: %s", cudaGetErrorString(e));
      }
      return gb::check_pdl_launch(
          gb::launch_pdl(route_topk_kernel<HT, WT>, dim3(T), dim3(threads), smem, stream,
                         dim3(1, 1, 1), (const HT*)h, (const WT*)w, logits, bias, T, E, K, top, mode, correction, groups, keep, ids, weights),
          "route_topk");
    });
  });
}

GB_EXPORT int gb_moe_gate_up(const void* h, int h_dtype, const void* w, int w_dtype, const int32_t* ids, void* act,
                             int act_dtype, int T, int top, int E, int F, int K, int kind, float limit,
                             const float* in_scale, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if ((size_t)K * sizeof(float) > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "moe_gate_up: width %d", K);
  return GB_DISPATCH_DTYPE(h_dtype, HT, [&]() -> int {
    return GB_DISPATCH_DTYPE(w_dtype, WT, [&]() -> int {
      return GB_DISPATCH_DTYPE(act_dtype, OT, [&]() -> int {
        moe_gate_up_kernel<HT, WT, OT><<<dim3(T, top), 128, (size_t)K * sizeof(float), stream>>>(
            (const HT*)h, (const WT*)w, ids, (OT*)act, top, E, F, K, kind, limit, in_scale);
        return gb::check_launch("moe_gate_up");
      });
    });
  });
}

// kind: 0 sigmoid, 1 silu, 2 relu^2, 3 tanh, 4 exact gelu.
GB_EXPORT int gb_moe_up(const void* h, int h_dtype, const void* w, int w_dtype, const int32_t* ids, void* act, int act_dtype,
                        int T, int top, int E, int F, int K, int kind, const float* in_scale, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if (kind < 0 || kind > 4) return gb::fail(GB_BAD_ARGUMENT, "moe_up: activation %d", kind);
  if ((size_t)K * sizeof(float) > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "moe_up: width %d", K);
  return GB_DISPATCH_DTYPE(h_dtype, HT, [&]() -> int {
    return GB_DISPATCH_DTYPE(w_dtype, WT, [&]() -> int {
      return GB_DISPATCH_DTYPE(act_dtype, OT, [&]() -> int {
        moe_up_kernel<HT, WT, OT><<<dim3(T, top), 128, (size_t)K * sizeof(float), stream>>>(
            (const HT*)h, (const WT*)w, ids, (OT*)act, top, E, F, K, kind, in_scale);
        return gb::check_launch("moe_up");
      });
    });
  });
}

GB_EXPORT int gb_moe_down(const void* act, int act_dtype, const void* w, int w_dtype, const int32_t* ids,
                          const float* weights, float* x, int T, int top, int E, int F, int N, float alpha,
                          const void* identity, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if ((size_t)top * F * sizeof(float) > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "moe_down: %d x %d activations", top, F);
  return GB_DISPATCH_DTYPE(act_dtype, AT, [&]() -> int {
    return GB_DISPATCH_DTYPE(w_dtype, WT, [&]() -> int {
      moe_down_kernel<AT, WT><<<T, 256, (size_t)top * F * sizeof(float), stream>>>(
          (const AT*)act, (const WT*)w, ids, weights, x, top, E, F, N, alpha, (const AT*)identity);
      return gb::check_launch("moe_down");
    });
  });
}
