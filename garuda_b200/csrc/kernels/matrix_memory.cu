// A matrix memory with exponential gates (mLSTM; Beck et al., "xLSTM: Extended Long Short-Term Memory", 2024):
// what surrounds its recurrence over a stretch of tokens, and the whole of it for single tokens. 32-bit arithmetic.
// Per head and token, with i and f the logarithms of the input and forget gates:
//     m' = max(f + m, i);   a = f + m - m';   s = exp(i - m')
//     S <- exp(a) S + s v k^T;   n <- exp(a) n + s k;   o = S q scale / (max(|n . q| scale, exp(-m')) + 1e-6)
//     out = o / sqrt(mean(o^2) + eps) * w * sigmoid(g)
//
//   memory_gates    the gates of a request's tokens and the running maximum over them (a scan: the token's map
//                   m -> max(f + m, i) composed with the one in front is (f1 + f2, max(f2 + i1, i2))); out: step
//                   [T, 2 H] = s, then a, which is what the state-space recurrence takes, and exp(-m')
//   memory_finish   from the recurrence's S q and n . q to `out`
//   memory_decode   all of it for one token per request, the shares of a head's rows in a thread-block cluster that
//                   adds up the head's mean square in distributed shared memory
//
// A request's state is one row: S of all heads [H, P, N] (P value channels, N key channels), n [H, N], m [H].
#include <cooperative_groups.h>

#include <type_traits>

#include "common.cuh"


namespace {

namespace cg = cooperative_groups;

__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
// min(z, 0) - ln(1 + exp(-|z|))
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

struct Gates {
  const float* i;          // logits of token 0, head 0; rows `stride` apart
  const float* f;
  const float* b_i;        // [H]
  const float* b_f;
  long long stride;
  float cap;
};

__device__ __forceinline__ void read_gates(const Gates& g, int t, int h, float& in, float& forget) {
  in = soft_cap(g.i[(size_t)t * g.stride + h] + g.b_i[h], g.cap);
  forget = log_sigmoid(soft_cap(g.f[(size_t)t * g.stride + h] + g.b_f[h], g.cap));
}

constexpr int SCAN_THREADS = 256, SCAN_PER = 4, SCAN_TILE = SCAN_THREADS * SCAN_PER;

// grid (H, R): a request's tokens in tiles, a thread SCAN_PER neighbouring ones.
__global__ void __launch_bounds__(SCAN_THREADS)
memory_gates_kernel(const Gates gates, const int32_t* __restrict__ cu_q, const int32_t* __restrict__ slots, float* __restrict__ m_state,
                    long long state_stride, float* __restrict__ step, float* __restrict__ floor_out, int H) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  __shared__ float warp_f[SCAN_THREADS / 32], warp_i[SCAN_THREADS / 32], carry_s;
  const int h = blockIdx.x, r = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = slots[r], t0 = cu_q[r], t1 = cu_q[r + 1];
  if (t0 >= t1) return;
  float* m_g = slot >= 0 ? m_state + (size_t)slot * state_stride + h : nullptr;
  float carry = m_g != nullptr ? *m_g : 0.f;                 // m in front of the tile
  for (int base = t0; base < t1; base += SCAN_TILE) {
    const int first = base + threadIdx.x * SCAN_PER;
    float in[SCAN_PER], fg[SCAN_PER];
    float F = 0.f, I = -INFINITY;                            // the thread's tokens as one map
#pragma unroll
    for (int k = 0; k < SCAN_PER; ++k) {
      in[k] = -INFINITY, fg[k] = 0.f;                        // (beyond the end: the map that changes nothing)
      if (first + k < t1) read_gates(gates, first + k, h, in[k], fg[k]);
    }
#pragma unroll
    for (int k = 0; k < SCAN_PER; ++k) {
      I = fmaxf(fg[k] + I, in[k]);
      F += fg[k];
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {                       // the maps up to and including this lane's
      const float f1 = __shfl_up_sync(0xffffffffu, F, o), i1 = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(F + i1, I);
        F += f1;
      }
    }
    if (lane == 31) warp_f[warp] = F, warp_i[warp] = I;
    __syncthreads();
    float m = carry;
    for (int w = 0; w < warp; ++w) m = fmaxf(warp_f[w] + m, warp_i[w]);
    {
      const float f1 = __shfl_up_sync(0xffffffffu, F, 1), i1 = __shfl_up_sync(0xffffffffu, I, 1);
      if (lane > 0) m = fmaxf(f1 + m, i1);
    }
#pragma unroll
    for (int k = 0; k < SCAN_PER; ++k) {
      const int t = first + k;
      if (t >= t1) break;
      const float before = fg[k] + m;
      m = fmaxf(before, in[k]);
      step[(size_t)t * 2 * H + h] = expf(in[k] - m);
      step[(size_t)t * 2 * H + H + h] = before - m;
      floor_out[(size_t)t * H + h] = expf(-m);
      if (t == min(t1, base + SCAN_TILE) - 1) carry_s = m;
    }
    __syncthreads();
    carry = carry_s;
  }
  if (m_g != nullptr && threadIdx.x == 0) *m_g = carry;
}

// A warp per (token, head), eight to a block.
template <typename OT>
__global__ void __launch_bounds__(256)
memory_finish_kernel(const float* __restrict__ y, const float* __restrict__ den, const float* __restrict__ floor_in,
                     const float* __restrict__ gate, long long gate_stride, const float* __restrict__ w, float scale, float eps,
                     OT* __restrict__ out, long long rows, int H, int P) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= rows) return;
  const long long t = i / H;
  const int h = (int)(i % H);
  const float* yr = y + i * P;
  const float by = scale / (fmaxf(fabsf(den[i]) * scale, floor_in[i]) + 1e-6f);
  float ss = 0.f;
  for (int c = lane; c < P; c += 32) {
    const float o = yr[c] * by;
    ss = fmaf(o, o, ss);
  }
  const float inv = 1.0f / sqrtf(gb::warp_sum(ss) / (float)P + eps);
  const float* gr = gate + t * gate_stride + (size_t)h * P;
  const float* wr = w + (size_t)h * P;
  OT* o = out + i * P;
  for (int c = lane; c < P; c += 32) o[c] = gb::from_float<OT>(((yr[c] * by) * inv) * wr[c] * sigmoidf_(gr[c]));
}

constexpr int DEC_THREADS = 256;

// grid (shares, H, R), clusters of (shares, 1, 1): one token per request (row t of the batch is request t). A block
// has `rows_per_block` rows of its head's S; ROW_LANES lanes a row, four neighbouring channels a lane at a time (VEC:
// as one 16-byte access). XT: what the queries, keys and values are rounded to, and the output's type.
template <int ROW_LANES, int QUADS, bool VEC, typename XT>
__global__ void __launch_bounds__(DEC_THREADS)
memory_decode_kernel(const float* __restrict__ rows, long long stride, const Gates gates, const float* __restrict__ gate,
                     long long gate_stride, const float* __restrict__ w, float scale, float eps, const int32_t* __restrict__ slots,
                     float* __restrict__ state, long long state_stride, int H, int N, int P, int rows_per_block,
                     XT* __restrict__ out) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  extern __shared__ __align__(16) float sm[];       // k, q [N rounded up to four each], v and then the read-out [rows]
  __shared__ float red[DEC_THREADS / 32], share_s;
  constexpr int GROUPS = DEC_THREADS / ROW_LANES;
  constexpr int BATCH = QUADS >= 4 ? 1 : (QUADS == 2 ? 2 : 4);
  cg::cluster_group cluster = cg::this_cluster();
  const int npad = (N + 3) / 4 * 4;
  float *sk = sm, *sq = sm + npad, *sv = sm + 2 * npad;
  const int h = blockIdx.y, t = blockIdx.z, p0 = blockIdx.x * rows_per_block, np = max(0, min(rows_per_block, P - p0));
  const int slot = slots[t], warp = threadIdx.x >> 5, lane32 = threadIdx.x & 31;
  const int group = threadIdx.x / ROW_LANES, lane = threadIdx.x % ROW_LANES;
  float* row_state = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
  float* S_g = row_state != nullptr ? row_state + ((size_t)h * P + p0) * N : nullptr;
  float* n_g = row_state != nullptr ? row_state + (size_t)H * P * N + (size_t)h * N : nullptr;
  float* m_g = row_state != nullptr ? row_state + (size_t)H * P * N + (size_t)H * N + h : nullptr;
  float S[BATCH][QUADS][4];
  auto fetch = [&](int base) {
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int p = base + i * GROUPS;
#pragma unroll
      for (int q = 0; q < QUADS; ++q) {
        const int c = (lane + q * ROW_LANES) * 4;
        if (VEC) {
          const float4 v = (S_g != nullptr && p < np && c < N) ? *reinterpret_cast<const float4*>(S_g + (size_t)p * N + c)
                                                               : make_float4(0.f, 0.f, 0.f, 0.f);
          S[i][q][0] = v.x, S[i][q][1] = v.y, S[i][q][2] = v.z, S[i][q][3] = v.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) S[i][q][e] = (S_g != nullptr && p < np && c + e < N) ? S_g[(size_t)p * N + c + e] : 0.f;
        }
      }
    }
  };
  fetch(group);                        // on its way while the rest is read
  const float* row = rows + (size_t)t * stride;           // v | k | q of all heads
  for (int i = threadIdx.x; i < 2 * npad + np; i += blockDim.x) {
    float v = 0.f;
    if (i >= 2 * npad) v = row[(size_t)h * P + p0 + i - 2 * npad];
    else if (i % npad < N) v = row[(size_t)H * P + (size_t)(i < npad ? 0 : H) * N + (size_t)h * N + i % npad];
    sm[i] = gb::to_float<XT>(gb::from_float<XT>(v));
  }
  float in, forget;
  read_gates(gates, t, h, in, forget);
  const float m_old = m_g != nullptr ? *m_g : 0.f;
  const float before = forget + m_old, m = fmaxf(before, in);
  const float put = expf(in - m), log_keep = before - m;
  // a slow decay as 1 + expm1: the second term holds what a rounded factor loses of the state at every token
  const bool slow = log_keep > -0.5f;
  const float keep = slow ? 1.0f : expf(log_keep), change = slow ? expm1f(log_keep) : 0.0f;
  __syncthreads();
  // the normalizer, in every block alike; the cluster's first stores it once all have read it
  float dot = 0.f;
  constexpr int N_PER = 2;                          // N is at most 512
  float n_new[N_PER];
#pragma unroll
  for (int i = 0; i < N_PER; ++i) {
    const int c = threadIdx.x + i * DEC_THREADS;
    n_new[i] = 0.f;
    if (c < N) {
      const float n = n_g != nullptr ? n_g[c] : 0.f;
      n_new[i] = fmaf(keep, n, fmaf(change, n, put * sk[c]));
      dot = fmaf(n_new[i], sq[c], dot);
    }
  }
  dot = gb::warp_sum(dot);
  if (lane32 == 0) red[warp] = dot;
  float b[QUADS][4], q4[QUADS][4];
#pragma unroll
  for (int q = 0; q < QUADS; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = (lane + q * ROW_LANES) * 4 + e;
      b[q][e] = c < N ? put * sk[c] : 0.f;
      q4[q][e] = c < N ? sq[c] : 0.f;
    }
  for (int base = group; base < (np + GROUPS - 1) / GROUPS * GROUPS; base += BATCH * GROUPS) {
    if (base != group) fetch(base);
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int p = base + i * GROUPS;
      const float v = p < np ? sv[p] : 0.f;
      float acc = 0.f;
#pragma unroll
      for (int q = 0; q < QUADS; ++q) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[i][q][e] = fmaf(keep, S[i][q][e], fmaf(change, S[i][q][e], v * b[q][e]));
          acc = fmaf(S[i][q][e], q4[q][e], acc);
        }
        const int c = (lane + q * ROW_LANES) * 4;
        if (S_g != nullptr && p < np) {
          if (VEC) {
            if (c < N) *reinterpret_cast<float4*>(S_g + (size_t)p * N + c) = make_float4(S[i][q][0], S[i][q][1], S[i][q][2], S[i][q][3]);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (c + e < N) S_g[(size_t)p * N + c + e] = S[i][q][e];
          }
        }
      }
#pragma unroll
      for (int o = ROW_LANES / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (lane == 0 && p < np) sv[p] = acc;          // the row's value has been read by this group alone
    }
  }
  __syncthreads();
  float den = 0.f;
#pragma unroll
  for (int i = 0; i < DEC_THREADS / 32; ++i) den += red[i];
  const float by = scale / (fmaxf(fabsf(den) * scale, expf(-m)) + 1e-6f);
  float ss = 0.f;
  for (int p = threadIdx.x; p < np; p += DEC_THREADS) {
    const float o = sv[p] * by;
    sv[p] = o;
    ss = fmaf(o, o, ss);
  }
  ss = gb::warp_sum(ss);
  __syncthreads();                     // red has been read
  if (lane32 == 0) red[warp] = ss;
  __syncthreads();
  if (threadIdx.x == 0) {
    float total = 0.f;
    for (int i = 0; i < DEC_THREADS / 32; ++i) total += red[i];
    share_s = total;
  }
  cluster.sync();                      // every block's share is there; every block has read n and m
  float total = 0.f;
  for (unsigned i = 0; i < cluster.num_blocks(); ++i) total += *cluster.map_shared_rank(&share_s, i);
  cluster.sync();                      // nobody leaves while its share may still be read
  const float inv = 1.0f / sqrtf(total / (float)P + eps);
  if (blockIdx.x == 0 && row_state != nullptr) {
#pragma unroll
    for (int i = 0; i < N_PER; ++i) {
      const int c = threadIdx.x + i * DEC_THREADS;
      if (c < N) n_g[c] = n_new[i];
    }
    if (threadIdx.x == 0) *m_g = m;
  }
  const size_t at = (size_t)h * P + p0;
  for (int p = threadIdx.x; p < np; p += DEC_THREADS)
    out[(size_t)t * H * P + at + p] = gb::from_float<XT>((sv[p] * inv) * w[at + p] * sigmoidf_(gate[(size_t)t * gate_stride + at + p]));
}

int check_sizes(const char* what, int H, int N, int P, float cap) {
  if (H < 1 || N < 1 || P < 1) return gb::fail(GB_BAD_ARGUMENT, "%s: %d heads of %d x %d", what, H, N, P);
  if (N > 512 || P > 8192) return gb::fail(GB_UNSUPPORTED, "%s: heads of %d x %d (at most 512 x 8192)", what, N, P);
  if (!(cap > 0.f)) return gb::fail(GB_BAD_ARGUMENT, "%s: gates capped at %g", what, cap);
  return GB_OK;
}

}  // namespace

// i, f: the gates' logits (row t, head h at [t * stride + h]); m_state: m of slot 0, head 0. Out: step [T, 2 H], floor [T, H].
GB_EXPORT int gb_memory_gates(const float* i, const float* f, long long stride, const float* b_i, const float* b_f, float cap,
                              const int32_t* cu_q, const int32_t* slots, float* m_state, long long state_stride, float* step,
                              float* floor_out, int R, int H, cudaStream_t stream) {
  if (R <= 0) return GB_OK;
  int rc = check_sizes("memory_gates", H, 1, 1, cap);
  if (rc != GB_OK) return rc;
  if (R > 65535) return gb::fail(GB_UNSUPPORTED, "memory_gates: %d requests", R);
  const Gates g = {i, f, b_i, b_f, stride, cap};
  return gb::check_pdl_launch(gb::launch_pdl(memory_gates_kernel, dim3(H, R), dim3(SCAN_THREADS), 0, stream, dim3(1, 1, 1), g, cu_q,
                                             slots, m_state, state_stride, step, floor_out, H),
                              "memory_gates");
}

// y [T, H P], den [T, H], floor [T, H] (exp(-m)), gate [T, >= H P] logits with rows gate_stride apart, w [H P]; out [T, H P].
GB_EXPORT int gb_memory_finish(const float* y, const float* den, const float* floor_in, const float* gate, long long gate_stride,
                               const float* w, float scale, float eps, void* out, int out_dtype, int T, int H, int P,
                               cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  int rc = check_sizes("memory_finish", H, 1, P, 1.f);
  if (rc != GB_OK) return rc;
  const long long rows = (long long)T * H, blocks = (rows + 7) / 8;
  if (blocks > 0x7fffffffLL) return gb::fail(GB_UNSUPPORTED, "memory_finish: %d tokens", T);
  return GB_DISPATCH_DTYPE(out_dtype, OT, [&]() -> int {
    return gb::check_pdl_launch(gb::launch_pdl(memory_finish_kernel<OT>, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1), y,
                                               den, floor_in, gate, gate_stride, w, scale, eps, (OT*)out, rows, H, P),
                                "memory_finish");
  });
}

// One token per request. rows: v | k | q of all heads, 32-bit, `stride` apart; i, f, gate: logits as above.
GB_EXPORT int gb_memory_decode(const float* rows, long long stride, const float* i, const float* f, long long gates_stride,
                               const float* b_i, const float* b_f, float cap, const float* gate, long long gate_stride, const float* w,
                               float scale, float eps, const int32_t* slots, float* state, long long state_stride, int R, int H,
                               int N, int P, void* out, int out_dtype, cudaStream_t stream) {
  if (R <= 0) return GB_OK;
  int rc = check_sizes("memory_decode", H, N, P, cap);
  if (rc != GB_OK) return rc;
  if (R > 65535 || H > 65535) return gb::fail(GB_UNSUPPORTED, "memory_decode: %d requests of %d heads", R, H);
  const Gates g = {i, f, b_i, b_f, gates_stride, cap};
  // a head's rows over the blocks of a cluster while (head, request) pairs alone leave SMs idle
  int shares = 1;
  while (shares < 8 && (long long)H * R * shares < 296 && P / (2 * shares) >= 8) shares *= 2;
  const int per_block = (P + shares - 1) / shares;
  const size_t smem = (size_t)(2 * ((N + 3) / 4 * 4) + per_block) * sizeof(float);
  if (smem > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "memory_decode: heads of %d x %d", N, P);
  const bool vec = N % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  return GB_DISPATCH_DTYPE(out_dtype, XT, [&]() -> int {
    auto go = [&](auto lanes, auto quads) -> int {
      constexpr int L = decltype(lanes)::value, Q = decltype(quads)::value;
      return gb::check_pdl_launch(
          gb::launch_pdl(vec ? memory_decode_kernel<L, Q, true, XT> : memory_decode_kernel<L, Q, false, XT>, dim3(shares, H, R),
                         dim3(DEC_THREADS), smem, stream, dim3(shares, 1, 1), rows, stride, g, gate, gate_stride, w, scale, eps, slots,
                         state, state_stride, H, N, P, per_block, (XT*)out),
          "memory_decode");
    };
    using std::integral_constant;
    if (N <= 16) return go(integral_constant<int, 4>(), integral_constant<int, 1>());
    if (N <= 32) return go(integral_constant<int, 8>(), integral_constant<int, 1>());
    if (N <= 64) return go(integral_constant<int, 16>(), integral_constant<int, 1>());
    if (N <= 128) return go(integral_constant<int, 32>(), integral_constant<int, 1>());
    if (N <= 256) return go(integral_constant<int, 32>(), integral_constant<int, 2>());
    return go(integral_constant<int, 32>(), integral_constant<int, 4>());
  });
}
