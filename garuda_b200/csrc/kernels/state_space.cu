// The selective state space with one decay per head and token (Mamba-2): a recurrent mixer whose state per
// request and head is a matrix S [vdim, dim] in 32-bit, behind a short causal convolution. Per token:
//     dt = softplus(d + dt_bias);   S <- exp(-rate dt) S + x (dt B)^T;   y = S C + skip x
// with x the head's vdim channels and B, C the dim channels of its group, convolved and through SiLU.
//
// Kernels, all 32-bit arithmetic:
//   ssd_prepare     convolution over the step's rows and the request's kept last inputs, bias, SiLU, the result
//                   rounded to the compute dtype; step sizes and the logarithms of the decays
//   ssd_recurrence  a request's tokens walked in order, any sizes: a warp owns rows of S, its lanes their channels
//   ssd_decode      both for steps of one token per request, a block per (request, head)
//   ssd_finish      y * silu(z), divided by the root mean square of its part of the row, times a weight; and the
//                   convolution's kept inputs moved on
// (ssd_chunk_mma.cu has the recurrence over long stretches of tokens as products on the tensor cores.)
//
// proj [T, P] is the projected 32-bit row: z from column cz, the convolved channels (x of all heads, B of all
// groups, C of all groups) from cx, d from cd. A request's state is one row: S of all heads, then the
// convolution's last taps - 1 inputs, oldest first.
#include <type_traits>

#include "common.cuh"

GB_DEFINE_LAST_ERROR()

namespace {

constexpr int MAX_TAPS = 16;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// A decay a = exp(log_a) as the two numbers that a state is moved on with, S <- keep S + (change S + input). A slow
// decay (a close to one) is 1 + expm1(log_a): the second term holds what a rounded `a` would lose, which over
// hundreds of tokens is the larger part of the state's error. A fast one is (a, 0).
__device__ __forceinline__ void decay_parts(float log_a, float& keep, float& change) {
  const bool slow = log_a > -0.5f;
  keep = slow ? 1.0f : expf(log_a);
  change = slow ? expm1f(log_a) : 0.0f;
}

// Input of channel c at `lag` tokens before token t (index j within its request's rows of this step): from the
// step's rows, or from the request's kept inputs [taps - 1, C] (oldest first).
__device__ __forceinline__ float conv_input(const float* __restrict__ rows, long long P, int t, int j, int lag, int c,
                                            const float* __restrict__ kept, int C, int taps) {
  if (j - lag >= 0) return rows[(size_t)(t - lag) * P + c];
  if (kept == nullptr) return 0.f;
  return kept[(size_t)(taps - 1 + j - lag) * C + c];
}

struct Conv {
  const float* rows;      // proj + cx
  long long P;            // floats between two rows
  const float* w;         // [C, taps]
  const float* b;         // [C] or null
  const float* kept;      // the kept inputs of slot 0, or null (one tap)
  long long kept_stride;  // floats between two slots
  int taps, C;
};

// bias + sum over taps in ascending order, then SiLU: the one order every kernel here takes
__device__ __forceinline__ float conv_silu(const Conv& cv, const float* kept, int t, int j, int c) {
  float acc = cv.b ? cv.b[c] : 0.f;
  for (int tap = 0; tap < cv.taps; ++tap)
    acc = fmaf(cv.w[(size_t)c * cv.taps + tap], conv_input(cv.rows, cv.P, t, j, cv.taps - 1 - tap, c, kept, cv.C, cv.taps), acc);
  return silu(acc);
}

constexpr int PREP_TOKENS = 8, PREP_THREADS = 128;

template <typename XT, int VEC>
__device__ __forceinline__ void store_vec(XT* to, const float (&v)[VEC]) {
  if (VEC == 2) gb::store_pair(to, v[0], v[VEC - 1]);
  else *to = gb::from_float<XT>(v[0]);
}

// grid (ceil(C / (VEC 128)) + 1, ceil(T / 8)): a thread convolves VEC neighbouring channels of eight tokens, all of
// their inputs asked for before the first is used. TAPS 0: any number of taps, every input looked up by itself.
// The last block of a row of blocks makes the tokens' step sizes dt and logarithms of decays -rate dt: step [T, 2 H].
template <int TAPS, int VEC, typename XT>
__global__ void __launch_bounds__(PREP_THREADS)
ssd_prepare_kernel(const Conv cv, const float* __restrict__ d_rows, const float* __restrict__ rate,
                   const float* __restrict__ dt_bias, const int32_t* __restrict__ token_req, const int32_t* __restrict__ cu_q,
                   const int32_t* __restrict__ slots, XT* __restrict__ act, float* __restrict__ step, int T, int H) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  const int t0 = blockIdx.y * PREP_TOKENS, n = min(PREP_TOKENS, T - t0);
  if (blockIdx.x == gridDim.x - 1) {
    for (int i = threadIdx.x; i < n * H; i += blockDim.x) {
      const int t = t0 + i / H, h = i % H;
      const float dt = softplus(d_rows[(size_t)t * cv.P + h] + dt_bias[h]);
      step[(size_t)t * 2 * H + h] = dt;
      step[(size_t)t * 2 * H + H + h] = -rate[h] * dt;
    }
    return;
  }
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= cv.C) return;
  const int r = token_req[t0], j0 = t0 - cu_q[r];
  if (TAPS > 0 && j0 >= TAPS - 1 && t0 + n <= cu_q[r + 1]) {      // the tile and its look-back lie in one request's rows
    constexpr int NT = TAPS > 0 ? TAPS : 1, IN = PREP_TOKENS + NT - 1;
    float in[IN][VEC], w[NT][VEC], b[VEC];
#pragma unroll
    for (int i = 0; i < IN; ++i) {
      const float* p = cv.rows + (size_t)(t0 - (NT - 1) + min(i, n + NT - 2)) * cv.P + c;
      if (VEC == 2) {
        const float2 v = *reinterpret_cast<const float2*>(p);
        in[i][0] = v.x, in[i][VEC - 1] = v.y;
      } else {
        in[i][0] = *p;
      }
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      b[v] = cv.b ? cv.b[c + v] : 0.f;
#pragma unroll
      for (int tap = 0; tap < NT; ++tap) w[tap][v] = cv.w[(size_t)(c + v) * NT + tap];
    }
#pragma unroll
    for (int tt = 0; tt < PREP_TOKENS; ++tt) {
      if (tt >= n) break;
      float out[VEC];
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        float acc = b[v];
#pragma unroll
        for (int tap = 0; tap < NT; ++tap) acc = fmaf(w[tap][v], in[tt + tap][v], acc);
        out[v] = silu(acc);
      }
      store_vec<XT, VEC>(act + (size_t)(t0 + tt) * cv.C + c, out);
    }
    return;
  }
  for (int tt = 0; tt < n; ++tt) {
    const int t = t0 + tt, rr = token_req[t], slot = slots[rr];
    const float* kept = slot >= 0 && cv.kept ? cv.kept + (size_t)slot * cv.kept_stride : nullptr;
    float out[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) out[v] = conv_silu(cv, kept, t, t - cu_q[rr], c + v);
    store_vec<XT, VEC>(act + (size_t)t * cv.C + c, out);
  }
}

// A head may keep one more row of state, driven by the constant input one in place of an x channel (the normalizer
// of a matrix memory): `state` is its place for head 0 in slot 0 ([H, dim], the slots as far apart as those of S; null: no such row), `y`
// [T, H] its read-out.
struct UnitRow {
  float* state;
  float* y;
};

constexpr int REC_WARPS = 4, REC_ROWS = 4, REC_TOKENS = 8;        // rows of S per warp; tokens staged at a time

// grid (H, R, ceil(vdim / 16), one more for a unit row), 128 threads. A warp owns four rows of S; lane l holds the channels l, l + 32, ...
// of each. A token's B, C, x, dt and decay come through shared memory, eight tokens at a time.
template <int PER, typename XT>
__global__ void __launch_bounds__(REC_WARPS * 32)
ssd_recurrence_kernel(const XT* __restrict__ act, int C, const float* __restrict__ step, const float* __restrict__ skip,
                      const int32_t* __restrict__ cu_q, const int32_t* __restrict__ slots, float* __restrict__ state,
                      long long state_stride, int H, int G, int dim, int vdim, float* __restrict__ y, const UnitRow unit) {
  gb::pdl_wait();
  constexpr int W = PER * 32;
  __shared__ float sb[REC_TOKENS][W], sc[REC_TOKENS][W], sx[REC_TOKENS][REC_WARPS * REC_ROWS], sdt[REC_TOKENS];
  __shared__ float s_keep[REC_TOKENS], s_change[REC_TOKENS];
  const bool is_unit = unit.state != nullptr && blockIdx.z == gridDim.z - 1;
  const int h = blockIdx.x, r = blockIdx.y, p0 = is_unit ? 0 : blockIdx.z * REC_WARPS * REC_ROWS;
  const int rows = is_unit ? 1 : vdim;             // of this block's state
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = slots[r], t0 = cu_q[r], t1 = cu_q[r + 1];
  const int off_b = H * vdim + h / (H / G) * dim, off_c = off_b + G * dim;
  const int row0 = p0 + warp * REC_ROWS;
  float* S_g = slot >= 0 ? (is_unit ? unit.state : state) + (size_t)slot * state_stride + (size_t)h * rows * dim : nullptr;
  float* y_g = is_unit ? unit.y + h : y + (size_t)h * vdim;
  const long long y_stride = is_unit ? H : (long long)H * vdim;
  float S[REC_ROWS][PER];
#pragma unroll
  for (int i = 0; i < REC_ROWS; ++i)
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int c = lane + 32 * k;
      S[i][k] = (S_g != nullptr && row0 + i < rows && c < dim) ? S_g[(size_t)(row0 + i) * dim + c] : 0.f;
    }
  const float dskip = is_unit || skip == nullptr ? 0.f : skip[h];
  for (int c0 = t0; c0 < t1; c0 += REC_TOKENS) {
    const int n = min(REC_TOKENS, t1 - c0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * W; i += blockDim.x) {
      const int tt = i / W, c = i % W;
      const XT* row = act + (size_t)(c0 + tt) * C;
      sb[tt][c] = c < dim ? gb::to_float<XT>(row[off_b + c]) : 0.f;
      sc[tt][c] = c < dim ? gb::to_float<XT>(row[off_c + c]) : 0.f;
    }
    for (int i = threadIdx.x; i < n * REC_WARPS * REC_ROWS; i += blockDim.x) {
      const int tt = i / (REC_WARPS * REC_ROWS), p = i % (REC_WARPS * REC_ROWS);
      if (is_unit) sx[tt][p] = p == 0 ? 1.f : 0.f;
      else sx[tt][p] = p0 + p < vdim ? gb::to_float<XT>(act[(size_t)(c0 + tt) * C + h * vdim + p0 + p]) : 0.f;
    }
    if (threadIdx.x < n) {
      const float* st = step + (size_t)(c0 + threadIdx.x) * 2 * H;
      sdt[threadIdx.x] = st[h];
      decay_parts(st[H + h], s_keep[threadIdx.x], s_change[threadIdx.x]);
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      const float keep = s_keep[tt], change = s_change[tt], dt = sdt[tt];
      float acc[REC_ROWS];
#pragma unroll
      for (int i = 0; i < REC_ROWS; ++i) acc[i] = 0.f;
#pragma unroll
      for (int k = 0; k < PER; ++k) {
        const float b = dt * sb[tt][lane + 32 * k], c = sc[tt][lane + 32 * k];
#pragma unroll
        for (int i = 0; i < REC_ROWS; ++i) {
          S[i][k] = fmaf(keep, S[i][k], fmaf(change, S[i][k], sx[tt][warp * REC_ROWS + i] * b));
          acc[i] = fmaf(S[i][k], c, acc[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < REC_ROWS; ++i) acc[i] = gb::warp_sum(acc[i]);
      float mine = acc[0];                 // lane i stores row i
#pragma unroll
      for (int i = 1; i < REC_ROWS; ++i) mine = lane == i ? acc[i] : mine;
      if (lane < REC_ROWS && row0 + lane < rows)
        y_g[(c0 + tt) * y_stride + row0 + lane] = fmaf(dskip, sx[tt][warp * REC_ROWS + lane], mine);
    }
  }
  gb::pdl_launch_dependents();         // only now: the next kernel's blocks would wait beside these for the whole walk
  if (S_g != nullptr) {
#pragma unroll
    for (int i = 0; i < REC_ROWS; ++i)
#pragma unroll
      for (int k = 0; k < PER; ++k) {
        const int c = lane + 32 * k;
        if (row0 + i < rows && c < dim) S_g[(size_t)(row0 + i) * dim + c] = S[i][k];
      }
  }
}

constexpr int DEC_THREADS = 256;

// One token per request (row t of the batch is request t): grid (H, R, shares of the head's rows). Every block
// convolves its head's x (its rows of it) and its group's B and C, then reads, decays, updates and writes its rows
// of S, ROW_LANES lanes a row, four neighbouring channels a lane at a time (VEC; else one), BATCH rows of a lane
// group in flight at once.
template <int ROW_LANES, int QUADS, bool VEC, typename XT>
__global__ void __launch_bounds__(DEC_THREADS)
ssd_decode_kernel(const Conv cv, const float* __restrict__ d_rows, const float* __restrict__ rate,
                  const float* __restrict__ dt_bias, const float* __restrict__ skip, const int32_t* __restrict__ slots,
                  float* __restrict__ state, long long state_stride, int H, int G, int dim, int vdim, int rows_per_block,
                  float* __restrict__ y) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  extern __shared__ __align__(16) float sm[];       // B [dim, rounded up], C [the same], x [rows]
  constexpr int GROUPS = DEC_THREADS / ROW_LANES;
  constexpr int BATCH = QUADS >= 4 ? 1 : (QUADS == 2 ? 2 : 4);
  const int dpad = (dim + 3) / 4 * 4;
  float *sb = sm, *sc = sm + dpad, *sx = sm + 2 * dpad;
  const int h = blockIdx.x, t = blockIdx.y, p0 = blockIdx.z * rows_per_block, np = min(rows_per_block, vdim - p0);
  const int slot = slots[t];
  const float* kept = slot >= 0 && cv.kept ? cv.kept + (size_t)slot * cv.kept_stride : nullptr;
  const int off_b = H * vdim + h / (H / G) * dim, off_c = off_b + G * dim;
  const int group = threadIdx.x / ROW_LANES, lane = threadIdx.x % ROW_LANES;
  float* S_g = slot >= 0 ? state + (size_t)slot * state_stride + (size_t)h * vdim * dim + (size_t)p0 * dim : nullptr;
  float S[BATCH][QUADS][4];
  auto fetch = [&](int base) {
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int p = base + i * GROUPS;
#pragma unroll
      for (int q = 0; q < QUADS; ++q) {
        const int c = (lane + q * ROW_LANES) * 4;
        if (VEC) {
          const float4 v = (S_g != nullptr && p < np && c < dim) ? *reinterpret_cast<const float4*>(S_g + (size_t)p * dim + c)
                                                                 : make_float4(0.f, 0.f, 0.f, 0.f);
          S[i][q][0] = v.x, S[i][q][1] = v.y, S[i][q][2] = v.z, S[i][q][3] = v.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) S[i][q][e] = (S_g != nullptr && p < np && c + e < dim) ? S_g[(size_t)p * dim + c + e] : 0.f;
        }
      }
    }
  };
  fetch(group);                        // on its way while the convolution runs
  for (int i = threadIdx.x; i < 2 * dpad + np; i += blockDim.x) {
    float v = 0.f;
    if (i >= 2 * dpad) v = conv_silu(cv, kept, t, 0, h * vdim + p0 + i - 2 * dpad);
    else if (i % dpad < dim) v = conv_silu(cv, kept, t, 0, (i < dpad ? off_b : off_c) + i % dpad);
    sm[i] = gb::to_float<XT>(gb::from_float<XT>(v));
  }
  const float dt = softplus(d_rows[(size_t)t * cv.P + h] + dt_bias[h]);
  float keep, change;
  decay_parts(-rate[h] * dt, keep, change);
  const float dskip = skip[h];
  __syncthreads();
  float b[QUADS][4], c4[QUADS][4];
#pragma unroll
  for (int q = 0; q < QUADS; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = (lane + q * ROW_LANES) * 4 + e;
      b[q][e] = c < dim ? dt * sb[c] : 0.f;
      c4[q][e] = c < dim ? sc[c] : 0.f;
    }
  for (int base = group; base < (np + GROUPS - 1) / GROUPS * GROUPS; base += BATCH * GROUPS) {
    if (base != group) fetch(base);
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int p = base + i * GROUPS;
      const float x = p < np ? sx[p] : 0.f;
      float acc = 0.f;
#pragma unroll
      for (int q = 0; q < QUADS; ++q) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[i][q][e] = fmaf(keep, S[i][q][e], fmaf(change, S[i][q][e], x * b[q][e]));
          acc = fmaf(S[i][q][e], c4[q][e], acc);
        }
        const int c = (lane + q * ROW_LANES) * 4;
        if (S_g != nullptr && p < np) {
          if (VEC) {
            if (c < dim) *reinterpret_cast<float4*>(S_g + (size_t)p * dim + c) = make_float4(S[i][q][0], S[i][q][1], S[i][q][2], S[i][q][3]);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (c + e < dim) S_g[(size_t)p * dim + c + e] = S[i][q][e];
          }
        }
      }
#pragma unroll
      for (int o = ROW_LANES / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (lane == 0 && p < np) y[(size_t)t * H * vdim + h * vdim + p0 + p] = fmaf(dskip, x, acc);
    }
  }
}

// Blocks [0, T * parts): one part of one token's row, v = y * silu(z), out = v / sqrt(mean(v^2) + eps) * w. The
// rest: a request's last taps - 1 inputs after this step, oldest first; a thread owns a channel and walks its entries in
// ascending order, reading only entries at or above the one it writes.
template <typename OT>
__global__ void __launch_bounds__(256)
ssd_finish_kernel(const float* __restrict__ y, const float* __restrict__ z_rows, long long P, const float* __restrict__ w,
                  float eps, OT* __restrict__ out, int T, int parts, int inner, const float* __restrict__ rows,
                  float* __restrict__ kept, long long kept_stride, const int32_t* __restrict__ cu_q,
                  const int32_t* __restrict__ slots, int C, int taps, int shift_blocks) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  if (blockIdx.x >= (unsigned)(T * parts)) {
    const int i = blockIdx.x - T * parts, r = i / shift_blocks, c = (i % shift_blocks) * blockDim.x + threadIdx.x;
    const int slot = slots[r];
    if (c >= C || slot < 0) return;
    const int t0 = cu_q[r], n = cu_q[r + 1] - t0, keep = taps - 1;
    float* k = kept + (size_t)slot * kept_stride;
    for (int e = 0; e < keep; ++e) {
      const int src = e + n;                  // index in (kept inputs, then the step's rows)
      k[(size_t)e * C + c] = src < keep ? k[(size_t)src * C + c] : rows[(size_t)(t0 + src - keep) * P + c];
    }
    return;
  }
  extern __shared__ float v_s[];          // [inner / parts]
  __shared__ float red[8];
  const int t = blockIdx.x / parts, part = blockIdx.x % parts, n = inner / parts;
  const float* yr = y + (size_t)t * inner + (size_t)part * n;
  const float* zr = z_rows + (size_t)t * P + (size_t)part * n;
  const float* wr = w + (size_t)part * n;
  float ss = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float v = yr[c] * silu(zr[c]);
    v_s[c] = v;                           // a thread reads back what it wrote itself
    ss = fmaf(v, v, ss);
  }
  ss = gb::warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < warps; ++i) total += red[i];
  const float scale = 1.0f / sqrtf(total / (float)n + eps);
  OT* o = out + (size_t)t * inner + (size_t)part * n;
  for (int c = threadIdx.x; c < n; c += blockDim.x) o[c] = gb::from_float<OT>((v_s[c] * scale) * wr[c]);
}

int check_sizes(const char* what, int H, int G, int dim, int vdim, int taps) {
  if (H < 1 || G < 1 || H % G) return gb::fail(GB_BAD_ARGUMENT, "%s: %d heads in %d groups", what, H, G);
  if (dim < 1 || vdim < 1) return gb::fail(GB_BAD_ARGUMENT, "%s: head sizes %d and %d", what, dim, vdim);
  if (dim > 512) return gb::fail(GB_UNSUPPORTED, "%s: a state of %d channels per row (at most 512)", what, dim);
  if (taps < 1 || taps > MAX_TAPS) return gb::fail(GB_UNSUPPORTED, "%s: %d taps (1 to %d)", what, taps, MAX_TAPS);
  return GB_OK;
}

}  // namespace

// proj [T, P] (see the head of this file); kept: the kept inputs of slot 0 (kept_stride floats between slots). Out: act [T, C]
// (x, B, C of all heads and groups, act_dtype) and step [T, 2 H] (dt, then -rate dt).
GB_EXPORT int gb_ssd_prepare(const float* proj, long long P, int cx, int cd, const float* conv_w, const float* conv_b, int taps,
                             const float* kept, long long kept_stride, const float* rate, const float* dt_bias,
                             const int32_t* token_req, const int32_t* cu_q, const int32_t* slots, void* act, int act_dtype,
                             float* step, int T, int H, int G, int dim, int vdim, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  int rc = check_sizes("ssd_prepare", H, G, dim, vdim, taps);
  if (rc != GB_OK) return rc;
  const int C = H * vdim + 2 * G * dim;
  if (P < cx + C || P < cd + H) return gb::fail(GB_BAD_ARGUMENT, "ssd_prepare: rows of %lld", P);
  if (T > 65535 * PREP_TOKENS) return gb::fail(GB_UNSUPPORTED, "ssd_prepare: %d tokens", T);
  const Conv cv = {proj + cx, P, conv_w, conv_b, taps > 1 ? kept : nullptr, kept_stride, taps, C};
  const bool pairs = C % 2 == 0 && P % 2 == 0 && (((uintptr_t)cv.rows & 7) | ((uintptr_t)act & 7)) == 0;
  const int per_block = PREP_THREADS * (pairs ? 2 : 1);
  const dim3 grid((C + per_block - 1) / per_block + 1, (T + PREP_TOKENS - 1) / PREP_TOKENS);
  return GB_DISPATCH_DTYPE(act_dtype, XT, [&]() -> int {
    auto go = [&](auto n) -> int {
      constexpr int TAPS = decltype(n)::value;
      return gb::check_pdl_launch(
          gb::launch_pdl(pairs ? ssd_prepare_kernel<TAPS, 2, XT> : ssd_prepare_kernel<TAPS, 1, XT>, grid, dim3(PREP_THREADS), 0, stream,
                         dim3(1, 1, 1), cv, proj + cd, rate, dt_bias, token_req, cu_q, slots, (XT*)act, step, T, H),
          "ssd_prepare");
    };
    using std::integral_constant;
    switch (taps) {
      case 1: return go(integral_constant<int, 1>());
      case 2: return go(integral_constant<int, 2>());
      case 3: return go(integral_constant<int, 3>());
      case 4: return go(integral_constant<int, 4>());
      default: return go(integral_constant<int, 0>());
    }
  });
}

// Walks every request's tokens in order; y [T, H vdim]. skip null: no skip term. unit_state, unit_y: see UnitRow.
GB_EXPORT int gb_ssd_recurrence(const void* act, int act_dtype, const float* step, const float* skip, const int32_t* cu_q,
                                const int32_t* slots, float* state, long long state_stride, int R, int H, int G, int dim,
                                int vdim, float* y, float* unit_state, float* unit_y, cudaStream_t stream) {
  if (R <= 0) return GB_OK;
  int rc = check_sizes("ssd_recurrence", H, G, dim, vdim, 1);
  if (rc != GB_OK) return rc;
  if ((unit_state == nullptr) != (unit_y == nullptr)) return gb::fail(GB_BAD_ARGUMENT, "ssd_recurrence: a unit row has a state and a read-out");
  if (R > 65535) return gb::fail(GB_UNSUPPORTED, "ssd_recurrence: %d requests", R);
  const UnitRow unit = {unit_state, unit_y};
  const int rows = REC_WARPS * REC_ROWS, C = H * vdim + 2 * G * dim;
  const dim3 grid(H, R, (vdim + rows - 1) / rows + (unit_state != nullptr));
  return GB_DISPATCH_DTYPE(act_dtype, XT, [&]() -> int {
    auto go = [&](auto per) -> int {
      return gb::check_pdl_launch(gb::launch_after(ssd_recurrence_kernel<decltype(per)::value, XT>, grid, dim3(REC_WARPS * 32), 0, stream,
                                                   dim3(1, 1, 1), (const XT*)act, C, step, skip, cu_q, slots, state, state_stride, H,
                                                   G, dim, vdim, y, unit),
                                  "ssd_recurrence");
    };
    if (dim <= 32) return go(std::integral_constant<int, 1>());
    if (dim <= 64) return go(std::integral_constant<int, 2>());
    if (dim <= 128) return go(std::integral_constant<int, 4>());
    if (dim <= 256) return go(std::integral_constant<int, 8>());
    return go(std::integral_constant<int, 16>());
  });
}

// One token per request. act_dtype: what the convolved activations are rounded to.
GB_EXPORT int gb_ssd_decode(const float* proj, long long P, int cx, int cd, const float* conv_w, const float* conv_b, int taps,
                            const float* kept, long long kept_stride, const float* rate, const float* dt_bias,
                            const float* skip, const int32_t* slots, float* state, long long state_stride, int R, int H, int G,
                            int dim, int vdim, int act_dtype, float* y, cudaStream_t stream) {
  if (R <= 0) return GB_OK;
  int rc = check_sizes("ssd_decode", H, G, dim, vdim, taps);
  if (rc != GB_OK) return rc;
  const int C = H * vdim + 2 * G * dim;
  if (P < cx + C || P < cd + H) return gb::fail(GB_BAD_ARGUMENT, "ssd_decode: rows of %lld", P);
  if (R > 65535) return gb::fail(GB_UNSUPPORTED, "ssd_decode: %d requests", R);
  const Conv cv = {proj + cx, P, conv_w, conv_b, taps > 1 ? kept : nullptr, kept_stride, taps, C};
  // a head's rows over several blocks while (head, request) pairs alone leave SMs idle
  int shares = 1;
  while (shares < 8 && (long long)H * R * shares < 148 && vdim / (2 * shares) >= 8) shares *= 2;
  const int rows = (vdim + shares - 1) / shares;
  const dim3 grid(H, R, (vdim + rows - 1) / rows);
  const size_t smem = (size_t)(2 * ((dim + 3) / 4 * 4) + rows) * sizeof(float);
  if (smem > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "ssd_decode: %d value channels per head", vdim);
  const bool vec = dim % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  return GB_DISPATCH_DTYPE(act_dtype, XT, [&]() -> int {
    auto go = [&](auto lanes, auto quads) -> int {
      constexpr int L = decltype(lanes)::value, Q = decltype(quads)::value;
      return gb::check_pdl_launch(
          gb::launch_pdl(vec ? ssd_decode_kernel<L, Q, true, XT> : ssd_decode_kernel<L, Q, false, XT>, grid, dim3(DEC_THREADS), smem,
                         stream, dim3(1, 1, 1), cv, proj + cd, rate, dt_bias, skip, slots, state, state_stride, H, G, dim, vdim,
                         rows, y),
          "ssd_decode");
    };
    using std::integral_constant;
    if (dim <= 16) return go(integral_constant<int, 4>(), integral_constant<int, 1>());
    if (dim <= 32) return go(integral_constant<int, 8>(), integral_constant<int, 1>());
    if (dim <= 64) return go(integral_constant<int, 16>(), integral_constant<int, 1>());
    if (dim <= 128) return go(integral_constant<int, 32>(), integral_constant<int, 1>());
    if (dim <= 256) return go(integral_constant<int, 32>(), integral_constant<int, 2>());
    return go(integral_constant<int, 32>(), integral_constant<int, 4>());
  });
}

// out [T, inner] from y [T, inner] and the gate z (columns cz .. of proj); the kept inputs of the batch's R requests
// are moved on by the step's rows (taps > 1).
GB_EXPORT int gb_ssd_finish(const float* y, const float* proj, long long P, int cz, int cx, const float* w, float eps, void* out,
                            int out_dtype, int T, int parts, int inner, float* kept, long long kept_stride,
                            const int32_t* cu_q, const int32_t* slots, int R, int C, int taps, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if (parts < 1 || inner % parts) return gb::fail(GB_BAD_ARGUMENT, "ssd_finish: %d channels in %d parts", inner, parts);
  const int n = inner / parts;
  if ((size_t)n * sizeof(float) > 48 * 1024) return gb::fail(GB_UNSUPPORTED, "ssd_finish: parts of %d channels (at most 12288)", n);
  const int threads = n >= 1024 ? 256 : (n >= 256 ? 128 : (n >= 64 ? 64 : 32));
  const int shift_blocks = taps > 1 ? (C + threads - 1) / threads : 0;
  const long long blocks = (long long)T * parts + (long long)R * shift_blocks;
  if (blocks > 0x7fffffffLL) return gb::fail(GB_UNSUPPORTED, "ssd_finish: %d tokens", T);
  return GB_DISPATCH_DTYPE(out_dtype, OT, [&]() -> int {
    return gb::check_pdl_launch(
        gb::launch_pdl(ssd_finish_kernel<OT>, dim3((unsigned)blocks), dim3(threads), (size_t)n * sizeof(float), stream, dim3(1, 1, 1), y,
                       proj + cz, P, w, eps, (OT*)out, T, parts, inner, proj + cx, kept, kept_stride, cu_q, slots, C, taps,
                       shift_blocks),
        "ssd_finish");
  });
}
