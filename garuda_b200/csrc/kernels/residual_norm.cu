// What stands between two sublayers' products in a layer with norms in front of and behind each sublayer, as one
// pass over the residual's row; and the normed embedding such a model starts from. 32-bit arithmetic.
//
//   residual_norm    x <- x + rms(y) * w_y (or + y, or nothing) + row;   out = rms(x) * w_out, or x, in out's dtype;
//                    y may be what routed experts leave for it: a row per (token, choice) pair, summed with the
//                    choices' weights as it is read
//   embedding_norm   x = rms(table[id]) * w;   pair = [x | x] in its dtype (the operand of a product that mixes the
//                    stream with the embedding's output: its first half is written again before every mix)
#include <type_traits>

#include "common.cuh"

GB_DEFINE_LAST_ERROR()

namespace {

inline bool host_aligned(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

// The block's sum of one value per thread, added up in the same order by every thread.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = gb::warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  __syncthreads();                  // `red` may still be read from the call before
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return gb::warp_sum(lane < warps ? red[lane] : 0.f);
}

__device__ __forceinline__ void store4(float* to, const float (&v)[4]) { *reinterpret_cast<float4*>(to) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* to, const float (&v)[4]) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 packed;
  packed.x = *reinterpret_cast<uint32_t*>(&lo);
  packed.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(to) = packed;
}

struct NormStep {
  float* x;                  // [T, d]
  const float* y;            // [T, d] or null
  const float* y_w;          // [d] or null: y is added as it is
  const float* row;          // [d] or null
  const float* out_w;        // [d] or null: out is x in its dtype
  float y_eps, out_eps;
  long long out_stride;
  int d;
  // routed experts' rows, added to y: sum_j weights[t][j] * rows[pair_row[t top + j]], j in the router's order; a pair without a row
  // stands for identity[t] (null: nothing). top 0: none.
  const float* rows;         // [num_rows, d]
  const int32_t* pair_row;
  const float* weights;      // [T, top]
  const __nv_bfloat16* identity;
  int top, num_rows;
};

// One block per token; a thread keeps PER groups of four neighbouring channels of the row in registers from the
// first read to the last write. VEC: rows start on 16 bytes and d is a multiple of four.
template <int PER, bool VEC, typename OT>
__global__ void __launch_bounds__(PER >= 4 ? 512 : 1024)
residual_norm_kernel(const NormStep p, OT* __restrict__ out) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  __shared__ float red[32];
  const size_t t = blockIdx.x;
  const int d = p.d;
  float* xr = p.x + t * d;
  auto load4 = [&](const float* from, int c, float (&v)[4]) {
    if (VEC) {
      const float4 q = *reinterpret_cast<const float4*>(from + c);
      v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = c + j < d ? from[c + j] : 0.f;
    }
  };
  float x[PER][4];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) x[k][j] = 0.f;
    if (c < d) load4(xr, c, x[k]);
  }
  const bool adds = p.y != nullptr || p.top > 0;
  if (adds) {
    float y[PER][4], ss = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * 4;
#pragma unroll
      for (int j = 0; j < 4; ++j) y[k][j] = 0.f;
      if (c < d && p.y != nullptr) load4(p.y + t * d, c, y[k]);
    }
#pragma unroll 2
    for (int e = 0; e < p.top; ++e) {
      const int from = p.pair_row[t * p.top + e];
      const float wt = p.weights[t * p.top + e];
#pragma unroll
      for (int k = 0; k < PER; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        if (c >= d) continue;
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (from >= 0 && from < p.num_rows) {
          load4(p.rows + (size_t)from * d, c, v);
        } else if (p.identity != nullptr) {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (VEC || c + j < d) v[j] = __bfloat162float(p.identity[t * d + c + j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) y[k][j] = fmaf(wt, v[j], y[k][j]);
      }
    }
#pragma unroll
    for (int k = 0; k < PER; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) ss = fmaf(y[k][j], y[k][j], ss);
    const float inv = p.y_w != nullptr ? 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.y_eps) : 1.0f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * 4;
      float w[4] = {1.f, 1.f, 1.f, 1.f};
      if (p.y_w != nullptr && c < d) load4(p.y_w, c, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) x[k][j] += (y[k][j] * inv) * w[j];
    }
  }
  if (p.row != nullptr) {
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * 4;
      if (c >= d) continue;
      float r[4];
      load4(p.row, c, r);
#pragma unroll
      for (int j = 0; j < 4; ++j) x[k][j] += r[j];
    }
  }
  if (adds || p.row != nullptr) {
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * 4;
      if (c >= d) continue;
      if (VEC) {
        store4(xr + c, x[k]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j < d) xr[c + j] = x[k][j];
      }
    }
  }
  if (out == nullptr) return;
  float inv = 1.0f;
  if (p.out_w != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (VEC || (threadIdx.x + k * blockDim.x) * 4 + j < d) ss = fmaf(x[k][j], x[k][j], ss);
    inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.out_eps);
  }
  OT* o = out + t * p.out_stride;
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 4;
    if (c >= d) continue;
    float w[4] = {1.f, 1.f, 1.f, 1.f}, v[4];
    if (p.out_w != nullptr) load4(p.out_w, c, w);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = (x[k][j] * inv) * w[j];
    if (VEC) {
      store4(o + c, v);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < d) o[c + j] = gb::from_float<OT>(v[j]);
    }
  }
}

// One block per token.
template <typename ET, typename OT>
__global__ void __launch_bounds__(256)
embedding_norm_kernel(const ET* __restrict__ table, const int32_t* __restrict__ ids, const float* __restrict__ w, float eps,
                      float* __restrict__ x, OT* __restrict__ pair, int d, int vocab) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  __shared__ float red[32];
  const size_t t = blockIdx.x;
  const int id = ids[t];
  const bool known = id >= 0 && id < vocab;          // refused on the host before any launch; never read out of range
  const ET* row = table + (size_t)(known ? id : 0) * d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float v = gb::to_float<ET>(row[c]);
    ss = fmaf(v, v, ss);
  }
  const float inv = known ? 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps) : 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float v = (gb::to_float<ET>(row[c]) * inv) * w[c];
    x[t * d + c] = v;
    if (pair != nullptr) pair[t * 2 * d + c] = pair[t * 2 * d + d + c] = gb::from_float<OT>(v);
  }
}

}  // namespace

// x [T, d]; y [T, d], y_w [d], row [d], out_w [d]: 32-bit, each may be null; out [T, d] with rows out_stride apart, or null.
// rows [num_rows, d] 32-bit, pair_row and weights [T, top], identity [T, d] bfloat16 or null: see NormStep (top 0: none of them).
GB_EXPORT int gb_residual_norm(float* x, const float* y, const float* y_w, float y_eps, const float* row, const float* out_w,
                               float out_eps, void* out, int out_dtype, long long out_stride, int T, int d, const float* rows,
                               const int32_t* pair_row, const float* weights, const void* identity, int top, int num_rows,
                               cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if (d < 1 || d > 16384) return gb::fail(GB_UNSUPPORTED, "residual_norm: rows of %d (1 to 16384)", d);
  if (out != nullptr && out_stride < d) return gb::fail(GB_BAD_ARGUMENT, "residual_norm: out rows %lld apart", out_stride);
  if (top < 0 || (top > 0 && (!rows || !pair_row || !weights))) return gb::fail(GB_BAD_ARGUMENT, "residual_norm: %d choices without their rows", top);
  const NormStep p = {x, y, y_w, row, out_w, y_eps, out_eps, out_stride, d, rows, pair_row, weights, (const __nv_bfloat16*)identity, top, num_rows};
  const int elem = out_dtype == GB_F32 ? 4 : 2;
  const bool vec = d % 4 == 0 && out_stride % 4 == 0 && host_aligned(x, 16) && host_aligned(y, 16) && host_aligned(y_w, 16) &&
                   host_aligned(row, 16) && host_aligned(out_w, 16) && host_aligned(out, 4 * elem) && host_aligned(rows, 16);
  const int quads = (d + 3) / 4;
  // few tokens: as many threads as the row has groups of four, up to two groups a thread; many: smaller blocks, more
  // of them to an SM
  int threads = T >= 296 ? (quads > 256 * 8 ? 512 : 256) : (quads > 1024 * 2 ? 512 : 1024);
  threads = quads < threads ? (quads + 31) / 32 * 32 : threads;
  const int per = (quads + threads - 1) / threads;
  return GB_DISPATCH_DTYPE(out_dtype, OT, [&]() -> int {
    auto go = [&](auto n) -> int {
      constexpr int PER = decltype(n)::value;
      return gb::check_pdl_launch(gb::launch_pdl(vec ? residual_norm_kernel<PER, true, OT> : residual_norm_kernel<PER, false, OT>, dim3(T),
                                                 dim3(threads), 0, stream, dim3(1, 1, 1), p, (OT*)out),
                                  "residual_norm");
    };
    using std::integral_constant;
    if (per <= 1) return go(integral_constant<int, 1>());
    if (per <= 2) return go(integral_constant<int, 2>());
    if (per <= 4) return go(integral_constant<int, 4>());
    return go(integral_constant<int, 8>());
  });
}

// table [vocab, d], w [d] 32-bit; x [T, d] 32-bit; pair [T, 2 d] or null.
GB_EXPORT int gb_embedding_norm(const void* table, int table_dtype, const int32_t* ids, const float* w, float eps, float* x, void* pair,
                                int pair_dtype, int T, int d, int vocab, cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  if (d < 1 || vocab < 1) return gb::fail(GB_BAD_ARGUMENT, "embedding_norm: a table of %d rows of %d", vocab, d);
  const int threads = d >= 256 ? 256 : (d + 31) / 32 * 32;
  return GB_DISPATCH_DTYPE(table_dtype, ET, [&]() -> int {
    return GB_DISPATCH_DTYPE(pair_dtype, OT, [&]() -> int {
      return gb::check_pdl_launch(gb::launch_pdl(embedding_norm_kernel<ET, OT>, dim3(T), dim3(threads), 0, stream, dim3(1, 1, 1),
                                                 (const ET*)table, ids, w, eps, x, (OT*)pair, d, vocab),
                                  "embedding_norm");
    });
  });
}
