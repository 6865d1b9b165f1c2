// Causal differential attention over the paged cache (Ye et al., "Differential Transformer", 2024), one warp per
// (token, head), 32-bit arithmetic throughout: the attention of the 32-bit path, and of sizes the tensor-core
// kernel does not take. With the two maps r = 1, 2 of a head over the same values:
//     p^r_j = softmax over the seen keys of (q^r . k^r_j) * scale;   o = sum_j (p^1_j - lambda p^2_j) v_j
//     out = o / sqrt(mean(o^2) + eps) * out_scale * sigmoid(gate)
// A query row is [map 1 | map 2], a cached key row too; seen: 0 <= i - j < window (0: every j <= i). Keys are walked 32
// at a time from the first seen, each map with a running maximum and sum, so the result for a token does not
// depend on what else is in the batch or on how its prompt was cut.
#include "common.cuh"

namespace {

constexpr int WARPS = 4;

template <typename T, int MAX_D>
__global__ void __launch_bounds__(WARPS * 32)
diff_attention_simple_kernel(const T* __restrict__ q, const T* __restrict__ k_pool, const T* __restrict__ v_pool,
                             const int32_t* __restrict__ block_table, int table_width, const int32_t* __restrict__ cu_q,
                             const int32_t* __restrict__ kv_lens, const int32_t* __restrict__ token_req, T* __restrict__ out, int Hq,
                             int Hkv, int dim, int vd, float scale, int window, int page_size, float lambda, float out_scale,
                             float eps, const float* __restrict__ gate, long long gate_stride) {
  __shared__ float q_s[WARPS][2 * MAX_D];
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * WARPS + warp;
  if (h >= Hq) return;
  const int r = token_req[t];
  const int pos = kv_lens[r] - (cu_q[r + 1] - cu_q[r]) + (t - cu_q[r]);
  const int start = window > 0 ? max(0, pos + 1 - window) : 0;
  const int kvh = h / (Hq / Hkv);
  const int32_t* table = block_table + (size_t)r * table_width;
  const T* qr = q + ((size_t)t * Hq + h) * 2 * dim;
  for (int c = lane; c < 2 * dim; c += 32) q_s[warp][c] = gb::to_float<T>(qr[c]);
  __syncwarp();

  constexpr int ACC = MAX_D / 32;
  const int nacc = (vd + 31) / 32;
  float acc[2][ACC], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int i = 0; i < ACC; ++i) acc[a][i] = 0.f;

  for (int base = start; base <= pos; base += 32) {
    const int j = base + lane;
    long long row = -1;  // this lane's key in the pool, in rows
    if (j <= pos) {
      const int page = table[j / page_size];
      if (page >= 0) row = ((long long)page * Hkv + kvh) * page_size + (j % page_size);
    }
    float p[2];
    float part[2][ACC];          // the block's keys summed by themselves, then added to the keys in front
    float corr[2];
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      float s = -INFINITY;
      if (row >= 0) {
        const T* kr = k_pool + row * 2 * dim + a * dim;
        const float* qa = q_s[warp] + a * dim;
        // eight interleaved sums, added up as a tree: less rounding than one sum of dim terms
        float d8[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        int c = 0;
        for (; c + 8 <= dim; c += 8)
#pragma unroll
          for (int e = 0; e < 8; ++e) d8[e] = fmaf(qa[c + e], gb::to_float<T>(kr[c + e]), d8[e]);
        for (int e = 0; c + e < dim; ++e) d8[0] = fmaf(qa[c + e], gb::to_float<T>(kr[c + e]), d8[0]);
        s = (((d8[0] + d8[1]) + (d8[2] + d8[3])) + ((d8[4] + d8[5]) + (d8[6] + d8[7]))) * scale;
      }
      const float m_new = fmaxf(m[a], gb::warp_max(s));
      p[a] = row >= 0 ? expf(s - m_new) : 0.f;
      corr[a] = m[a] == -INFINITY ? 0.f : expf(m[a] - m_new);
      l[a] = l[a] * corr[a] + gb::warp_sum(p[a]);
      m[a] = m_new;
#pragma unroll
      for (int i = 0; i < ACC; ++i) part[a][i] = 0.f;
    }
    const int n_here = min(32, pos - base + 1);
    for (int jj = 0; jj < n_here; ++jj) {
      const float p1 = __shfl_sync(0xffffffffu, p[0], jj), p2 = __shfl_sync(0xffffffffu, p[1], jj);
      const long long rj = __shfl_sync(0xffffffffu, row, jj);
      if (rj < 0) continue;
      const T* vr = v_pool + rj * vd;
#pragma unroll
      for (int i = 0; i < ACC; ++i) {
        const int c = lane + 32 * i;
        if (i < nacc && c < vd) {
          const float v = gb::to_float<T>(vr[c]);
          part[0][i] = fmaf(p1, v, part[0][i]);
          part[1][i] = fmaf(p2, v, part[1][i]);
        }
      }
    }
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int i = 0; i < ACC; ++i) acc[a][i] = fmaf(acc[a][i], corr[a], part[a][i]);
  }
  const float inv1 = l[0] > 0.f ? 1.0f / l[0] : 0.f, inv2 = l[1] > 0.f ? lambda / l[1] : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ACC; ++i) {
    acc[0][i] = acc[0][i] * inv1 - acc[1][i] * inv2;           // channels beyond vd stay zero
    ss = fmaf(acc[0][i], acc[0][i], ss);
  }
  float by = out_scale / sqrtf(gb::warp_sum(ss) / (float)vd + eps);
  if (gate != nullptr) by *= 1.0f / (1.0f + expf(-gate[(size_t)t * gate_stride + h]));
  T* o = out + ((size_t)t * Hq + h) * vd;
#pragma unroll
  for (int i = 0; i < ACC; ++i) {
    const int c = lane + 32 * i;
    if (i < nacc && c < vd) o[c] = gb::from_float<T>(acc[0][i] * by);
  }
}

}  // namespace

// q [T, Hq, 2 dim], k_pool [pages, Hkv, page_size, 2 dim], v_pool [pages, Hkv, page_size, vd], out [T, Hq vd], one dtype;
// gate: 32-bit logits [T, Hq] with rows gate_stride apart, or null.
GB_EXPORT int gb_diff_attention_simple(const void* q, const void* k_pool, const void* v_pool, int dtype, const int32_t* block_table,
                                       int table_width, const int32_t* cu_q, const int32_t* kv_lens, const int32_t* token_req,
                                       void* out, int T, int Hq, int Hkv, int dim, int vd, float scale, int window, int page_size,
                                       float lambda, float out_scale, float eps, const float* gate, long long gate_stride,
                                       cudaStream_t stream) {
  if (T <= 0) return GB_OK;
  constexpr int WIDEST = 512;
  if (dim < 1 || vd < 1 || dim > WIDEST || vd > WIDEST)
    return gb::fail(GB_UNSUPPORTED, "diff_attention: maps of %d and values of %d channels (1 to %d)", dim, vd, WIDEST);
  if (Hkv < 1 || Hq % Hkv) return gb::fail(GB_BAD_ARGUMENT, "diff_attention: %d query heads for %d kv heads", Hq, Hkv);
  if (window < 0 || page_size < 1) return gb::fail(GB_BAD_ARGUMENT, "diff_attention: a window of %d, pages of %d", window, page_size);
  dim3 grid(T, (Hq + WARPS - 1) / WARPS);
  return GB_DISPATCH_DTYPE(dtype, TT, [&]() -> int {
    auto kernel = dim <= 128 && vd <= 128 ? diff_attention_simple_kernel<TT, 128> : diff_attention_simple_kernel<TT, WIDEST>;
    kernel<<<grid, WARPS * 32, 0, stream>>>((const TT*)q, (const TT*)k_pool, (const TT*)v_pool, block_table, table_width, cu_q, kv_lens,
                                            token_req, (TT*)out, Hq, Hkv, dim, vd, scale, window, page_size, lambda, out_scale, eps,
                                            gate, gate_stride);
    return gb::check_launch("diff_attention");
  });
}
