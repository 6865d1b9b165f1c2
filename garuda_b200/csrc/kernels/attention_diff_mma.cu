// bfloat16 differential attention over the paged cache on the tensor cores (mma.sync m16n8k16, 32-bit accumulation),
// flash-style: every head has two softmax maps over the same values, of which the second, times lambda, is taken
// off the first (Ye et al., "Differential Transformer", 2024).
//     p^r_ij = softmax over 0 <= i - j < window (0: every j <= i) of (q^r_i . k^r_j) * scale,   r = 1, 2
//     o_i = sum_j (p^1_ij - lambda p^2_ij) v_j;   out_i = o_i / sqrt(mean(o_i^2) + eps) * out_scale * sigmoid(gate_i)
// A query row is [map 1 | map 2] and so is a cached key row, so a tile of keys and values is brought to shared memory
// once for both maps. The eight warps of a CTA are (map) x (a share of the work); each runs an ordinary online softmax
// over its map, and the maps meet at the end, in 32-bit and in shared memory: difference, norm and gate are the
// epilogue, and neither map is rounded before the other is taken off it. The rows of a query tile are (token,
// head-of-group) pairs of one key/value head of one request. Two shapes of one kernel:
//  * TILE (prompt portions): 64 rows per CTA, 16 per warp of each map, every warp walks all key tiles.
//  * DECODE (a request with at most 16 rows): the four warps of a map take a quarter of every tile's keys each for the
//    same rows; `splits` CTAs share a request's tiles and leave partial results in the caller's scratch, which a
//    second kernel merges in split order.
//
// Compiled per (GB_MAP_DIM = channels of one map, GB_VALUE_DIM), multiples of 16 up to 128.
#include "attention_mma_core.cuh"
#include "common.cuh"

#ifndef GB_MAP_DIM
#define GB_MAP_DIM 64
#endif
#ifndef GB_VALUE_DIM
#define GB_VALUE_DIM 128
#endif

namespace {

using namespace attn_mma;

constexpr int D = GB_MAP_DIM, KD = 2 * D, VD = GB_VALUE_DIM;
static_assert(D % 16 == 0 && D >= 16 && D <= 128 && VD % 16 == 0 && VD >= 16 && VD <= 128, "widths are multiples of 16 up to 128");
constexpr int LDK = KD + 8, LDV = VD + 8, LDO = VD + 4;
constexpr int THREADS = 256, MERGE_THREADS = 128;
constexpr int ROWS_TILE = 64, ROWS_DECODE = 16;
constexpr int MAX_SPLITS = 32;
constexpr int PR = VD + 2;                 // floats of a row's partial result: sums, maximum, denominator
constexpr float LOG2E = 1.4426950408889634f;
constexpr size_t TILES_BYTES = (size_t)(ROWS_TILE * LDK + 2 * KT * (LDK + LDV)) * sizeof(__nv_bfloat16);
constexpr size_t PARTS_BYTES = (size_t)8 * ROWS_DECODE * PR * sizeof(float);
constexpr size_t SMEM = TILES_BYTES > PARTS_BYTES ? TILES_BYTES : PARTS_BYTES;
static_assert((size_t)ROWS_TILE * LDO * sizeof(float) <= SMEM, "the second map's rows fit where the tiles were");

using KeyTile = PaddedTile<D, LDK>;
using ValueTile = PaddedTile<VD, LDV>;

struct Params {
  const __nv_bfloat16* q;        // [T, Hq, KD]
  const __nv_bfloat16* k_pool;   // [pages, Hkv, page_size, KD]
  const __nv_bfloat16* v_pool;   // [pages, Hkv, page_size, VD]
  __nv_bfloat16* out;            // [T, Hq * VD]
  const int32_t* block_table;
  const int32_t* cu_q;
  const int32_t* kv_lens;
  float* partials;               // [R, Hkv, splits, 2 maps, ROWS_DECODE, PR] (DECODE with splits > 1)
  int table_width, Hq, Hkv, g, window, page_size, splits;
  float scale_log2, lambda, out_scale, eps;
  const float* gate;             // logits [T, Hq], rows gate_stride apart, or null
  long long gate_stride;
};

__device__ __forceinline__ void cp_async_16(void* smem, const void* gmem, bool valid) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s), "l"(gmem), "r"(bytes) : "memory");
}

// Keys [tile_start, tile_start + 64) of one kv head, keys of both maps and values, 16 bytes per copy. Keys outside
// [lo, hi] or without a page become zeros (a reused page may hold anything, and zero times a NaN is a NaN).
__device__ __forceinline__ void load_kv_tile(__nv_bfloat16* ks, __nv_bfloat16* vs, int64_t* where, const Params& p, const int32_t* table,
                                             int kvh, int tile_start, int lo, int hi) {
  __syncthreads();        // the copies of the tile in front have read `where`
  if (threadIdx.x < KT) {
    const int j = tile_start + threadIdx.x;
    int64_t w = -1;
    if (j <= hi && j >= lo) {
      const int page = table[j / p.page_size];
      if (page >= 0) w = ((int64_t)page * p.Hkv + kvh) * p.page_size + (j % p.page_size);
    }
    where[threadIdx.x] = w;
  }
  __syncthreads();
  constexpr int CK = KD / 8, CV = VD / 8;
  for (int c = threadIdx.x; c < KT * CK; c += THREADS) {
    const int row = c / CK, ch = c % CK;
    const int64_t w = where[row];
    cp_async_16(ks + row * LDK + ch * 8, p.k_pool + (w >= 0 ? (size_t)w * KD + ch * 8 : 0), w >= 0);
  }
  for (int c = threadIdx.x; c < KT * CV; c += THREADS) {
    const int row = c / CV, ch = c % CV;
    const int64_t w = where[row];
    cp_async_16(vs + row * LDV + ch * 8, p.v_pool + (w >= 0 ? (size_t)w * VD + ch * 8 : 0), w >= 0);
  }
}

// What a row's difference is multiplied by: the norm, the constant and the gate.
__device__ __forceinline__ float row_factor(const Params& p, float sum_of_squares, int token, int head) {
  float by = p.out_scale / sqrtf(sum_of_squares / (float)VD + p.eps);
  if (p.gate != nullptr) by *= 1.0f / (1.0f + expf(-p.gate[(size_t)token * p.gate_stride + head]));
  return by;
}

// One channel of the parts' sums of one map: parts `stride` floats apart. Returns the quotient.
__device__ __forceinline__ float merged(const float* part, size_t stride, int n, int c, float scale_log2) {
  float m = -INFINITY;
#pragma unroll 8
  for (int s = 0; s < n; ++s) m = fmaxf(m, part[s * stride + VD]);
  float o = 0.f, l = 0.f;
#pragma unroll 8
  for (int s = 0; s < n; ++s) {
    const float ms = part[s * stride + VD];
    const float f = ms == -INFINITY ? 0.f : fast_exp2((ms - m) * scale_log2);
    o = fmaf(part[s * stride + c], f, o);
    l = fmaf(part[s * stride + VD + 1], f, l);
  }
  return l > 0.f ? o / l : 0.f;
}

// grid (x, Hkv, R): TILE: x a tile of 64 rows of the request; DECODE: x one of p.splits shares of the keys.
template <bool DECODE>
__global__ void __launch_bounds__(THREADS, (D <= 64 && VD <= 64) ? 2 : 1)
diff_attention_kernel(const Params p) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [ROWS_TILE][LDK]
  __nv_bfloat16* kv = qs + ROWS_TILE * LDK;                          // 2 stages x ([KT][LDK], [KT][LDV])
  __shared__ int64_t where[KT];
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  const int r = blockIdx.z, kvh = blockIdx.y;
  const int q_begin = p.cu_q[r], q_len = p.cu_q[r + 1] - q_begin;
  const bool small = q_len * p.g <= ROWS_DECODE;
  if (small != DECODE || q_len <= 0) return;
  const int tokens_per_tile = DECODE ? q_len : ROWS_TILE / p.g;
  const int tok0 = DECODE ? 0 : blockIdx.x * tokens_per_tile;
  if (tok0 >= q_len) return;
  const int kv_len = p.kv_lens[r];
  const int32_t* table = p.block_table + (size_t)r * p.table_width;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, map = warp >> 2, share = warp & 3;
  const int ntok = min(tokens_per_tile, q_len - tok0);
  const int nrows = ntok * p.g;
  const int pos0 = kv_len - q_len + tok0;
  auto first_seen = [&](int pos) { return p.window > 0 ? max(0, pos + 1 - p.window) : 0; };
  const int lo = first_seen(pos0), hi = pos0 + ntok - 1;
  const int last_start = first_seen(hi);             // the first position that the tile's last row reads
  const int tile_begin = lo / KT, tile_end = hi / KT + 1;
  int w_begin = tile_begin, w_end = tile_end;
  if (DECODE && p.splits > 1) {
    const int per = (tile_end - tile_begin + p.splits - 1) / p.splits;
    w_begin = min(tile_end, tile_begin + (int)blockIdx.x * per);
    w_end = min(tile_end, w_begin + per);
  }
  auto load = [&](int w, int stage) {
    __nv_bfloat16* ks = kv + stage * KT * (LDK + LDV);
    load_kv_tile(ks, ks + KT * LDK, where, p, table, kvh, w * KT, lo, hi);
  };
  // queries: row = token_local * g + head_of_group
  for (int c = threadIdx.x; c < ROWS_TILE * (KD / 8); c += THREADS) {
    const int row = c / (KD / 8), ch = c % (KD / 8);
    const bool valid = row < nrows;
    const int tok = valid ? row / p.g : 0, gh = valid ? row % p.g : 0;
    cp_async_16(qs + row * LDK + ch * 8, p.q + ((size_t)(q_begin + tok0 + tok) * p.Hq + kvh * p.g + gh) * KD + ch * 8, valid);
  }
  if (w_begin < w_end) load(w_begin, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  const int my_rows = DECODE ? 0 : share * 16;         // first row of the warp's 16
  int row_pos[2], row_start[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = my_rows + lane / 4 + 8 * i;
    row_pos[i] = row < nrows ? pos0 + row / p.g : -1;
    row_start[i] = row < nrows ? first_seen(row_pos[i]) : 0;
  }
  WarpState<VD> st;
  st.reset();
  uint32_t qf[D / 16][4];
  const bool works = DECODE || my_rows < nrows;       // a warp whose rows are all padding only copies
  for (int w = w_begin; w < w_end; ++w) {
    const int stage = (w - w_begin) & 1;
    const __nv_bfloat16* ks = kv + stage * KT * (LDK + LDV) + map * D;
    const __nv_bfloat16* vs = kv + stage * KT * (LDK + LDV) + KT * LDK;
    if (w + 1 < w_end) load(w + 1, stage ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    if (w == w_begin) {
#pragma unroll
      for (int kk = 0; kk < D / 16; ++kk)
        ldmatrix_x4(qf[kk], qs + (my_rows + (lane % 16)) * LDK + map * D + kk * 16 + (lane / 16) * 8);
    }
    if (works) {
      // no mask where the tile lies wholly before the first row's position and inside the last row's window
      const bool full = w * KT + KT - 1 <= pos0 && w * KT >= last_start;
      if (DECODE)
        process_tile<D, 16>(st, qf, KeyTile{ks + share * 16 * LDK}, ValueTile{vs + share * 16 * LDV}, w * KT + share * 16, row_pos,
                            row_start, p.scale_log2, full);
      else
        process_tile<D, KT>(st, qf, KeyTile{ks}, ValueTile{vs}, w * KT, row_pos, row_start, p.scale_log2, full);
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    st.l[i] += __shfl_xor_sync(0xffffffffu, st.l[i], 1);
    st.l[i] += __shfl_xor_sync(0xffffffffu, st.l[i], 2);
  }
  __syncthreads();                                     // the tiles are no longer read
  if (!DECODE) {
    float* second = reinterpret_cast<float*>(smem_raw);       // [ROWS_TILE][LDO]: lambda times the second map's rows
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = my_rows + lane / 4 + 8 * i;
      const float inv = st.l[i] > 0.f ? (map == 1 ? p.lambda : 1.0f) / st.l[i] : 0.f;
#pragma unroll
      for (int n = 0; n < VD / 8; ++n) {
        st.o[n][2 * i] *= inv;
        st.o[n][2 * i + 1] *= inv;
        if (map == 1) *reinterpret_cast<float2*>(second + row * LDO + n * 8 + (lane % 4) * 2) = make_float2(st.o[n][2 * i], st.o[n][2 * i + 1]);
      }
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = my_rows + lane / 4 + 8 * i;
      float ss = 0.f;
#pragma unroll
      for (int n = 0; n < VD / 8; ++n) {
        const float2 b = *reinterpret_cast<const float2*>(second + row * LDO + n * 8 + (lane % 4) * 2);
        st.o[n][2 * i] -= b.x;
        st.o[n][2 * i + 1] -= b.y;
        ss = fmaf(st.o[n][2 * i], st.o[n][2 * i], fmaf(st.o[n][2 * i + 1], st.o[n][2 * i + 1], ss));
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (row >= nrows) continue;
      const int token = q_begin + tok0 + row / p.g, head = kvh * p.g + row % p.g;
      const float by = row_factor(p, ss, token, head);
      __nv_bfloat16* dst = p.out + ((size_t)token * p.Hq + head) * VD;
#pragma unroll
      for (int n = 0; n < VD / 8; ++n)
        *reinterpret_cast<uint32_t*>(dst + n * 8 + (lane % 4) * 2) = pack_bf16(st.o[n][2 * i] * by, st.o[n][2 * i + 1] * by);
    }
    return;
  }
  // DECODE: the warps' states over their quarters of the keys, merged in warp order
  float* part = reinterpret_cast<float*>(smem_raw);       // [2 maps][4][ROWS_DECODE][PR]
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float* pr = part + ((size_t)warp * ROWS_DECODE + lane / 4 + 8 * i) * PR;
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
      pr[n * 8 + (lane % 4) * 2] = st.o[n][2 * i];
      pr[n * 8 + (lane % 4) * 2 + 1] = st.o[n][2 * i + 1];
    }
    if (lane % 4 == 0) {
      pr[VD] = st.m[i];
      pr[VD + 1] = st.l[i];
    }
  }
  __syncthreads();
  if (p.splits > 1) {
    for (int idx = threadIdx.x; idx < 2 * ROWS_DECODE * VD; idx += THREADS) {
      const int a = idx / (ROWS_DECODE * VD), row = idx / VD % ROWS_DECODE, c = idx % VD;
      if (row >= nrows) continue;
      const float* from = part + ((size_t)a * 4 * ROWS_DECODE + row) * PR;
      float m = -INFINITY, o = 0.f, l = 0.f;
      for (int w = 0; w < 4; ++w) m = fmaxf(m, from[(size_t)w * ROWS_DECODE * PR + VD]);
      for (int w = 0; w < 4; ++w) {
        const float* pr = from + (size_t)w * ROWS_DECODE * PR;
        const float f = pr[VD] == -INFINITY ? 0.f : fast_exp2((pr[VD] - m) * p.scale_log2);
        o = fmaf(pr[c], f, o);
        l = fmaf(pr[VD + 1], f, l);
      }
      float* dst = p.partials + (((((size_t)r * p.Hkv + kvh) * p.splits + blockIdx.x) * 2 + a) * ROWS_DECODE + row) * PR;
      dst[c] = o;
      if (c == 0) {
        dst[VD] = m;
        dst[VD + 1] = l;
      }
    }
    return;
  }
  for (int row = warp; row < nrows; row += THREADS / 32) {
    const float *one = part + (size_t)row * PR, *two = one + (size_t)4 * ROWS_DECODE * PR;
    float o[(VD + 31) / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < (VD + 31) / 32; ++i) {
      const int c = lane + 32 * i;
      o[i] = 0.f;
      if (c < VD)
        o[i] = merged(one, (size_t)ROWS_DECODE * PR, 4, c, p.scale_log2) - p.lambda * merged(two, (size_t)ROWS_DECODE * PR, 4, c, p.scale_log2);
      ss = fmaf(o[i], o[i], ss);
    }
    const int token = q_begin + row / p.g, head = kvh * p.g + row % p.g;
    const float by = row_factor(p, gb::warp_sum(ss), token, head);
#pragma unroll
    for (int i = 0; i < (VD + 31) / 32; ++i) {
      const int c = lane + 32 * i;
      if (c < VD) p.out[((size_t)token * p.Hq + head) * VD + c] = __float2bfloat16_rn(o[i] * by);
    }
  }
}

// grid (Hkv, R, rows of a request), a thread per channel: the shares of a decode request's keys for one row, merged in
// split order.
__global__ void __launch_bounds__(MERGE_THREADS)
diff_attention_merge_kernel(const Params p) {
  gb::pdl_launch_dependents();
  gb::pdl_wait();
  __shared__ float red[MERGE_THREADS / 32];
  const int kvh = blockIdx.x, r = blockIdx.y, row = blockIdx.z;
  const int q_begin = p.cu_q[r], q_len = p.cu_q[r + 1] - q_begin;
  if (q_len * p.g > ROWS_DECODE || q_len <= 0 || row >= q_len * p.g) return;
  const size_t stride = (size_t)2 * ROWS_DECODE * PR;
  const float* one = p.partials + ((size_t)r * p.Hkv + kvh) * p.splits * stride + (size_t)row * PR;
  const int c = threadIdx.x;
  float o = 0.f;
  if (c < VD) o = merged(one, stride, p.splits, c, p.scale_log2) - p.lambda * merged(one + (size_t)ROWS_DECODE * PR, stride, p.splits, c, p.scale_log2);
  const float part = gb::warp_sum(o * o);
  if ((c & 31) == 0) red[c >> 5] = part;
  __syncthreads();
  const int token = q_begin + row / p.g, head = kvh * p.g + row % p.g;
  const float by = row_factor(p, (red[0] + red[1]) + (red[2] + red[3]), token, head);
  if (c < VD) p.out[((size_t)token * p.Hq + head) * VD + c] = __float2bfloat16_rn(o * by);
}

}  // namespace

GB_DEFINE_LAST_ERROR()

// Bytes of scratch for `splits` CTAs per decode request (0 for one).
GB_EXPORT long long gb_diff_attention_scratch_bytes(int R, int kv_heads, int splits) {
  return splits > 1 ? (long long)R * kv_heads * splits * 2 * ROWS_DECODE * PR * (long long)sizeof(float) : 0;
}

// q [T, Hq, 2 D], k_pool [pages, Hkv, page_size, 2 D], v_pool [pages, Hkv, page_size, VD], out [T, Hq * VD], bfloat16, 16-byte
// aligned. A split that holds no key of a request leaves a partial with maximum -inf, which the merge skips.
GB_EXPORT int gb_diff_attention(const void* q, const void* k_pool, const void* v_pool, void* out, const int32_t* block_table,
                                int table_width, const int32_t* cu_q, const int32_t* kv_lens, int T, int R, int Hq, int Hkv, float scale,
                                int window, int page_size, int max_q_len, int min_q_len, int splits, void* scratch,
                                long long scratch_bytes, float lambda, float out_scale, float eps, const float* gate,
                                long long gate_stride, cudaStream_t stream) {
  if (T <= 0 || R <= 0) return GB_OK;
  if (Hkv < 1 || Hq % Hkv) return gb::fail(GB_BAD_ARGUMENT, "diff_attention: %d query heads for %d kv heads", Hq, Hkv);
  if (!(scale > 0.f) || window < 0 || page_size < 1) return gb::fail(GB_BAD_ARGUMENT, "diff_attention: scale %g, window %d, pages of %d", scale, window, page_size);
  const int g = Hq / Hkv;
  if (g > ROWS_TILE) return gb::fail(GB_UNSUPPORTED, "diff_attention: a group of %d query heads per kv head", g);
  if (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)out) & 15) return gb::fail(GB_BAD_ARGUMENT, "diff_attention: operands start on 16 bytes");
  splits = splits < 1 ? 1 : (splits > MAX_SPLITS ? MAX_SPLITS : splits);
  if (splits > 1 && (scratch == nullptr || scratch_bytes < gb_diff_attention_scratch_bytes(R, Hkv, splits)))
    return gb::fail(GB_BAD_ARGUMENT, "diff_attention: %d splits need more scratch", splits);
  Params p;
  p.q = (const __nv_bfloat16*)q; p.k_pool = (const __nv_bfloat16*)k_pool; p.v_pool = (const __nv_bfloat16*)v_pool;
  p.out = (__nv_bfloat16*)out; p.block_table = block_table; p.cu_q = cu_q; p.kv_lens = kv_lens;
  p.partials = (float*)scratch;
  p.table_width = table_width; p.Hq = Hq; p.Hkv = Hkv; p.g = g; p.window = window; p.page_size = page_size; p.splits = splits;
  p.scale_log2 = scale * LOG2E; p.lambda = lambda; p.out_scale = out_scale; p.eps = eps;
  p.gate = gate; p.gate_stride = gate_stride;
  static gb::OncePerDevice configured;
  if (configured.needed()) {
    for (auto k : {diff_attention_kernel<false>, diff_attention_kernel<true>}) {
      const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
      if (e != cudaSuccess) return gb::fail(GB_CUDA_ERROR, "diff_attention: %s", cudaGetErrorString(e));
    }
    configured.done();
  }
  if (min_q_len * g <= ROWS_DECODE) {
    int rc = gb::check_pdl_launch(gb::launch_pdl(diff_attention_kernel<true>, dim3(splits, Hkv, R), dim3(THREADS), SMEM, stream,
                                                 dim3(1, 1, 1), p), "diff_attention (decode)");
    if (rc) return rc;
    if (splits > 1) {
      rc = gb::check_pdl_launch(gb::launch_pdl(diff_attention_merge_kernel, dim3(Hkv, R, min(max_q_len * g, ROWS_DECODE)), dim3(MERGE_THREADS), 0,
                                               stream, dim3(1, 1, 1), p), "diff_attention (merge)");
      if (rc) return rc;
    }
  }
  if (max_q_len * g > ROWS_DECODE) {
    const int tokens_per_tile = ROWS_TILE / g;
    dim3 grid((max_q_len + tokens_per_tile - 1) / tokens_per_tile, Hkv, R);
    return gb::check_pdl_launch(gb::launch_pdl(diff_attention_kernel<false>, grid, dim3(THREADS), SMEM, stream, dim3(1, 1, 1), p),
                                "diff_attention (tile)");
  }
  return GB_OK;
}
