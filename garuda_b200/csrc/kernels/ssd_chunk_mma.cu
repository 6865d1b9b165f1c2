// The state-space recurrence of state_space.cu over long stretches of tokens, as products on the tensor cores
// (mma.sync m16n8k16, 32-bit accumulation). Per head, with L_i the sum of the decays' logarithms of a chunk's
// tokens up to i and S the state in front of the chunk:
//     M_ij = exp(L_i - L_j) dt_j (C_i . B_j)   for j <= i, else 0
//     y_i  = sum_j M_ij x_j + exp(L_i) S C_i + skip x_i
//     S   <- exp(L_last) S + sum_j exp(L_last - L_j) dt_j x_j B_j^T
// (the state-space duality of Dao and Gu, "Transformers are SSMs", 2024, with the chunks in order).
//
// x, B and C arrive as bfloat16 and enter the products as they are. Everything else that enters one is 32-bit
// (M, the decayed x, the state): it is written as a sum of three bfloat16 numbers, hi + mid + lo, which together hold
// a 32-bit float's 24 bits, and the three products are added up in the 32-bit accumulators. The state itself never
// leaves its 32-bit accumulators from a request's first token of the step to its last.
//
// A CTA walks one request's chunks of 64 tokens in order for one head and a slice of 32 (or 16) of its vdim rows of
// S. Its eight warps are (16 rows of the slice) x (a share of every product's inner dimension: of the state's
// channels for S C and the update, of the chunk's tokens for M x), so every warp owns its piece of S, in the layout in
// which accumulators are again operands, and nothing of S is ever exchanged; the shares of y are added up in
// shared memory. The next chunk is on its way (cp.async) while one is computed.
//
// A sum of many log decays loses the low bits of the differences that the products take, so L_i is kept as two floats.
// A head may keep one more row of state whose input is the constant one (the normalizer of a matrix memory): a slice
// of its own, of which one row counts.
//
// Compiled per (GB_STATE_DIM = channels of S, GB_HEAD_DIM = rows of S), multiples of 16.
#include "attention_mma_core.cuh"
#include "common.cuh"

#ifndef GB_STATE_DIM
#define GB_STATE_DIM 128
#endif
#ifndef GB_HEAD_DIM
#define GB_HEAD_DIM 64
#endif

namespace {

using attn_mma::ldmatrix_x4;
using attn_mma::ldmatrix_x4_trans;
using attn_mma::mma_16816;
using attn_mma::pack_bf16;

constexpr int N = GB_STATE_DIM, P = GB_HEAD_DIM;
static_assert(N % 16 == 0 && N >= 16 && N <= 256 && P % 16 == 0 && P >= 16, "sizes are multiples of 16, at most 256 state channels");
constexpr int Q = 64;                              // tokens of a chunk
constexpr int PS = P % 32 == 0 ? 32 : 16;          // rows of S of a CTA
constexpr int WARPS = 8, THREADS = WARPS * 32;
constexpr int PR = PS / 16, KS = WARPS / PR;       // row blocks of 16; warps that share the inner dimension
constexpr int NT = N / 16, MT = (NT + KS - 1) / KS;      // blocks of 16 state channels, at most so many a warp
constexpr int SPLIT = 3;                           // bfloat16 parts of a 32-bit operand
constexpr int LDN = N + 8, LDX = PS + 8, LDM = Q + 8, LDY = PS + 4;

struct Stage {
  __nv_bfloat16 b[Q][LDN], c[Q][LDN], x[Q][LDX];
};
struct Smem {
  Stage stage[2];
  union {
    __nv_bfloat16 m[SPLIT][Q][LDM];                // M in its three parts
    float y[2][Q][LDY];                            // the warps' shares of the chunk's y, added up in two places
  };
  float grow[2][Q];                                // exp(L_i)
  float fade[2][Q];                                // exp(L_last - L_j) dt_j
  float log_sum[2][Q], log_rest[2][Q];             // L_i, and what it lost in rounding
  float dt[2][Q];
};

__device__ __forceinline__ void cp_async_16(void* smem, const void* gmem, bool valid) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s), "l"(gmem), "r"(bytes) : "memory");
}

// Two 32-bit values as SPLIT packed pairs of bfloat16 whose sums are the values.
__device__ __forceinline__ void split_pair(float a, float b, uint32_t (&out)[SPLIT]) {
#pragma unroll
  for (int s = 0; s < SPLIT; ++s) {
    out[s] = pack_bf16(a, b);
    if (s + 1 < SPLIT) {
      a -= __uint_as_float(out[s] << 16);
      b -= __uint_as_float(out[s] & 0xffff0000u);
    }
  }
}

// The lower-triangle blocks (16 x 16) of M, row block first, shared out to the warps so that none has more than two.
__device__ __forceinline__ int m_block(int warp, int k, int& ib, int& jb) {
  const int id = warp + k * WARPS;                 // 0 .. 9
  if (id >= 10) return 0;
  ib = id < 1 ? 0 : id < 3 ? 1 : id < 6 ? 2 : 3;
  jb = id - ib * (ib + 1) / 2;
  return 1;
}

// grid (H, P / PS, one more for a unit row, R). act [T, C]: x of all heads, B of all groups, C of all groups; step [T, 2 H]: dt, log of the decay.
__global__ void __launch_bounds__(THREADS, N <= 128 ? 2 : 1)
ssd_chunk_kernel(const __nv_bfloat16* __restrict__ act, int C, const float* __restrict__ step, const float* __restrict__ skip,
                 const int32_t* __restrict__ cu_q, const int32_t* __restrict__ slots, float* __restrict__ state,
                 long long state_stride, int H, int G, float* __restrict__ y, float* __restrict__ unit_state, float* __restrict__ unit_y) {
  extern __shared__ __align__(16) unsigned char raw[];
  Smem& sm = *reinterpret_cast<Smem*>(raw);
  gb::pdl_wait();
  const bool unit = blockIdx.y == P / PS;
  const int h = blockIdx.x, p0 = blockIdx.y * PS, r = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3;
  const int pr = warp % PR, kh = warp / PR;
  const int slot = slots[r], t0 = cu_q[r], t1 = cu_q[r + 1];
  const int off_b = H * P + h / (H / G) * N, off_c = off_b + G * N, off_x = h * P + p0;
  if (t0 >= t1) return;

  auto load = [&](int chunk, int st) {
    const int base = t0 + chunk * Q;
    Stage& s = sm.stage[st];
    for (int i = threadIdx.x; i < Q * (N / 8); i += THREADS) {
      const int row = i / (N / 8), ch = (i % (N / 8)) * 8;
      const bool ok = base + row < t1;
      const __nv_bfloat16* src = act + (size_t)(ok ? base + row : t0) * C + ch;
      cp_async_16(&s.b[row][ch], src + off_b, ok);
      cp_async_16(&s.c[row][ch], src + off_c, ok);
    }
    for (int i = threadIdx.x; i < (unit ? 0 : Q * (PS / 8)); i += THREADS) {
      const int row = i / (PS / 8), ch = (i % (PS / 8)) * 8;
      const bool ok = base + row < t1;
      cp_async_16(&s.x[row][ch], act + (size_t)(ok ? base + row : t0) * C + off_x + ch, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // (Tokens beyond a request's last are zeros in every operand: a short chunk runs the same instructions, which the
  // compiler may then interleave freely.) The last warp: a chunk's running sums of log decays (lane l has tokens 2 l and 2 l + 1; beyond the end: dt 0,
  // decay one), from values asked for a chunk ahead.
  float d[2], a[2];
  auto ask_decays = [&](int chunk) {
    const int t = t0 + chunk * Q + 2 * lane;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      d[e] = t + e < t1 ? step[(size_t)(t + e) * 2 * H + h] : 0.f;
      a[e] = t + e < t1 ? step[(size_t)(t + e) * 2 * H + H + h] : 0.f;
    }
  };
  auto decays = [&](int st) {
    double run = (double)a[0] + a[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    const double last = __shfl_sync(0xffffffffu, run, 31);
    double before = __shfl_up_sync(0xffffffffu, run, 1);
    if (lane == 0) before = 0.0;
    const double l[2] = {before + a[0], run};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = 2 * lane + e;
      sm.log_sum[st][i] = (float)l[e];
      sm.log_rest[st][i] = (float)(l[e] - (float)l[e]);
      sm.dt[st][i] = d[e];
      sm.grow[st][i] = expf((float)l[e]);
      sm.fade[st][i] = expf((float)(last - l[e])) * d[e];
    }
  };

  // the warp's piece of S^T: rows pr * 16 .., channel blocks kh, kh + KS, ...; two accumulator tiles of 8 channels each
  float S[MT][2][4];
  float* S_g = slot >= 0 ? (unit ? unit_state + (size_t)slot * state_stride + (size_t)h * N
                                 : state + (size_t)slot * state_stride + ((size_t)h * P + p0 + pr * 16) * N) : nullptr;
  const int S_rows = unit ? (pr == 0 ? 1 : 0) : 16;             // rows of the warp's piece that there are
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = (kh + m * KS) * 16 + half * 8 + 2 * tig + (e & 1), row = g + (e >> 1) * 8;
        S[m][half][e] = (S_g != nullptr && row < S_rows && kh + m * KS < NT) ? S_g[(size_t)row * N + n] : 0.f;
      }
  const float dskip = unit || skip == nullptr ? 0.f : skip[h];
  if (unit)                       // its input, for every chunk (tokens beyond a request's last have step zero)
    for (int i = threadIdx.x; i < 2 * Q * PS; i += THREADS)
      sm.stage[i / (Q * PS)].x[i / PS % Q][i % PS] = __float2bfloat16_rn(i % PS == 0 ? 1.f : 0.f);
  const int chunks = (t1 - t0 + Q - 1) / Q;
  load(0, 0);
  if (warp == WARPS - 1) {
    ask_decays(0);
    decays(0);
    ask_decays(1);
  }
  for (int ck = 0; ck < chunks; ++ck) {
    const int st = ck & 1;
    const Stage& s = sm.stage[st];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();           // this chunk has landed; everyone is done with the chunk in front (its buffers, y's shares)
    if (ck + 1 < chunks) load(ck + 1, st ^ 1);
    // ---- M, its lower triangle
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      int ib, jb;
      if (!m_block(warp, k, ib, jb)) continue;
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int kk = 0; kk < NT; ++kk) {
        uint32_t a[4], b[4];
        ldmatrix_x4(a, &s.c[ib * 16 + (lane & 15)][kk * 16 + (lane >> 4) * 8]);
        ldmatrix_x4(b, &s.b[jb * 16 + (lane & 7) + (lane >> 4) * 8][kk * 16 + ((lane >> 3) & 1) * 8]);
        mma_16816(acc[0], a, b[0], b[1]);
        mma_16816(acc[1], a, b[2], b[3]);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int up = 0; up < 2; ++up) {
          const int i = ib * 16 + g + up * 8, j = jb * 16 + half * 8 + 2 * tig;
          const float li = sm.log_sum[st][i], li_rest = sm.log_rest[st][i];
          float v[2];
#pragma unroll
          for (int e = 0; e < 2; ++e)
            v[e] = j + e <= i ? acc[half][up * 2 + e] * (expf((li - sm.log_sum[st][j + e]) + (li_rest - sm.log_rest[st][j + e])) * sm.dt[st][j + e]) : 0.f;
          uint32_t parts[SPLIT];
          split_pair(v[0], v[1], parts);
#pragma unroll
          for (int q = 0; q < SPLIT; ++q) *reinterpret_cast<uint32_t*>(&sm.m[q][i][j]) = parts[q];
        }
    }
    // ---- the state's part of y^T: rows of the slice x tokens, this warp's channels
    float acc[Q / 8][4];
#pragma unroll
    for (int i = 0; i < Q / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int nb = kh + m * KS;
      if (nb >= NT) break;
      uint32_t a[SPLIT][4];
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int up = 0; up < 2; ++up) {
          uint32_t parts[SPLIT];
          split_pair(S[m][half][up * 2], S[m][half][up * 2 + 1], parts);
#pragma unroll
          for (int q = 0; q < SPLIT; ++q) a[q][half * 2 + up] = parts[q];
        }
#pragma unroll
      for (int ib = 0; ib < Q / 16; ++ib) {
        uint32_t b[4];
        ldmatrix_x4(b, &s.c[ib * 16 + (lane & 7) + (lane >> 4) * 8][nb * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int q = SPLIT - 1; q >= 0; --q) {          // the small parts first
          mma_16816(acc[2 * ib], a[q], b[0], b[1]);
          mma_16816(acc[2 * ib + 1], a[q], b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < Q / 8; ++i) {
      const float g0 = sm.grow[st][i * 8 + 2 * tig], g1 = sm.grow[st][i * 8 + 2 * tig + 1];
      acc[i][0] *= g0, acc[i][1] *= g1, acc[i][2] *= g0, acc[i][3] *= g1;
    }
    // ---- the state moves on: S <- exp(L_last) S + (fade x)^T B
    {
      const float whole = sm.grow[st][Q - 1];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[m][half][e] *= whole;
#pragma unroll
      for (int jb = 0; jb < Q / 16; ++jb) {
        uint32_t xt[4], a[SPLIT][4];
        ldmatrix_x4_trans(xt, &s.x[jb * 16 + (lane & 7) + (lane >> 4) * 8][pr * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int j = jb * 16 + (i >> 1) * 8 + 2 * tig;
          uint32_t parts[SPLIT];
          split_pair(__uint_as_float(xt[i] << 16) * sm.fade[st][j], __uint_as_float(xt[i] & 0xffff0000u) * sm.fade[st][j + 1], parts);
#pragma unroll
          for (int q = 0; q < SPLIT; ++q) a[q][i] = parts[q];
        }
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const int nb = kh + m * KS;
          if (nb >= NT) break;
          uint32_t b[4];
          ldmatrix_x4_trans(b, &s.b[jb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][nb * 16 + (lane >> 4) * 8]);
#pragma unroll
          for (int q = SPLIT - 1; q >= 0; --q) {
            mma_16816(S[m][0], a[q], b[0], b[1]);
            mma_16816(S[m][1], a[q], b[2], b[3]);
          }
        }
      }
    }
    if (ck + 1 < chunks && warp == WARPS - 1) {
      decays(st ^ 1);
      ask_decays(ck + 2);
    }
    __syncthreads();           // M is whole
    // ---- the chunk's own part of y^T: x^T M^T over this warp's token blocks
#pragma unroll
    for (int k = 0; k < (Q / 16 + KS - 1) / KS; ++k) {
      const int jb = (k & 1) ? (k + 1) * KS - 1 - kh : k * KS + kh;       // blocks early and late in turn: they differ in length
      if (jb >= Q / 16) continue;
      uint32_t xt[4];
      ldmatrix_x4_trans(xt, &s.x[jb * 16 + (lane & 7) + (lane >> 4) * 8][pr * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
      for (int ib = 0; ib < Q / 16; ++ib) {
        if (ib < jb) continue;
#pragma unroll
        for (int q = SPLIT - 1; q >= 0; --q) {
          uint32_t b[4];
          ldmatrix_x4(b, &sm.m[q][ib * 16 + (lane & 7) + (lane >> 4) * 8][jb * 16 + ((lane >> 3) & 1) * 8]);
          mma_16816(acc[2 * ib], xt, b[0], b[1]);
          mma_16816(acc[2 * ib + 1], xt, b[2], b[3]);
        }
      }
    }
    __syncthreads();           // M has been read: its place takes the shares of y
    for (int turn = 0; turn < KS / 2; ++turn) {
      if (kh >> 1 == turn) {
#pragma unroll
        for (int i = 0; i < Q / 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float& to = sm.y[kh & 1][i * 8 + 2 * tig + (e & 1)][pr * 16 + g + (e >> 1) * 8];
            to = turn == 0 ? acc[i][e] : to + acc[i][e];
          }
      }
      __syncthreads();
    }
    const int n = min(Q, t1 - t0 - ck * Q);
    if (unit) {
      if (threadIdx.x < n) unit_y[(size_t)(t0 + ck * Q + threadIdx.x) * H + h] = sm.y[0][threadIdx.x][0] + sm.y[1][threadIdx.x][0];
      continue;
    }
    for (int i = threadIdx.x; i < n * PS; i += THREADS) {
      const int t = i / PS, p = i % PS;
      y[(size_t)(t0 + ck * Q + t) * H * P + off_x + p] = fmaf(dskip, __bfloat162float(s.x[t][p]), sm.y[0][t][p] + sm.y[1][t][p]);
    }
  }
  gb::pdl_launch_dependents();
  if (S_g != nullptr) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int n = (kh + m * KS) * 16 + half * 8 + 2 * tig + (e & 1), row = g + (e >> 1) * 8;
          if (row < S_rows && kh + m * KS < NT) S_g[(size_t)row * N + n] = S[m][half][e];
        }
  }
}

}  // namespace

GB_DEFINE_LAST_ERROR()

// act [T, C] bfloat16 (16-byte aligned, C a multiple of 8), step [T, 2 H], y [T, H P]; skip, state and the unit row as for
// gb_ssd_recurrence.
GB_EXPORT int gb_ssd_chunk(const void* act, const float* step, const float* skip, const int32_t* cu_q, const int32_t* slots,
                           float* state, long long state_stride, int R, int H, int G, float* y, float* unit_state, float* unit_y,
                           cudaStream_t stream) {
  if (R <= 0) return GB_OK;
  if (H < 1 || G < 1 || H % G) return gb::fail(GB_BAD_ARGUMENT, "ssd_chunk: %d heads in %d groups", H, G);
  if ((unit_state == nullptr) != (unit_y == nullptr)) return gb::fail(GB_BAD_ARGUMENT, "ssd_chunk: a unit row has a state and a read-out");
  if (R > 65535 || ((uintptr_t)act & 15)) return gb::fail(GB_UNSUPPORTED, "ssd_chunk: %d requests, rows at %p", R, act);
  static gb::OncePerDevice configured;
  if (configured.needed()) {
    const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(Smem));
    if (e != cudaSuccess) return gb::fail(GB_CUDA_ERROR, "ssd_chunk: %s", cudaGetErrorString(e));
    configured.done();
  }
  const int C = H * P + 2 * G * N;
  return gb::check_pdl_launch(gb::launch_after(ssd_chunk_kernel, dim3(H, P / PS + (unit_state != nullptr), R), dim3(THREADS), sizeof(Smem), stream,
                                               dim3(1, 1, 1), (const __nv_bfloat16*)act, C, step, skip, cu_q, slots, state, state_stride, H, G, y,
                                               unit_state, unit_y),
                              "ssd_chunk");
}
