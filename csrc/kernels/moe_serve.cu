// Mixture of experts for serving, on one GPU and without a host round trip: the router's choice, the grouping of tokens by
// expert, and the grouped tcgen05 product for prompts.  (Decode steps use the grouped form of the weight-streaming product in
// gemm_skinny.cu, fp32 the one in gemm_simt.cu; dispatch between GPUs is in moe_fused.cu.)
//
// Scores are sigmoids of the router's logits; a correction per expert takes part in the choice of the `top` largest but not
// in the weights, which are the chosen scores as they are.  The chosen (token, expert) pairs get slots: every expert owns a
// run of whole blocks of `block_rows` slots, so that a block of the grouped product has one matrix.  All sizes on the host are
// upper bounds; the number of blocks in use stays on the device.
#include "lt_cuda.h"
#include "gemm_sm100.cuh"
#include "common/scalar.cuh"

namespace lt {

constexpr int kMoeMaxExperts = 1024;

struct MoePlan {
  float* weight;       // [N, top]
  int* slot;           // [N, top]
  int* src;            // [max_blocks * block_rows] token of a slot (only slots in use are written), or nullptr
  int* group;          // [max_blocks] expert of a block
  int* group_rows;     // [max_blocks] slots of the block in use
  int* live;           // number of blocks in use
};

// The `top` best experts of a token, one warp: lane l holds experts l, l + 32, ..  `take(j, expert, score)` runs on lane 0.
template <int EPL, class Take>
__device__ __forceinline__ void choose_experts(const float* __restrict__ logits, const float* __restrict__ correction, int E, int top,
                                               Take take) {
  const int lane = threadIdx.x & 31;
  float s[EPL], c[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    const int e = i * 32 + lane;
    s[i] = e < E ? sigmoid_f(logits[e]) : 0.f;
    c[i] = e < E ? s[i] + correction[e] : -INFINITY;
  }
  unsigned taken = 0u;                                     // bit i: this lane's i-th expert is out
#pragma unroll
  for (int i = 0; i < EPL; ++i)
    if (i * 32 + lane >= E) taken |= 1u << i;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY, score = 0.f;
    int at = kMoeMaxExperts;                               // no expert
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (!(taken >> i & 1u) && (at == kMoeMaxExperts || c[i] > best)) { best = c[i]; score = s[i]; at = i * 32 + lane; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b2 = __shfl_xor_sync(0xffffffffu, best, o), s2 = __shfl_xor_sync(0xffffffffu, score, o);
      const int a2 = __shfl_xor_sync(0xffffffffu, at, o);
      if (a2 != kMoeMaxExperts && (at == kMoeMaxExperts || b2 > best || (b2 == best && a2 < at))) { best = b2; score = s2; at = a2; }
    }
    if (at == kMoeMaxExperts) at = j;                      // logits that are not numbers: some expert, so that slots stay valid
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    if (lane == 0) take(j, at, score);
  }
}

// Exclusive scan of the experts' block counts: first[e] = first block of expert e, *total = blocks in all.  1024 threads or a
// divisor of it; cnt and first in shared memory.
__device__ __forceinline__ void scan_blocks(const int* cnt, int* first, int* total, int E, int block_rows, int* warp_sums) {
  const int per = (kMoeMaxExperts + blockDim.x - 1) / blockDim.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  int mine = 0;
  for (int i = 0; i < per; ++i) {
    const int e = threadIdx.x * per + i;
    if (e < E) mine += (cnt[e] + block_rows - 1) / block_rows;
  }
  int v = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int u = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v += u;
  }
  if (lane == 31) warp_sums[warp] = v;
  __syncthreads();
  int base = 0, all = 0;
  for (int i = 0; i < nw; ++i) {
    if (i < warp) base += warp_sums[i];
    all += warp_sums[i];
  }
  int at = base + v - mine;
  for (int i = 0; i < per; ++i) {
    const int e = threadIdx.x * per + i;
    if (e < E) {
      first[e] = at;
      at += (cnt[e] + block_rows - 1) / block_rows;
    }
  }
  if (threadIdx.x == 0) *total = all;
  __syncthreads();
}

__device__ __forceinline__ void write_groups(const MoePlan& p, const int* cnt, const int* first, int total, int E, int block_rows) {
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    for (int b = 0, left = cnt[e]; left > 0; ++b, left -= block_rows) {
      p.group[first[e] + b] = e;
      p.group_rows[first[e] + b] = min(left, block_rows);
    }
  if (threadIdx.x == 0) *p.live = total;
}

// Few tokens: everything in one CTA.
template <int EPL>
__global__ void __launch_bounds__(1024) moe_plan_small_kernel(const float* __restrict__ logits, const float* __restrict__ correction,
                                                              MoePlan p, int N, int E, int top, int block_rows) {
  extern __shared__ int2 chosen[];                         // [N * top] expert, position among the expert's tokens
  __shared__ int cnt[kMoeMaxExperts], first[kMoeMaxExperts], warp_sums[32], total;
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int n = threadIdx.x >> 5; n < N; n += blockDim.x >> 5)
    choose_experts<EPL>(logits + (long long)n * E, correction, E, top, [&](int j, int e, float s) {
      p.weight[n * top + j] = s;
      chosen[n * top + j] = make_int2(e, atomicAdd(&cnt[e], 1));
    });
  __syncthreads();
  scan_blocks(cnt, first, &total, E, block_rows, warp_sums);
  for (int i = threadIdx.x; i < N * top; i += blockDim.x) {
    const int slot = first[chosen[i].x] * block_rows + chosen[i].y;
    p.slot[i] = slot;
    if (p.src) p.src[slot] = i / top;
  }
  write_groups(p, cnt, first, total, E, block_rows);
}

// Many tokens, first pass: choice, and a position for every pair among its expert's tokens.  counts [E] starts at zero.
constexpr int kMoeTokensPerCta = 32;
template <int EPL>
__global__ void __launch_bounds__(256) moe_choose_kernel(const float* __restrict__ logits, const float* __restrict__ correction,
                                                         float* __restrict__ weight, int2* __restrict__ pairs, int* __restrict__ counts,
                                                         int N, int E, int top) {
  extern __shared__ int2 chosen[];                         // [tokens of this CTA * top]
  __shared__ int cnt[kMoeMaxExperts];
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  const int n0 = blockIdx.x * kMoeTokensPerCta, n1 = min(N, n0 + kMoeTokensPerCta);
  for (int n = n0 + (threadIdx.x >> 5); n < n1; n += blockDim.x >> 5)
    choose_experts<EPL>(logits + (long long)n * E, correction, E, top, [&](int j, int e, float s) {
      weight[(long long)n * top + j] = s;
      chosen[(n - n0) * top + j] = make_int2(e, atomicAdd(&cnt[e], 1));
    });
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    if (cnt[e]) cnt[e] = atomicAdd(counts + e, cnt[e]);    // where this CTA's tokens start
  __syncthreads();
  for (int i = threadIdx.x; i < (n1 - n0) * top; i += blockDim.x)
    pairs[(long long)n0 * top + i] = make_int2(chosen[i].x, cnt[chosen[i].x] + chosen[i].y);
}

// Second pass: slots, the block table, and (x given) the tokens' rows copied to their slots, one warp per token.
__global__ void __launch_bounds__(256) moe_place_kernel(const int2* __restrict__ pairs, const int* __restrict__ counts, MoePlan p,
                                                        const uint4* __restrict__ x, uint4* __restrict__ xs, int row_units, int N, int E,
                                                        int top, int block_rows) {
  __shared__ int cnt[kMoeMaxExperts], first[kMoeMaxExperts], warp_sums[32], total;
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = counts[e];
  __syncthreads();
  scan_blocks(cnt, first, &total, E, block_rows, warp_sums);
  const int lane = threadIdx.x & 31;
  for (int n = blockIdx.x * 8 + (threadIdx.x >> 5); n < N; n += gridDim.x * 8) {
    for (int j = lane; j < top; j += 32) {
      const int2 c = pairs[(long long)n * top + j];
      const int slot = first[c.x] * block_rows + c.y;
      p.slot[(long long)n * top + j] = slot;
      if (p.src) p.src[slot] = n;
    }
    if (x) {
      __syncwarp();
      for (int u = lane; u < row_units; u += 32 * 4) {
        uint4 v[4];
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (u + 32 * k < row_units) v[k] = x[(long long)n * row_units + u + 32 * k];
        for (int j = 0; j < top; ++j) {
          uint4* dst = xs + (long long)p.slot[(long long)n * top + j] * row_units;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (u + 32 * k < row_units) dst[u + 32 * k] = v[k];
        }
      }
    }
  }
  if (blockIdx.x == 0) write_groups(p, cnt, first, total, E, block_rows);
}

// C[slots, N] = A[slots, K] @ W[expert of the slot's 128-row block]^T, gated or not; only the blocks in use are computed.
template <int BLOCK_N, int EPI>
__global__ void __launch_bounds__(kGemmThreads, 1)
moe_grouped_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB,
                        const __grid_constant__ CUtensorMap tmC, const GemmParams p, const int* __restrict__ live) {
  __shared__ GemmParams q;
  if (threadIdx.x == 0) {
    q = p;
    q.dp_tiles = min(p.num_tiles, *live * p.n_blocks);
  }
  __syncthreads();
  gemm_body<BLOCK_N, 0, 0, 0, false, EPI>(&tmA, &tmB, q, NoGate(), NoDone(), 0, &tmC);
}

template <int BLOCK_N, int EPI>
static int launch_grouped(const CUtensorMap& tmA, const CUtensorMap& tmB, const CUtensorMap& tmC, const GemmParams& p, const int* live,
                          int grid, cudaStream_t st) {
  static bool configured = false;
  auto kern = moe_grouped_gemm_kernel<BLOCK_N, EPI>;
  if (!configured) {
    LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, GemmCfg<BLOCK_N>::kStagedSmemBytes));
    configured = true;
  }
  kern<<<grid, kGemmThreads, GemmCfg<BLOCK_N>::kStagedSmemBytes, st>>>(tmA, tmB, tmC, p, live);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // namespace lt

#define LT_MOE_BY_EXPERTS(E, CALL)                                                  \
  do {                                                                              \
    if (E <= 32) { constexpr int EPL = 1; CALL; }                                   \
    else if (E <= 64) { constexpr int EPL = 2; CALL; }                              \
    else if (E <= 128) { constexpr int EPL = 4; CALL; }                             \
    else if (E <= 256) { constexpr int EPL = 8; CALL; }                             \
    else { constexpr int EPL = 32; CALL; }                                          \
  } while (0)

extern "C" {

// logits [N, E] fp32 -> weight [N, top], slot [N, top], src, and the block table (see MoePlan).  max_blocks is at least
// min(N top, E) + N top / block_rows.  pairs (int2 [N * top]) and counts (int [E], zero) are scratch for more than 64 tokens; with
// x (bf16 rows of row_bytes, a multiple of 16) the tokens' rows are also copied to xs[slot] - more than 64 tokens only.
int lt_moe_plan(const float* logits, const float* correction, float* weight, int* slot, int* src, int* group, int* group_rows, int* live,
                void* pairs, int* counts, const void* x, void* xs, int row_bytes, int N, int E, int top, int block_rows, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  if (E < 1 || E > kMoeMaxExperts || top < 1 || top > E || top > 128 || block_rows < 1) return -4;
  MoePlan p{weight, slot, src, group, group_rows, live};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (N <= 64) {
    if (x) return -4;
    const int smem = N * top * 8;
    LT_MOE_BY_EXPERTS(E, {
      LT_RETURN_IF_CUDA(cudaFuncSetAttribute(moe_plan_small_kernel<EPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 128 * 8));
      (moe_plan_small_kernel<EPL><<<1, 1024, smem, st>>>(logits, correction, p, N, E, top, block_rows));
    });
    LT_LAUNCH_CHECK();
    return 0;
  }
  if (!pairs || !counts || (x && (!xs || (row_bytes & 15) || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(xs) & 15))))
    return -4;
  const int smem = kMoeTokensPerCta * top * 8;
  LT_MOE_BY_EXPERTS(E, (moe_choose_kernel<EPL><<<(N + kMoeTokensPerCta - 1) / kMoeTokensPerCta, 256, smem, st>>>(
                           logits, correction, weight, static_cast<int2*>(pairs), counts, N, E, top)));
  LT_LAUNCH_CHECK();
  int grid = (N + 7) / 8;
  if (grid > sm_count() * 8) grid = sm_count() * 8;
  moe_place_kernel<<<grid, 256, 0, st>>>(static_cast<const int2*>(pairs), counts, p, static_cast<const uint4*>(x), static_cast<uint4*>(xs),
                                         row_bytes / 16, N, E, top, block_rows);
  LT_LAUNCH_CHECK();
  return 0;
}

// C [max_blocks * 128, N] bf16 = A @ W[group[block]]^T for the first *live blocks of 128 rows; K and N multiples of 8.  act 0: W [experts,
// N, K]; 1 (GELU) or 2 (SiLU): W [experts, 2 N, K], gate rows, then up rows, and C = act(gate) * up.
int lt_moe_grouped_gemm(const void* A, const void* W, void* C, const int* group, const int* live, int max_blocks, int experts, int N,
                        int K, int act, void* stream) {
  using namespace lt;
  if (max_blocks < 1 || (K & 7) || (N & 7) || act < 0 || act > 2) return -int(kStatusBadArgument);
  const int slots = max_blocks * kBlockM, sms = sm_count(), rows = act ? 2 * N : N;
  const int block_n = act ? 256 : pick_block_n(slots, N, sms);
  const int out_n = act ? 128 : block_n;
  GemmParams p{};
  p.M = slots; p.N = N; p.K = K;
  p.C = C; p.ldc = N; p.alpha = 1.f;
  p.glu_act = act;
  p.status = device_status_word();
  fill_tiles(p, out_n);
  p.raster = 2;
  p.group_of_mblk = group;
  p.b_group_rows = rows;
  CUtensorMap tmA, tmB, tmC;
  int r = make_operand_maps(&tmA, &tmB, A, W, slots, experts * rows, K, K, K, 0, 0, out_n);
  if (r) return r;
  r = make_staged_map(&tmC, C, slots, N, N);
  if (r) return 3000 + r;
  const int grid = sms < p.num_tiles ? sms : p.num_tiles;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (act) return launch_grouped<256, kEpiGlu>(tmA, tmB, tmC, p, live, grid, st);
  return block_n == 256 ? launch_grouped<256, kEpiStaged>(tmA, tmB, tmC, p, live, grid, st)
                        : launch_grouped<128, kEpiStaged>(tmA, tmB, tmC, p, live, grid, st);
}

}  // extern "C"
