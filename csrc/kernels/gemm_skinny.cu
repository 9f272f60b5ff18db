// Weight-streaming GEMM for 9 to 128 rows (decode with a batch of sequences): y[M, N] = x[M, K] @ W[N, K]^T (+ residual).
//
// With this few rows the multiplication is bound by reading W once (a 1.1B model's weights stream in 0.3 ms), but a
// 128-row tcgen05 tile wastes most of its rows and, worse, a 2048-column output gives a persistent tile kernel 8 or 16
// tiles for 148 SMs.  Here a CTA of eight warps owns 32 output columns and a slice of K; every warp walks its share of the
// slice in 32-element chunks with 8 to 16 sixteen-byte weight loads in flight per lane and feeds them to the warp-level
// tensor-core instruction (mma.sync m16n8k16: 16 rows of x by 8 columns of W; tcgen05's smallest tile is 64 rows and needs a
// TMEM / barrier set-up that costs more than these microsecond kernels run).  The K dimension inside a chunk is permuted
// the same way for both operands so that each lane's 16 contiguous bytes are exactly its fragments of two instructions.
// The eight warps' partial sums are folded through shared memory; when several CTAs share a column group (narrow
// outputs: more CTAs than column groups are needed to fill the GPU) each writes its partial to a workspace and the CTA
// that arrives last at the group's counter adds them in a fixed order, so the result does not depend on arrival order
// and nothing ever waits.
//
// Three variants share the loop: a batch of equal products at fixed offsets (one per attention head), rows grouped by expert
// (a mixture of experts in a decode step: blocks of 16, 32 or 64 rows, each block with the matrix of its expert, its
// rows picked out of the tokens by a table), and a gated epilogue: w holds gate rows, then up rows, a CTA owns 16 of
// each, and y = act(gate) * up leaves the kernel, so that the wide intermediate is never stored.
// The reference runs every Linear through cublasSgemm whatever the row count
// (src/ops/linear.cpp:176-192).
#include "lt_cuda.h"
#include "common/host.h"
#include "common/ptx.cuh"
#include "common/scalar.cuh"

#include <atomic>
#include <map>
#include <mutex>
#include <utility>

namespace lt {

constexpr int kSkWarps = 8;
constexpr int kSkCols = 32;   // output columns per CTA: four 8-column fragments per warp
constexpr size_t kSkWsBytes = 12u << 20;
constexpr int kSkCounters = 4096;

__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                               uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

struct SkinnyParams {
  const __nv_bfloat16* x;
  long long ldx;
  const __nv_bfloat16* w;
  long long ldw;
  __nv_bfloat16* y;
  long long ldy;
  const __nv_bfloat16* residual;
  long long ldr;
  int M, N, K, chunks_per_cta;   // gated: N counts results, w has 2 N rows
  float* ws;
  unsigned* counters;
  int act;                       // gated: 1 GELU (tanh form), 2 SiLU
  long long sx, sw, sy;          // batch: element offsets of the next product; grouped: sw of the next expert's matrix
  const int* group;              // grouped: expert of every block of 16 MT rows
  const int* group_rows;         // rows of the block that exist
  const int* live;               // number of blocks
  const int* src;                // row of x for every row of y; nullptr: the same row
};

enum { kSkPlain = 0, kSkBatch = 1, kSkGrouped = 2 };

// MT = number of 16-row blocks of x (rows past M read as zero).  Grid: (column groups, K splits, products or row blocks).
template <int MT, int MODE, bool GLU>
__global__ void __launch_bounds__(kSkWarps * 32, (MODE != kSkPlain || GLU) && MT == 1 ? 2 : 1)
gemm_skinny_kernel(const SkinnyParams p) {
  extern __shared__ float red[];   // [4 slots][MT * 16 registers][32 lanes]
  constexpr int R = MT * 16;
  constexpr int U = MT <= 2 ? 4 : 2;   // chunks whose weight loads are in flight together
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, q = lane & 3;
  const int n0 = blockIdx.x * (GLU ? kSkCols / 2 : kSkCols);
  const int nchunks = p.K >> 5;
  const int c_begin = blockIdx.y * p.chunks_per_cta;
  const int c_end = min(nchunks, c_begin + p.chunks_per_cta);
  const int N = p.N;
  int M = p.M;
  const __nv_bfloat16* x = p.x;
  const __nv_bfloat16* w = p.w;
  __nv_bfloat16* y = p.y;
  if constexpr (MODE == kSkBatch) {
    x += blockIdx.z * p.sx;
    w += blockIdx.z * p.sw;
    y += blockIdx.z * p.sy;
  }
  if constexpr (MODE == kSkGrouped) {
    if (int(blockIdx.z) >= *p.live) return;
    M = p.group_rows[blockIdx.z];
    w += p.group[blockIdx.z] * p.sw;
    y += (long long)blockIdx.z * R * p.ldy;
  }
  // the rows of x this lane reads
  const __nv_bfloat16* xrow[MT][2];
  if constexpr (MODE == kSkGrouped) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = m * 16 + g + h * 8;
        long long at = (long long)blockIdx.z * R + r;
        if (p.src) at = r < M ? p.src[at] : 0;
        xrow[m][h] = x + at * p.ldx + q * 8;
      }
  }
  const __nv_bfloat16* xbase = x + q * 8;
  const long long ldx = p.ldx;

  float acc[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int f = 0; f < 4; ++f)
#pragma unroll
      for (int r = 0; r < 4; ++r) acc[m][f][r] = 0.f;

  const __nv_bfloat16* wrow[4];
  bool wok[4];
#pragma unroll
  for (int f = 0; f < 4; ++f) {
    const int n = n0 + (GLU ? f & 1 : f) * 8 + g;
    wok[f] = n < N;
    wrow[f] = w + (long long)(wok[f] ? n + (GLU && f >= 2 ? N : 0) : 0) * p.ldw + q * 8;
  }

  for (int c = c_begin + warp; c < c_end; c += kSkWarps * U) {
    uint4 wv[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int cc = c + u * kSkWarps;
#pragma unroll
      for (int f = 0; f < 4; ++f)
        wv[u][f] = (cc < c_end && wok[f]) ? ld_nc_v4(wrow[f] + (long long)cc * 32) : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int cc = c + u * kSkWarps;
      if (cc >= c_end) break;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int r0 = m * 16 + g, r1 = r0 + 8;
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
        const __nv_bfloat16 *x0, *x1;
        if constexpr (MODE == kSkGrouped) { x0 = xrow[m][0]; x1 = xrow[m][1]; }
        else { x0 = xbase + (long long)r0 * ldx; x1 = xbase + (long long)r1 * ldx; }
        const uint4 xlo = r0 < M ? __ldg(reinterpret_cast<const uint4*>(x0 + cc * 32)) : zero;
        const uint4 xhi = r1 < M ? __ldg(reinterpret_cast<const uint4*>(x1 + cc * 32)) : zero;
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          // physical k = q * 8 + j * 4 + {0, 1} plays logical k = q * 2 + {0, 1}, physical + 2 plays logical + 8, for A and B alike
          mma_bf16_16816(acc[m][f], xlo.x, xhi.x, xlo.y, xhi.y, wv[u][f].x, wv[u][f].y);
          mma_bf16_16816(acc[m][f], xlo.z, xhi.z, xlo.w, xhi.w, wv[u][f].z, wv[u][f].w);
        }
      }
    }
  }

  // fold the eight warps' partial sums: 4-7 into 0-3, 2-3 into 0-1, 1 into 0
#pragma unroll 1
  for (int half = kSkWarps / 2; half >= 1; half >>= 1) {
    if (warp >= half && warp < 2 * half) {
      float* dst = red + (size_t)(warp - half) * R * 32 + lane;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int f = 0; f < 4; ++f)
#pragma unroll
          for (int r = 0; r < 4; ++r) dst[((m * 4 + f) * 4 + r) * 32] = acc[m][f][r];
    }
    __syncthreads();
    if (warp < half) {
      const float* src = red + (size_t)warp * R * 32 + lane;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int f = 0; f < 4; ++f)
#pragma unroll
          for (int r = 0; r < 4; ++r) acc[m][f][r] += src[((m * 4 + f) * 4 + r) * 32];
    }
    __syncthreads();
  }
  if (warp != 0) return;

  const int splits = gridDim.y;
  if (splits > 1) {
    float* mine = p.ws + ((size_t)blockIdx.y * gridDim.x + blockIdx.x) * (R * 32) + lane;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int f = 0; f < 4; ++f)
#pragma unroll
        for (int r = 0; r < 4; ++r) mine[((m * 4 + f) * 4 + r) * 32] = acc[m][f][r];
    __threadfence();
    __syncwarp();
    unsigned prev = 0;
    if (lane == 0) prev = atomicAdd(p.counters + blockIdx.x, 1u);
    prev = __shfl_sync(0xffffffffu, prev, 0);
    if (prev != unsigned(splits - 1)) return;   // not the last CTA of this column group
    __threadfence();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int f = 0; f < 4; ++f)
#pragma unroll
        for (int r = 0; r < 4; ++r) acc[m][f][r] = 0.f;
    for (int s = 0; s < splits; ++s) {   // every part from the workspace, in index order: the sum is the same whoever is last
      const float* part = p.ws + ((size_t)s * gridDim.x + blockIdx.x) * (R * 32) + lane;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int f = 0; f < 4; ++f)
#pragma unroll
          for (int r = 0; r < 4; ++r) acc[m][f][r] += __ldcg(part + ((m * 4 + f) * 4 + r) * 32);
    }
    if (lane == 0) p.counters[blockIdx.x] = 0u;   // ready for the next launch on this stream
  }

#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int f = 0; f < (GLU ? 2 : 4); ++f) {
      const int col = n0 + f * 8 + q * 2;
      if (col >= N) continue;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = m * 16 + g + h * 8;
        if (row >= M) continue;
        float v0 = acc[m][f][h * 2], v1 = acc[m][f][h * 2 + 1];
        if constexpr (GLU) {
          const float u0 = acc[m][f + 2][h * 2], u1 = acc[m][f + 2][h * 2 + 1];
          v0 = (p.act == 1 ? gelu_tanh_f(v0) : silu_quick_f(v0)) * u0;
          v1 = (p.act == 1 ? gelu_tanh_f(v1) : silu_quick_f(v1)) * u1;
        } else if (p.residual) {
          const float2 rv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p.residual + (long long)row * p.ldr + col));
          v0 += rv.x;
          v1 += rv.y;
        }
        *reinterpret_cast<uint32_t*>(y + (long long)row * p.ldy + col) = pack_bf16x2(v0, v1);
      }
    }
  }
}

struct SkinnyWs {
  float* ws = nullptr;
  unsigned* counters = nullptr;
};
static std::mutex g_sk_mu;
// Measured under graph replay (Llama-1.1B shapes, 32 and 128 rows): the hand-over of partial sums through L2 costs about 3 us, more
// than a 2048-deep K loop on a third of the SMs, so by default K is split only when a warp still keeps 16 chunks (K >= 8192).
static std::atomic<int> g_sk_target{1};       // CTAs per SM the K split aims for (lt_gemm_skinny_set_target)
static std::atomic<int> g_sk_min_chunks{16};  // 32-element chunks a warp keeps at least when K is split
static std::map<std::pair<int, cudaStream_t>, SkinnyWs> g_sk_ws;

// Workspace of the K split, one per (device, stream): launches on one stream are serialised and the last CTA of a
// column group resets its counter.  Not allocated while the stream records a graph (the launch then runs unsplit).
static bool get_skinny_ws(cudaStream_t st, SkinnyWs* out) {
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess) return false;
  std::lock_guard<std::mutex> lock(g_sk_mu);
  auto key = std::make_pair(dev, st);
  auto it = g_sk_ws.find(key);
  if (it != g_sk_ws.end()) { *out = it->second; return out->ws != nullptr; }
  cudaStreamCaptureStatus cap = cudaStreamCaptureStatusNone;
  if (cudaStreamIsCapturing(st, &cap) != cudaSuccess || cap != cudaStreamCaptureStatusNone) {
    cudaGetLastError();
    return false;
  }
  void* base = nullptr;
  if (cudaMalloc(&base, kSkWsBytes + kSkCounters * sizeof(unsigned)) != cudaSuccess) {
    cudaGetLastError();
    g_sk_ws[key] = SkinnyWs{};
    return false;
  }
  SkinnyWs w;
  w.ws = static_cast<float*>(base);
  w.counters = reinterpret_cast<unsigned*>(static_cast<char*>(base) + kSkWsBytes);
  if (cudaMemsetAsync(w.counters, 0, kSkCounters * sizeof(unsigned), st) != cudaSuccess) {
    cudaGetLastError();
    cudaFree(base);
    g_sk_ws[key] = SkinnyWs{};
    return false;
  }
  g_sk_ws[key] = w;
  *out = w;
  return true;
}

template <int MT, int MODE, bool GLU>
static int launch_skinny(SkinnyParams p, int z, cudaStream_t st) {
  static bool configured = false;
  constexpr int smem = 4 * MT * 16 * 32 * 4;
  auto kern = gemm_skinny_kernel<MT, MODE, GLU>;
  if (!configured) {
    LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    configured = true;
  }
  const int sms = sm_count();
  const int cols = GLU ? kSkCols / 2 : kSkCols;
  const int groups = (p.N + cols - 1) / cols;
  const int nchunks = p.K / 32;
  int splits = MODE == kSkPlain ? (g_sk_target.load() * sms + groups - 1) / groups : 1;
  const int mc = g_sk_min_chunks.load();
  const int max_splits = nchunks / (mc * kSkWarps) > 1 ? nchunks / (mc * kSkWarps) : 1;   // at least `mc` chunks per warp
  if (splits > max_splits) splits = max_splits;
  SkinnyWs wsp;
  if (splits > 1) {
    const size_t need = size_t(splits) * groups * (MT * 16 * 32) * sizeof(float);
    if (groups > kSkCounters || need > kSkWsBytes || !get_skinny_ws(st, &wsp)) splits = 1;
  }
  int per = (nchunks + splits - 1) / splits;
  splits = (nchunks + per - 1) / per;
  p.chunks_per_cta = per;
  p.ws = wsp.ws;
  p.counters = wsp.counters;
  kern<<<dim3(groups, splits, z), kSkWarps * 32, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

template <int MODE, bool GLU>
static int skinny_by_rows(const SkinnyParams& p, int rows, int z, cudaStream_t st) {
  if (rows <= 16) return launch_skinny<1, MODE, GLU>(p, z, st);
  if (rows <= 32) return launch_skinny<2, MODE, GLU>(p, z, st);
  if (rows <= 64) return launch_skinny<4, MODE, GLU>(p, z, st);
  if constexpr (MODE == kSkGrouped) return -int(kStatusBadArgument);
  else return launch_skinny<8, MODE, GLU>(p, z, st);
}

static bool skinny_ok(const SkinnyParams& p) {
  return p.N > 0 && p.K > 0 && !(p.K & 31) && !(p.N & 7) && !(p.ldx & 7) && !(p.ldw & 7) && !(p.ldy & 1) && !(p.ldr & 1) &&
         !(p.sx & 7) && !(p.sw & 7) && !(p.sy & 1) && !(reinterpret_cast<uintptr_t>(p.x) & 15) && !(reinterpret_cast<uintptr_t>(p.w) & 15) &&
         !(reinterpret_cast<uintptr_t>(p.y) & 3) && !(reinterpret_cast<uintptr_t>(p.residual) & 3);
}

}  // namespace lt

extern "C" {

// How many CTAs per SM the K split of narrow outputs aims for (default 1; 1 to 8) and how many 32-element chunks of K a
// warp keeps at least (default 16; 1 to 16).
int lt_gemm_skinny_set_target(int ctas_per_sm, int min_chunks_per_warp) {
  lt::g_sk_target.store(ctas_per_sm < 1 ? 1 : (ctas_per_sm > 8 ? 8 : ctas_per_sm));
  lt::g_sk_min_chunks.store(min_chunks_per_warp < 1 ? 1 : (min_chunks_per_warp > 16 ? 16 : min_chunks_per_warp));
  return 0;
}

// y[M, N] = x[M, K] @ w[N, K]^T (+ residual[M, N]), all bf16; 1 <= M <= 128, K a multiple of 32, N a multiple of 8, operand
// rows 16-byte aligned, y / residual rows 4-byte aligned.
int lt_gemm_skinny_bf16(const void* x, long long ldx, const void* w, long long ldw, void* y, long long ldy, const void* residual,
                        long long ldr, int M, int N, int K, void* stream) {
  using namespace lt;
  SkinnyParams p{};
  p.x = static_cast<const __nv_bfloat16*>(x); p.ldx = ldx;
  p.w = static_cast<const __nv_bfloat16*>(w); p.ldw = ldw;
  p.y = static_cast<__nv_bfloat16*>(y); p.ldy = ldy;
  p.residual = static_cast<const __nv_bfloat16*>(residual); p.ldr = ldr;
  p.M = M; p.N = N; p.K = K;
  if (M < 1 || M > 128 || !skinny_ok(p)) return -int(kStatusBadArgument);
  return skinny_by_rows<kSkPlain, false>(p, M, 1, static_cast<cudaStream_t>(stream));
}

// y[M, N] = act(x @ gate^T) * (x @ up^T), w [2 N, K] = gate rows, then up rows; act 1: GELU (tanh form), 2: SiLU.  Otherwise as above.
int lt_gemm_skinny_glu(const void* x, long long ldx, const void* w, void* y, int M, int N, int K, int act, void* stream) {
  using namespace lt;
  SkinnyParams p{};
  p.x = static_cast<const __nv_bfloat16*>(x); p.ldx = ldx;
  p.w = static_cast<const __nv_bfloat16*>(w); p.ldw = K;
  p.y = static_cast<__nv_bfloat16*>(y); p.ldy = N;
  p.M = M; p.N = N; p.K = K; p.act = act;
  if (M < 1 || M > 128 || act < 1 || act > 2 || !skinny_ok(p)) return -int(kStatusBadArgument);
  return skinny_by_rows<kSkPlain, true>(p, M, 1, static_cast<cudaStream_t>(stream));
}

// A batch of products y_b = x_b @ w_b^T: x_b at offset b * sx, w_b [N, K] one after another, y_b at offset b * sy.
int lt_gemm_skinny_batch(const void* x, long long ldx, long long sx, const void* w, void* y, long long ldy, long long sy, int batch,
                         int M, int N, int K, void* stream) {
  using namespace lt;
  SkinnyParams p{};
  p.x = static_cast<const __nv_bfloat16*>(x); p.ldx = ldx; p.sx = sx;
  p.w = static_cast<const __nv_bfloat16*>(w); p.ldw = K; p.sw = (long long)N * K;
  p.y = static_cast<__nv_bfloat16*>(y); p.ldy = ldy; p.sy = sy;
  p.M = M; p.N = N; p.K = K;
  if (M < 1 || M > 128 || batch < 1 || batch > 65535 || !skinny_ok(p)) return -int(kStatusBadArgument);
  return skinny_by_rows<kSkBatch, false>(p, M, batch, static_cast<cudaStream_t>(stream));
}

// Rows grouped by expert in blocks of block_rows (16, 32 or 64): block b (of *live, at most max_blocks) takes rows of x
// src[b block_rows ..] (src nullptr: the same rows of x), group_rows[b] of them, times the matrix of expert group[b], into
// rows b block_rows .. of y.  act 0: w [experts, N, K]; else gated as in lt_gemm_skinny_glu, w [experts, 2 N, K].
int lt_gemm_skinny_grouped(const void* x, long long ldx, const void* w, void* y, const int* group, const int* group_rows,
                           const int* live, const int* src, int max_blocks, int block_rows, int N, int K, int act, void* stream) {
  using namespace lt;
  SkinnyParams p{};
  p.x = static_cast<const __nv_bfloat16*>(x); p.ldx = ldx;
  p.w = static_cast<const __nv_bfloat16*>(w); p.ldw = K; p.sw = (long long)(act ? 2 * N : N) * K;
  p.y = static_cast<__nv_bfloat16*>(y); p.ldy = N;
  p.N = N; p.K = K; p.act = act;
  p.group = group; p.group_rows = group_rows; p.live = live; p.src = src;
  if (max_blocks < 1 || max_blocks > 65535 || act < 0 || act > 2 || (block_rows != 16 && block_rows != 32 && block_rows != 64) ||
      !skinny_ok(p))
    return -int(kStatusBadArgument);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return act ? skinny_by_rows<kSkGrouped, true>(p, block_rows, max_blocks, st) : skinny_by_rows<kSkGrouped, false>(p, block_rows, max_blocks, st);
}

}  // extern "C"
