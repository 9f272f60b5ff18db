// GEMM on the CUDA cores for what the tensor-core kernels do not take: true fp32 operands (no reduced-precision mode) and
// bf16 operands whose pitch or inner extent TMA cannot describe.  Optionally a batch of equal products at fixed element
// offsets (a block-diagonal matrix is one), or rows grouped by expert (a mixture of experts).  Also the narrow projection with
// fp32 results (gates of a recurrence, a router).
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

constexpr int kStTile = 64, kStK = 16;

// Rows in blocks of kStTile, each with the matrix of one expert (see lt_gemm_simt_grouped).
struct StGroups {
  const int* group;
  const int* rows;
  const int* live;
  const int* src;
};

// C[M, N] = alpha * A[M, K] @ B[N, K]^T; 256 threads, 4 x 4 results each, fp32 accumulation in blocks of kStK (a sum of short
// sums: the rounding error grows with the number of blocks, not with K).
template <typename T, typename TO, bool GROUPED>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ B, TO* __restrict__ C, int M, int N, int K, long long lda,
                 long long ldb, long long ldc, long long sa, long long sb, long long sc, float alpha, const StGroups gr) {
  __shared__ float As[kStK][kStTile + 4], Bs[kStK][kStTile + 4];
  __shared__ int row_of[kStTile];
  if constexpr (GROUPED) {
    if (int(blockIdx.y) >= *gr.live) return;
    M = blockIdx.y * kStTile + gr.rows[blockIdx.y];
    B += gr.group[blockIdx.y] * sb;
    if (threadIdx.x < kStTile) {
      const int m = blockIdx.y * kStTile + threadIdx.x;
      row_of[threadIdx.x] = !gr.src ? m : m < M ? gr.src[m] : 0;
    }
    __syncthreads();
  } else {
    A += blockIdx.z * sa;
    B += blockIdx.z * sb;
    C += blockIdx.z * sc;
  }
  const int m0 = blockIdx.y * kStTile, n0 = blockIdx.x * kStTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kStK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * 256;
      const int r = e >> 4, k = k0 + (e & 15);
      As[e & 15][r] = (m0 + r < M && k < K) ? ldf(A + (GROUPED ? row_of[r] : m0 + r) * lda + k) : 0.f;
      Bs[e & 15][r] = (n0 + r < N && k < K) ? ldf(B + (n0 + r) * ldb + k) : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};
#pragma unroll
    for (int k = 0; k < kStK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = As[k][ty * 4 + i]; b[i] = Bs[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(a[i], b[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) stf(C + m * ldc + n, acc[i][j] * alpha);
    }
}

// y[R, J] (fp32) = x[R, K] @ w[J, K]^T for a narrow w: a CTA makes a 4 x 8 patch, its eight warps share K (so that a
// handful of rows is not bound by the latency of one long walk) and fold their sums through shared memory.
constexpr int kRdR = 4, kRdJ = 8;
template <typename T, int V>
__global__ void __launch_bounds__(256)
rows_dot_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, float* __restrict__ y, int R, int J, int K) {
  __shared__ float part[8][kRdR * kRdJ];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = blockIdx.x * kRdR, j0 = blockIdx.y * kRdJ;
  float acc[kRdR * kRdJ] = {};
  for (int k = threadIdx.x * V; k < K; k += 256 * V) {
    float xv[kRdR][V];
    // rows past the end read the last row; their results are dropped
#pragma unroll
    for (int i = 0; i < kRdR; ++i) {
      const T* src = x + min(r0 + i, R - 1) * ldx + k;
      if constexpr (V == 8) ldf8(src, xv[i]);
      else xv[i][0] = ldf(src);
    }
#pragma unroll
    for (int c = 0; c < kRdJ; ++c) {
      const T* src = w + (long long)min(j0 + c, J - 1) * K + k;
      float wv[V];
      if constexpr (V == 8) ldf8(src, wv);
      else wv[0] = ldf(src);
#pragma unroll
      for (int r = 0; r < kRdR; ++r)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[r * kRdJ + c] = fmaf(xv[r][v], wv[v], acc[r * kRdJ + c]);
    }
  }
  part[warp][lane] = warp_sum_each<kRdR * kRdJ>(acc);
  __syncthreads();
  if (warp == 0) {
    const int r = r0 + lane / kRdJ, c = j0 + lane % kRdJ;
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) v += part[i][lane];
    if (r < R && c < J) y[(long long)r * J + c] = v;
  }
}

}  // namespace lt

extern "C" {

// Operands fp32 (in_fp32 = 1) or bf16, C fp32 or bf16; batch products at element offsets sa, sb, sc.
int lt_gemm_simt(int in_fp32, int out_fp32, const void* A, const void* B, void* C, int M, int N, int K, long long lda,
                 long long ldb, long long ldc, int batch, long long sa, long long sb, long long sc, float alpha, void* stream) {
  using namespace lt;
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0) return 0;
  const int mb = (M + kStTile - 1) / kStTile;
  if (batch > 65535 || mb > 65535) return -4;
  dim3 grid((N + kStTile - 1) / kStTile, mb, batch);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
#define LT_ST(TI, TO) gemm_simt_kernel<TI, TO, false><<<grid, 256, 0, st>>>( \
      static_cast<const TI*>(A), static_cast<const TI*>(B), static_cast<TO*>(C), M, N, K, lda, ldb, ldc, sa, sb, sc, alpha, StGroups{})
  if (in_fp32 && out_fp32) LT_ST(float, float);
  else if (!in_fp32 && out_fp32) LT_ST(bf, float);
  else if (!in_fp32) LT_ST(bf, bf);
  else return -4;
#undef LT_ST
  LT_LAUNCH_CHECK();
  return 0;
}

// Rows grouped by expert in blocks of 64: block b (of *live, at most max_blocks) takes rows src[64 b ..] of A (src nullptr: the same
// rows), group_rows[b] of them, times B[group[b]] ([experts, N, K]), into rows 64 b .. of C.  A, B and C of one type.
int lt_gemm_simt_grouped(int fp32, const void* A, long long lda, const void* B, void* C, const int* group, const int* group_rows,
                         const int* live, const int* src, int max_blocks, int N, int K, void* stream) {
  using namespace lt;
  if (max_blocks < 1 || max_blocks > 65535 || N < 1 || K < 1) return -4;
  dim3 grid((N + kStTile - 1) / kStTile, max_blocks);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const StGroups gr{group, group_rows, live, src};
  using bf = __nv_bfloat16;
#define LT_SG(T) gemm_simt_kernel<T, T, true><<<grid, 256, 0, st>>>(static_cast<const T*>(A), static_cast<const T*>(B), static_cast<T*>(C), \
                                                                    0, N, K, lda, K, N, 0, (long long)N * K, 0, 1.f, gr)
  if (fp32) LT_SG(float);
  else LT_SG(bf);
#undef LT_SG
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_rows_dot(int fp32, const void* x, long long ldx, const void* w, float* y, int R, int J, int K, void* stream) {
  using namespace lt;
  if (R <= 0 || J <= 0) return 0;
  dim3 grid((R + kRdR - 1) / kRdR, (J + kRdJ - 1) / kRdJ);
  if (grid.y > 65535) return -4;
  const bool v8 = K % 8 == 0 && ldx % 8 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
#define LT_RD(T, V) rows_dot_kernel<T, V><<<grid, 256, 0, st>>>(static_cast<const T*>(x), ldx, static_cast<const T*>(w), y, R, J, K)
  if (fp32) { if (v8) LT_RD(float, 8); else LT_RD(float, 1); }
  else { if (v8) LT_RD(bf, 8); else LT_RD(bf, 1); }
#undef LT_RD
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
