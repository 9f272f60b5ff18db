// GEMM on the CUDA cores for what the tensor-core kernels do not take: true fp32 operands (no reduced-precision mode) and
// bf16 operands whose pitch or inner extent TMA cannot describe.  Optionally a batch of equal products at fixed element
// offsets (a block-diagonal matrix is one).  Also the narrow projection with fp32 results (gates of a recurrence).
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

constexpr int kStTile = 64, kStK = 16;

// C[M, N] = alpha * A[M, K] @ B[N, K]^T; 256 threads, 4 x 4 results each, fp32 accumulation in blocks of kStK (a sum of short
// sums: the rounding error grows with the number of blocks, not with K).
template <typename T, typename TO>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ B, TO* __restrict__ C, int M, int N, int K, long long lda,
                 long long ldb, long long ldc, long long sa, long long sb, long long sc, float alpha) {
  __shared__ float As[kStK][kStTile + 4], Bs[kStK][kStTile + 4];
  A += blockIdx.z * sa;
  B += blockIdx.z * sb;
  C += blockIdx.z * sc;
  const int m0 = blockIdx.y * kStTile, n0 = blockIdx.x * kStTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kStK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * 256;
      const int r = e >> 4, k = k0 + (e & 15);
      As[e & 15][r] = (m0 + r < M && k < K) ? ldf(A + (m0 + r) * lda + k) : 0.f;
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

// y[R, J] (fp32) = x[R, K] @ w[J, K]^T for a narrow w: a CTA makes a 4 x 4 patch, its eight warps share K (so that a
// handful of rows is not bound by the latency of one long walk) and fold their sums through shared memory.
constexpr int kRdTile = 4;
template <typename T, int V>
__global__ void __launch_bounds__(256)
rows_dot_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, float* __restrict__ y, int R, int J, int K) {
  __shared__ float part[8][kRdTile * kRdTile];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = blockIdx.x * kRdTile, j0 = blockIdx.y * kRdTile;
  const T* xp[kRdTile];
  const T* wp[kRdTile];
#pragma unroll
  for (int i = 0; i < kRdTile; ++i) {            // rows past the end read the last row; their results are dropped
    xp[i] = x + min(r0 + i, R - 1) * ldx;
    wp[i] = w + (long long)min(j0 + i, J - 1) * K;
  }
  float acc[kRdTile][kRdTile] = {};
#pragma unroll 2
  for (int k = threadIdx.x * V; k < K; k += 256 * V) {
    float xv[kRdTile][V], wv[kRdTile][V];
#pragma unroll
    for (int i = 0; i < kRdTile; ++i) {
      if constexpr (V == 4) {
        const float4 a = ldf4(xp[i] + k), b = ldf4(wp[i] + k);
        xv[i][0] = a.x; xv[i][1] = a.y; xv[i][2] = a.z; xv[i][3] = a.w;
        wv[i][0] = b.x; wv[i][1] = b.y; wv[i][2] = b.z; wv[i][3] = b.w;
      } else {
        xv[i][0] = ldf(xp[i] + k);
        wv[i][0] = ldf(wp[i] + k);
      }
    }
#pragma unroll
    for (int r = 0; r < kRdTile; ++r)
#pragma unroll
      for (int c = 0; c < kRdTile; ++c)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[r][c] = fmaf(xv[r][v], wv[c][v], acc[r][c]);
  }
#pragma unroll
  for (int r = 0; r < kRdTile; ++r)
#pragma unroll
    for (int c = 0; c < kRdTile; ++c) {
      const float v = warp_sum(acc[r][c]);
      if (lane == 0) part[warp][r * kRdTile + c] = v;
    }
  __syncthreads();
  if (threadIdx.x < kRdTile * kRdTile) {
    const int r = r0 + threadIdx.x / kRdTile, c = j0 + threadIdx.x % kRdTile;
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) v += part[i][threadIdx.x];
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
#define LT_ST(TI, TO) gemm_simt_kernel<TI, TO><<<grid, 256, 0, st>>>(static_cast<const TI*>(A), static_cast<const TI*>(B), \
                                                                     static_cast<TO*>(C), M, N, K, lda, ldb, ldc, sa, sb, sc, alpha)
  if (in_fp32 && out_fp32) LT_ST(float, float);
  else if (!in_fp32 && out_fp32) LT_ST(bf, float);
  else if (!in_fp32) LT_ST(bf, bf);
  else return -4;
#undef LT_ST
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_rows_dot(int fp32, const void* x, long long ldx, const void* w, float* y, int R, int J, int K, void* stream) {
  using namespace lt;
  if (R <= 0 || J <= 0) return 0;
  dim3 grid((R + kRdTile - 1) / kRdTile, (J + kRdTile - 1) / kRdTile);
  if (grid.y > 65535) return -4;
  const bool v4 = K % 4 == 0 && ldx % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
#define LT_RD(T, V) rows_dot_kernel<T, V><<<grid, 256, 0, st>>>(static_cast<const T*>(x), ldx, static_cast<const T*>(w), y, R, J, K)
  if (fp32) { if (v4) LT_RD(float, 4); else LT_RD(float, 1); }
  else { if (v4) LT_RD(bf, 4); else LT_RD(bf, 1); }
#undef LT_RD
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
