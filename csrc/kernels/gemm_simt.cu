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

// y[R, J] (fp32) = x[R, K] @ w[J, K]^T for a narrow w: a CTA takes four rows, its eight warps share the J columns, two at
// a time, so that a row of w is read once per four rows of x.
constexpr int kRdRows = 4;
template <typename T, int V>
__global__ void __launch_bounds__(256)
rows_dot_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, float* __restrict__ y, int R, int J, int K) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = blockIdx.x * kRdRows;
  for (int j = (blockIdx.y * 8 + warp) * 2; j < J; j += gridDim.y * 16) {
    const bool two = j + 1 < J;
    float acc[2][kRdRows] = {};
    for (int k = lane * V; k < K; k += 32 * V) {
      float wv[2][V];
      if constexpr (V == 4) {
        const float4 a = ldf4(w + (long long)j * K + k);
        const float4 b = two ? ldf4(w + (long long)(j + 1) * K + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        wv[0][0] = a.x; wv[0][1] = a.y; wv[0][2] = a.z; wv[0][3] = a.w;
        wv[1][0] = b.x; wv[1][1] = b.y; wv[1][2] = b.z; wv[1][3] = b.w;
      } else {
        wv[0][0] = ldf(w + (long long)j * K + k);
        wv[1][0] = two ? ldf(w + (long long)(j + 1) * K + k) : 0.f;
      }
#pragma unroll
      for (int r = 0; r < kRdRows; ++r) {
        if (r0 + r >= R) break;
        float xv[V];
        if constexpr (V == 4) {
          const float4 a = ldf4(x + (r0 + r) * ldx + k);
          xv[0] = a.x; xv[1] = a.y; xv[2] = a.z; xv[3] = a.w;
        } else {
          xv[0] = ldf(x + (r0 + r) * ldx + k);
        }
#pragma unroll
        for (int v = 0; v < V; ++v) {
          acc[0][r] = fmaf(wv[0][v], xv[v], acc[0][r]);
          acc[1][r] = fmaf(wv[1][v], xv[v], acc[1][r]);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < kRdRows; ++r) {
      const float a = warp_sum(acc[0][r]), b = warp_sum(acc[1][r]);
      if (lane == 0 && r0 + r < R) {
        y[(long long)(r0 + r) * J + j] = a;
        if (two) y[(long long)(r0 + r) * J + j + 1] = b;
      }
    }
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
  const int rb = (R + kRdRows - 1) / kRdRows;
  int jb = 1;
  if (rb < 148) jb = (J + 15) / 16;
  dim3 grid(rb, jb);
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
