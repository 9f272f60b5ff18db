// A single fp32 residual whose sublayers are normed on both sides, in one pass over the residual.
//
// Between two sublayers every token needs the finished sublayer's output y (RMS-normed over the model width, weighted, times
// one multiplier) added to its residual row, and the RMS norm of the result as the next sublayer's input - or the row
// itself, rounded, where the next reader wants it unnormed.  y is one row, the weighted sum of a token's expert rows (each
// token of a mixture of experts has `top` rows somewhere in an expert-ordered buffer), or both.  One CTA owns a token and
// keeps residual and y in registers, so each is read once.  The first call of a model starts the residual as the
// embedding row; the last one takes the wanted rows only and keeps nothing.
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

struct ResidualParams {
  float* x;                 // [tokens, width]
  const int* tokens;        // with `embed`: the residual starts as embed[tokens[row]]
  const void* embed;
  const void* y;            // [tokens, width] at pitch ldy, or nullptr
  long long ldy;
  const void* z;            // expert rows [., width], or nullptr
  const int* z_slot;        // [tokens, top] row of z
  const float* z_weight;    // [tokens, top]
  int top;
  const float* y_norm;      // nullptr: y is added as it is
  float mult;
  const float* norm;        // nullptr: h is the residual itself
  float eps;
  void* h;
  const int* rows;          // which tokens to take (nullptr: all, in order)
  int width, write_x;
};

// V: elements per access (1 or 4).  NC: accesses per thread.
constexpr int max_threads(int V) { return V == 4 ? 512 : 1024; }
template <typename T, int V, int NC>
__global__ void __launch_bounds__(max_threads(V)) residual_norm_kernel(const ResidualParams p) {
  __shared__ float red[64];
  const int W = p.width, nt = blockDim.x;
  const long long row = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float x[NC][V], y[NC][V];
  auto load = [&](const T* src, float (&v)[V]) {
    if constexpr (V == 4) {
      const float4 f = ldf4(src);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
      v[0] = ldf(src);
    }
  };
  const float* xr = p.x + row * W;
  const T* er = p.embed ? static_cast<const T*>(p.embed) + (long long)p.tokens[row] * W : nullptr;
  const T* yr = p.y ? static_cast<const T*>(p.y) + row * p.ldy : nullptr;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * nt + threadIdx.x) * V;
#pragma unroll
    for (int v = 0; v < V; ++v) x[i][v] = y[i][v] = 0.f;
    if (c < W) {
      if (er) load(er + c, x[i]);
      else if constexpr (V == 4) {
        const float4 f = ldf4(xr + c);
        x[i][0] = f.x; x[i][1] = f.y; x[i][2] = f.z; x[i][3] = f.w;
      } else {
        x[i][0] = xr[c];
      }
      if (yr) load(yr + c, y[i]);
    }
  }
  // Few rows leave every load's latency in the open: there the norms' weights, and eight expert rows at a time, are on their way
  // together.  (With many rows that costs more in registers than it hides.)
  constexpr bool kEarly = NC == 1;
  [[maybe_unused]] float wy[V], wn[V];
  if constexpr (kEarly) {
    const int c = threadIdx.x * V;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      wy[v] = p.y_norm && c + v < W ? p.y_norm[c + v] : 1.f;
      wn[v] = p.norm && c + v < W ? p.norm[c + v] : 1.f;
    }
  }
  if (p.z) {
    constexpr int kRows = kEarly ? 8 : 1;
    for (int j0 = 0; j0 < p.top; j0 += kRows) {
      const T* zr[kRows];
      float a[kRows];
#pragma unroll
      for (int j = 0; j < kRows; ++j) {
        const bool in = j0 + j < p.top;
        zr[j] = static_cast<const T*>(p.z) + (in ? (long long)p.z_slot[row * p.top + j0 + j] * W : 0);
        a[j] = in ? p.z_weight[row * p.top + j0 + j] : 0.f;
      }
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = (i * nt + threadIdx.x) * V;
        if (c < W) {
          float z[kRows][V];
#pragma unroll
          for (int j = 0; j < kRows; ++j)
            if (j0 + j < p.top) load(zr[j] + c, z[j]);
#pragma unroll
          for (int j = 0; j < kRows; ++j)
            if (j0 + j < p.top) {
#pragma unroll
              for (int v = 0; v < V; ++v) y[i][v] = fmaf(a[j], z[j][v], y[i][v]);
            }
        }
      }
    }
  }
  if (p.y || p.z) {
    float f = p.mult;
    if (p.y_norm) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NC; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) ss = fmaf(y[i][v], y[i][v], ss);
      f *= 1.f / sqrtf(block_sum2(ss, 0.f, red).x / W + p.eps);
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * nt + threadIdx.x) * V;
      if (c < W) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          if constexpr (kEarly) x[i][v] = fmaf(f, y[i][v] * wy[v], x[i][v]);
          else x[i][v] = fmaf(f, p.y_norm ? y[i][v] * p.y_norm[c + v] : y[i][v], x[i][v]);
        }
      }
    }
  }
  if (p.write_x) {
    float* xw = p.x + row * W;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * nt + threadIdx.x) * V;
      if (c < W) {
        if constexpr (V == 4) stf4(xw + c, make_float4(x[i][0], x[i][1], x[i][2], x[i][3]));
        else xw[c] = x[i][0];
      }
    }
  }
  float inv = 1.f;
  if (p.norm) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) ss = fmaf(x[i][v], x[i][v], ss);
    inv = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / W + p.eps);
  }
  T* h = static_cast<T*>(p.h) + (long long)blockIdx.x * W;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * nt + threadIdx.x) * V;
    if (c < W) {
      float o[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        if constexpr (kEarly) o[v] = x[i][v] * inv * wn[v];
        else o[v] = p.norm ? x[i][v] * inv * p.norm[c + v] : x[i][v];
      }
      if constexpr (V == 4) stf4(h + c, make_float4(o[0], o[1], o[2], o[3]));
      else stf(h + c, o[0]);
    }
  }
}

template <typename T, int V>
static int launch_residual(const ResidualParams& p, int rows, cudaStream_t st) {
  const int pieces = (p.width + V - 1) / V;
  // many rows: a few accesses per thread in flight and cheap block sums; few rows: more threads, shorter latency
  int nc = rows >= 2 * sm_count() ? 4 : 1;
  while (nc < 8 && pieces > max_threads(V) * nc) nc *= 2;
  if (pieces > max_threads(V) * nc) return -4;
  const int threads = ((pieces + nc - 1) / nc + 31) / 32 * 32;
  switch (nc) {
    case 1: residual_norm_kernel<T, V, 1><<<rows, threads, 0, st>>>(p); break;
    case 2: residual_norm_kernel<T, V, 2><<<rows, threads, 0, st>>>(p); break;
    case 4: residual_norm_kernel<T, V, 4><<<rows, threads, 0, st>>>(p); break;
    default: residual_norm_kernel<T, V, 8><<<rows, threads, 0, st>>>(p); break;
  }
  LT_LAUNCH_CHECK();
  return 0;
}

}  // namespace lt

extern "C" {

int lt_residual_norm(int fp32, float* x, const int* tokens, const void* embed, const void* y, long long ldy, const void* z,
                     const int* z_slot, const float* z_weight, int top, const float* y_norm, float mult, const float* norm, float eps,
                     void* h, const int* rows, int n_rows, int width, int write_x, void* stream) {
  using namespace lt;
  if (width < 1 || (!x && !embed) || (write_x && !x) || (z && (!z_slot || !z_weight || top < 1))) return -4;
  if (n_rows == 0) return 0;
  ResidualParams p{x, tokens, embed, y, ldy, z, z_slot, z_weight, top, y_norm, mult, norm, eps, h, rows, width, write_x};
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = width % 4 == 0 && ldy % 4 == 0 && al(x) && al(embed) && al(y) && al(z) && al(h);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (fp32) return vec ? launch_residual<float, 4>(p, n_rows, st) : launch_residual<float, 1>(p, n_rows, st);
  return vec ? launch_residual<__nv_bfloat16, 4>(p, n_rows, st) : launch_residual<__nv_bfloat16, 1>(p, n_rows, st);
}

}  // extern "C"
