// Hyper-connected residual streams with the RMS norm of the next sublayer, in one pass over the streams.
//
// A model with hyper-connections keeps `streams` residual copies x_1 .. x_s per token.  Between two sublayers every token
// needs: the update of all streams with the finished sublayer's output y,
//     x_t <- sum_s mix[s, t] x_s + out[t] y,
// the mixed input of the next one, u = sum_s in[s] x_s, and its RMS norm.  One CTA owns a token: the streams are read and
// written once (fp32), u stays in shared memory between the sum of squares and the normalisation.  y may be one branch or
// the half sum of two branches that are RMS-normed over the model width first.  The first sublayer of a model starts the
// streams as copies of the embedding row; the last call reads u as the plain sum of the streams (no `in`) and keeps nothing.
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

constexpr int kHyperMaxStreams = 16;

struct HyperParams {
  float* x;                 // [tokens, streams, width]
  const int* tokens;        // with `embed`: the streams start as embed[tokens[row]]
  const void* embed;
  const void* y1;           // finished sublayer (nullptr: nothing to add)
  const void* y2;
  long long ldy1, ldy2;
  const float* n1;          // RMS weights of the two branches (nullptr: y1 is added as it is)
  const float* n2;
  const float* mix;         // [streams, streams] as [from, to]
  const float* out;         // [streams]
  const float* in;          // [streams] or nullptr: ones
  const float* norm;        // [width]
  float eps;
  void* h;
  long long ldh;
  const int* rows;          // which tokens of x to take (nullptr: all, in order)
  int width, streams, write_x;
};

// S: number of streams, 0 = read it from the parameters.  V: elements per access.
template <typename T, int S, int V>
__global__ void __launch_bounds__(256) hyper_norm_kernel(const HyperParams p) {
  extern __shared__ float u_s[];                      // [width]
  __shared__ float red[64];
  __shared__ float mix_s[kHyperMaxStreams * kHyperMaxStreams], out_s[kHyperMaxStreams], in_s[kHyperMaxStreams];
  constexpr int MS = S > 0 ? S : kHyperMaxStreams;
  const int ns = S > 0 ? S : p.streams;
  const int W = p.width;
  const bool update = p.y1 != nullptr;
  const long long row = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  for (int i = threadIdx.x; i < ns * ns; i += blockDim.x) mix_s[i] = update ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < ns; i += blockDim.x) {
    out_s[i] = update ? p.out[i] : 0.f;
    in_s[i] = p.in ? p.in[i] : 1.f;
  }
  const T* y1 = update ? static_cast<const T*>(p.y1) + row * p.ldy1 : nullptr;
  const T* y2 = p.n1 ? static_cast<const T*>(p.y2) + row * p.ldy2 : nullptr;
  float r1 = 0.f, r2 = 0.f;
  if (update && p.n1) {
    float a = 0.f, b = 0.f;
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
      if constexpr (V == 4) {
        const float4 f = ldf4(y1 + c), g = ldf4(y2 + c);
        a += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
        b += g.x * g.x + g.y * g.y + g.z * g.z + g.w * g.w;
      } else {
        const float f = ldf(y1 + c), g = ldf(y2 + c);
        a += f * f;
        b += g * g;
      }
    }
    const float2 s = block_sum2(a, b, red);
    r1 = 0.5f / sqrtf(s.x / W + p.eps);
    r2 = 0.5f / sqrtf(s.y / W + p.eps);
  }
  __syncthreads();
  float* xr = p.x ? p.x + row * (long long)ns * W : nullptr;
  const T* er = p.embed ? static_cast<const T*>(p.embed) + (long long)p.tokens[row] * W : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float xs[MS][V], y[V];
#pragma unroll
    for (int s = 0; s < MS; ++s) {
      if (s < ns) {
        if constexpr (V == 4) {
          const float4 f = er ? ldf4(er + c) : *reinterpret_cast<const float4*>(xr + (long long)s * W + c);
          xs[s][0] = f.x; xs[s][1] = f.y; xs[s][2] = f.z; xs[s][3] = f.w;
        } else {
          xs[s][0] = er ? ldf(er + c) : xr[(long long)s * W + c];
        }
      }
    }
    if (update) {
      if constexpr (V == 4) {
        const float4 f = ldf4(y1 + c);
        y[0] = f.x; y[1] = f.y; y[2] = f.z; y[3] = f.w;
      } else {
        y[0] = ldf(y1 + c);
      }
      if (p.n1) {
        float z[V];
        if constexpr (V == 4) {
          const float4 f = ldf4(y2 + c);
          z[0] = f.x; z[1] = f.y; z[2] = f.z; z[3] = f.w;
        } else {
          z[0] = ldf(y2 + c);
        }
#pragma unroll
        for (int v = 0; v < V; ++v) y[v] = y[v] * r1 * p.n1[c + v] + z[v] * r2 * p.n2[c + v];
      }
    }
    float u[V];
#pragma unroll
    for (int v = 0; v < V; ++v) u[v] = 0.f;
#pragma unroll
    for (int t = 0; t < MS; ++t) {
      if (t < ns) {
        float nx[V];
#pragma unroll
        for (int v = 0; v < V; ++v) nx[v] = xs[t][v];
        if (update) {
#pragma unroll
          for (int v = 0; v < V; ++v) nx[v] = out_s[t] * y[v];
#pragma unroll
          for (int s = 0; s < MS; ++s) {
            if (s < ns) {
#pragma unroll
              for (int v = 0; v < V; ++v) nx[v] = fmaf(mix_s[s * ns + t], xs[s][v], nx[v]);
            }
          }
        }
        if (p.write_x) {
          if constexpr (V == 4) *reinterpret_cast<float4*>(xr + (long long)t * W + c) = make_float4(nx[0], nx[1], nx[2], nx[3]);
          else xr[(long long)t * W + c] = nx[0];
        }
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = fmaf(in_s[t], nx[v], u[v]);
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) {
      u_s[c + v] = u[v];
      ss += u[v] * u[v];
    }
  }
  const float inv = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / W + p.eps);
  T* h = static_cast<T*>(p.h) + (long long)blockIdx.x * p.ldh;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {      // every thread reads back what it wrote itself
    if constexpr (V == 4) {
      stf4(h + c, make_float4(u_s[c] * inv * p.norm[c], u_s[c + 1] * inv * p.norm[c + 1], u_s[c + 2] * inv * p.norm[c + 2],
                              u_s[c + 3] * inv * p.norm[c + 3]));
    } else {
      stf(h + c, u_s[c] * inv * p.norm[c]);
    }
  }
}

template <typename T, int S>
static int launch_hyper(const HyperParams& p, int rows, bool vec, cudaStream_t st) {
  const size_t smem = size_t(p.width) * 4;
  auto kern = vec ? hyper_norm_kernel<T, S, S == 0 ? 1 : 4> : hyper_norm_kernel<T, S, 1>;
  if (smem > 48 * 1024) LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
  const int per = vec ? 4 : 1;
  int threads = ((p.width + per - 1) / per + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  kern<<<rows, threads, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

template <typename T>
static int hyper_dispatch(const HyperParams& p, int rows, bool vec, cudaStream_t st) {
  switch (p.streams) {
    case 1: return launch_hyper<T, 1>(p, rows, vec, st);
    case 2: return launch_hyper<T, 2>(p, rows, vec, st);
    case 3: return launch_hyper<T, 3>(p, rows, vec, st);
    case 4: return launch_hyper<T, 4>(p, rows, vec, st);
    default: return launch_hyper<T, 0>(p, rows, false, st);      // any other number: scalar accesses keep the streams in registers
  }
}

}  // namespace lt

extern "C" {

int lt_hyper_norm(int fp32, void* x, const int* tokens, const void* embed, const void* y1, long long ldy1, const float* n1,
                  const void* y2, long long ldy2, const float* n2, const float* mix, const float* out, const float* in,
                  const float* norm, float eps, void* h, long long ldh, const int* rows, int n_rows, int width, int streams,
                  int write_x, void* stream) {
  using namespace lt;
  if (streams < 1 || streams > kHyperMaxStreams || width < 1 || width > 49152 || (!x && !embed) || (write_x && !x)) return -4;
  if (n_rows == 0) return 0;
  HyperParams p{};
  p.x = static_cast<float*>(x);
  p.tokens = tokens; p.embed = embed;
  p.y1 = y1; p.ldy1 = ldy1; p.n1 = n1;
  p.y2 = y2; p.ldy2 = ldy2; p.n2 = n2;
  p.mix = mix; p.out = out; p.in = in; p.norm = norm; p.eps = eps;
  p.h = h; p.ldh = ldh; p.rows = rows; p.width = width; p.streams = streams; p.write_x = write_x;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = width % 4 == 0 && ldh % 4 == 0 && ldy1 % 4 == 0 && ldy2 % 4 == 0 && al(x) && al(embed) && al(y1) && al(y2) && al(h);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return fp32 ? hyper_dispatch<float>(p, n_rows, vec, st) : hyper_dispatch<__nv_bfloat16>(p, n_rows, vec, st);
}

}  // extern "C"
