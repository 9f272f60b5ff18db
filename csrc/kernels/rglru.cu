// Gated linear recurrence (RG-LRU) with the short causal convolution in front of it.
//
//   u_t = conv(x_t + bx)                          per channel, `taps` taps, zeros before the sequence
//   r_t = sigmoid(ra u_t + ra.b), i_t = sigmoid(ri u_t + ri.b)      block-diagonal matrices
//   log a_t = -8 r_t softplus(lam);   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t;   out_t = S_t gelu(y_t + by)
//
// Prompts run as three launches: the convolution, the block-diagonal product (the tensor-core GEMM with one block per
// column group, logits in fp32) and a scan in which a CTA owns 16 channels, splits 128 tokens over its threads, composes the
// affine maps of the pieces in shared memory and carries the state through the whole prompt in one pass.  A decode step is
// one kernel: a CTA owns a slice of one block's outputs, rebuilds the block's u for its sequences in shared memory, streams
// its rows of ra and ri once for all of them and finishes the recurrence.
//
// State per sequence slot (fp32): S [width], and the newest convolution inputs x + bx in a ring of `taps` rows addressed by
// position modulo taps, so that a step writes a row that no other CTA of the same step reads.
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

constexpr int kRgMaxTaps = 32;

// u[n, c] for tokens start .. start + N - 1 of one sequence; earlier inputs come from the ring.
constexpr int kConvTokens = 8;
template <typename T>
__global__ void __launch_bounds__(128)
conv_causal_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ xb, const float* __restrict__ w,
                   const float* __restrict__ b, const float* __restrict__ ring, T* __restrict__ u, int N, int C, int taps, int start) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int t0 = blockIdx.y * kConvTokens;
  const float bx = xb ? xb[c] : 0.f;
  float acc[kConvTokens];
#pragma unroll
  for (int i = 0; i < kConvTokens; ++i) acc[i] = b[c];
  // input at t0 + d meets tap (taps - 1 - i + d) of output t0 + i
  for (int d = -(taps - 1); d < kConvTokens; ++d) {
    const int t = t0 + d, pos = start + t;
    if (t >= N) break;
    float v = 0.f;
    if (t >= 0) v = ldf(x + t * ldx + c) + bx;
    else if (pos >= 0) v = ring[(long long)(pos % taps) * C + c];
#pragma unroll
    for (int i = 0; i < kConvTokens; ++i) {
      const int tap = taps - 1 - i + d;
      if (tap >= 0 && tap < taps) acc[i] = fmaf(v, w[(long long)c * taps + tap], acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kConvTokens; ++i)
    if (t0 + i < N) stf(u + (long long)(t0 + i) * C + c, acc[i]);
}

struct RglruGate {
  float a, b;     // S <- a S + b
};
__device__ __forceinline__ RglruGate rglru_gate(float r_logit, float i_logit, float u, float sp) {
  const float log_a = -8.f * sigmoid_f(r_logit) * sp;
  // 1 - a^2 without cancellation where a is close to 1
  return RglruGate{expf(log_a), sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i_logit) * u};
}

constexpr int kScanCh = 16, kScanSeg = 16, kScanLen = 8;
template <typename T>
__global__ void __launch_bounds__(kScanCh * kScanSeg)
rglru_scan_kernel(const T* __restrict__ u, const float* __restrict__ gates, const float* __restrict__ rb, const float* __restrict__ ib,
                  const float* __restrict__ sp, const T* __restrict__ y, long long ldy, const float* __restrict__ yb,
                  const T* __restrict__ x, long long ldx, const float* __restrict__ xb, float* __restrict__ state,
                  float* __restrict__ ring, T* __restrict__ out, int N, int C, int bw, int taps, int start) {
  __shared__ float sA[kScanSeg][kScanCh], sB[kScanSeg][kScanCh];
  const int ch = threadIdx.x % kScanCh, seg = threadIdx.x / kScanCh;
  const int c = blockIdx.x * kScanCh + ch;
  const bool ok = c < C;
  const int cc = ok ? c : C - 1;
  const int gcol = (cc / bw) * 2 * bw + cc % bw;            // column of r in the gates of block c / bw; i is bw further
  const float my_sp = sp[cc], my_rb = rb[cc], my_ib = ib[cc], my_yb = yb[cc];
  float h = start > 0 ? state[cc] : 0.f;                     // every thread of the channel carries the same value
  float cu[kScanLen], cr[kScanLen], ci[kScanLen], cy[kScanLen];
  auto load = [&](int base) {
#pragma unroll
    for (int k = 0; k < kScanLen; ++k) {
      const int t = base + seg * kScanLen + k;
      if (t < N) {
        cu[k] = ldf(u + (long long)t * C + cc);
        cr[k] = gates[(long long)t * 2 * C + gcol];
        ci[k] = gates[(long long)t * 2 * C + gcol + bw];
        cy[k] = ldf(y + t * ldy + cc);
      }
    }
  };
  load(0);
  for (int base = 0; base < N; base += kScanSeg * kScanLen) {
    RglruGate g[kScanLen];
    float yy[kScanLen], A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < kScanLen; ++k) {
      const int t = base + seg * kScanLen + k;
      g[k] = t < N ? rglru_gate(cr[k] + my_rb, ci[k] + my_ib, cu[k], my_sp) : RglruGate{1.f, 0.f};
      yy[k] = cy[k] + my_yb;
      A *= g[k].a;
      B = fmaf(g[k].a, B, g[k].b);
    }
    if (base + kScanSeg * kScanLen < N) load(base + kScanSeg * kScanLen);      // in flight during the exchange below
    sA[seg][ch] = A;
    sB[seg][ch] = B;
    __syncthreads();
    float hs = h;
#pragma unroll
    for (int s = 0; s < kScanSeg; ++s) {
      if (s == seg) hs = h;
      h = fmaf(sA[s][ch], h, sB[s][ch]);
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kScanLen; ++k) {
      const int t = base + seg * kScanLen + k;
      hs = fmaf(g[k].a, hs, g[k].b);
      if (ok && t < N) stf(out + (long long)t * C + c, hs * gelu_tanh_f(yy[k]));
    }
  }
  if (ok && seg == 0) state[c] = h;
  // the newest inputs of the convolution, for what follows
  for (int t = max(0, N - taps) + seg; ok && t < N; t += kScanSeg)
    ring[(long long)((start + t) % taps) * C + c] = ldf(x + t * ldx + c) + (xb ? xb[c] : 0.f);
}

struct RglruStep {
  const void* x;            // [S, C] projections at pitch ldx (before the bias), likewise y
  const void* y;
  long long ldx, ldy;
  const float* xb;
  const float* yb;
  const float* conv_w;
  const float* conv_b;
  const void* gates;        // [blocks, 2 bw, bw] as [block, rows of ra | rows of ri, in]
  const float* rb;
  const float* ib;
  const float* sp;          // softplus(lam)
  float* state;             // [slots, C]
  float* ring;              // [slots, taps, C]
  const int* slots;         // [S]
  const int* positions;     // [S]
  void* out;                // [S, C]
  int S, C, bw, taps, rows_per_cta;
};

constexpr int kStepSeqs = 16, kStepWarps = 8;
template <typename T>
__global__ void __launch_bounds__(kStepWarps * 32) rglru_step_kernel(const RglruStep p) {
  extern __shared__ float u_s[];      // [kStepSeqs][bw]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slices = (p.bw + p.rows_per_cta - 1) / p.rows_per_cta;
  const int blk = blockIdx.x / slices, j0 = (blockIdx.x % slices) * p.rows_per_cta, j1 = min(p.bw, j0 + p.rows_per_cta);
  const int s0 = blockIdx.y * kStepSeqs, ns = min(kStepSeqs, p.S - s0);
  const int c0 = blk * p.bw;
  for (int i = threadIdx.x; i < ns * p.bw; i += blockDim.x) {
    const int s = s0 + i / p.bw, j = i % p.bw, c = c0 + j;
    const int pos = p.positions[s];
    float* ring = p.ring + (long long)p.slots[s] * p.taps * p.C;
    const float now = ldf(static_cast<const T*>(p.x) + s * p.ldx + c) + (p.xb ? p.xb[c] : 0.f);
    float acc = p.conv_b[c];
    for (int k = 0; k < p.taps - 1; ++k) {
      const int q = pos - (p.taps - 1) + k;
      if (q >= 0) acc = fmaf(ring[(long long)(q % p.taps) * p.C + c], p.conv_w[(long long)c * p.taps + k], acc);
    }
    acc = fmaf(now, p.conv_w[(long long)c * p.taps + p.taps - 1], acc);
    u_s[i] = round_as(static_cast<const T*>(nullptr), acc);
    if (j >= j0 && j < j1) ring[(long long)(pos % p.taps) * p.C + c] = now;      // the row of position - taps: read by nobody
  }
  __syncthreads();
  for (int j = j0 + warp; j < j1; j += kStepWarps) {
    const T* wr = static_cast<const T*>(p.gates) + ((long long)blk * 2 * p.bw + j) * p.bw;
    const T* wi = wr + (long long)p.bw * p.bw;
    float ar[kStepSeqs], ai[kStepSeqs];
#pragma unroll
    for (int s = 0; s < kStepSeqs; ++s) ar[s] = ai[s] = 0.f;
    for (int k = lane; k < p.bw; k += 32) {
      const float a = ldf(wr + k), b = ldf(wi + k);
#pragma unroll
      for (int s = 0; s < kStepSeqs; ++s) {
        if (s < ns) {
          const float f = u_s[s * p.bw + k];
          ar[s] = fmaf(a, f, ar[s]);
          ai[s] = fmaf(b, f, ai[s]);
        }
      }
    }
    float rl = 0.f, il = 0.f;
#pragma unroll
    for (int s = 0; s < kStepSeqs; ++s) {
      if (s < ns) {
        const float a = warp_sum(ar[s]), b = warp_sum(ai[s]);
        if (lane == s) { rl = a; il = b; }
      }
    }
    if (lane < ns) {
      const int s = s0 + lane, c = c0 + j;
      const RglruGate g = rglru_gate(rl + p.rb[c], il + p.ib[c], u_s[lane * p.bw + j], p.sp[c]);
      float* st = p.state + (long long)p.slots[s] * p.C + c;
      const float prev = p.positions[s] > 0 ? *st : 0.f;
      const float h = fmaf(g.a, prev, g.b);
      *st = h;
      stf(static_cast<T*>(p.out) + (long long)s * p.C + c,
          h * gelu_tanh_f(ldf(static_cast<const T*>(p.y) + s * p.ldy + c) + p.yb[c]));
    }
  }
}

}  // namespace lt

extern "C" {

// ring: the slot's [taps, C] rows.
int lt_conv_causal(int fp32, const void* x, long long ldx, const float* xb, const float* w, const float* b, const float* ring,
                   void* u, int N, int C, int taps, int start, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  if (taps < 1 || taps > kRgMaxTaps) return -4;
  const int tb = (N + kConvTokens - 1) / kConvTokens;
  if (tb > 65535) return -4;
  dim3 grid((C + 127) / 128, tb);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (fp32) conv_causal_kernel<float><<<grid, 128, 0, st>>>(static_cast<const float*>(x), ldx, xb, w, b, ring, static_cast<float*>(u), N, C, taps, start);
  else conv_causal_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(x), ldx, xb, w, b, ring, static_cast<__nv_bfloat16*>(u), N, C, taps, start);
  LT_LAUNCH_CHECK();
  return 0;
}

// gates [N, 2 C] fp32: per block bw logits of r, then bw of i.  state [C], ring [taps, C] of the sequence's slot.
int lt_rglru_scan(int fp32, const void* u, const float* gates, const float* rb, const float* ib, const float* sp, const void* y,
                  long long ldy, const float* yb, const void* x, long long ldx, const float* xb, float* state, float* ring, void* out,
                  int N, int C, int bw, int taps, int start, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  if (bw < 1 || C % bw != 0 || taps < 1 || taps > kRgMaxTaps) return -4;
  const int grid = (C + kScanCh - 1) / kScanCh;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LT_SCAN(T) rglru_scan_kernel<T><<<grid, kScanCh * kScanSeg, 0, st>>>( \
      static_cast<const T*>(u), gates, rb, ib, sp, static_cast<const T*>(y), ldy, yb, static_cast<const T*>(x), ldx, xb, state, ring, \
      static_cast<T*>(out), N, C, bw, taps, start)
  if (fp32) LT_SCAN(float);
  else LT_SCAN(__nv_bfloat16);
#undef LT_SCAN
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_rglru_step(int fp32, const void* x, long long ldx, const float* xb, const float* conv_w, const float* conv_b, const void* gates,
                  const float* rb, const float* ib, const float* sp, const void* y, long long ldy, const float* yb,
                  float* state, float* ring, const int* slots, const int* positions, void* out, int S, int C, int bw, int taps,
                  void* stream) {
  using namespace lt;
  if (S == 0) return 0;
  const int smem = kStepSeqs * bw * 4;
  if (bw < 1 || C % bw != 0 || taps < 1 || smem > 200 * 1024) return -4;
  const int blocks = C / bw, groups = (S + kStepSeqs - 1) / kStepSeqs;
  // rows per CTA: whole warps of work, about two CTAs per SM
  int rows = bw;
  while (rows > kStepWarps && blocks * groups * ((bw + rows - 1) / rows) < 2 * sm_count()) rows = (rows + 1) / 2;
  if (rows < kStepWarps) rows = bw < kStepWarps ? bw : kStepWarps;
  RglruStep p{x, y, ldx, ldy, xb, yb, conv_w, conv_b, gates, rb, ib, sp, state, ring, slots, positions, out, S, C, bw, taps, rows};
  dim3 grid(blocks * ((bw + rows - 1) / rows), groups);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (smem > 48 * 1024) {
    LT_RETURN_IF_CUDA(cudaFuncSetAttribute(rglru_step_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    LT_RETURN_IF_CUDA(cudaFuncSetAttribute(rglru_step_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  }
  if (fp32) rglru_step_kernel<float><<<grid, kStepWarps * 32, smem, st>>>(p);
  else rglru_step_kernel<__nv_bfloat16><<<grid, kStepWarps * 32, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
