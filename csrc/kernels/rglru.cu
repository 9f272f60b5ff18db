// Gated linear recurrence (RG-LRU) with the short causal convolution in front of it.
//
//   u_t = conv(x_t + bx)                          per channel, `taps` taps, zeros before the sequence
//   r_t = sigmoid(ra u_t + ra.b), i_t = sigmoid(ri u_t + ri.b)      block-diagonal matrices
//   log a_t = -8 r_t softplus(lam);   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t;   out_t = S_t gelu(y_t + by)
//
// Prompts run as three launches: the convolution, the block-diagonal product (the tensor-core GEMM with one block per
// column group, logits in fp32) and a scan in which a CTA owns 16 channels, splits 256 tokens over its threads, composes the
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

// u[n, c] for tokens start .. start + N - 1 of one sequence; earlier inputs come from the ring.  A thread walks
// kConvTokens tokens of V channels; with TAPS known the weights and the last inputs stay in registers.
constexpr int kConvTokens = 8;
template <typename T, int TAPS, int V>
__global__ void __launch_bounds__(128)
conv_causal_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ xb, const float* __restrict__ w,
                   const float* __restrict__ b, const float* __restrict__ ring, T* __restrict__ u, int N, int C, int taps, int start) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int t0 = blockIdx.y * kConvTokens;
  auto input = [&](int t, float (&v)[V]) {
    const int pos = start + t;
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = 0.f;
    if (t >= N) return;
    if (t >= 0) {
      if constexpr (V == 4) {
        const float4 f = ldf4(x + t * ldx + c);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
      } else {
        v[0] = ldf(x + t * ldx + c);
      }
      if (xb)
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] += xb[c + k];
    } else if (pos >= 0) {
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = ring[(long long)(pos % taps) * C + c + k];
    }
  };
  float acc[kConvTokens][V];
#pragma unroll
  for (int i = 0; i < kConvTokens; ++i)
#pragma unroll
    for (int k = 0; k < V; ++k) acc[i][k] = b[c + k];
  if constexpr (TAPS > 0) {
    float wt[V][TAPS];
#pragma unroll
    for (int k = 0; k < V; ++k)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) wt[k][j] = w[(long long)(c + k) * TAPS + j];
#pragma unroll
    for (int d = -(TAPS - 1); d < kConvTokens; ++d) {
      float v[V];
      input(t0 + d, v);
#pragma unroll
      for (int i = 0; i < kConvTokens; ++i) {
        const int tap = TAPS - 1 - i + d;                    // which tap of output t0 + i this input meets
        if (tap >= 0 && tap < TAPS)
#pragma unroll
          for (int k = 0; k < V; ++k) acc[i][k] = fmaf(v[k], wt[k][tap], acc[i][k]);
      }
    }
  } else {
    for (int d = -(taps - 1); d < kConvTokens; ++d) {
      float v[V];
      input(t0 + d, v);
#pragma unroll
      for (int i = 0; i < kConvTokens; ++i) {
        const int tap = taps - 1 - i + d;
        if (tap >= 0 && tap < taps)
#pragma unroll
          for (int k = 0; k < V; ++k) acc[i][k] = fmaf(v[k], w[(long long)(c + k) * taps + tap], acc[i][k]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kConvTokens; ++i)
    if (t0 + i < N) {
      if constexpr (V == 4) stf4(u + (long long)(t0 + i) * C + c, make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]));
      else stf(u + (long long)(t0 + i) * C + c, acc[i][0]);
    }
}

struct RglruGate {
  float a, b;     // S <- a S + b
};
// fp32 activations: the library functions.
__device__ __forceinline__ RglruGate rglru_gate(const float*, float r_logit, float i_logit, float u, float sp) {
  const float log_a = -8.f * sigmoid_f(r_logit) * sp;
  // 1 - a^2 without cancellation where a is close to 1
  return RglruGate{expf(log_a), sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i_logit) * u};
}
__device__ __forceinline__ float gelu_branch(const float*, float z) { return gelu_tanh_f(z); }
// bf16 activations: the same in fp32 on the fast exponential and divide (a few units in the last place of fp32).
__device__ __forceinline__ float fast_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ RglruGate rglru_gate(const __nv_bfloat16*, float r_logit, float i_logit, float u, float sp) {
  const float log_a = -8.f * fast_sigmoid(r_logit) * sp;
  const float a = __expf(log_a), x = -2.f * log_a;
  // 1 - exp(-x): its power series where the difference would cancel
  const float series = x * (1.f - x * (0.5f - x * (1.f / 6 - x * (1.f / 24 - x * (1.f / 120 - x * (1.f / 720))))));
  const float rest = x < 0.25f ? series : 1.f - a * a;
  return RglruGate{a, sqrtf(rest) * fast_sigmoid(i_logit) * u};
}
__device__ __forceinline__ float gelu_branch(const __nv_bfloat16*, float z) {
  // (1 + tanh(y)) / 2 is sigmoid(2 y)
  return z * fast_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}

constexpr int kScanCh = 16, kScanSeg = 32, kScanLen = 8;
template <typename T>
__global__ void __launch_bounds__(kScanCh * kScanSeg, 1)
rglru_scan_kernel(const T* __restrict__ u, const float* __restrict__ gates, const float* __restrict__ rb, const float* __restrict__ ib,
                  const float* __restrict__ sp, const T* __restrict__ y, long long ldy, const float* __restrict__ yb,
                  const T* __restrict__ x, long long ldx, const float* __restrict__ xb, float* __restrict__ state,
                  float* __restrict__ ring, T* __restrict__ out, int N, int C, int bw, int taps, int start) {
  __shared__ float2 part[kScanSeg][kScanCh];                 // (A, B) of every segment: S <- A S + B
  __shared__ float enter[kScanSeg + 1][kScanCh];             // the state before every segment, and after the last
  const int ch = threadIdx.x % kScanCh, seg = threadIdx.x / kScanCh;
  const int c = blockIdx.x * kScanCh + ch;
  const bool ok = c < C;
  const int cc = ok ? c : C - 1;
  const int gcol = (cc / bw) * 2 * bw + cc % bw;            // column of r in the gates of block c / bw; i is bw further
  const float my_sp = sp[cc], my_rb = rb[cc], my_ib = ib[cc], my_yb = yb[cc];
  constexpr int kStep = kScanSeg * kScanLen;
  const T* tag = nullptr;
  if (seg == 0) enter[0][ch] = start > 0 ? state[cc] : 0.f;
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
  for (int base = 0; base < N; base += kStep) {
    RglruGate g[kScanLen];
    float yy[kScanLen], A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < kScanLen; ++k) {
      const int t = base + seg * kScanLen + k;
      g[k] = t < N ? rglru_gate(tag, cr[k] + my_rb, ci[k] + my_ib, cu[k], my_sp) : RglruGate{1.f, 0.f};
      yy[k] = cy[k] + my_yb;
      A *= g[k].a;
      B = fmaf(g[k].a, B, g[k].b);
    }
    if (base + kStep < N) load(base + kStep);                 // in flight during the exchange below
    part[seg][ch] = make_float2(A, B);
    __syncthreads();
    if (seg == 0) {                                           // one thread per channel walks the segments
      float h = enter[0][ch];
#pragma unroll
      for (int s = 0; s < kScanSeg; ++s) {
        enter[s][ch] = h;
        const float2 m = part[s][ch];
        h = fmaf(m.x, h, m.y);
      }
      enter[kScanSeg][ch] = h;
    }
    __syncthreads();
    float hs = enter[seg][ch];
#pragma unroll
    for (int k = 0; k < kScanLen; ++k) {
      const int t = base + seg * kScanLen + k;
      hs = fmaf(g[k].a, hs, g[k].b);
      if (ok && t < N) stf(out + (long long)t * C + c, hs * gelu_branch(tag, yy[k]));
    }
    // segment 0 moves on to the next step's entry state only after it has used its own (same thread)
    if (seg == 0) enter[0][ch] = enter[kScanSeg][ch];
  }
  if (ok && seg == 0) state[c] = enter[0][ch];
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
  // where the earlier inputs of every sequence lie in its ring (-1: before its start), and where the new one goes
  __shared__ int tap_row[kStepSeqs][kRgMaxTaps];
  for (int i = threadIdx.x; i < ns * p.taps; i += blockDim.x) {
    const int s = i / p.taps, k = i % p.taps, q = p.positions[s0 + s] - (p.taps - 1) + k;
    tap_row[s][k] = q >= 0 ? p.slots[s0 + s] * p.taps + q % p.taps : -1;
  }
  __syncthreads();
#pragma unroll 4
  for (int i = threadIdx.x; i < ns * p.bw; i += blockDim.x) {
    const int s = i / p.bw, j = i % p.bw, c = c0 + j;
    const float now = ldf(static_cast<const T*>(p.x) + (s0 + s) * p.ldx + c) + (p.xb ? p.xb[c] : 0.f);
    float acc = p.conv_b[c];
    const float* w = p.conv_w + (long long)c * p.taps;
#pragma unroll 4
    for (int k = 0; k < p.taps - 1; ++k) {
      const int row = tap_row[s][k];
      if (row >= 0) acc = fmaf(p.ring[(long long)row * p.C + c], w[k], acc);
    }
    acc = fmaf(now, w[p.taps - 1], acc);
    u_s[i] = round_as(static_cast<const T*>(nullptr), acc);
  }
  // the new input goes into the row of position - taps, which nobody reads in this step (a loop of its own: stores between
  // the loads above would keep them from overlapping)
  for (int i = threadIdx.x; i < ns * (j1 - j0); i += blockDim.x) {
    const int s = i / (j1 - j0), c = c0 + j0 + i % (j1 - j0);
    p.ring[(long long)tap_row[s][p.taps - 1] * p.C + c] = ldf(static_cast<const T*>(p.x) + (s0 + s) * p.ldx + c) + (p.xb ? p.xb[c] : 0.f);
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
      const RglruGate g = rglru_gate(static_cast<const T*>(nullptr), rl + p.rb[c], il + p.ib[c], u_s[lane * p.bw + j], p.sp[c]);
      float* st = p.state + (long long)p.slots[s] * p.C + c;
      const float prev = p.positions[s] > 0 ? *st : 0.f;
      const float h = fmaf(g.a, prev, g.b);
      *st = h;
      stf(static_cast<T*>(p.out) + (long long)s * p.C + c,
          h * gelu_branch(static_cast<const T*>(nullptr), ldf(static_cast<const T*>(p.y) + s * p.ldy + c) + p.yb[c]));
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
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool v4 = C % 4 == 0 && ldx % 4 == 0 && (fp32 ? al(x) : (reinterpret_cast<uintptr_t>(x) & 7) == 0) && al(u);
  const int per = v4 ? 512 : 128;
  dim3 grid((C + per - 1) / per, tb);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LT_CONV(T, TAPS, V) conv_causal_kernel<T, TAPS, V><<<grid, 128, 0, st>>>( \
      static_cast<const T*>(x), ldx, xb, w, b, ring, static_cast<T*>(u), N, C, taps, start)
#define LT_CONV_T(T)                                    \
  if (v4 && taps == 4) LT_CONV(T, 4, 4);                \
  else if (v4 && taps == 3) LT_CONV(T, 3, 4);           \
  else if (v4 && taps == 2) LT_CONV(T, 2, 4);           \
  else if (v4) LT_CONV(T, 0, 4);                        \
  else LT_CONV(T, 0, 1)
  if (fp32) { LT_CONV_T(float); }
  else { LT_CONV_T(__nv_bfloat16); }
#undef LT_CONV_T
#undef LT_CONV
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
  if (bw < 1 || C % bw != 0 || taps < 1 || taps > kRgMaxTaps || smem > 200 * 1024) return -4;
  const int blocks = C / bw, groups = (S + kStepSeqs - 1) / kStepSeqs;
  // rows per CTA: whole warps of work, about one CTA per SM (each rebuilds u of its block)
  int rows = bw;
  while (rows > kStepWarps && blocks * groups * ((bw + rows - 1) / rows) < sm_count()) rows = (rows + 1) / 2;
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
