// Gated linear recurrence (RG-LRU) with the short causal convolution in front of it.
//
//   u_t = conv(x_t + bx)                          per channel, `taps` taps, zeros before the sequence
//   r_t = sigmoid(ra u_t + ra.b), i_t = sigmoid(ri u_t + ri.b)      block-diagonal matrices
//   log a_t = -8 r_t softplus(lam);   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t;   out_t = S_t gelu(y_t + by)
//
// Prompts: the convolution, the block-diagonal product (the tensor-core GEMM with one block per column group, logits in
// fp32) and a scan in three launches (maps of 32-token pieces, a walk over the pieces, the pieces).  A decode step is
// two: the convolution, and the block-diagonal product with everything that follows it.
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
constexpr int kConvTokens = 16;
template <typename T, int TAPS, int V>
__global__ void __launch_bounds__(128)
conv_causal_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ xb, const float* __restrict__ w,
                   const float* __restrict__ b, const float* __restrict__ ring, T* __restrict__ u, int N, int C, int taps, int start) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int t0 = blockIdx.y * kConvTokens;
  float bx[V], bias[V];
#pragma unroll
  for (int k = 0; k < V; ++k) { bx[k] = xb ? xb[c + k] : 0.f; bias[k] = b[c + k]; }
  auto input = [&](int t, float (&v)[V]) {
    const int pos = start + t;
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = 0.f;
    if (t >= N) return;
    if (t >= 0) {
      if constexpr (V == 4) {
        const float4 f = ldf4(x + t * ldx + c);
        v[0] = f.x + bx[0]; v[1] = f.y + bx[1]; v[2] = f.z + bx[2]; v[3] = f.w + bx[3];
      } else {
        v[0] = ldf(x + t * ldx + c) + bx[0];
      }
    } else if (pos >= 0) {
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = ring[(long long)(pos % taps) * C + c + k];
    }
  };
  auto put = [&](int t, const float (&a)[V]) {
    if (t >= N) return;
    if constexpr (V == 4) stf4(u + (long long)t * C + c, make_float4(a[0], a[1], a[2], a[3]));
    else stf(u + (long long)t * C + c, a[0]);
  };
  if constexpr (TAPS > 1) {
    float wt[V][TAPS], past[TAPS - 1][V];          // past[j]: the input j + 1 tokens back
#pragma unroll
    for (int k = 0; k < V; ++k)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) wt[k][j] = w[(long long)(c + k) * TAPS + j];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(t0 - 1 - j, past[j]);
#pragma unroll
    for (int i = 0; i < kConvTokens; ++i) {
      float v[V], acc[V];
      input(t0 + i, v);
#pragma unroll
      for (int k = 0; k < V; ++k) {
        acc[k] = bias[k];
#pragma unroll
        for (int j = TAPS - 2; j >= 0; --j) acc[k] = fmaf(past[j][k], wt[k][TAPS - 2 - j], acc[k]);
        acc[k] = fmaf(v[k], wt[k][TAPS - 1], acc[k]);
#pragma unroll
        for (int j = TAPS - 2; j > 0; --j) past[j][k] = past[j - 1][k];
        past[0][k] = v[k];
      }
      put(t0 + i, acc);
    }
  } else {
    for (int i = 0; i < kConvTokens; ++i) {
      float acc[V];
#pragma unroll
      for (int k = 0; k < V; ++k) acc[k] = bias[k];
      for (int j = 0; j < taps; ++j) {
        float v[V];
        input(t0 + i - (taps - 1) + j, v);
#pragma unroll
        for (int k = 0; k < V; ++k) acc[k] = fmaf(v[k], w[(long long)(c + k) * taps + j], acc[k]);
      }
      put(t0 + i, acc);
    }
  }
}

struct RglruGate {
  float a, b;     // S <- a S + b
};
// Both forms work from d = 1 - a: where a is close to 1 the state remembers for thousands of tokens, and an a that is wrong in
// its last place the same way at every token adds up; 1 - d rounds once.  1 - a^2 = d (2 - d) does not cancel.
// fp32 activations: the library functions.
__device__ __forceinline__ RglruGate rglru_gate(const float*, float r_logit, float i_logit, float u, float sp) {
  const float d = -expm1f(-8.f * sigmoid_f(r_logit) * sp);
  return RglruGate{1.f - d, sqrtf(d * (2.f - d)) * sigmoid_f(i_logit) * u};
}
__device__ __forceinline__ float gelu_branch(const float*, float z) { return gelu_tanh_f(z); }
// bf16 activations: the same in fp32 on the fast exponential and divide (a few units in the last place of fp32).
__device__ __forceinline__ float fast_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ RglruGate rglru_gate(const __nv_bfloat16*, float r_logit, float i_logit, float u, float sp) {
  const float x = 8.f * fast_sigmoid(r_logit) * sp;                  // -log a
  // 1 - exp(-x): its power series where the difference would cancel
  const float series = x * (1.f - x * (0.5f - x * (1.f / 6 - x * (1.f / 24 - x * (1.f / 120 - x * (1.f / 720))))));
  const float d = x < 0.25f ? series : 1.f - __expf(-x);
  float root;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(d * (2.f - d)));
  return RglruGate{1.f - d, root * fast_sigmoid(i_logit) * u};
}
__device__ __forceinline__ float gelu_branch(const __nv_bfloat16*, float z) {
  // (1 + tanh(y)) / 2 is sigmoid(2 y)
  return z * fast_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}

// The scan over a prompt: pieces of kScanLen tokens.  Pass 0 composes the affine map of every piece, pass 1 (below) walks the
// pieces, pass 2 runs every piece from its entry state.  The gates are evaluated twice, but every pass runs with the whole
// GPU on it, and the second reading mostly comes from L2.
constexpr int kScanLen = 32;
struct RglruScan {
  const void* u;             // [N, C]
  const float* gates;        // [N, 2 C]: per block bw logits of r, then bw of i
  const float* rb;
  const float* ib;
  const float* sp;
  const void* y;
  long long ldy;
  const float* yb;
  float2* maps;              // [pieces, C]: S <- x S + y
  float* entry;              // [pieces, C]
  void* out;
  int N, C, bw;
};
template <typename T, int V, int PASS>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const RglruScan p) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= p.C) return;
  const int t0 = blockIdx.y * kScanLen, t1 = min(p.N, t0 + kScanLen);
  const T* tag = nullptr;
  float sp[V], rb[V], ib[V], yb[V], A[V], h[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    sp[v] = p.sp[c + v]; rb[v] = p.rb[c + v]; ib[v] = p.ib[c + v];
    yb[v] = PASS == 2 ? p.yb[c + v] : 0.f;
    A[v] = 1.f;
    h[v] = PASS == 2 ? p.entry[(long long)blockIdx.y * p.C + c + v] : 0.f;
  }
  const T* u = static_cast<const T*>(p.u) + c;
  const T* y = static_cast<const T*>(p.y) + c;
  const float* gr = p.gates + (c / p.bw) * 2 * p.bw + c % p.bw;
  T* out = static_cast<T*>(p.out) + c;
  constexpr int kAhead = V == 4 ? 2 : 4;                      // tokens per group; the next group's loads run under this one's math
  struct Group {
    float u[kAhead][V], r[kAhead][V], i[kAhead][V], y[kAhead][V];
  };
  Group buf[2];
  auto load = [&](Group& g, int tb) {
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      const long long t = min(tb + k, t1 - 1);
      if constexpr (V == 4) {
        *reinterpret_cast<float4*>(g.u[k]) = ldf4(u + t * p.C);
        *reinterpret_cast<float4*>(g.r[k]) = ldf4(gr + t * 2 * p.C);
        *reinterpret_cast<float4*>(g.i[k]) = ldf4(gr + t * 2 * p.C + p.bw);
        if (PASS == 2) *reinterpret_cast<float4*>(g.y[k]) = ldf4(y + t * p.ldy);
      } else {
        g.u[k][0] = ldf(u + t * p.C);
        g.r[k][0] = gr[t * 2 * p.C];
        g.i[k][0] = gr[t * 2 * p.C + p.bw];
        if (PASS == 2) g.y[k][0] = ldf(y + t * p.ldy);
      }
    }
  };
  auto run = [&](const Group& cur, int tb) {
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      if (tb + k >= t1) break;
      float o[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const RglruGate g = rglru_gate(tag, cur.r[k][v] + rb[v], cur.i[k][v] + ib[v], cur.u[k][v], sp[v]);
        h[v] = fmaf(g.a, h[v], g.b);
        if (PASS == 0) A[v] *= g.a;
        else o[v] = h[v] * gelu_branch(tag, cur.y[k][v] + yb[v]);
      }
      if (PASS == 2) {
        if constexpr (V == 4) stf4(out + (long long)(tb + k) * p.C, make_float4(o[0], o[1], o[2], o[3]));
        else stf(out + (long long)(tb + k) * p.C, o[0]);
      }
    }
  };
  load(buf[0], t0);
#pragma unroll 1
  for (int tb = t0; tb < t1; tb += 2 * kAhead) {
    load(buf[1], tb + kAhead);
    run(buf[0], tb);
    load(buf[0], tb + 2 * kAhead);
    run(buf[1], tb + kAhead);
  }
  if (PASS == 0)
#pragma unroll
    for (int v = 0; v < V; ++v) p.maps[(long long)blockIdx.y * p.C + c + v] = make_float2(A[v], h[v]);
}

// Pass 1: entry states of the pieces and the state after the last; also puts the newest convolution inputs into the ring.
// A CTA owns 16 channels; 32 threads per channel take a run of pieces each, compose it, and run it again from its entry state.
constexpr int kWalkCh = 16, kWalkSeg = 32;
template <typename T>
__global__ void __launch_bounds__(kWalkCh * kWalkSeg)
rglru_walk_kernel(const float2* __restrict__ maps, float* __restrict__ entry, float* __restrict__ state, const T* __restrict__ x,
                  long long ldx, const float* __restrict__ xb, float* __restrict__ ring, int N, int C, int pieces, int taps, int start) {
  __shared__ float2 run_s[kWalkSeg][kWalkCh];
  const int ch = threadIdx.x % kWalkCh, seg = threadIdx.x / kWalkCh;
  const int c = blockIdx.x * kWalkCh + ch;
  const bool ok = c < C;
  const float2* mp = maps + (ok ? c : C - 1);
  const int per = (pieces + kWalkSeg - 1) / kWalkSeg, p0 = seg * per, p1 = min(pieces, p0 + per);
  float A = 1.f, B = 0.f;
#pragma unroll 8
  for (int q = p0; q < p1; ++q) {
    const float2 m = mp[(long long)q * C];
    A *= m.x;
    B = fmaf(m.x, B, m.y);
  }
  run_s[seg][ch] = make_float2(A, B);
  float h = start > 0 && ok ? state[c] : 0.f;
  __syncthreads();
  float mine = h;
#pragma unroll
  for (int s = 0; s < kWalkSeg; ++s) {
    if (s == seg) mine = h;
    const float2 m = run_s[s][ch];
    h = fmaf(m.x, h, m.y);
  }
  if (!ok) return;
#pragma unroll 8
  for (int q = p0; q < p1; ++q) {
    const float2 m = mp[(long long)q * C];
    entry[(long long)q * C + c] = mine;
    mine = fmaf(m.x, mine, m.y);
  }
  if (seg == 0) state[c] = h;               // every thread of the channel has read the old one before the barrier
  for (int t = max(0, N - taps) + seg; t < N; t += kWalkSeg)
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
  void* u;                  // [S, C] scratch
  void* out;                // [S, C]
  int S, C, bw, taps;
};

// First half of a step: the convolution of every (sequence, channel); the new input goes into the ring row of position - taps,
// which the step does not read.
template <typename T>
__global__ void __launch_bounds__(128) conv_step_kernel(const RglruStep p) {
  const int c = blockIdx.x * 128 + threadIdx.x, s = blockIdx.y;
  if (c >= p.C) return;
  const int pos = p.positions[s];
  float* ring = p.ring + (long long)p.slots[s] * p.taps * p.C + c;
  const float now = ldf(static_cast<const T*>(p.x) + s * p.ldx + c) + (p.xb ? p.xb[c] : 0.f);
  const float* w = p.conv_w + (long long)c * p.taps;
  float acc = p.conv_b[c];
#pragma unroll 4
  for (int k = 0; k < p.taps - 1; ++k) {
    const int q = pos - (p.taps - 1) + k;
    if (q >= 0) acc = fmaf(ring[(long long)(q % p.taps) * p.C], w[k], acc);
  }
  stf(static_cast<T*>(p.u) + (long long)s * p.C + c, fmaf(now, w[p.taps - 1], acc));
  ring[(long long)(pos % p.taps) * p.C] = now;
}

// What is left once both gate logits are known.
template <typename T>
__device__ __forceinline__ void rglru_finish(const RglruStep& p, int s, int c, float r_logit, float i_logit, float u, float old, float y) {
  const T* tag = nullptr;
  const RglruGate g = rglru_gate(tag, r_logit + p.rb[c], i_logit + p.ib[c], u, p.sp[c]);
  const float h = fmaf(g.a, old, g.b);
  p.state[(long long)p.slots[s] * p.C + c] = h;
  stf(static_cast<T*>(p.out) + (long long)s * p.C + c, h * gelu_branch(tag, y + p.yb[c]));
}

// Second half, bf16: a warp makes both gates of 8 channels for 16 sequences on the tensor core (mma.sync m16n8k16; the logits
// come out in fp32) straight from global memory: a lane's 16 contiguous bytes of u and of the matrices are its fragments of
// two instructions, with K permuted alike for both.  bw a multiple of 32.
__device__ __forceinline__ void rg_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__global__ void __launch_bounds__(64) rglru_gates_mma_kernel(const RglruStep p) {
  const int lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int c0 = (blockIdx.x * 2 + (threadIdx.x >> 5)) * 8, s0 = blockIdx.y * 16;
  if (c0 >= p.C) return;
  const int blk = c0 / p.bw, j0 = c0 % p.bw;
  // the four (sequence, channel) pairs whose results this lane gets: rows g and g + 8, columns 2 q and 2 q + 1
  float old[4], y[4], uu[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int s = min(s0 + g + (e >> 1) * 8, p.S - 1), c = c0 + q * 2 + (e & 1);
    old[e] = p.positions[s] > 0 ? p.state[(long long)p.slots[s] * p.C + c] : 0.f;
    y[e] = ldf(static_cast<const __nv_bfloat16*>(p.y) + s * p.ldy + c);
    uu[e] = ldf(static_cast<const __nv_bfloat16*>(p.u) + (long long)s * p.C + c);
  }
  const __nv_bfloat16* u_lo = static_cast<const __nv_bfloat16*>(p.u) + (long long)min(s0 + g, p.S - 1) * p.C + blk * p.bw + q * 8;
  const __nv_bfloat16* u_hi = static_cast<const __nv_bfloat16*>(p.u) + (long long)min(s0 + g + 8, p.S - 1) * p.C + blk * p.bw + q * 8;
  const __nv_bfloat16* wr = static_cast<const __nv_bfloat16*>(p.gates) + ((long long)blk * 2 * p.bw + j0 + g) * p.bw + q * 8;
  const __nv_bfloat16* wi = wr + (long long)p.bw * p.bw;
  float dr[4] = {}, di[4] = {};
#pragma unroll 4
  for (int k = 0; k < p.bw; k += 32) {
    const uint4 lo = *reinterpret_cast<const uint4*>(u_lo + k), hi = *reinterpret_cast<const uint4*>(u_hi + k);
    const uint4 br = __ldg(reinterpret_cast<const uint4*>(wr + k)), bi = __ldg(reinterpret_cast<const uint4*>(wi + k));
    rg_mma(dr, lo.x, hi.x, lo.y, hi.y, br.x, br.y);
    rg_mma(dr, lo.z, hi.z, lo.w, hi.w, br.z, br.w);
    rg_mma(di, lo.x, hi.x, lo.y, hi.y, bi.x, bi.y);
    rg_mma(di, lo.z, hi.z, lo.w, hi.w, bi.z, bi.w);
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int s = s0 + g + (e >> 1) * 8;
    if (s < p.S) rglru_finish<__nv_bfloat16>(p, s, c0 + q * 2 + (e & 1), dr[e], di[e], uu[e], old[e], y[e]);
  }
}

// The same for fp32 and for other block sizes: a warp per (sequence, channel).
template <typename T>
__global__ void __launch_bounds__(128) rglru_gates_kernel(const RglruStep p) {
  const int lane = threadIdx.x & 31, c = blockIdx.x * 4 + (threadIdx.x >> 5), s = blockIdx.y;
  if (c >= p.C) return;
  const int blk = c / p.bw;
  const T* u = static_cast<const T*>(p.u) + (long long)s * p.C + blk * p.bw;
  const T* wr = static_cast<const T*>(p.gates) + ((long long)blk * 2 * p.bw + c % p.bw) * p.bw;
  float r = 0.f, i = 0.f;
  for (int k = lane; k < p.bw; k += 32) {
    const float f = ldf(u + k);
    r = fmaf(ldf(wr + k), f, r);
    i = fmaf(ldf(wr + (long long)p.bw * p.bw + k), f, i);
  }
  r = warp_sum(r);
  i = warp_sum(i);
  if (lane == 0) {
    const float old = p.positions[s] > 0 ? p.state[(long long)p.slots[s] * p.C + c] : 0.f;
    rglru_finish<T>(p, s, c, r, i, ldf(u + c % p.bw), old, ldf(static_cast<const T*>(p.y) + s * p.ldy + c));
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
// scratch: 3 * C * ceil(N / 32) floats.
int lt_rglru_scan(int fp32, const void* u, const float* gates, const float* rb, const float* ib, const float* sp, const void* y,
                  long long ldy, const float* yb, const void* x, long long ldx, const float* xb, float* state, float* ring, void* out,
                  float* scratch, int N, int C, int bw, int taps, int start, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  const int pieces = (N + kScanLen - 1) / kScanLen;
  if (bw < 1 || C % bw != 0 || taps < 1 || taps > kRgMaxTaps || pieces > 65535) return -4;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  RglruScan p{u, gates, rb, ib, sp, y, ldy, yb, reinterpret_cast<float2*>(scratch), scratch + 2ll * C * pieces, out, N, C, bw};
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool v4 = bw % 4 == 0 && ldy % 4 == 0 && al(u) && al(gates) && al(out) && (reinterpret_cast<uintptr_t>(y) & (fp32 ? 15 : 7)) == 0;
  const int per = v4 ? 512 : 128;
  dim3 grid((C + per - 1) / per, pieces);
#define LT_SCAN(T)                                                                                                        \
  if (v4) rglru_scan_kernel<T, 4, 0><<<grid, 128, 0, st>>>(p);                                                            \
  else rglru_scan_kernel<T, 1, 0><<<grid, 128, 0, st>>>(p);                                                               \
  LT_LAUNCH_CHECK();                                                                                                      \
  rglru_walk_kernel<T><<<(C + kWalkCh - 1) / kWalkCh, kWalkCh * kWalkSeg, 0, st>>>(p.maps, p.entry, state, static_cast<const T*>(x), ldx, xb, ring, N, C, pieces, taps, start); \
  LT_LAUNCH_CHECK();                                                                                                      \
  if (v4) rglru_scan_kernel<T, 4, 2><<<grid, 128, 0, st>>>(p);                                                            \
  else rglru_scan_kernel<T, 1, 2><<<grid, 128, 0, st>>>(p)
  if (fp32) { LT_SCAN(float); }
  else { LT_SCAN(__nv_bfloat16); }
#undef LT_SCAN
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_rglru_step(int fp32, const void* x, long long ldx, const float* xb, const float* conv_w, const float* conv_b, const void* gates,
                  const float* rb, const float* ib, const float* sp, const void* y, long long ldy, const float* yb,
                  float* state, float* ring, const int* slots, const int* positions, void* u, void* out, int S, int C, int bw, int taps,
                  void* stream) {
  using namespace lt;
  if (S == 0) return 0;
  if (bw < 1 || C % bw != 0 || taps < 1 || S > 65535) return -4;
  RglruStep p{x, y, ldx, ldy, xb, yb, conv_w, conv_b, gates, rb, ib, sp, state, ring, slots, positions, u, out, S, C, bw, taps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 cg((C + 127) / 128, S);
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (fp32) {
    conv_step_kernel<float><<<cg, 128, 0, st>>>(p);
    LT_LAUNCH_CHECK();
    rglru_gates_kernel<float><<<dim3((C + 3) / 4, S), 128, 0, st>>>(p);
  } else {
    conv_step_kernel<__nv_bfloat16><<<cg, 128, 0, st>>>(p);
    LT_LAUNCH_CHECK();
    if (bw % 32 == 0 && al(u) && al(gates)) rglru_gates_mma_kernel<<<dim3((C / 8 + 1) / 2, (S + 15) / 16), 64, 0, st>>>(p);
    else rglru_gates_kernel<__nv_bfloat16><<<dim3((C + 3) / 4, S), 128, 0, st>>>(p);
  }
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
