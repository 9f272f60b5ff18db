// Around windowed attention on a paged cache: query / key norm over the whole projection, interleaved rotary embedding (any
// number of leading dimensions, any table of frequencies, a gain on cos and sin) and the cache write in one kernel; the
// copy of a window's keys out of the blocks; per-head output gates; and attention on the CUDA cores for fp32 activations
// and for head sizes outside the tensor-core kernels.
//
// Caches are [num_blocks, kv_heads, block_size, padded head size]; keys and values may have different sizes.  The padding
// columns of q, k and v are written as zeros here, so that a tensor-core kernel of the next larger size can run on them.
#include "lt_cuda.h"
#include "common/host.h"
#include "common/scalar.cuh"

namespace lt {

struct QkvParams {
  const void* proj;          // [N, ld]: q at column q_off, k at k_off, v at v_off
  long long ld;
  int q_off, k_off, v_off;
  int H, G, D, E, DP, EP;    // heads, kv heads, query/key size, value size, padded sizes
  const float* q_norm;       // [H * D] or nullptr
  const float* k_norm;       // [G * D] or nullptr
  float eps;
  const int* positions;      // [N]
  const int* slots;          // [N] block * block_size + offset
  const double* freq;        // [rot_dims / 2] angle per token
  int rot_dims;
  float gain;
  void* q_out;               // [N, H, DP]
  void* k_cache;
  void* v_cache;
  int block_size;
  void* k_lin;               // [N, G, DP] or nullptr: the new keys / values once more, one after another
  void* v_lin;
};

constexpr int kQkvThreads = 256;
// V: elements per access of the projection row (8: bf16 in 16-byte pieces; segment offsets and sizes are multiples of it).
template <typename T, int V>
__global__ void __launch_bounds__(kQkvThreads) qkv_rope_kernel(const QkvParams p) {
  extern __shared__ float2 cs[];         // [rot_dims / 2] (cos, sin) of this token, then the row: q, k, v as fp32
  __shared__ float red[64];
  float* q_s = reinterpret_cast<float*>(cs + p.rot_dims / 2);
  const int nq = p.H * p.D, nk = p.G * p.D, nv = p.G * p.E;
  float* k_s = q_s + nq;
  float* v_s = k_s + nk;
  const int n = blockIdx.x;
  const T* row = static_cast<const T*>(p.proj) + n * p.ld;
  const int pos = p.positions[n], slot = p.slots[n];
  float sum[2] = {0.f, 0.f};
  auto fetch = [&](const T* src, float* dst, int count, float& acc) {
    for (int i = threadIdx.x * V; i < count; i += kQkvThreads * V) {
      if constexpr (V == 8) {
        const float4 a = ldf4(src + i), b = ldf4(src + i + 4);
        *reinterpret_cast<float4*>(dst + i) = a;
        *reinterpret_cast<float4*>(dst + i + 4) = b;
        acc += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w + b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
      } else {
        const float f = ldf(src + i);
        dst[i] = f;
        acc += f * f;
      }
    }
  };
  float unused = 0.f;
  fetch(row + p.q_off, q_s, nq, sum[0]);
  fetch(row + p.k_off, k_s, nk, sum[1]);
  fetch(row + p.v_off, v_s, nv, unused);
  for (int i = threadIdx.x; i < p.rot_dims / 2; i += kQkvThreads) {
    // the angle can be far outside a period: reduce it in double before the fp32 sine
    const double turns = double(pos) * p.freq[i] * 0.15915494309189535;
    float s, c;
    sincospif(float(2.0 * (turns - rint(turns))), &s, &c);
    cs[i] = make_float2(c * p.gain, s * p.gain);
  }
  const float2 s2 = block_sum2(sum[0], sum[1], red);          // also publishes the row and the angles
  const float rq = p.q_norm ? 1.f / sqrtf(s2.x / nq + p.eps) : 1.f;
  const float rk = p.k_norm ? 1.f / sqrtf(s2.y / nk + p.eps) : 1.f;
  // the pair (d, d + 1) of one head of q or k
  auto pair = [&](const float* src, const float* w, int h, int d, float r) -> float2 {
    const int c = h * p.D + d;
    float u = d < p.D ? src[c] * r : 0.f, v = d + 1 < p.D ? src[c + 1] * r : 0.f;
    if (w) {
      if (d < p.D) u *= w[c];
      if (d + 1 < p.D) v *= w[c + 1];
    }
    if (d < p.rot_dims) {
      const float2 t = cs[d >> 1];
      return make_float2(u * t.x - v * t.y, v * t.x + u * t.y);
    }
    return make_float2(u, v);
  };
  const int dq = p.DP / 4;                  // DP and EP are multiples of 8
  T* q_out = static_cast<T*>(p.q_out) + (long long)n * p.H * p.DP;
  for (int i = threadIdx.x; i < p.H * dq; i += kQkvThreads) {
    const int h = i / dq, d = (i % dq) * 4;
    const float2 a = pair(q_s, p.q_norm, h, d, rq), b = pair(q_s, p.q_norm, h, d + 2, rq);
    stf4(q_out + h * p.DP + d, make_float4(a.x, a.y, b.x, b.y));
  }
  const int blk = slot / p.block_size, off = slot % p.block_size;
  for (int i = threadIdx.x; i < p.G * dq; i += kQkvThreads) {
    const int g = i / dq, d = (i % dq) * 4;
    const float2 a = pair(k_s, p.k_norm, g, d, rk), b = pair(k_s, p.k_norm, g, d + 2, rk);
    const float4 f = make_float4(a.x, a.y, b.x, b.y);
    stf4(static_cast<T*>(p.k_cache) + (((long long)blk * p.G + g) * p.block_size + off) * p.DP + d, f);
    if (p.k_lin) stf4(static_cast<T*>(p.k_lin) + ((long long)n * p.G + g) * p.DP + d, f);
  }
  const int eq = p.EP / 4;
  for (int i = threadIdx.x; i < p.G * eq; i += kQkvThreads) {
    const int g = i / eq, e = (i % eq) * 4;
    const float* v = v_s + g * p.E;
    const float4 f = make_float4(e < p.E ? v[e] : 0.f, e + 1 < p.E ? v[e + 1] : 0.f, e + 2 < p.E ? v[e + 2] : 0.f, e + 3 < p.E ? v[e + 3] : 0.f);
    stf4(static_cast<T*>(p.v_cache) + (((long long)blk * p.G + g) * p.block_size + off) * p.EP + e, f);
    if (p.v_lin) stf4(static_cast<T*>(p.v_lin) + ((long long)n * p.G + g) * p.EP + e, f);
  }
}

// Rows [pos0, pos0 + n) of one sequence out of its blocks into [n, G, D] arrays.
__global__ void kv_gather_kernel(const uint4* __restrict__ k_cache, const uint4* __restrict__ v_cache, uint4* __restrict__ k_lin,
                                 uint4* __restrict__ v_lin, const int* __restrict__ table, int pos0, int G, int ku, int vu,
                                 int block_size) {
  const int pos = pos0 + blockIdx.x;
  const long long blk = table[pos / block_size];
  const int off = pos % block_size;
  for (int i = threadIdx.x; i < G * (ku + vu); i += blockDim.x) {
    const bool is_k = i < G * ku;
    const int j = is_k ? i : i - G * ku, w = is_k ? ku : vu;
    const int g = j / w, u = j % w;
    const long long src = ((blk * G + g) * block_size + off) * w + u, dst = ((long long)blockIdx.x * G + g) * w + u;
    if (is_k) k_lin[dst] = k_cache[src];
    else v_lin[dst] = v_cache[src];
  }
}

// One warp per (row, query head): scores of 32 keys at a time (a lane per key), online softmax, value columns over the lanes.
// Rows are tokens of one sequence (table_stride 0) or one token of every sequence.
constexpr int kWaWarps = 4;
template <typename T>
__global__ void __launch_bounds__(kWaWarps * 32)
window_attn_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                   const int* __restrict__ tables, long long table_stride, const int* __restrict__ positions, T* __restrict__ o,
                   const T* __restrict__ gate, long long ldg, int N, int H, int G, int D, int E, int DP, int EP, int block_size,
                   int window, float scale) {
  extern __shared__ float wa_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* q_s = wa_smem + warp * (DP + EP);
  float* acc = q_s + DP;
  const long long item = (long long)blockIdx.x * kWaWarps + warp;
  if (item >= (long long)N * H) return;
  const int n = int(item / H), h = int(item % H), g = h / (H / G);
  const int pos = positions[n];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int* bt = tables + n * table_stride;
  for (int d = lane; d < D; d += 32) q_s[d] = ldf(q + ((long long)n * H + h) * DP + d);
  for (int e = lane; e < E; e += 32) acc[e] = 0.f;
  __syncwarp();
  float m = -INFINITY, l = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    const int j = j0 + lane;
    const bool live = j <= pos;
    float s = -INFINITY;
    long long base = 0;
    if (live) {
      base = ((long long)bt[j / block_size] * G + g) * block_size + j % block_size;
      float d0 = 0.f, d1 = 0.f;
      const T* kr = k_cache + base * DP;
      int d = 0;
      for (; d + 3 < D; d += 4) {
        const float4 kv = ldf4(kr + d);
        d0 = fmaf(kv.x, q_s[d], d0); d1 = fmaf(kv.y, q_s[d + 1], d1);
        d0 = fmaf(kv.z, q_s[d + 2], d0); d1 = fmaf(kv.w, q_s[d + 3], d1);
      }
      for (; d < D; ++d) d0 = fmaf(ldf(kr + d), q_s[d], d0);
      s = (d0 + d1) * scale;
    }
    const float nm = fmaxf(m, warp_max(s));
    const float keep = m == -INFINITY ? 0.f : expf(m - nm);
    const float p = live ? expf(s - nm) : 0.f;
    l = l * keep + warp_sum(p);
    m = nm;
    const int nk = min(32, pos - j0 + 1);
    for (int e0 = 0; e0 < E; e0 += 32) {                    // whole warp in every pass: the shuffles below need all lanes
      const int e = e0 + lane;
      float a = e < E ? acc[e] * keep : 0.f;
      for (int t = 0; t < nk; ++t) {
        const float pt = __shfl_sync(0xffffffffu, p, t);
        const long long bt_row = __shfl_sync(0xffffffffu, base, t);
        if (e < E) a = fmaf(pt, ldf(v_cache + bt_row * EP + e), a);
      }
      if (e < E) acc[e] = a;
    }
  }
  const float f = (gate ? sigmoid_f(ldf(gate + n * ldg + h)) : 1.f) / l;
  for (int e = lane; e < E; e += 32) stf(o + ((long long)n * H + h) * E + e, acc[e] * f);
}

// out[n, h, e] = o[n, h, e] * sigmoid(gate[n, h]) for e < E, packed.
template <typename T>
__global__ void head_gate_kernel(const T* __restrict__ o, const T* __restrict__ gate, long long ldg, T* __restrict__ out,
                                 long long rows, int H, int E, int EP) {
  const long long total = rows * H * E;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int e = int(i % E);
    const long long nh = i / E;
    const float g = sigmoid_f(ldf(gate + (nh / H) * ldg + nh % H));
    stf(out + i, ldf(o + nh * EP + e) * g);
  }
}

// The same, eight bf16 columns per thread (E and EP multiples of 8).
__global__ void head_gate8_kernel(const uint4* __restrict__ o, const __nv_bfloat16* __restrict__ gate, long long ldg,
                                  uint4* __restrict__ out, long long rows, int H, int eu, int epu) {
  const long long total = rows * H * eu;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int u = int(i % eu);
    const long long nh = i / eu;
    const float g = sigmoid_f(__bfloat162float(gate[(nh / H) * ldg + nh % H]));
    uint4 v = o[nh * epu + u];
    __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 f = __bfloat1622float2(b[k]);
      b[k] = __floats2bfloat162_rn(f.x * g, f.y * g);
    }
    out[i] = v;
  }
}

}  // namespace lt

extern "C" {

int lt_qkv_rope(int fp32, const void* proj, long long ld, int n, int q_off, int k_off, int v_off, int H, int G, int D, int E, int DP,
                int EP, const float* q_norm, const float* k_norm, float eps, const int* positions, const int* slots,
                const double* freq, int rot_dims, float gain, void* q_out, void* k_cache, void* v_cache, int block_size,
                void* k_lin, void* v_lin, void* stream) {
  using namespace lt;
  if (n == 0) return 0;
  const long long smem = (long long)rot_dims * 4 + ((long long)H * D + (long long)G * (D + E)) * 4;
  if (G < 1 || H % G != 0 || DP < D || EP < E || (DP & 7) || (EP & 7) || rot_dims > D || (rot_dims & 1) || smem > 220 * 1024) return -4;
  QkvParams p{proj, ld, q_off, k_off, v_off, H, G, D, E, DP, EP, q_norm, k_norm, eps, positions, slots, freq, rot_dims, gain,
              q_out, k_cache, v_cache, block_size, k_lin, v_lin};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v8 = !fp32 && ((ld | q_off | k_off | v_off | (H * D) | (G * D) | (G * E)) & 7) == 0 && (rot_dims & 3) == 0 &&
                  (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  auto kern = fp32 ? qkv_rope_kernel<float, 1> : v8 ? qkv_rope_kernel<__nv_bfloat16, 8> : qkv_rope_kernel<__nv_bfloat16, 1>;
  if (smem > 48 * 1024) LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
  kern<<<n, kQkvThreads, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

// Head sizes here are bytes of one (token, head) row; multiples of 16.
int lt_kv_gather(const void* k_cache, const void* v_cache, void* k_lin, void* v_lin, const int* table, int pos0, int n, int G,
                 int k_bytes, int v_bytes, int block_size, void* stream) {
  using namespace lt;
  if (n <= 0) return 0;
  if ((k_bytes & 15) || (v_bytes & 15)) return -4;
  kv_gather_kernel<<<n, 128, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(k_cache), static_cast<const uint4*>(v_cache), static_cast<uint4*>(k_lin), static_cast<uint4*>(v_lin),
      table, pos0, G, k_bytes / 16, v_bytes / 16, block_size);
  LT_LAUNCH_CHECK();
  return 0;
}

// o [N, H, E]; gate [N, H] logits at pitch ldg or nullptr; window 0: every earlier key.
int lt_window_attn(int fp32, const void* q, const void* k_cache, const void* v_cache, const int* tables, long long table_stride,
                   const int* positions, void* o, const void* gate, long long ldg, int N, int H, int G, int D, int E, int DP, int EP,
                   int block_size, int window, float scale, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  if (G < 1 || H % G != 0 || (DP & 3) || DP + EP > 3072) return -4;
  const int smem = kWaWarps * (DP + EP) * 4;
  const long long items = (long long)N * H;
  const unsigned grid = unsigned((items + kWaWarps - 1) / kWaWarps);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LT_WA(T) window_attn_kernel<T><<<grid, kWaWarps * 32, smem, st>>>( \
      static_cast<const T*>(q), static_cast<const T*>(k_cache), static_cast<const T*>(v_cache), tables, table_stride, positions, \
      static_cast<T*>(o), static_cast<const T*>(gate), ldg, N, H, G, D, E, DP, EP, block_size, window, scale)
  if (fp32) LT_WA(float);
  else LT_WA(__nv_bfloat16);
#undef LT_WA
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_head_gate(int fp32, const void* o, const void* gate, long long ldg, void* out, long long rows, int H, int E, int EP,
                 void* stream) {
  using namespace lt;
  const long long total = rows * H * E;
  if (total == 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v8 = !fp32 && E % 8 == 0 && EP % 8 == 0;
  long long blocks = ((v8 ? total / 8 : total) + 255) / 256;
  const long long cap = (long long)sm_count() * 16;
  if (blocks > cap) blocks = cap;
  const unsigned nb = unsigned(blocks);
  if (fp32) head_gate_kernel<float><<<nb, 256, 0, st>>>(static_cast<const float*>(o), static_cast<const float*>(gate), ldg, static_cast<float*>(out), rows, H, E, EP);
  else if (v8) head_gate8_kernel<<<nb, 256, 0, st>>>(static_cast<const uint4*>(o), static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<uint4*>(out), rows, H, E / 8, EP / 8);
  else head_gate_kernel<__nv_bfloat16><<<nb, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(o), static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<__nv_bfloat16*>(out), rows, H, E, EP);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
