// Matrix memory with exponential gates (mLSTM): per head a state S [D, E], a key sum n [D] and a running maximum m,
//
//   i = cap tanh((wi h + bi) / cap)      f = logsigmoid(cap tanh((wf h + bf) / cap))
//   m_t = max(f + m_(t-1), i),  S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,  n_t likewise with k alone
//   o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6),  then RMS norm per head, a weight and a sigmoid gate.
//
// Prompts run chunk by chunk of 128 tokens.  With F the running sum of f inside a chunk, a_s = i_s - F_s and
// M_t = max(m at the chunk's start, max_{s <= t} a_s), everything a chunk needs is a difference of these:
//   weight of token s at token t     exp(a_s - M_t)          m_t = F_t + M_t
//   weight of the state before it    exp(m_start - M_t)
// so no exponent is ever positive.  Four kernels: gates (a, F, the running maxima and m at chunk starts), chunk states (the
// K^T V of every chunk, tensor cores), a scan over chunks (elementwise, fp32) and the outputs (tensor cores; the head norm
// and the gate in the epilogue).  The state stays fp32; where it, the decayed keys or the token weights enter a bf16
// tensor-core product they are split into a high and a low bf16 part and multiplied twice, which keeps 16 bits of them.
// mma.sync is used rather than tcgen05: the operands are made on the fly from fp32 values.
//
// A decode step is one kernel over (sequence, head, column slice): the slice of S is read, updated, used and written once.
//
// State per slot (fp32): S [H, D, E]; n [2, H, D] and m [2, H], where bank p & 1 holds the value before position p, so that
// the CTAs of a step that share a head read one bank while one of them writes the other.
#include "lt_cuda.h"
#include "common/host.h"
#include "common/ptx.cuh"
#include "common/scalar.cuh"

namespace lt {

constexpr int kMlChunk = 128;     // tokens per chunk
constexpr int kMlRows = 64;       // rows and columns of the tiles

__device__ __forceinline__ float mlstm_input_gate(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float mlstm_forget_gate(float x, float cap) { return log_sigmoid_f(cap * tanhf(x / cap)); }

// ------------------------------------------------------------------------------------------------ gates of a prompt
// logits [N, 2 H] fp32 (i then f).  Writes a, F and the running maximum of a inside the chunk ([H, N] each) and m at the
// start of every chunk ([H, chunks + 1]).
__global__ void __launch_bounds__(256)
mlstm_gates_kernel(const float* __restrict__ logits, const float* __restrict__ ib, const float* __restrict__ fb, float cap,
                   const float* __restrict__ m_state, float* __restrict__ a_out, float* __restrict__ f_out,
                   float* __restrict__ c_out, float* __restrict__ m_out, int N, int H, int chunks) {
  extern __shared__ float last_s[];      // [chunks] F at a chunk's last token, [chunks] largest a of the chunk
  const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float bi = ib[h], bf = fb[h];
  for (int c = warp; c < chunks; c += 8) {
    const int t0 = c * kMlChunk;
    float run = 0.f, top = -INFINITY;
    for (int s = 0; s < kMlChunk; s += 32) {
      const int t = t0 + s + lane;
      float f = 0.f, i = -INFINITY;
      if (t < N) {
        i = mlstm_input_gate(logits[(long long)t * 2 * H + h] + bi, cap);
        f = mlstm_forget_gate(logits[(long long)t * 2 * H + H + h] + bf, cap);
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float g = __shfl_up_sync(0xffffffffu, f, o);
        if (lane >= o) f += g;
      }
      f += run;
      float mx = i - f;
      const float a = mx;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float g = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, g);
      }
      mx = fmaxf(mx, top);
      if (t < N) {
        a_out[(long long)h * N + t] = a;
        f_out[(long long)h * N + t] = f;
        c_out[(long long)h * N + t] = mx;
      }
      run = __shfl_sync(0xffffffffu, f, 31);
      top = __shfl_sync(0xffffffffu, mx, 31);
    }
    // (tokens past the end add nothing to F and -inf to the maximum)
    if (lane == 0) { last_s[c] = run; last_s[chunks + c] = top; }
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    float m = m_state ? m_state[h] : 0.f;
    for (int c = 0; c < chunks; ++c) {
      m_out[(long long)h * (chunks + 1) + c] = m;
      m = last_s[c] + fmaxf(m, last_s[chunks + c]);
    }
    m_out[(long long)h * (chunks + 1) + chunks] = m;
  }
}

// ------------------------------------------------------------------------------------------------ tensor-core pieces
constexpr int kMlPitch = kMlRows + 8;     // bf16 elements per shared-memory row of a 64-wide tile: conflict-free ldmatrix

__device__ __forceinline__ void ldsm4(const __nv_bfloat16* p, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(const __nv_bfloat16* p, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(v);
  lo = __float2bfloat16(v - __bfloat162float(hi));
}
__device__ __forceinline__ void split4(float4 v, __nv_bfloat16* hi, __nv_bfloat16* lo) {
  const float4 h = make_float4(__bfloat162float(__float2bfloat16(v.x)), __bfloat162float(__float2bfloat16(v.y)),
                               __bfloat162float(__float2bfloat16(v.z)), __bfloat162float(__float2bfloat16(v.w)));
  stf4(hi, h);
  stf4(lo, make_float4(v.x - h.x, v.y - h.y, v.z - h.z, v.w - h.w));
}

// Eight neighbouring bf16 of a row, zeros outside the valid columns.
__device__ __forceinline__ uint4 load8(const __nv_bfloat16* row, int c, int cols, bool row_ok, bool aligned) {
  if (!row_ok || c >= cols) return make_uint4(0u, 0u, 0u, 0u);
  if (aligned && c + 8 <= cols) return *reinterpret_cast<const uint4*>(row + c);
  uint4 v;
  __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&v);
#pragma unroll
  for (int i = 0; i < 8; ++i) e[i] = c + i < cols ? row[c + i] : __float2bfloat16(0.f);
  return v;
}

// ------------------------------------------------------------------------------------------------ chunk states
// U[h, c] [D, E] = sum_s exp(a_s - M_last) k_s v_s^T and nU[h, c] [D].  One CTA per 64 rows of U: the decayed keys are split
// into their two parts once and stay in shared memory while 128 columns of V at a time pass by (the next ones are loaded
// into registers under the products).  Eight warps as 2 row halves x 4 column quarters of 32 x 32.
constexpr int kMlWide = 128, kMlWidePitch = kMlWide + 8;
constexpr size_t kMlStateSmem = (2 * size_t(kMlChunk) * kMlPitch + size_t(kMlChunk) * kMlWidePitch) * 2;

__global__ void __launch_bounds__(256, 2)
mlstm_chunk_state_kernel(const __nv_bfloat16* __restrict__ k, const __nv_bfloat16* __restrict__ v, long long ld,
                         const float* __restrict__ a, const float* __restrict__ cmax, const float* __restrict__ m_start,
                         float* __restrict__ U, float* __restrict__ nU, int N, int D, int E, int chunks, int aligned) {
  extern __shared__ __align__(16) uint8_t ml_smem[];
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(ml_smem);          // [128][pitch]: high parts of w_s k_s
  __nv_bfloat16* kl = kh + kMlChunk * kMlPitch;
  __nv_bfloat16* vs = kl + kMlChunk * kMlPitch;                            // [128][wide pitch]
  __shared__ float w_s[kMlChunk];
  const int c = blockIdx.x, h = blockIdx.y, d0 = blockIdx.z * kMlRows;
  const int t0 = c * kMlChunk, len = min(kMlChunk, N - t0);
  const float m_last = fmaxf(m_start[(long long)h * (chunks + 1) + c], cmax[(long long)h * N + t0 + len - 1]);
  if (int(threadIdx.x) < kMlChunk) w_s[threadIdx.x] = int(threadIdx.x) < len ? expf(a[(long long)h * N + t0 + threadIdx.x] - m_last) : 0.f;
  const __nv_bfloat16* kp = k + (long long)t0 * ld + (long long)h * D;
  const __nv_bfloat16* vp = v + (long long)t0 * ld + (long long)h * E;
  uint4 vr[8];
  auto fetch = [&](int e0) {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = threadIdx.x + j * 256, r = i >> 4, cc = (i & 15) * 8;
      vr[j] = load8(vp + r * ld, e0 + cc, E, r < len, aligned);
    }
  };
  fetch(0);
  __syncthreads();
  for (int i = threadIdx.x; i < kMlChunk * 8; i += 256) {
    const int r = i >> 3, cc = (i & 7) * 8;
    const uint4 raw = load8(kp + r * ld, d0 + cc, D, r < len, aligned);
    const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&raw);
    uint4 hi, lo;
    __nv_bfloat16 *ph = reinterpret_cast<__nv_bfloat16*>(&hi), *pl = reinterpret_cast<__nv_bfloat16*>(&lo);
#pragma unroll
    for (int j = 0; j < 8; ++j) split_bf16(__bfloat162float(e[j]) * w_s[r], ph[j], pl[j]);
    *reinterpret_cast<uint4*>(kh + r * kMlPitch + cc) = hi;
    *reinterpret_cast<uint4*>(kl + r * kMlPitch + cc) = lo;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lj = lane >> 3, lr = lane & 7;
  const int wd = (warp >> 2) * 32, we = (warp & 3) * 32;
  const int g = lane >> 2, q = lane & 3;
  float* out = U + ((long long)h * chunks + c) * D * E;
  const bool e2 = (E & 1) == 0;
  for (int e0 = 0; e0 < E; e0 += kMlWide) {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = threadIdx.x + j * 256, r = i >> 4, cc = (i & 15) * 8;
      *reinterpret_cast<uint4*>(vs + r * kMlWidePitch + cc) = vr[j];
    }
    __syncthreads();
    if (e0 + kMlWide < E) fetch(e0 + kMlWide);
    float acc[2][4][4] = {};
#pragma unroll
    for (int ks = 0; ks < kMlChunk; ks += 16) {
      uint32_t b[2][4];
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) ldsm4t(vs + (ks + (lj & 1) * 8 + lr) * kMlWidePitch + we + nb * 16 + (lj >> 1) * 8, b[nb]);
#pragma unroll
      for (int mb = 0; mb < 2; ++mb) {
        const int off = (ks + (lj >> 1) * 8 + lr) * kMlPitch + wd + mb * 16 + (lj & 1) * 8;
        uint32_t ah[4], al[4];
        ldsm4t(kh + off, ah);
        ldsm4t(kl + off, al);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) {
          mma16816(acc[mb][nb], ah, b[nb >> 1][(nb & 1) * 2], b[nb >> 1][(nb & 1) * 2 + 1]);
          mma16816(acc[mb][nb], al, b[nb >> 1][(nb & 1) * 2], b[nb >> 1][(nb & 1) * 2 + 1]);
        }
      }
    }
#pragma unroll
    for (int mb = 0; mb < 2; ++mb)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int r = 0; r < 4; r += 2) {
          const int d = d0 + wd + mb * 16 + g + (r >> 1) * 8, e = e0 + we + nb * 8 + q * 2;
          if (d < D && e < E) {
            float* dst = out + (long long)d * E + e;
            if (e2) {
              *reinterpret_cast<float2*>(dst) = make_float2(acc[mb][nb][r], acc[mb][nb][r + 1]);
            } else {
              dst[0] = acc[mb][nb][r];
              if (e + 1 < E) dst[1] = acc[mb][nb][r + 1];
            }
          }
        }
    __syncthreads();
  }
  if (threadIdx.x < kMlRows && d0 + int(threadIdx.x) < D) {
    float s = 0.f;
    for (int r = 0; r < len; ++r)
      s += __bfloat162float(kh[r * kMlPitch + threadIdx.x]) + __bfloat162float(kl[r * kMlPitch + threadIdx.x]);
    nU[((long long)h * chunks + c) * D + d0 + threadIdx.x] = s;
  }
}

// ------------------------------------------------------------------------------------------------ scan over chunks
// In place: U[h, c] becomes the state at the start of chunk c; the state after the last chunk goes back to the slot.
template <int V>
__global__ void __launch_bounds__(256)
mlstm_chunk_scan_kernel(float* __restrict__ U, float* __restrict__ nU, const float* __restrict__ cmax,
                        const float* __restrict__ m_start, float* __restrict__ S, const float* __restrict__ n_in,
                        float* __restrict__ n_out, float* __restrict__ m_out, int N, int D, int E, int chunks, int fresh) {
  extern __shared__ float keep_s[];      // [chunks]
  const int h = blockIdx.y;
  for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
    const float m = m_start[(long long)h * (chunks + 1) + c];
    const float top = fmaxf(m, cmax[(long long)h * N + min(N, (c + 1) * kMlChunk) - 1]);
    keep_s[c] = expf(m - top);
  }
  if (blockIdx.x == 0 && threadIdx.x == 0) m_out[h] = m_start[(long long)h * (chunks + 1) + chunks];
  __syncthreads();
  const long long DE = (long long)D * E;
  const unsigned s_blocks = unsigned((DE + 256 * V - 1) / (256 * V));        // the blocks after these take n
  // One column of V values through all chunks: eight chunks are read ahead of their use.
  auto walk = [&](float* u, long long stride, const float* first, float* last) {
    float cur[V], nx[8][V];
    auto ld = [&](const float* p, float (&d)[V]) {
      if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        d[0] = f.x; d[1] = f.y; d[2] = f.z; d[3] = f.w;
      } else {
        d[0] = *p;
      }
    };
    auto st = [&](float* p, const float (&d)[V]) {
      if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(d[0], d[1], d[2], d[3]);
      else *p = d[0];
    };
    if (fresh) {
#pragma unroll
      for (int v = 0; v < V; ++v) cur[v] = 0.f;
    } else {
      ld(first, cur);
    }
    for (int c0 = 0; c0 < chunks; c0 += 8) {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < chunks) ld(u + (c0 + j) * stride, nx[j]);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < chunks) {
          st(u + (c0 + j) * stride, cur);
          const float k = keep_s[c0 + j];
#pragma unroll
          for (int v = 0; v < V; ++v) cur[v] = fmaf(k, cur[v], nx[j][v]);
        }
    }
    st(last, cur);
  };
  if (blockIdx.x < s_blocks) {
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
    if (i < DE) walk(U + (long long)h * chunks * DE + i, DE, S + (long long)h * DE + i, S + (long long)h * DE + i);
  } else {
    const long long d = ((long long)(blockIdx.x - s_blocks) * 256 + threadIdx.x) * V;
    if (d < D) walk(nU + (long long)h * chunks * D + d, D, n_in + (long long)h * D + d, n_out + (long long)h * D + d);
  }
}

// ------------------------------------------------------------------------------------------------ outputs of a prompt
struct MlstmOut {
  const __nv_bfloat16* q;
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;
  long long ld;
  const float* a;
  const float* f;
  const float* cmax;
  const float* m_start;
  const float* S0;               // [H, chunks, D, E] states at chunk starts
  const float* n0;               // [H, chunks, D]
  const float* norm;             // [H * E]
  const __nv_bfloat16* gate;     // [N, H * E] logits at pitch ldg
  long long ldg;
  float* o;                      // scratch [N, H * E]
  __nv_bfloat16* out;            // [N, H * E]
  float qscale, eps;
  int N, H, D, E, chunks, fresh, aligned;
};

constexpr int kMlPPitch = kMlChunk + 8;
static size_t mlstm_out_smem(int D) {
  const int dp = (D + 63) / 64 * 64 + 8;
  return size_t(kMlRows) * dp * 2 + 2 * size_t(kMlRows) * kMlPPitch * 2 + 4 * size_t(kMlRows) * kMlPitch * 2;
}

// One CTA: 64 tokens (half a chunk) of one head, eight warps as 4 row blocks of 16 x 2 column halves of 32.
__global__ void __launch_bounds__(256, 2) mlstm_out_kernel(const MlstmOut p) {
  extern __shared__ __align__(16) uint8_t ml_smem[];
  const int D = p.D, E = p.E;
  const int dp = (D + 63) / 64 * 64 + 8;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(ml_smem);      // [64][dp]
  __nv_bfloat16* ph = qs + kMlRows * dp;                               // [64][kMlPPitch] token weights, high and low parts
  __nv_bfloat16* pl = ph + kMlRows * kMlPPitch;
  __nv_bfloat16* tiles = pl + kMlRows * kMlPPitch;                     // two buffers of two 64 x 64 tiles (high and low parts)
  __shared__ float a_s[kMlChunk], top_s[kMlRows], inter_s[kMlRows], den_s[2][kMlRows], inv_s[kMlRows], sq_s[2][kMlRows];
  const int h = blockIdx.y, c = blockIdx.x >> 1, half = blockIdx.x & 1;
  const int t0 = c * kMlChunk, r0 = half * kMlRows;                    // chunk start, first row inside it
  const int len = min(kMlChunk, p.N - t0);                             // tokens of this chunk
  if (r0 >= len) return;
  const int rows = min(kMlRows, len - r0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lj = lane >> 3, lr = lane & 7;
  const int g = lane >> 2, q4 = lane & 3;
  const int wr = (warp >> 1) * 16, wc = (warp & 1) * 32, wh = warp & 1;
  const long long hn = (long long)h * p.N;
  const float m0 = p.m_start[(long long)h * (p.chunks + 1) + c];
  const bool have_state = !(p.fresh && c == 0);
  for (int i = threadIdx.x; i < kMlChunk; i += blockDim.x) a_s[i] = i < len ? p.a[hn + t0 + i] : -INFINITY;
  for (int i = threadIdx.x; i < kMlRows; i += blockDim.x) {
    const float top = i < rows ? fmaxf(m0, p.cmax[hn + t0 + r0 + i]) : 0.f;
    top_s[i] = top;
    inter_s[i] = i < rows && have_state ? expf(m0 - top) * p.qscale : 0.f;
  }
  const __nv_bfloat16* qp = p.q + (long long)(t0 + r0) * p.ld + (long long)h * D;
  for (int i = threadIdx.x; i < kMlRows * ((dp - 8) / 8); i += blockDim.x) {
    const int r = i / ((dp - 8) / 8), cc = (i % ((dp - 8) / 8)) * 8;
    *reinterpret_cast<uint4*>(qs + r * dp + cc) = load8(qp + r * p.ld, cc, D, r < rows, p.aligned);
  }
  __syncthreads();

  // Tiles come through registers: the next one is loaded while the current one is multiplied, then stored into the other
  // buffer, so that a tile costs one barrier.
  constexpr int kTile = kMlRows * kMlPitch;
  uint4 reg[4];
  auto fetch_bf = [&](const __nv_bfloat16* src, int rows_ok, int c0, int cols) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = threadIdx.x + j * 256, r = i >> 3;
      reg[j] = load8(src + r * p.ld, c0 + (i & 7) * 8, cols, r < rows_ok, p.aligned);
    }
  };
  auto store_bf = [&](__nv_bfloat16* dst) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = threadIdx.x + j * 256;
      *reinterpret_cast<uint4*>(dst + (i >> 3) * kMlPitch + (i & 7) * 8) = reg[j];
    }
  };
  const int nd = (D + 63) / 64;

  // ---- token weights: (q . k) qscale exp(a_s - M_t) for s <= t, and their row sums
  float sum_lo = 0.f, sum_hi = 0.f;
  const __nv_bfloat16* kp = p.k + (long long)t0 * p.ld + (long long)h * D;
  const int k_stages = (half + 1) * nd;
  auto fetch_k = [&](int st) {
    const int kb = st / nd;
    fetch_bf(kp + (long long)kb * kMlRows * p.ld, len - kb * kMlRows, (st % nd) * 64, D);
  };
  fetch_k(0);
  store_bf(tiles);
  __syncthreads();
  for (int kb = 0, st = 0; kb <= half; ++kb) {
    float acc[4][4] = {};
    for (int dd = 0; dd < nd; ++dd, ++st) {
      if (st + 1 < k_stages) fetch_k(st + 1);
      const __nv_bfloat16* t = tiles + (st & 1) * 2 * kTile;
#pragma unroll
      for (int ks = 0; ks < 64; ks += 16) {
        uint32_t a[4], b[2][4];
        ldsm4(qs + (wr + (lj & 1) * 8 + lr) * dp + dd * 64 + ks + (lj >> 1) * 8, a);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) ldsm4(t + (wc + nb * 16 + (lj >> 1) * 8 + lr) * kMlPitch + ks + (lj & 1) * 8, b[nb]);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) mma16816(acc[nb], a, b[nb >> 1][(nb & 1) * 2], b[nb >> 1][(nb & 1) * 2 + 1]);
      }
      if (st + 1 < k_stages) store_bf(tiles + ((st + 1) & 1) * 2 * kTile);
      __syncthreads();
    }
#pragma unroll
    for (int nb = 0; nb < 4; ++nb)
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int row = wr + g + (r >> 1) * 8, s = kb * kMlRows + wc + nb * 8 + q4 * 2 + (r & 1);
        const float w = s <= r0 + row && s < len && row < rows ? acc[nb][r] * p.qscale * expf(a_s[s] - top_s[row]) : 0.f;
        if (r < 2) sum_lo += w;
        else sum_hi += w;
        split_bf16(w, ph[row * kMlPPitch + s], pl[row * kMlPPitch + s]);
      }
  }
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 1);
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 2);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 1);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 2);
  if (q4 == 0) { den_s[wh][wr + g] = sum_lo; den_s[wh][wr + g + 8] = sum_hi; }
  // n . q of the state before the chunk: four threads per row
  float nq = 0.f;
  if (have_state) {
    const float* n0 = p.n0 + ((long long)h * p.chunks + c) * D;
    const int r = threadIdx.x >> 2;
    for (int d = threadIdx.x & 3; d < D; d += 4) nq = fmaf(n0[d], __bfloat162float(qs[r * dp + d]), nq);
  }
  nq += __shfl_xor_sync(0xffffffffu, nq, 1);
  nq += __shfl_xor_sync(0xffffffffu, nq, 2);
  __syncthreads();
  if ((threadIdx.x & 3) == 0) {
    const int r = threadIdx.x >> 2;
    const float m = r < rows ? p.f[hn + t0 + r0 + r] + top_s[r] : 0.f;
    const float den = fabsf(den_s[0][r] + den_s[1][r] + inter_s[r] * nq);
    inv_s[r] = 1.f / (fmaxf(den, expf(-m)) + 1e-6f);
  }
  __syncthreads();

  // ---- outputs, 64 columns at a time: the state before the chunk (nd slices of it), then the chunk's own tokens
  float sq_lo = 0.f, sq_hi = 0.f;
  const float* S0 = p.S0 + ((long long)h * p.chunks + c) * D * E;
  const __nv_bfloat16* vp = p.v + (long long)t0 * p.ld + (long long)h * E;
  const bool e4 = E % 4 == 0;
  const int ns = have_state ? nd : 0, per = ns + half + 1;
  const int o_stages = ((E + 63) / 64) * per;
  auto fetch_o = [&](int st) {
    const int e0 = (st / per) * 64, k = st % per;
    if (k >= ns) {
      fetch_bf(vp + (long long)(k - ns) * kMlRows * p.ld, len - (k - ns) * kMlRows, e0, E);
      return;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = threadIdx.x + j * 256, r = k * 64 + (i >> 4), cc = e0 + (i & 15) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < D && cc < E) {
        const float* src = S0 + (long long)r * E + cc;
        if (e4) {
          v = *reinterpret_cast<const float4*>(src);
        } else {
          v.x = src[0];
          if (cc + 1 < E) v.y = src[1];
          if (cc + 2 < E) v.z = src[2];
          if (cc + 3 < E) v.w = src[3];
        }
      }
      reg[j] = make_uint4(__float_as_uint(v.x), __float_as_uint(v.y), __float_as_uint(v.z), __float_as_uint(v.w));
    }
  };
  auto store_o = [&](int st) {
    __nv_bfloat16* t = tiles + (st & 1) * 2 * kTile;
    if (st % per >= ns) {
      store_bf(t);
      return;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = threadIdx.x + j * 256, off = (i >> 4) * kMlPitch + (i & 15) * 4;
      split4(make_float4(__uint_as_float(reg[j].x), __uint_as_float(reg[j].y), __uint_as_float(reg[j].z), __uint_as_float(reg[j].w)), t + off,
             t + kTile + off);
    }
  };
  fetch_o(0);
  store_o(0);
  __syncthreads();
  for (int e0 = 0, st = 0; e0 < E; e0 += 64) {
    float acc[4][4] = {};
    for (int k = 0; k < per; ++k, ++st) {
      if (st + 1 < o_stages) fetch_o(st + 1);
      const __nv_bfloat16* t = tiles + (st & 1) * 2 * kTile;
      if (k < ns) {
#pragma unroll
        for (int ks = 0; ks < 64; ks += 16) {
          uint32_t a[4];
          ldsm4(qs + (wr + (lj & 1) * 8 + lr) * dp + k * 64 + ks + (lj >> 1) * 8, a);
#pragma unroll
          for (int nb = 0; nb < 2; ++nb) {
            uint32_t bh[4], bl[4];
            const int off = (ks + (lj & 1) * 8 + lr) * kMlPitch + wc + nb * 16 + (lj >> 1) * 8;
            ldsm4t(t + off, bh);
            ldsm4t(t + kTile + off, bl);
            mma16816(acc[nb * 2], a, bh[0], bh[1]);
            mma16816(acc[nb * 2 + 1], a, bh[2], bh[3]);
            mma16816(acc[nb * 2], a, bl[0], bl[1]);
            mma16816(acc[nb * 2 + 1], a, bl[2], bl[3]);
          }
        }
        if (k == ns - 1) {
          const float il = inter_s[wr + g], ih = inter_s[wr + g + 8];
#pragma unroll
          for (int nb = 0; nb < 4; ++nb) {
            acc[nb][0] *= il; acc[nb][1] *= il;
            acc[nb][2] *= ih; acc[nb][3] *= ih;
          }
        }
      } else {
#pragma unroll
        for (int ks = 0; ks < 64; ks += 16) {
          uint32_t ah[4], al[4];
          const int aoff = (wr + (lj & 1) * 8 + lr) * kMlPPitch + (k - ns) * kMlRows + ks + (lj >> 1) * 8;
          ldsm4(ph + aoff, ah);
          ldsm4(pl + aoff, al);
#pragma unroll
          for (int nb = 0; nb < 2; ++nb) {
            uint32_t b[4];
            ldsm4t(t + (ks + (lj & 1) * 8 + lr) * kMlPitch + wc + nb * 16 + (lj >> 1) * 8, b);
            mma16816(acc[nb * 2], ah, b[0], b[1]);
            mma16816(acc[nb * 2 + 1], ah, b[2], b[3]);
            mma16816(acc[nb * 2], al, b[0], b[1]);
            mma16816(acc[nb * 2 + 1], al, b[2], b[3]);
          }
        }
      }
      if (st + 1 < o_stages) store_o(st + 1);
      __syncthreads();
    }
    const float dl = inv_s[wr + g], dh = inv_s[wr + g + 8];
#pragma unroll
    for (int nb = 0; nb < 4; ++nb)
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int row = wr + g + (r >> 1) * 8, e = e0 + wc + nb * 8 + q4 * 2 + (r & 1);
        const float o = acc[nb][r] * (r < 2 ? dl : dh);
        if (r < 2) sq_lo += o * o;
        else sq_hi += o * o;
        if (row < rows && e < E) p.o[((long long)(t0 + r0 + row) * p.H + h) * E + e] = o;
      }
  }
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 1);
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 2);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 1);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 2);
  if (q4 == 0) { sq_s[wh][wr + g] = sq_lo; sq_s[wh][wr + g + 8] = sq_hi; }
  __syncthreads();                                       // also makes this CTA's rows of o visible to all its threads
  // ---- head norm, weight and gate
  for (int row = warp; row < rows; row += 8) {
    const float inv = 1.f / sqrtf((sq_s[0][row] + sq_s[1][row]) / E + p.eps);
    const long long t = t0 + r0 + row;
    const float* o = p.o + (t * p.H + h) * E;
    const __nv_bfloat16* gt = p.gate + t * p.ldg + (long long)h * E;
    __nv_bfloat16* out = p.out + (t * p.H + h) * E;
    for (int e = lane; e < E; e += 32)
      out[e] = __float2bfloat16(o[e] * inv * p.norm[(long long)h * E + e] * sigmoid_f(__bfloat162float(gt[e])));
  }
}

// ------------------------------------------------------------------------------------------------ decode step
struct MlstmStep {
  const void* q;
  const void* k;
  const void* v;
  long long ld;
  const float* logits;         // [rows, 2 H]
  const float* ib;
  const float* fb;
  float* S;                    // [slots, H, D, E]
  float* n;                    // [slots, 2, H, D]
  float* m;                    // [slots, 2, H]
  const int* slots;
  const int* positions;
  float* o;                    // [rows, H * E]
  float cap, qscale;
  int H, D, E;
};

// One token of every sequence: CTA = (column slice of 16 V, head, sequence), 16 threads across the columns, 16 along D.
template <typename T, int V>
__global__ void __launch_bounds__(256) mlstm_step_kernel(const MlstmStep p) {
  extern __shared__ float st_smem[];
  __shared__ float red[64];
  __shared__ float part[16][16 * V + 1];
  const int D = p.D, E = p.E, H = p.H;
  float* k_s = st_smem;
  float* q_s = k_s + D;
  const int h = blockIdx.y, s = blockIdx.z;
  const int slot = p.slots[s], pos = p.positions[s];
  const bool fresh = pos == 0;
  const int bank = pos & 1;
  const T* kp = static_cast<const T*>(p.k) + s * p.ld + (long long)h * D;
  const T* qp = static_cast<const T*>(p.q) + s * p.ld + (long long)h * D;
  const T* vp = static_cast<const T*>(p.v) + s * p.ld + (long long)h * E;
  const float i = mlstm_input_gate(p.logits[(long long)s * 2 * H + h] + p.ib[h], p.cap);
  const float f = mlstm_forget_gate(p.logits[(long long)s * 2 * H + H + h] + p.fb[h], p.cap);
  const float m0 = fresh ? 0.f : p.m[((long long)slot * 2 + bank) * H + h];
  const float m1 = fmaxf(f + m0, i);
  const float keep = fresh ? 0.f : expf(f + m0 - m1), add = expf(i - m1);
  const float* n_in = p.n + (((long long)slot * 2 + bank) * H + h) * D;
  float* n_out = p.n + (((long long)slot * 2 + (bank ^ 1)) * H + h) * D;
  float dot = 0.f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    const float kk = ldf(kp + d) * add, qq = ldf(qp + d) * p.qscale;
    k_s[d] = kk;
    q_s[d] = qq;
    const float nn = (fresh ? 0.f : keep * n_in[d]) + kk;
    dot = fmaf(nn, qq, dot);
    if (blockIdx.x == 0) n_out[d] = nn;
  }
  if (blockIdx.x == 0 && threadIdx.x == 0) p.m[((long long)slot * 2 + (bank ^ 1)) * H + h] = m1;
  dot = block_sum2(dot, 0.f, red).x;
  const float inv = 1.f / (fmaxf(fabsf(dot), expf(-m1)) + 1e-6f);
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int e = blockIdx.x * 16 * V + tx * V;
  float acc[V];
#pragma unroll
  for (int j = 0; j < V; ++j) acc[j] = 0.f;
  if (e < E) {
    float* Sp = p.S + ((long long)slot * H + h) * D * E + e;
    float vv[V];
#pragma unroll
    for (int j = 0; j < V; ++j) vv[j] = ldf(vp + e + j);
#pragma unroll 8
    for (int d = ty; d < D; d += 16) {
      if constexpr (V == 4) {
        float4 st = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(Sp + (long long)d * E);
        const float kk = k_s[d], qq = q_s[d];
        st.x = fmaf(keep, st.x, kk * vv[0]);
        st.y = fmaf(keep, st.y, kk * vv[1]);
        st.z = fmaf(keep, st.z, kk * vv[2]);
        st.w = fmaf(keep, st.w, kk * vv[3]);
        *reinterpret_cast<float4*>(Sp + (long long)d * E) = st;
        acc[0] = fmaf(qq, st.x, acc[0]);
        acc[1] = fmaf(qq, st.y, acc[1]);
        acc[2] = fmaf(qq, st.z, acc[2]);
        acc[3] = fmaf(qq, st.w, acc[3]);
      } else {
        const float st = (fresh ? 0.f : keep * Sp[(long long)d * E]) + k_s[d] * vv[0];
        Sp[(long long)d * E] = st;
        acc[0] = fmaf(q_s[d], st, acc[0]);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) part[ty][tx * V + j] = acc[j];
  __syncthreads();
  for (int j = threadIdx.x; j < 16 * V; j += blockDim.x) {
    const int col = blockIdx.x * 16 * V + j;
    if (col < E) {
      float sum = 0.f;
#pragma unroll
      for (int y = 0; y < 16; ++y) sum += part[y][j];
      p.o[((long long)s * H + h) * E + col] = sum * inv;
    }
  }
}

// The recurrence token by token for a whole prompt of one sequence (fp32 activations): CTA = (16 columns, head), the slice
// of S in shared memory.
template <typename T>
__global__ void __launch_bounds__(128) mlstm_seq_kernel(const MlstmStep p, int N, int start, int slot) {
  extern __shared__ float st_smem[];
  __shared__ float red[64];
  __shared__ float part[8][17];
  const int D = p.D, E = p.E, H = p.H, h = blockIdx.y;
  float* S_s = st_smem;            // [D][16]
  float* n_s = S_s + D * 16;
  float* k_s = n_s + D;
  float* q_s = k_s + D;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int e = blockIdx.x * 16 + tx;
  const bool fresh = start == 0;
  const int bank = start & 1, bank1 = (start + N) & 1;
  float* Sp = p.S + ((long long)slot * H + h) * D * E + e;
  for (int d = ty; d < D; d += 8) S_s[d * 16 + tx] = fresh || e >= E ? 0.f : Sp[(long long)d * E];
  for (int d = threadIdx.x; d < D; d += 128) n_s[d] = fresh ? 0.f : p.n[(((long long)slot * 2 + bank) * H + h) * D + d];
  float m = fresh ? 0.f : p.m[((long long)slot * 2 + bank) * H + h];
  __syncthreads();
  for (int t = 0; t < N; ++t) {
    const float i = mlstm_input_gate(p.logits[(long long)t * 2 * H + h] + p.ib[h], p.cap);
    const float f = mlstm_forget_gate(p.logits[(long long)t * 2 * H + H + h] + p.fb[h], p.cap);
    const float m1 = fmaxf(f + m, i);
    const float keep = expf(f + m - m1), add = expf(i - m1);
    m = m1;
    float dot = 0.f;
    for (int d = threadIdx.x; d < D; d += 128) {
      const float kk = ldf(static_cast<const T*>(p.k) + t * p.ld + (long long)h * D + d) * add;
      const float qq = ldf(static_cast<const T*>(p.q) + t * p.ld + (long long)h * D + d) * p.qscale;
      k_s[d] = kk;
      q_s[d] = qq;
      n_s[d] = fmaf(keep, n_s[d], kk);
      dot = fmaf(n_s[d], qq, dot);
    }
    dot = block_sum2(dot, 0.f, red).x;
    const float inv = 1.f / (fmaxf(fabsf(dot), expf(-m1)) + 1e-6f);
    const float vv = e < E ? ldf(static_cast<const T*>(p.v) + t * p.ld + (long long)h * E + e) : 0.f;
    float acc = 0.f;
    for (int d = ty; d < D; d += 8) {
      const float st = fmaf(keep, S_s[d * 16 + tx], k_s[d] * vv);
      S_s[d * 16 + tx] = st;
      acc = fmaf(q_s[d], st, acc);
    }
    part[ty][tx] = acc;
    __syncthreads();
    if (ty == 0 && e < E) {
      float sum = 0.f;
#pragma unroll
      for (int y = 0; y < 8; ++y) sum += part[y][tx];
      p.o[((long long)t * H + h) * E + e] = sum * inv;
    }
    __syncthreads();
  }
  if (e < E)
    for (int d = ty; d < D; d += 8) Sp[(long long)d * E] = S_s[d * 16 + tx];
  if (blockIdx.x == 0) {
    for (int d = threadIdx.x; d < D; d += 128) p.n[(((long long)slot * 2 + bank1) * H + h) * D + d] = n_s[d];
    if (threadIdx.x == 0) p.m[((long long)slot * 2 + bank1) * H + h] = m;
  }
}

// out[row, h, :] = rms(o[row, h, :]) * w[h, :] * sigmoid(gate[row, h, :]); one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate, long long ldg,
                      T* __restrict__ out, long long items, int H, int E, float eps) {
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31, h = int(item % H);
  const long long row = item / H;
  const float* src = o + item * E;
  float ss = 0.f;
  for (int e = lane; e < E; e += 32) ss += src[e] * src[e];
  const float inv = 1.f / sqrtf(warp_sum(ss) / E + eps);
  for (int e = lane; e < E; e += 32)
    stf(out + item * E + e, src[e] * inv * w[(long long)h * E + e] * sigmoid_f(ldf(gate + row * ldg + (long long)h * E + e)));
}

}  // namespace lt

extern "C" {

// One prompt chunk of one sequence, bf16.  q, k [N, H * D] and v [N, H * E] at pitch ld; logits [N, 2 H] fp32; S [H, D, E],
// n [2, H, D], m [2, H] of the sequence's slot; scratch: a, f, cmax [H, N], m_start [H, chunks + 1], U [H, chunks, D, E],
// nU [H, chunks, D], o [N, H * E], all fp32, chunks = ceil(N / 128).  out [N, H * E].
int lt_mlstm_prefill(const void* q, const void* k, const void* v, long long ld, const float* logits, const float* ib,
                     const float* fb, float cap, float qscale, const float* norm, float eps, const void* gate, long long ldg,
                     float* S, float* n, float* m, float* a, float* f, float* cmax, float* m_start, float* U, float* nU, float* o,
                     void* out, int N, int H, int D, int E, int start, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  const int chunks = (N + kMlChunk - 1) / kMlChunk;
  const size_t smem_out = mlstm_out_smem(D);
  const size_t smem_state = kMlStateSmem;
  const size_t smem_scan = size_t(chunks) * 4;
  const int dt = (D + kMlRows - 1) / kMlRows;
  if (smem_out > 220 * 1024 || H > 65535 || dt > 65535 || 2 * smem_scan > 48 * 1024) return -4;      // 6144 chunks: 786432 tokens at a time
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int aligned = ld % 8 == 0 && D % 8 == 0 && E % 8 == 0 && al(q) && al(k) && al(v);
  const int bank = start & 1, bank1 = (start + N) & 1, fresh = start == 0;
  mlstm_gates_kernel<<<H, 256, 2 * smem_scan, st>>>(logits, ib, fb, cap, fresh ? nullptr : m + (long long)bank * H, a, f, cmax, m_start, N, H, chunks);
  LT_LAUNCH_CHECK();
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem_state)));
  mlstm_chunk_state_kernel<<<dim3(chunks, H, dt), 256, smem_state, st>>>(
      static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), ld, a, cmax, m_start, U, nU, N, D, E, chunks, aligned);
  LT_LAUNCH_CHECK();
  const bool v4 = D % 4 == 0;                 // then D E and every offset are multiples of 4 too
  const long long per = v4 ? 1024 : 256;
  const unsigned sb = unsigned(((long long)D * E + per - 1) / per + (D + per - 1) / per);
  if (v4) {
    mlstm_chunk_scan_kernel<4><<<dim3(sb, H), 256, smem_scan, st>>>(U, nU, cmax, m_start, S, n + (long long)bank * H * D, n + (long long)bank1 * H * D, m + (long long)bank1 * H, N, D, E, chunks, fresh);
  } else {
    mlstm_chunk_scan_kernel<1><<<dim3(sb, H), 256, smem_scan, st>>>(U, nU, cmax, m_start, S, n + (long long)bank * H * D, n + (long long)bank1 * H * D, m + (long long)bank1 * H, N, D, E, chunks, fresh);
  }
  LT_LAUNCH_CHECK();
  MlstmOut p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), ld, a, f, cmax,
             m_start, U, nU, norm, static_cast<const __nv_bfloat16*>(gate), ldg, o, static_cast<__nv_bfloat16*>(out), qscale, eps, N, H, D, E,
             chunks, fresh, aligned};
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(mlstm_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem_out)));
  mlstm_out_kernel<<<dim3(2 * chunks, H), 256, smem_out, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

// One token of S sequences (seq_len 0), or seq_len tokens of one sequence one after another (its slot and first position
// given as slot / start): o [rows, H * E] fp32, before the head norm.
int lt_mlstm_step(int fp32, const void* q, const void* k, const void* v, long long ld, const float* logits, const float* ib,
                  const float* fb, float cap, float qscale, float* S, float* n, float* m, const int* slots, const int* positions,
                  float* o, int rows, int H, int D, int E, int seq_len, int slot, int start, void* stream) {
  using namespace lt;
  if (rows == 0 && seq_len == 0) return 0;
  if (H > 65535 || rows > 65535 || D > 2048) return -4;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  MlstmStep p{q, k, v, ld, logits, ib, fb, S, n, m, slots, positions, o, cap, qscale, H, D, E};
  if (seq_len > 0) {
    const int smem = (D * 16 + 3 * D) * 4;
    auto kern = fp32 ? mlstm_seq_kernel<float> : mlstm_seq_kernel<__nv_bfloat16>;
    if (smem > 48 * 1024) LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    kern<<<dim3((E + 15) / 16, H), 128, smem, st>>>(p, seq_len, start, slot);
  } else {
    const bool v4 = E % 4 == 0;
    const int cols = v4 ? 64 : 16;
    dim3 grid((E + cols - 1) / cols, H, rows);
    const int smem = 2 * D * 4;
    if (fp32) {
      if (v4) mlstm_step_kernel<float, 4><<<grid, 256, smem, st>>>(p);
      else mlstm_step_kernel<float, 1><<<grid, 256, smem, st>>>(p);
    } else {
      if (v4) mlstm_step_kernel<__nv_bfloat16, 4><<<grid, 256, smem, st>>>(p);
      else mlstm_step_kernel<__nv_bfloat16, 1><<<grid, 256, smem, st>>>(p);
    }
  }
  LT_LAUNCH_CHECK();
  return 0;
}

int lt_head_norm_gate(int fp32, const float* o, const float* w, const void* gate, long long ldg, void* out, long long rows, int H,
                      int E, float eps, void* stream) {
  using namespace lt;
  const long long items = rows * H;
  if (items == 0) return 0;
  const unsigned grid = unsigned((items + 3) / 4);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (fp32) head_norm_gate_kernel<float><<<grid, 128, 0, st>>>(o, w, static_cast<const float*>(gate), ldg, static_cast<float*>(out), items, H, E, eps);
  else head_norm_gate_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(o, w, static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<__nv_bfloat16*>(out), items, H, E, eps);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
