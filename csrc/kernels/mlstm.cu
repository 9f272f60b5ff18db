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
// so no exponent is ever positive.  Four kernels: gates (a, F and the running maxima of every chunk), chunk states (the K^T V
// of every chunk relative to its own largest a, tensor cores), a scan over chunks (m and the states at chunk starts, fp32)
// and the outputs (tensor cores; the head norm and the gate in the epilogue).  The state stays fp32; where it, the decayed keys or the token weights enter a bf16
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
// logits [N, 2 H] fp32 (i then f); one warp per (chunk, head).  Writes a, F and the running maximum of a inside the chunk
// ([H, N] each) and, per chunk, F at its last token and its largest a ([H, chunks] pairs).
__global__ void __launch_bounds__(128)
mlstm_gates_kernel(const float* __restrict__ logits, const float* __restrict__ ib, const float* __restrict__ fb, float cap,
                   float* __restrict__ a_out, float* __restrict__ f_out, float* __restrict__ c_out, float2* __restrict__ last, int N,
                   int H, int chunks) {
  const int h = blockIdx.y, c = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (c >= chunks) return;
  const float bi = ib[h], bf = fb[h];
  constexpr int kParts = kMlChunk / 32;
  float li[kParts], lf[kParts];
#pragma unroll
  for (int k = 0; k < kParts; ++k) {
    const int t = min(c * kMlChunk + k * 32 + lane, N - 1);
    li[k] = logits[(long long)t * 2 * H + h] + bi;
    lf[k] = logits[(long long)t * 2 * H + H + h] + bf;
  }
  float run = 0.f, top = -INFINITY;
#pragma unroll
  for (int k = 0; k < kParts; ++k) {
    const int t = c * kMlChunk + k * 32 + lane;
    // tokens past the end add nothing to F and -inf to the maximum
    float f = t < N ? mlstm_forget_gate(lf[k], cap) : 0.f;
    const float i = t < N ? mlstm_input_gate(li[k], cap) : -INFINITY;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float g = __shfl_up_sync(0xffffffffu, f, o);
      if (lane >= o) f += g;
    }
    f += run;
    const float a = i - f;
    float mx = a;
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
  if (lane == 0) last[(long long)h * chunks + c] = make_float2(run, top);
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

// out = o * inv * w * sigmoid(gate) over a row, by one warp.  vec: everything aligned to four elements.  The loads of 512 columns
// are requested before the first of them is used.
template <typename T>
__device__ __forceinline__ void norm_gate_row(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate,
                                              T* __restrict__ out, int E, float inv, bool vec) {
  const int lane = threadIdx.x & 31;
  if (!vec) {
    for (int e = lane; e < E; e += 32) stf(out + e, o[e] * inv * w[e] * sigmoid_f(ldf(gate + e)));
    return;
  }
  for (int e0 = lane * 4; e0 < E; e0 += 512) {
    float4 a[4], b[4], c[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int e = min(e0 + k * 128, E - 4);
      a[k] = *reinterpret_cast<const float4*>(o + e);
      b[k] = *reinterpret_cast<const float4*>(w + e);
      c[k] = ldf4(gate + e);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (e0 + k * 128 < E)
        stf4(out + e0 + k * 128, make_float4(a[k].x * inv * b[k].x * sigmoid_f(c[k].x), a[k].y * inv * b[k].y * sigmoid_f(c[k].y),
                                             a[k].z * inv * b[k].z * sigmoid_f(c[k].z), a[k].w * inv * b[k].w * sigmoid_f(c[k].w)));
  }
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

// The same into shared memory: an asynchronous 16-byte copy where the piece is whole and aligned.
__device__ __forceinline__ void copy8(__nv_bfloat16* dst, const __nv_bfloat16* row, int c, int cols, bool row_ok, bool aligned) {
  if (row_ok && aligned && c + 8 <= cols)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(row + c) : "memory");
  else
    *reinterpret_cast<uint4*>(dst) = load8(row, c, cols, row_ok, false);
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// ------------------------------------------------------------------------------------------------ chunk states
// U[h, c] [D, EP] = sum_s exp(a_s - largest a of the chunk) k_s v_s^T and nU[h, c] [D]; EP: E rounded up to 8, zeros behind.
// One CTA per 64 rows of U: the decayed keys are split
// into their two parts once and stay in shared memory while 128 columns of V at a time pass by (the next ones are loaded
// into registers under the products).  Eight warps as 2 row halves x 4 column quarters of 32 x 32.
constexpr int kMlWide = 128, kMlWidePitch = kMlWide + 8;
constexpr size_t kMlStateSmem = (2 * size_t(kMlChunk) * kMlPitch + size_t(kMlChunk) * kMlWidePitch) * 2;

__global__ void __launch_bounds__(256, 2)
mlstm_chunk_state_kernel(const __nv_bfloat16* __restrict__ k, const __nv_bfloat16* __restrict__ v, long long ld,
                         const float* __restrict__ a, const float2* __restrict__ last, float* __restrict__ U, float* __restrict__ nU,
                         int N, int D, int E, int EP, int chunks, int aligned) {
  extern __shared__ __align__(16) uint8_t ml_smem[];
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(ml_smem);          // [128][pitch]: high parts of w_s k_s
  __nv_bfloat16* kl = kh + kMlChunk * kMlPitch;
  __nv_bfloat16* vs = kl + kMlChunk * kMlPitch;                            // [128][wide pitch]
  __shared__ float w_s[kMlChunk];
  const int c = blockIdx.x, h = blockIdx.y, d0 = blockIdx.z * kMlRows;
  const int t0 = c * kMlChunk, len = min(kMlChunk, N - t0);
  const float m_last = last[(long long)h * chunks + c].y;
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
  float* out = U + ((long long)h * chunks + c) * D * EP;
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
          if (d < D && e < EP) *reinterpret_cast<float2*>(out + (long long)d * EP + e) = make_float2(acc[mb][nb][r], acc[mb][nb][r + 1]);
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
// In place: U[h, c] becomes the state at the start of chunk c, as eight high parts and eight low parts (bf16) where eight
// fp32 values were; the state after the last chunk goes back to the slot.  nU likewise, in fp32.  m_start [H, chunks + 1]; its last
// entry is m after the portion, which the output kernel puts into the slot: here other blocks still read the slot's m, and the
// old and the new value share a bank when the portion's length is even.
__global__ void __launch_bounds__(256)
mlstm_chunk_scan_kernel(float* __restrict__ U, float* __restrict__ nU, const float2* __restrict__ last, const float* __restrict__ m_in,
                        float* __restrict__ m_start, float* __restrict__ S, const float* __restrict__ n_in, float* __restrict__ n_out,
                        int D, int E, int EP, int chunks, int fresh) {
  extern __shared__ float2 mix_s[];      // [chunks]: S <- x S + y U
  const int h = blockIdx.y;
  for (int c = threadIdx.x; c < chunks; c += blockDim.x) mix_s[c] = last[(long long)h * chunks + c];
  __syncthreads();
  if (threadIdx.x == 0) {
    float m = fresh ? 0.f : m_in[h];
    for (int c = 0; c < chunks; ++c) {
      const float2 l = mix_s[c];
      const float top = fmaxf(m, l.y);
      if (blockIdx.x == 0) m_start[(long long)h * (chunks + 1) + c] = m;
      mix_s[c] = make_float2(m - top, l.y - top);
      m = l.x + top;
    }
    if (blockIdx.x == 0) m_start[(long long)h * (chunks + 1) + chunks] = m;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < chunks; c += blockDim.x) mix_s[c] = make_float2(expf(mix_s[c].x), expf(mix_s[c].y));
  __syncthreads();
  const long long DE = (long long)D * EP;
  const unsigned s_blocks = unsigned((DE + 2047) / 2048);          // the blocks after these take n
  if (blockIdx.x >= s_blocks) {
    const int d = (blockIdx.x - s_blocks) * 256 + threadIdx.x;
    if (d >= D) return;
    float cur = fresh ? 0.f : n_in[(long long)h * D + d];
    float* u = nU + (long long)h * chunks * D + d;
    for (int c0 = 0; c0 < chunks; c0 += 8) {
      float nx[8];
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < chunks) nx[j] = u[(long long)(c0 + j) * D];
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < chunks) {
          u[(long long)(c0 + j) * D] = cur;
          cur = fmaf(mix_s[c0 + j].x, cur, mix_s[c0 + j].y * nx[j]);
        }
    }
    n_out[(long long)h * D + d] = cur;
    return;
  }
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * 8;
  if (i >= DE) return;
  const int e = int(i % EP);
  float* st = S + ((long long)h * D + i / EP) * E + e;
  float cur[8];
#pragma unroll
  for (int v = 0; v < 8; ++v) cur[v] = fresh || e + v >= E ? 0.f : st[v];
  float* u = U + (long long)h * chunks * DE + i;
  constexpr int kAhead = 4;
  float nx[2][kAhead][8];
  auto load = [&](float (&b)[kAhead][8], int c0) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < chunks) ldf8(u + (c0 + j) * DE, b[j]);
  };
  auto step = [&](const float (&b)[kAhead][8], int c0) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < chunks) {
        uint4 hi, lo;
        __nv_bfloat16 *ph = reinterpret_cast<__nv_bfloat16*>(&hi), *pl = reinterpret_cast<__nv_bfloat16*>(&lo);
#pragma unroll
        for (int v = 0; v < 8; ++v) split_bf16(cur[v], ph[v], pl[v]);
        uint4* dst = reinterpret_cast<uint4*>(u + (c0 + j) * DE);
        dst[0] = hi;
        dst[1] = lo;
        const float2 m = mix_s[c0 + j];
#pragma unroll
        for (int v = 0; v < 8; ++v) cur[v] = fmaf(m.x, cur[v], m.y * b[j][v]);
      }
  };
  load(nx[0], 0);
  for (int c0 = 0; c0 < chunks; c0 += 2 * kAhead) {
    load(nx[1], c0 + kAhead);
    step(nx[0], c0);
    load(nx[0], c0 + 2 * kAhead);
    step(nx[1], c0 + kAhead);
  }
#pragma unroll
  for (int v = 0; v < 8; ++v)
    if (e + v < E) st[v] = cur[v];
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
  const float* m_start;          // [H, chunks + 1]
  float* m_out;                  // [H]
  const __nv_bfloat16* S0;       // [H, chunks, D, EP / 8, 16] states at chunk starts: eight high parts, eight low parts
  const float* n0;               // [H, chunks, D]
  const float* norm;             // [H * E]
  const __nv_bfloat16* gate;     // [N, H * E] logits at pitch ldg
  long long ldg;
  float* o;                      // scratch [N, H * E]
  __nv_bfloat16* out;            // [N, H * E]
  float qscale, eps;
  int N, H, D, E, EP, chunks, fresh, aligned;
};

constexpr int kMlPPitch = kMlChunk + 8;
static size_t mlstm_out_smem(int D, int rows, int stages) {
  const int dp = (D + 63) / 64 * 64 + 8;
  return size_t(rows) * dp * 2 + 2 * size_t(rows) * kMlPPitch * 2 + size_t(stages) * 2 * kMlRows * kMlPitch * 2;
}

// One CTA: ROWS tokens of one chunk of one head; a warp has 16 rows and 32 of the 64 columns of a tile.  All tiles (keys,
// then per 64 output columns the slices of the state before the chunk and the values) go through one ring of STAGES buffers
// filled by asynchronous copies.
template <int ROWS, int STAGES>
__global__ void __launch_bounds__(ROWS * 4, ROWS == 128 ? 1 : 2) mlstm_out_kernel(const MlstmOut p) {
  extern __shared__ __align__(16) uint8_t ml_smem[];
  constexpr int kThreads = ROWS * 4, kParts = kMlChunk / ROWS, kTile = kMlRows * kMlPitch;
  const int D = p.D, E = p.E;
  const int nd = (D + 63) / 64, dp = nd * 64 + 8;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(ml_smem);      // [ROWS][dp]
  __nv_bfloat16* ph = qs + ROWS * dp;                                  // [ROWS][kMlPPitch] token weights, high and low parts
  __nv_bfloat16* pl = ph + ROWS * kMlPPitch;
  __nv_bfloat16* tiles = pl + ROWS * kMlPPitch;                        // [STAGES][2][64][pitch]
  __shared__ float a_s[kMlChunk], top_s[ROWS], inter_s[ROWS], den_s[2][ROWS], inv_s[ROWS], sq_s[2][ROWS];
  const int h = blockIdx.y, c = blockIdx.x / kParts;
  const int t0 = c * kMlChunk, r0 = (blockIdx.x % kParts) * ROWS;      // chunk start, first row inside it
  const int len = min(kMlChunk, p.N - t0);                             // tokens of this chunk
  if (r0 >= len) return;
  const int rows = min(ROWS, len - r0);
  const int kblocks = (r0 + rows + 63) / 64;                           // key blocks that some row sees
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lj = lane >> 3, lr = lane & 7;
  const int g = lane >> 2, q4 = lane & 3;
  const int wr = (warp >> 1) * 16, wc = (warp & 1) * 32, wh = warp & 1;
  const long long hn = (long long)h * p.N;
  const float m0 = p.m_start[(long long)h * (p.chunks + 1) + c];
  if (blockIdx.x == 0 && threadIdx.x == 0) p.m_out[h] = p.m_start[(long long)h * (p.chunks + 1) + p.chunks];
  const bool have_state = !(p.fresh && c == 0);

  // ---- the tiles in order of use
  const __nv_bfloat16* kp = p.k + (long long)t0 * p.ld + (long long)h * D;
  const __nv_bfloat16* vp = p.v + (long long)t0 * p.ld + (long long)h * E;
  const __nv_bfloat16* S0 = p.S0 + ((long long)h * p.chunks + c) * D * p.EP * 2;
  const int ns = have_state ? nd : 0, per = ns + kblocks;
  const int k_stages = kblocks * nd, stages = k_stages + (E + 63) / 64 * per;
  auto issue = [&](int st) {
    if (st < stages) {
      __nv_bfloat16* t = tiles + (st % STAGES) * 2 * kTile;
      const int o = st - k_stages, k = o % per;
      if (st < k_stages || k >= ns) {
        const bool key = st < k_stages;
        const int kb = key ? st / nd : k - ns;
        const __nv_bfloat16* src = (key ? kp : vp) + (long long)kb * kMlRows * p.ld;
        const int c0 = key ? (st % nd) * 64 : o / per * 64, cols = key ? D : E, ok = len - kb * kMlRows;
        for (int i = threadIdx.x; i < kMlRows * 8; i += kThreads) {
          const int r = i >> 3, cc = (i & 7) * 8;
          copy8(t + r * kMlPitch + cc, src + r * p.ld, c0 + cc, cols, r < ok, p.aligned);
        }
      } else {
        const int e0 = o / per * 64;
        for (int i = threadIdx.x; i < kMlRows * 16; i += kThreads) {       // 16-byte pieces: part 0 high, 1 low
          const int r = i >> 4, part = i & 1, cc = ((i >> 1) & 7) * 8, d = k * 64 + r;
          copy8(t + part * kTile + r * kMlPitch + cc, S0 + (long long)d * p.EP * 2 + (e0 + cc) * 2 + part * 8, 0, 8, d < D && e0 + cc < p.EP, true);
        }
      }
    }
    copy_commit();
  };
  for (int st = 0; st < STAGES - 1; ++st) issue(st);

  for (int i = threadIdx.x; i < kMlChunk; i += kThreads) a_s[i] = i < len ? p.a[hn + t0 + i] : -INFINITY;
  for (int i = threadIdx.x; i < ROWS; i += kThreads) {
    const float top = i < rows ? fmaxf(m0, p.cmax[hn + t0 + r0 + i]) : 0.f;
    top_s[i] = top;
    inter_s[i] = i < rows && have_state ? expf(m0 - top) * p.qscale : 0.f;
  }
  const __nv_bfloat16* qp = p.q + (long long)(t0 + r0) * p.ld + (long long)h * D;
  for (int i = threadIdx.x; i < ROWS * nd * 8; i += kThreads) {
    const int r = i / (nd * 8), cc = (i % (nd * 8)) * 8;
    *reinterpret_cast<uint4*>(qs + r * dp + cc) = load8(qp + r * p.ld, cc, D, r < rows, p.aligned);
  }
  int st = 0;
  // The tile of stage st is there and everybody is done with the one before it, whose buffer is filled again.
  auto acquire = [&]() -> const __nv_bfloat16* {
    copy_wait<STAGES - 2>();
    __syncthreads();
    issue(st + STAGES - 1);
    return tiles + (st++ % STAGES) * 2 * kTile;
  };

  // ---- token weights: (q . k) qscale exp(a_s - M_t) for s <= t, and their row sums
  float sum_lo = 0.f, sum_hi = 0.f;
  for (int kb = 0; kb < kblocks; ++kb) {
    float acc[4][4] = {};
    for (int dd = 0; dd < nd; ++dd) {
      const __nv_bfloat16* t = acquire();
#pragma unroll
      for (int ks = 0; ks < 64; ks += 16) {
        uint32_t a[4], b[2][4];
        ldsm4(qs + (wr + (lj & 1) * 8 + lr) * dp + dd * 64 + ks + (lj >> 1) * 8, a);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) ldsm4(t + (wc + nb * 16 + (lj >> 1) * 8 + lr) * kMlPitch + ks + (lj & 1) * 8, b[nb]);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) mma16816(acc[nb], a, b[nb >> 1][(nb & 1) * 2], b[nb >> 1][(nb & 1) * 2 + 1]);
      }
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
#pragma unroll 8
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
  const float il = inter_s[wr + g], ih = inter_s[wr + g + 8], dl = inv_s[wr + g], dh = inv_s[wr + g + 8];
  for (int e0 = 0; e0 < E; e0 += 64) {
    float acc[4][4] = {};
    for (int k = 0; k < ns; ++k) {
      const __nv_bfloat16* t = acquire();
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
    }
#pragma unroll
    for (int nb = 0; nb < 4; ++nb) {
      acc[nb][0] *= il; acc[nb][1] *= il;
      acc[nb][2] *= ih; acc[nb][3] *= ih;
    }
    for (int kb = 0; kb < kblocks; ++kb) {
      const __nv_bfloat16* t = acquire();
#pragma unroll
      for (int ks = 0; ks < 64; ks += 16) {
        uint32_t ah[4], al[4];
        const int aoff = (wr + (lj & 1) * 8 + lr) * kMlPPitch + kb * kMlRows + ks + (lj >> 1) * 8;
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
  copy_wait<0>();
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 1);
  sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 2);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 1);
  sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 2);
  if (q4 == 0) { sq_s[wh][wr + g] = sq_lo; sq_s[wh][wr + g + 8] = sq_hi; }
  __syncthreads();                                       // also makes this CTA's rows of o visible to all its threads
  // ---- head norm, weight and gate: a warp per row
  for (int row = warp; row < rows; row += kThreads / 32) {
    const float inv = 1.f / sqrtf((sq_s[0][row] + sq_s[1][row]) / E + p.eps);
    const long long t = t0 + r0 + row;
    norm_gate_row(p.o + (t * p.H + h) * E, p.norm + (long long)h * E, p.gate + t * p.ldg + (long long)h * E, p.out + (t * p.H + h) * E, E, inv,
                  p.aligned && (p.ldg & 3) == 0);
  }
}

template <int ROWS, int STAGES>
static int launch_mlstm_out(const MlstmOut& p, cudaStream_t st) {
  const size_t smem = mlstm_out_smem(p.D, ROWS, STAGES);
  auto kern = mlstm_out_kernel<ROWS, STAGES>;
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
  kern<<<dim3(p.chunks * (kMlChunk / ROWS), p.H), ROWS * 4, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
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
                      T* __restrict__ out, long long items, int H, int E, float eps, int vec) {
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31, h = int(item % H);
  const long long row = item / H;
  const float* src = o + item * E;
  float ss = 0.f;
#pragma unroll 4
  for (int e = lane; e < E; e += 32) ss += src[e] * src[e];
  const float inv = 1.f / sqrtf(warp_sum(ss) / E + eps);
  norm_gate_row(src, w + (long long)h * E, gate + row * ldg + (long long)h * E, out + item * E, E, inv, vec != 0);
}

}  // namespace lt

extern "C" {

// One prompt portion of one sequence, bf16.  q, k [N, H * D] and v [N, H * E] at pitch ld; logits [N, 2 H] fp32; S [H, D, E],
// n [2, H, D], m [2, H] of the sequence's slot; scratch (fp32, 16-byte aligned): a, f, cmax [H, N], last [H, chunks, 2],
// m_start [H, chunks + 1], U [H, chunks, D, E rounded up to 8], nU [H, chunks, D], o [N, H * E], chunks = ceil(N / 128).
// out [N, H * E].
int lt_mlstm_prefill(const void* q, const void* k, const void* v, long long ld, const float* logits, const float* ib,
                     const float* fb, float cap, float qscale, const float* norm, float eps, const void* gate, long long ldg,
                     float* S, float* n, float* m, float* a, float* f, float* cmax, float* last, float* m_start, float* U, float* nU,
                     float* o, void* out, int N, int H, int D, int E, int start, void* stream) {
  using namespace lt;
  if (N == 0) return 0;
  const int chunks = (N + kMlChunk - 1) / kMlChunk, EP = (E + 7) / 8 * 8;
  const size_t smem_scan = size_t(chunks) * 8, limit = 227 * 1024 - 4096;      // the kernels' static shared memory stays below 4 KB
  const int dt = (D + kMlRows - 1) / kMlRows;
  if (mlstm_out_smem(D, 64, 2) > limit || H > 65535 || dt > 65535 || smem_scan > 48 * 1024) return -4;   // 786432 tokens at a time
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int aligned = ld % 8 == 0 && D % 8 == 0 && E % 8 == 0 && al(q) && al(k) && al(v) && al(gate) && al(norm) && al(out) && al(o);
  const int bank = start & 1, bank1 = (start + N) & 1, fresh = start == 0;
  float2* ends = reinterpret_cast<float2*>(last);
  mlstm_gates_kernel<<<dim3((chunks + 3) / 4, H), 128, 0, st>>>(logits, ib, fb, cap, a, f, cmax, ends, N, H, chunks);
  LT_LAUNCH_CHECK();
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(kMlStateSmem)));
  mlstm_chunk_state_kernel<<<dim3(chunks, H, dt), 256, kMlStateSmem, st>>>(
      static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), ld, a, ends, U, nU, N, D, E, EP, chunks, aligned);
  LT_LAUNCH_CHECK();
  const unsigned sb = unsigned(((long long)D * EP + 2047) / 2048 + (D + 255) / 256);
  mlstm_chunk_scan_kernel<<<dim3(sb, H), 256, smem_scan, st>>>(U, nU, ends, m + (long long)bank * H, m_start, S, n + (long long)bank * H * D,
                                                              n + (long long)bank1 * H * D, D, E, EP, chunks, fresh);
  LT_LAUNCH_CHECK();
  MlstmOut p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), ld, a, f, cmax,
             m_start, m + (long long)bank1 * H, reinterpret_cast<const __nv_bfloat16*>(U), nU, norm, static_cast<const __nv_bfloat16*>(gate), ldg, o,
             static_cast<__nv_bfloat16*>(out), qscale, eps, N, H, D, E, EP, chunks, fresh, aligned};
  // whole chunks per CTA share the tiles among more rows, where they fit and fill the GPU
  if ((long long)chunks * H >= sm_count() * 3 / 4) {
    if (mlstm_out_smem(D, 128, 4) <= limit) return launch_mlstm_out<128, 4>(p, st);
    if (mlstm_out_smem(D, 128, 3) <= limit) return launch_mlstm_out<128, 3>(p, st);
  }
  if (mlstm_out_smem(D, 64, 4) <= limit) return launch_mlstm_out<64, 4>(p, st);
  return launch_mlstm_out<64, 2>(p, st);
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
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const int vec = E % 4 == 0 && ldg % 4 == 0 && al(o) && al(w) && al(gate) && al(out);
  if (fp32) head_norm_gate_kernel<float><<<grid, 128, 0, st>>>(o, w, static_cast<const float*>(gate), ldg, static_cast<float*>(out), items, H, E, eps, vec);
  else head_norm_gate_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(o, w, static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<__nv_bfloat16*>(out), items, H, E, eps, vec);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
