// Latent attention on a paged cache.  A token is kept as one row: its normed latent (kv_rank columns, padded to `c`) and one
// rotated key part shared by all heads (padded to `r`).  Keys and values of a head are linear maps of the latent, so a
// decode step moves the query to the latent's side once and then attends to the rows themselves: every head reads the same
// row, as key over its c + r columns and as value over its first c.
//
//   latent_rope_kernel     rotation of the queries' shared-position part, norm of the latent, rotation of the key part,
//                          cache write
//   latent_decode_kernel   split-K decode attention of up to 32 heads per CTA on the rows of a sequence's pages
//   latent_merge_kernel    combines the splits
#include "lt_cuda.h"
#include "common/host.h"
#include "common/ptx.cuh"
#include "common/scalar.cuh"

namespace lt {

struct RopeParams {
  void* proj;                // [N, ld]: heads of d + r columns from column 0, the latent and the key part from c_off
  long long ld;
  int H, d, r, rot;          // rot <= r rotated columns
  int c_off, rank, c;        // c_off < 0: queries only
  const float* c_norm;       // [rank]
  float eps;
  const int* positions;
  const int* slots;          // block * block_size + offset: the row of the cache [blocks, 1, block_size, c + r]
  const double* freq;        // [rot / 2] angle per token
  float gain;
  void* q_out;               // [N, H, q_ld]: rotated part at column q_col; nullptr: in place
  int q_ld, q_col;
  void* cache;
  void* lin;                 // [N, c + r] or nullptr: the row once more
};

constexpr int kRopeThreads = 128;
constexpr int kRopeMaxPairs = 1024;

__device__ __forceinline__ float2 ldf2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ldf2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void stf2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void stf2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

template <typename T>
__global__ void __launch_bounds__(kRopeThreads) latent_rope_kernel(const RopeParams p) {
  extern __shared__ float2 cs[];         // [rot / 2] (cos, sin) of this token
  __shared__ float red[64];
  const int n = blockIdx.x;
  T* row = static_cast<T*>(p.proj) + n * p.ld;
  const int pos = p.positions[n];
  for (int i = threadIdx.x; i < p.rot / 2; i += kRopeThreads) {
    // the angle can be far outside a period: reduce it in double before the fp32 sine
    const double turns = double(pos) * p.freq[i] * 0.15915494309189535;
    float s, c;
    sincospif(float(2.0 * (turns - rint(turns))), &s, &c);
    cs[i] = make_float2(c * p.gain, s * p.gain);
  }
  float ss = 0.f;
  if (p.c_off >= 0)
    for (int i = threadIdx.x; i < p.rank; i += kRopeThreads) {
      const float f = ldf(row + p.c_off + i);
      ss = fmaf(f, f, ss);
    }
  const float sum = block_sum2(ss, 0.f, red).x;            // also publishes the angles
  auto turn = [&](float2 v, int i) -> float2 {             // pair i; pairs past the rotated part are zeros
    if (2 * i >= p.rot) return make_float2(0.f, 0.f);
    const float2 t = cs[i];
    return make_float2(v.x * t.x - v.y * t.y, v.y * t.x + v.x * t.y);
  };
  const int pr = p.r / 2;
  T* q_out = p.q_out ? static_cast<T*>(p.q_out) + (long long)n * p.H * p.q_ld + p.q_col : row + p.d;
  const int q_ld = p.q_out ? p.q_ld : p.d + p.r;
  for (int i = threadIdx.x; i < p.H * pr; i += kRopeThreads) {
    const int h = i / pr, k = i - h * pr;
    stf2(q_out + (long long)h * q_ld + 2 * k, turn(ldf2(row + (long long)h * (p.d + p.r) + p.d + 2 * k), k));
  }
  if (p.c_off < 0) return;
  const float inv = 1.f / sqrtf(sum / p.rank + p.eps);
  const int width = p.c + p.r;
  T* out = static_cast<T*>(p.cache) + (long long)p.slots[n] * width;
  T* lin = p.lin ? static_cast<T*>(p.lin) + (long long)n * width : nullptr;
  const T* src = row + p.c_off;
  for (int i = threadIdx.x; i < width / 2; i += kRopeThreads) {
    float2 v;
    if (2 * i < p.c) {
      v.x = 2 * i < p.rank ? ldf(src + 2 * i) * inv * p.c_norm[2 * i] : 0.f;
      v.y = 2 * i + 1 < p.rank ? ldf(src + 2 * i + 1) * inv * p.c_norm[2 * i + 1] : 0.f;
    } else {
      const int k = i - p.c / 2;
      const bool live = 2 * k < p.rot;
      v = turn(live ? make_float2(ldf(src + p.rank + 2 * k), ldf(src + p.rank + 2 * k + 1)) : make_float2(0.f, 0.f), k);
    }
    stf2(out + 2 * i, v);
    if (lin) stf2(lin + 2 * i, v);
  }
}

// ------------------------------------------------------------------------------------------------------------ decode
// One CTA of eight warps per (sequence, group of up to 16 MT heads, split of the visible keys).  Tiles of 64 rows arrive by
// plain bulk copies, one per row (rows of a sequence lie in pages), at a pitch of 16 bytes more than a row, so that
// ldmatrix meets no bank conflicts; a ring of `stages` tiles is filled ahead.  Per tile:
//   scores   warp = 16 keys x one half of the c + r columns (mma.sync m16n8k16: heads x keys), halves added through shared
//            memory; the query block stays in shared memory
//   softmax  256 / (16 MT) threads per head: running maximum and sum in registers, weights as bf16 operands to shared
//   values   warp = an eighth of the c columns: accumulators in registers, rows read transposed from the same tile
// tcgen05 is not the tool here: its 64- or 128-row tiles would be mostly empty at 16 or 32 heads, 512 value columns of them
// would fill the tensor memory, and the kernel is bound by streaming the rows.
constexpr int kLdThreads = 256;
constexpr int kLdKeys = 64;
constexpr int kLdMaxStages = 4;
constexpr int kLdSPitch = kLdKeys + 4;      // floats
constexpr int kLdPPitch = kLdKeys + 8;      // bf16

struct LatentDecodeParams {
  const __nv_bfloat16* q;        // [S, H, w]
  const __nv_bfloat16* cache;    // [rows, w], w = c + r, a multiple of 64
  const int* tables;             // [S, max_blocks]
  const int* ctx;                // [S] keys of the sequence, the query's own included
  float* part;                   // [S * H, splits, c] unnormalised outputs
  float* stat;                   // [S * H, splits, 2] maximum (log2 domain) and sum
  __nv_bfloat16* out;            // [S, H, c]
  int H, c, w, block_size, max_blocks, splits, window, stages;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void ld_ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ld_bulk(uint32_t smem_dst, const void* gsrc, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_dst), "l"(gsrc), "r"(bytes), "r"(bar) : "memory");
}

// Shared memory of a CTA: tiles, query block, score halves, weights, per-head factors, barriers.
__host__ __device__ inline int ld_smem_bytes(int w, int heads, int stages) {
  const int pitch = w * 2 + 16;
  return stages * kLdKeys * pitch + heads * pitch + 2 * heads * kLdSPitch * 4 + heads * kLdPPitch * 2 + 3 * heads * 4 + kLdMaxStages * 8 + 16;
}

// MT: 16-head blocks of a CTA (1 or 2).
template <int MT>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LatentDecodeParams p) {
  constexpr int MH = MT * 16;
  constexpr int TPH = kLdThreads / MH;           // threads per head in the softmax
  constexpr int KPT = kLdKeys / TPH;             // keys of each
  extern __shared__ __align__(128) uint8_t ld_smem[];
  const int pitch = p.w * 2 + 16, tile_bytes = kLdKeys * pitch;
  uint8_t* q_s = ld_smem + p.stages * tile_bytes;
  float* s_s = reinterpret_cast<float*>(q_s + MH * pitch);                             // [2][MH][kLdSPitch]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_s + 2 * MH * kLdSPitch);     // [MH][kLdPPitch]
  float* f_s = reinterpret_cast<float*>(p_s + MH * kLdPPitch);                         // [MH] rescale of the tile
  float* m_s = f_s + MH;                                                               // [MH] final maximum, then sum
  float* l_s = m_s + MH;
  const uint32_t bars = smem_u32(l_s + MH);
  __shared__ int abort_s, drain_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sp = blockIdx.x, h0 = blockIdx.y * MH, s = blockIdx.z;
  const int heads = min(MH, p.H - h0);
  const int ctx = p.ctx[s];
  const int lo = p.window > 0 ? max(0, ctx - p.window) : 0;
  const int per = ((ctx - lo + p.splits - 1) / p.splits + kLdKeys - 1) / kLdKeys * kLdKeys;
  const int t0 = lo + sp * per, t1 = min(ctx, t0 + per);
  if (t0 >= t1) {                                // nothing left for this split
    if (threadIdx.x < heads) {
      float* st = p.stat + (((long long)s * p.H + h0 + threadIdx.x) * p.splits + sp) * 2;
      st[0] = -INFINITY;
      st[1] = 0.f;
    }
    return;
  }
  const int tiles = (t1 - t0 + kLdKeys - 1) / kLdKeys;
  const int* bt = p.tables + (long long)s * p.max_blocks;
  if (threadIdx.x == 0) {
    abort_s = 0; drain_s = 0;
    for (int i = 0; i < p.stages; ++i) mbar_init(bars + 8u * i, 1);
    fence_barrier_init();
    fence_proxy_async();
  }
  {
    const int units = p.w / 8;
    const __nv_bfloat16* q = p.q + ((long long)s * p.H + h0) * p.w;
    for (int i = threadIdx.x; i < MH * units; i += kLdThreads) {
      const int h = i / units, u = i - h * units;
      *reinterpret_cast<uint4*>(q_s + h * pitch + u * 16) =
          h < heads ? *reinterpret_cast<const uint4*>(q + (long long)h * p.w + u * 8) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  __syncthreads();
  volatile int* abort_flag = &abort_s;
  // the rows of tile i into its stage, two per lane of warp 0; past the last key that key's row again (its weight is zero)
  auto request = [&](int i) {
    const uint32_t bar = bars + 8u * (i % p.stages);
    if (lane == 0) mbar_expect_tx(bar, uint32_t(kLdKeys * p.w * 2));
    __syncwarp();
    const uint32_t dst = smem_u32(ld_smem) + (i % p.stages) * tile_bytes;
#pragma unroll
    for (int k = 0; k < kLdKeys / 32; ++k) {
      const int r = k * 32 + lane, pos = min(t0 + i * kLdKeys + r, t1 - 1);
      const long long src = (long long)bt[pos / p.block_size] * p.block_size + pos % p.block_size;
      ld_bulk(dst + r * pitch, p.cache + src * p.w, uint32_t(p.w * 2), bar);
    }
  };
  if (warp == 0)
    for (int i = 0; i < p.stages - 1 && i < tiles; ++i) request(i);

  const int nch = p.c / 64;                      // 8-column blocks per warp in the value product (up to 8)
  float o[MT][8][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int r = 0; r < 4; ++r) o[m][n][r] = 0.f;
  const int g = lane >> 2, qd = lane & 3;
  const int my_head = threadIdx.x / TPH, sub = threadIdx.x % TPH;
  float m_run = -INFINITY, l_run = 0.f;
  const int kg = warp & 3, half = warp >> 2, ksteps = p.w / 32;       // per half
  const uint32_t q_addr = smem_u32(q_s) + (lane & 15) * pitch + (lane >> 4) * 16 + half * (p.w / 2) * 2;
  bool ok = true;

  for (int i = 0; i < tiles; ++i) {
    if (warp == 0 && i + p.stages - 1 < tiles) request(i + p.stages - 1);      // its stage was read in iteration i - 1
    const uint32_t tile = smem_u32(ld_smem) + (i % p.stages) * tile_bytes;
    const bool got = mbar_wait(bars + 8u * (i % p.stages), uint32_t(i / p.stages) & 1u, abort_flag, p.status, kStatusTimeoutFull);
    if (got) {
      float sc[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int r = 0; r < 4; ++r) sc[m][n][r] = 0.f;
      const uint32_t k_addr = tile + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 16 + half * (p.w / 2) * 2;
#pragma unroll 4
      for (int ks = 0; ks < ksteps; ++ks) {
        uint32_t b[4];
        ld_ldsm_x4(k_addr + ks * 32, b);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          ld_ldsm_x4(q_addr + m * 16 * pitch + ks * 32, a);
          ld_mma(sc[m][0], a, b[0], b[1]);
          ld_mma(sc[m][1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* dst = s_s + (half * MH + m * 16 + g) * kLdSPitch + kg * 16 + n * 8 + qd * 2;
          *reinterpret_cast<float2*>(dst) = make_float2(sc[m][n][0], sc[m][n][1]);
          *reinterpret_cast<float2*>(dst + 8 * kLdSPitch) = make_float2(sc[m][n][2], sc[m][n][3]);
        }
    }
    __syncthreads();
    if (*abort_flag) { ok = false; break; }      // the same for all: the flag is written before the barrier or not at all
    {
      const float* s0 = s_s + my_head * kLdSPitch + sub * KPT;
      const float* s1 = s0 + MH * kLdSPitch;
      const int live = t1 - t0 - i * kLdKeys - sub * KPT;            // keys of this thread that exist
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < KPT; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(s0 + k), b = *reinterpret_cast<const float4*>(s1 + k);
        v[k] = (a.x + b.x) * p.scale_log2; v[k + 1] = (a.y + b.y) * p.scale_log2;
        v[k + 2] = (a.z + b.z) * p.scale_log2; v[k + 3] = (a.w + b.w) * p.scale_log2;
      }
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        if (k >= live) v[k] = -INFINITY;
        mx = fmaxf(mx, v[k]);
      }
#pragma unroll
      for (int d = 1; d < TPH; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float m_new = fmaxf(m_run, mx);      // finite: every tile has a key
      const float f = exp2f(m_run - m_new);
      float sum = 0.f;
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = exp2f(v[k] - m_new);
        sum += v[k];
      }
#pragma unroll
      for (int d = 1; d < TPH; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      l_run = l_run * f + sum;
      m_run = m_new;
      __nv_bfloat16* dst = p_s + my_head * kLdPPitch + sub * KPT;
#pragma unroll
      for (int k = 0; k < KPT; k += 4) stf4(dst + k, make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]));
      if (sub == 0) f_s[my_head] = f;
    }
    __syncthreads();
    {
      float f[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m) { f[m][0] = f_s[m * 16 + g]; f[m][1] = f_s[m * 16 + g + 8]; }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          o[m][n][0] *= f[m][0]; o[m][n][1] *= f[m][0];
          o[m][n][2] *= f[m][1]; o[m][n][3] *= f[m][1];
        }
      const uint32_t p_addr = smem_u32(p_s) + (lane & 15) * (kLdPPitch * 2) + (lane >> 4) * 16;
      const uint32_t v_addr = tile + lane * pitch + warp * nch * 16;
#pragma unroll
      for (int kh = 0; kh < 2; ++kh) {           // 32 keys
        uint32_t a[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int k = 0; k < 2; ++k) ld_ldsm_x4(p_addr + m * 16 * (kLdPPitch * 2) + (kh * 2 + k) * 32, a[m][k]);
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          if (n < nch) {
            uint32_t b[4];
            ld_ldsm_x4_trans(v_addr + kh * 32 * pitch + n * 16, b);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              ld_mma(o[m][n], a[m][0], b[0], b[1]);
              ld_mma(o[m][n], a[m][1], b[2], b[3]);
            }
          }
        }
      }
    }
    __syncthreads();                             // the stage, the scores and the weights may be written again
  }
  if (!ok) {
    // a copy never arrived: the other requested stages get one more bounded wait each before the CTA leaves
    if (warp == 0)
      for (int st = 0; st < p.stages; ++st) {
        mbar_wait(bars + 8u * st, 0u, &drain_s, p.status, kStatusTimeoutFull);
        mbar_wait(bars + 8u * st, 1u, &drain_s, p.status, kStatusTimeoutFull);
      }
    return;
  }
  if (sub == 0) { m_s[my_head] = m_run; l_s[my_head] = l_run; }
  __syncthreads();
  if (p.splits > 1 && threadIdx.x < heads) {
    float* st = p.stat + (((long long)s * p.H + h0 + threadIdx.x) * p.splits + sp) * 2;
    st[0] = m_s[threadIdx.x];
    st[1] = l_s[threadIdx.x];
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = m * 16 + e * 8 + g;
      if (h >= heads) continue;
      const long long row = (long long)s * p.H + h0 + h;
      const float inv = 1.f / l_s[h];
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        if (n < nch) {
          const int col = (warp * nch + n) * 8 + qd * 2;
          const float2 v = make_float2(o[m][n][e * 2], o[m][n][e * 2 + 1]);
          if (p.splits > 1) stf2(p.part + (row * p.splits + sp) * p.c + col, v);
          else stf2(p.out + row * p.c + col, make_float2(v.x * inv, v.y * inv));
        }
      }
    }
}

// out[row, :] from the splits of one (sequence, head).
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part, const float* __restrict__ stat,
                                                           __nv_bfloat16* __restrict__ out, int splits, int c) {
  const long long row = blockIdx.x;
  const float2* st = reinterpret_cast<const float2*>(stat) + row * splits;
  float m = -INFINITY, l = 0.f;
  for (int i = 0; i < splits; ++i) m = fmaxf(m, st[i].x);
  for (int i = 0; i < splits; ++i) l += st[i].y > 0.f ? st[i].y * exp2f(st[i].x - m) : 0.f;
  const float inv = 1.f / l;
  for (int col = threadIdx.x * 4; col < c; col += 128 * 4) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < splits; ++i) {
      if (st[i].y > 0.f) {                       // a split without keys has written no outputs
        const float f = exp2f(st[i].x - m);
        const float4 v = ldf4(part + (row * splits + i) * c + col);
        a.x = fmaf(f, v.x, a.x); a.y = fmaf(f, v.y, a.y); a.z = fmaf(f, v.z, a.z); a.w = fmaf(f, v.w, a.w);
      }
    }
    stf4(out + row * c + col, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv));
  }
}

template <int MT>
static int launch_latent_decode(LatentDecodeParams& p, int S, cudaStream_t st) {
  constexpr int MH = MT * 16;
  p.stages = kLdMaxStages;
  while (p.stages > 2 && ld_smem_bytes(p.w, MH, p.stages) > 227 * 1024) --p.stages;
  const int smem = ld_smem_bytes(p.w, MH, p.stages);
  if (smem > 227 * 1024) return -4;
  auto kern = latent_decode_kernel<MT>;
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(p.splits, (p.H + MH - 1) / MH, S), kLdThreads, smem, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // namespace lt

extern "C" {

// proj [n, ld]: rotates columns d .. d + rot of each of H heads of d + r columns (in place, or into q_out [n, H, q_ld] at column
// q_col, the padding up to r as zeros); with c_off >= 0 also norms the latent at c_off (rank columns) and rotates the key part
// behind it, and writes both, padded to c and r columns, to row slots[n] of the cache (and row n of lin).
int lt_latent_rope(int fp32, void* proj, long long ld, int n, int H, int d, int r, int rot, int c_off, int rank, int c,
                   const float* c_norm, float eps, const int* positions, const int* slots, const double* freq, float gain, void* q_out,
                   int q_ld, int q_col, void* cache, void* lin, void* stream) {
  using namespace lt;
  if (n == 0) return 0;
  if (H < 1 || rot > r || (rot & 1) || rot > 2 * kRopeMaxPairs || ((d | r | c | q_ld | q_col) & 1) || (ld & 1) ||
      (c_off >= 0 && (rank > c || rank < 1 || !c_norm || !cache || !slots)))
    return -4;
  RopeParams p{proj, ld, H, d, r, rot, c_off, rank, c, c_norm, eps, positions, slots, freq, gain, q_out, q_ld, q_col, cache, lin};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (fp32) latent_rope_kernel<float><<<n, kRopeThreads, rot * 4, st>>>(p);
  else latent_rope_kernel<__nv_bfloat16><<<n, kRopeThreads, rot * 4, st>>>(p);
  LT_LAUNCH_CHECK();
  return 0;
}

// out [S, H, c] = attention of q [S, H, w] over the rows of each sequence's pages (the newest `window`, 0: all); c and w multiples
// of 64, c <= 512.  part [S * H, splits, c] and stat [S * H, splits, 2] are scratch (unused with one split).
int lt_latent_decode(const void* q, const void* cache, const int* tables, const int* ctx, float* part, float* stat, void* out, int S,
                     int H, int c, int w, int block_size, int max_blocks, int splits, int window, float scale, void* stream) {
  using namespace lt;
  if (S == 0) return 0;
  if (H < 1 || c < 64 || c > 512 || (c & 63) || (w & 63) || w < c || w > 1024 || splits < 1 || splits > 65535 || S > 65535 ||
      (splits > 1 && (!part || !stat)) || (reinterpret_cast<uintptr_t>(cache) & 15) || (reinterpret_cast<uintptr_t>(q) & 15))
    return -4;
  LatentDecodeParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(cache), tables, ctx, part, stat,
                       static_cast<__nv_bfloat16*>(out), H, c, w, block_size, max_blocks, splits, window, 0,
                       scale * 1.4426950408889634f, device_status_word()};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rc = H <= 16 ? launch_latent_decode<1>(p, S, st) : launch_latent_decode<2>(p, S, st);
  if (rc != 0 || splits == 1) return rc;
  latent_merge_kernel<<<S * H, 128, 0, st>>>(part, stat, static_cast<__nv_bfloat16*>(out), splits, c);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
