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
#include <cuda.h>
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
// One CTA per (sequence, group of up to 16 MT heads, split of the visible keys): eight warps make scores and weights, eight
// more the values, one tile of 32 rows behind.  Tiles arrive by TMA tensor copies, one per page (issuing a copy costs its warp
// on the order of a hundred cycles, so rows or 64-column panels one by one would bound the kernel): the map sees a row as panels
// of 64 columns, and a copy lands as [panel][row][64 columns] in the 128-byte-swizzled layout, so that ldmatrix meets no bank
// conflicts.  Per tile:
//   scores   warp = 16 keys x a quarter of the c + r columns (mma.sync m16n8k16: heads x keys), the quarters added through
//            shared memory; a warp's part of the query block stays in its registers
//   softmax  256 / (16 MT) threads per head: running maximum and sum in registers, weights as bf16 operands to shared
//   values   warp = an eighth of the c columns: accumulators in registers, rows read transposed from the same tile
// mbarriers hand over tiles (ring of `stages`), weights (two buffers) and both back.  A second kernel merges the splits (measured:
// quicker than merging them as a thread-block cluster through distributed shared memory).
// tcgen05 is not used: with 16 or 32 heads its 128-row tiles would be mostly empty, and 512 value columns of them would fill
// the tensor memory.
constexpr int kLdThreads = 512;
constexpr int kLdRole = 256;                // threads of each half
constexpr int kLdKeys = 32;
constexpr int kLdMaxStages = 6;
constexpr int kLdMaxSplits = 64;
constexpr int kLdMaxKs = 9;                 // 16-column steps of a quarter: w up to 576
constexpr int kLdSPitch = kLdKeys + 8;      // floats
constexpr int kLdPPitch = kLdKeys + 8;      // bf16

struct LatentDecodeParams {
  const __nv_bfloat16* q;        // [S, H, w], w = c + r, a multiple of 64
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
// Barrier of the eight warps that make the scores: true where all of them say so.
__device__ __forceinline__ bool ld_bar_and(bool v) {
  int r;
  asm volatile("{\n.reg .pred p, q;\nsetp.ne.s32 p, %1, 0;\nbar.red.and.pred q, 1, 256, p;\nselp.s32 %0, 1, 0, q;\n}" : "=r"(r) : "r"(int(v)) : "memory");
  return r != 0;
}

// Shared memory of a CTA: slack for alignment, tiles, score quarters, weights, per-head numbers, barriers.
__host__ __device__ inline int ld_smem_bytes(int w, int heads, int stages) {
  return 1024 + stages * kLdKeys * w * 2 + 2 * (4 * heads * kLdSPitch * 4 + heads * kLdPPitch * 2 + heads * 4) + 2 * heads * 4 +
         (2 * kLdMaxStages + 4) * 8;
}

// MT: 16-head blocks of a CTA (1 or 2).  FULL: the largest row (w 576, c 512), whose loops have no conditions, so that loads run
// ahead of the products.
template <int MT, bool FULL>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap, const LatentDecodeParams p) {
  constexpr int MH = MT * 16;
  constexpr int TPH = kLdRole / MH;              // threads per head in the softmax
  constexpr int KPT = kLdKeys / TPH;             // keys of each
  extern __shared__ uint8_t ld_raw[];
  uint8_t* ld_smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ld_raw) + 1023) & ~uintptr_t(1023));
  const int tile_bytes = kLdKeys * p.w * 2;
  float* s_s = reinterpret_cast<float*>(ld_smem + p.stages * tile_bytes);              // [2][4][MH][kLdSPitch]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_s + 2 * 4 * MH * kLdSPitch); // [2][MH][kLdPPitch]
  float* f_s = reinterpret_cast<float*>(p_s + 2 * MH * kLdPPitch);                     // [2][MH] rescale of the tile
  float* m_s = f_s + 2 * MH;                                                           // [MH] final maximum, then sum
  float* l_s = m_s + MH;
  const uint32_t bars = smem_u32(l_s + MH);
  auto full = [&](int st) { return bars + 8u * st; };                                  // the tile has arrived
  auto empty = [&](int st) { return bars + 8u * (kLdMaxStages + st); };                // nobody needs the tile any more
  auto p_full = [&](int b) { return bars + 8u * (2 * kLdMaxStages + b); };             // weights and rescale factors are there
  auto p_free = [&](int b) { return bars + 8u * (2 * kLdMaxStages + 2 + b); };
  __shared__ int abort_s, drain_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sp = blockIdx.x, h0 = blockIdx.y * MH, s = blockIdx.z;
  const int heads = min(MH, p.H - h0);
  const int ctx = p.ctx[s];
  const int lo = p.window > 0 ? max(0, ctx - p.window) : 0;
  const int base = lo & ~(kLdKeys - 1);          // tiles start on multiples of 32 keys, and so on a page or its half, quarter, ..
  const int per = ((ctx - base + p.splits - 1) / p.splits + kLdKeys - 1) / kLdKeys * kLdKeys;
  const int t0 = base + sp * per, t1 = min(ctx, t0 + per);
  const int tiles = t1 > t0 ? (t1 - t0 + kLdKeys - 1) / kLdKeys : 0;      // 0: nothing left for this split
  const int run = min(p.block_size, kLdKeys), run_log = 31 - __clz(run), panels = p.w / 64, run_bytes = run * panels * 128;
  // where 16-byte unit u of row r of a tile lies
  auto unit_at = [&](int r, int u) {
    return (r >> run_log) * run_bytes + ((((u >> 3) << run_log) + (r & (run - 1))) << 7) + (((u & 7) ^ (r & 7)) << 4);
  };
  if (threadIdx.x == 0) {
    abort_s = 0; drain_s = 0;
    for (int i = 0; i < p.stages; ++i) { mbar_init(full(i), 1); mbar_init(empty(i), kLdRole / 32); }
    for (int b = 0; b < 2; ++b) { mbar_init(p_full(b), kLdRole / 32); mbar_init(p_free(b), kLdRole / 32); }
    fence_barrier_init();
    fence_proxy_async();
  }
  __syncthreads();
  volatile int* abort_flag = &abort_s;
  const int g = lane >> 2, qd = lane & 3;
  const int nch = FULL ? 8 : p.c / 64;           // 8-column blocks per warp in the value product (up to 8)
  const int my_head = (threadIdx.x % kLdRole) / TPH, sub = threadIdx.x % TPH;
  float m_run = -INFINITY, l_run = 0.f;
  float o[MT][8][4];
  bool ok = true;

  if (warp < kLdRole / 32) {
    // ------------------------------------------------------------------ scores and weights
    const int kg = warp & 1, quarter = warp >> 1, nks = FULL ? kLdMaxKs : p.w / 64;
    // A fragments of this warp's part of the query block: rows = heads (g and g + 8 of every block), zero past the last
    uint32_t qa[MT][kLdMaxKs][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const bool lo_ok = m * 16 + g < heads, hi_ok = m * 16 + g + 8 < heads;
      const __nv_bfloat16* q0 = p.q + ((long long)s * p.H + h0 + (lo_ok ? m * 16 + g : 0)) * p.w + quarter * (p.w / 4) + qd * 2;
      const __nv_bfloat16* q1 = p.q + ((long long)s * p.H + h0 + (hi_ok ? m * 16 + g + 8 : 0)) * p.w + quarter * (p.w / 4) + qd * 2;
#pragma unroll
      for (int ks = 0; ks < kLdMaxKs; ++ks) {
        const bool in = ks < nks;
        qa[m][ks][0] = in && lo_ok ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16) : 0u;
        qa[m][ks][1] = in && hi_ok ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16) : 0u;
        qa[m][ks][2] = in && lo_ok ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 8) : 0u;
        qa[m][ks][3] = in && hi_ok ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 8) : 0u;
      }
    }
    const int key = kg * 16 + (lane & 7) + ((lane >> 4) << 3), u0 = quarter * (p.w / 32) + ((lane >> 3) & 1);
    const int key_at = unit_at(key, 0) & ~127;
    int st = 0;
    uint32_t phase = 0;
    for (int i = 0; i < tiles; ++i) {
      const int b = i & 1;
      const uint32_t tile = smem_u32(ld_smem) + st * tile_bytes + key_at;
      ok = ok && mbar_wait(full(st), phase, abort_flag, p.status, kStatusTimeoutFull);
      if (++st == p.stages) { st = 0; phase ^= 1u; }
      if (__all_sync(0xffffffffu, ok)) {
        float sc[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int r = 0; r < 4; ++r) sc[m][n][r] = 0.f;
#pragma unroll
        for (int ks = 0; ks < kLdMaxKs; ++ks) {
          if (ks < nks) {
            uint32_t kb[4];
            const int u = u0 + ks * 2;            // 16-byte unit of the row
            ld_ldsm_x4(tile + ((u >> 3) << (run_log + 7)) + (((u & 7) ^ (key & 7)) << 4), kb);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              ld_mma(sc[m][0], qa[m][ks], kb[0], kb[1]);
              ld_mma(sc[m][1], qa[m][ks], kb[2], kb[3]);
            }
          }
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            float* dst = s_s + ((b * 4 + quarter) * MH + m * 16 + g) * kLdSPitch + kg * 16 + n * 8 + qd * 2;
            *reinterpret_cast<float2*>(dst) = make_float2(sc[m][n][0], sc[m][n][1]);
            *reinterpret_cast<float2*>(dst + 8 * kLdSPitch) = make_float2(sc[m][n][2], sc[m][n][3]);
          }
      }
      // the quarters are there; a wait that ran out in one warp ends the loop in all
      if (!ld_bar_and(ok)) { ok = false; break; }
      const float* sr = s_s + (b * 4 * MH + my_head) * kLdSPitch + sub * KPT;
      const int first = t0 + i * kLdKeys + sub * KPT;                // this thread's keys that are visible: in [lo, t1)
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < KPT; ++k) v[k] = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if constexpr (KPT == 4) {
          const float4 a = *reinterpret_cast<const float4*>(sr + j * MH * kLdSPitch);
          v[0] += a.x; v[1] += a.y; v[2] += a.z; v[3] += a.w;
        } else {
          const float2 a = *reinterpret_cast<const float2*>(sr + j * MH * kLdSPitch);
          v[0] += a.x; v[1] += a.y;
        }
      }
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = first + k < t1 && first + k >= lo ? v[k] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[k]);
      }
      // The reference the exponents are taken from moves only when a score passes it by more than 2^8 (and for the first tile).
      const bool over = mx > m_run + 8.f;
      float f = 1.f;
      if (__any_sync(0xffffffffu, over)) {
#pragma unroll
        for (int d = 1; d < TPH; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
        if (mx > m_run + 8.f) {
          f = exp2f(m_run - mx);                 // zero for the first tile
          l_run *= f;
          m_run = mx;
        }
      }
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = exp2f(v[k] - m_run);
        l_run += v[k];                           // this thread's share of the sum
      }
      if (i >= 2) ok = mbar_wait(p_free(b), uint32_t((i >> 1) - 1) & 1u, abort_flag, p.status, kStatusTimeoutEmpty);
      __nv_bfloat16* dst = p_s + (b * MH + my_head) * kLdPPitch + sub * KPT;
      if constexpr (KPT == 4) stf4(dst, make_float4(v[0], v[1], v[2], v[3]));
      else stf2(dst, make_float2(v[0], v[1]));
      if (sub == 0) f_s[b * MH + my_head] = f;
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full(b));
    }
  } else {
    // ------------------------------------------------------------------ values, and the copies (first warp of these)
    const int pw = warp - kLdRole / 32;
    const int* bt = p.tables + (long long)s * p.max_blocks;
    // Lane l brings the l-th run of rows of every tile: the block of the table it lies in, and where in the block.
    int blk = (t0 + lane * run) / p.block_size, in_blk = (t0 + lane * run) % p.block_size, asked = 0, ask_st = 0;
    auto next_row = [&]() {                      // its first row of the next tile in the cache (-1: none), then one tile on
      const int row = lane < kLdKeys >> run_log && t0 + asked * kLdKeys + lane * run < t1 ? bt[blk] * p.block_size + in_blk : -1;
      if (run < kLdKeys) blk += kLdKeys >> run_log;
      else if ((in_blk += kLdKeys) == p.block_size) { in_blk = 0; ++blk; }
      return row;
    };
    auto request = [&](int row) {                // pages are allocated whole: runs come whole
      const int rows = min(kLdKeys, ((t1 - t0 - asked * kLdKeys + run - 1) >> run_log) << run_log);
      if (lane == 0) mbar_expect_tx(full(ask_st), uint32_t(rows * p.w * 2));
      __syncwarp();
      if (row >= 0) tma_load_3d(smem_u32(ld_smem) + ask_st * tile_bytes + lane * run_bytes, &tmap, full(ask_st), 0, row, 0);
      ++asked;
      if (++ask_st == p.stages) ask_st = 0;
    };
    int row = -1;                                // of the next tile to ask for
    if (pw == 0) {
      for (int i = 0; i < p.stages - 1 && i < tiles; ++i) request(next_row());
      row = next_row();
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int r = 0; r < 4; ++r) o[m][n][r] = 0.f;
    const int lane_at = unit_at(lane, 0) & ~127;
    int st = 0, old_st = 0;
    uint32_t phase = 0, old_phase = 0;
    for (int i = 0; i < tiles; ++i) {
      const int b = i & 1;
      if (pw == 0 && asked < tiles) {                          // into the stage of tile i - 1
        if (i > 0) ok = mbar_wait(empty(old_st), old_phase, abort_flag, p.status, kStatusTimeoutEmpty);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        request(row);
        row = next_row();                                      // on its way until the next request
      }
      ok = mbar_wait(full(st), phase, abort_flag, p.status, kStatusTimeoutFull) &&
           mbar_wait(p_full(b), uint32_t(i >> 1) & 1u, abort_flag, p.status, kStatusTimeoutFull);
      if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
      const int tail = t1 - t0 - i * kLdKeys;
      if (tail < kLdKeys) {
        // rows past the last key may hold anything: zeros where this warp reads, so that zero weights do not meet a NaN
        if (lane >= tail)
          for (int n = 0; n < nch; ++n)
            *reinterpret_cast<uint4*>(ld_smem + st * tile_bytes + unit_at(lane, pw * nch + n)) = make_uint4(0u, 0u, 0u, 0u);
        __syncwarp();
      }
      bool same = true;
      float f[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        f[m][0] = f_s[b * MH + m * 16 + g];
        f[m][1] = f_s[b * MH + m * 16 + g + 8];
        same = same && f[m][0] == 1.f && f[m][1] == 1.f;
      }
      if (!__all_sync(0xffffffffu, same)) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 8; ++n) {
            o[m][n][0] *= f[m][0]; o[m][n][1] *= f[m][0];
            o[m][n][2] *= f[m][1]; o[m][n][3] *= f[m][1];
          }
      }
      const uint32_t tile = smem_u32(ld_smem) + st * tile_bytes + lane_at;
      const uint32_t p_addr = smem_u32(p_s) + b * MH * kLdPPitch * 2 + (lane & 15) * (kLdPPitch * 2) + (lane >> 4) * 16;
      uint32_t a[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int k = 0; k < 2; ++k) ld_ldsm_x4(p_addr + m * 16 * (kLdPPitch * 2) + k * 32, a[m][k]);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {           // two column blocks at a time: four products between dependent ones
        if (n < nch) {
          uint32_t vb[2][4];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int u = pw * nch + n + e;
            if (n + e < nch) ld_ldsm_x4_trans(tile + ((u >> 3) << (run_log + 7)) + (((u & 7) ^ (lane & 7)) << 4), vb[e]);
          }
#pragma unroll
          for (int k = 0; k < 2; ++k)
#pragma unroll
            for (int e = 0; e < 2; ++e)
#pragma unroll
              for (int m = 0; m < MT; ++m)
                if (n + e < nch) ld_mma(o[m][n + e], a[m][k], vb[e][2 * k], vb[e][2 * k + 1]);
        }
      }
      __syncwarp();
      if (lane == 0) { mbar_arrive(p_free(b)); mbar_arrive(empty(st)); }
      old_st = st;
      old_phase = phase;
      if (++st == p.stages) { st = 0; phase ^= 1u; }
    }
  }
  if (*abort_flag && warp == 0) {
    // a copy never arrived: the other requested stages get one more bounded wait each before the CTA goes on
    for (int st = 0; st < p.stages; ++st) {
      mbar_wait(full(st), 0u, &drain_s, p.status, kStatusTimeoutFull);
      mbar_wait(full(st), 1u, &drain_s, p.status, kStatusTimeoutFull);
    }
  }
#pragma unroll
  for (int d = 1; d < TPH; d <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, d);
  const bool maker = warp >= kLdRole / 32;       // holds outputs; the others hold maxima and sums
  const int pw = maker ? warp - kLdRole / 32 : 0;
  if (!maker && sub == 0) {
    m_s[my_head] = ok ? m_run : -INFINITY;
    l_s[my_head] = ok ? l_run : 0.f;
  }
  __syncthreads();
  if (p.splits > 1 && threadIdx.x < heads) {
    float* st = p.stat + (((long long)s * p.H + h0 + threadIdx.x) * p.splits + sp) * 2;
    st[0] = m_s[threadIdx.x];
    st[1] = l_s[threadIdx.x];
  }
  if (tiles == 0 || !maker) return;
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
          const int col = (pw * nch + n) * 8 + qd * 2;
          const float2 v = make_float2(o[m][n][e * 2], o[m][n][e * 2 + 1]);
          if (p.splits > 1) stf2(p.part + (row * p.splits + sp) * p.c + col, v);
          else stf2(p.out + row * p.c + col, make_float2(v.x * inv, v.y * inv));
        }
      }
    }
}

// out[row, :] from the splits of one (sequence, head): a thread per four columns, eight splits in flight.
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part, const float* __restrict__ stat,
                                                           __nv_bfloat16* __restrict__ out, int splits, int c) {
  __shared__ float share[kLdMaxSplits];
  const long long row = blockIdx.x;
  const float2* st = reinterpret_cast<const float2*>(stat) + row * splits;
  if (threadIdx.x < 32) {
    float m = -INFINITY, l = 0.f;
    for (int i = threadIdx.x; i < splits; i += 32) m = fmaxf(m, st[i].x);
    m = warp_max(m);
    for (int i = threadIdx.x; i < splits; i += 32) {
      const float2 v = st[i];
      const float f = v.y > 0.f ? exp2f(v.x - m) : 0.f;
      share[i] = f;
      l = fmaf(v.y, f, l);
    }
    l = warp_sum(l);
    for (int i = threadIdx.x; i < splits; i += 32) share[i] /= l;
  }
  __syncthreads();
  for (int col = threadIdx.x * 4; col < c; col += 128 * 4) {
    const float* src = part + row * splits * c + col;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i0 = 0; i0 < splits; i0 += 8) {
      float4 v[8];
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        f[i] = i0 + i < splits ? share[i0 + i] : 0.f;
        if (f[i] > 0.f) v[i] = ldf4(src + (long long)(i0 + i) * c);    // a split without keys has written no outputs
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (f[i] > 0.f) {
          a.x = fmaf(f[i], v[i].x, a.x); a.y = fmaf(f[i], v[i].y, a.y); a.z = fmaf(f[i], v[i].z, a.z); a.w = fmaf(f[i], v[i].w, a.w);
        }
    }
    stf4(out + row * c + col, a);
  }
}

template <int MT, bool FULL>
static int launch_latent_decode(const CUtensorMap& tmap, LatentDecodeParams& p, int S, cudaStream_t st) {
  constexpr int MH = MT * 16;
  p.stages = kLdMaxStages;
  while (p.stages > 2 && ld_smem_bytes(p.w, MH, p.stages) > 227 * 1024) --p.stages;
  const int smem = ld_smem_bytes(p.w, MH, p.stages);
  if (smem > 227 * 1024) return -4;
  auto kern = latent_decode_kernel<MT, FULL>;
  LT_RETURN_IF_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(p.splits, (p.H + MH - 1) / MH, S), kLdThreads, smem, st>>>(tmap, p);
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
// of 64, c <= 512, w <= 576; block_size 8, 16 or a multiple of 32; the cache has num_blocks blocks.  part [S * H, splits, c] and stat [S * H, splits, 2] are scratch (unused with one split).
// splits <= 64.
int lt_latent_decode(const void* q, const void* cache, const int* tables, const int* ctx, float* part, float* stat, void* out, int S,
                     int H, int c, int w, int num_blocks, int block_size, int max_blocks, int splits, int window, float scale, void* stream) {
  using namespace lt;
  if (S == 0) return 0;
  if (H < 1 || c < 64 || c > 512 || (c & 63) || (w & 63) || w < c || w > 64 * kLdMaxKs || splits < 1 || splits > kLdMaxSplits || S > 65535 ||
      (block_size != 8 && block_size != 16 && block_size % 32 != 0) || num_blocks < 1 || (splits > 1 && (!part || !stat)) || (reinterpret_cast<uintptr_t>(cache) & 15) || (reinterpret_cast<uintptr_t>(q) & 15))
    return -4;
  LatentDecodeParams p{static_cast<const __nv_bfloat16*>(q), tables, ctx, part, stat,
                       static_cast<__nv_bfloat16*>(out), H, c, w, block_size, max_blocks, splits, window, 0,
                       scale * 1.4426950408889634f, device_status_word()};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  CUtensorMap tmap;
  const int r = encode_tmap_3d(&tmap, cache, 2, 64, (uint64_t)num_blocks * block_size, w / 64, (uint64_t)w * 2, 128, 64,
                               block_size < kLdKeys ? block_size : kLdKeys, w / 64, 1);
  if (r) return 1000 + r;
  const bool full = c == 512 && w == 64 * kLdMaxKs;
  const int rc = H <= 16 ? (full ? launch_latent_decode<1, true>(tmap, p, S, st) : launch_latent_decode<1, false>(tmap, p, S, st))
                         : (full ? launch_latent_decode<2, true>(tmap, p, S, st) : launch_latent_decode<2, false>(tmap, p, S, st));
  if (rc != 0 || splits == 1) return rc;
  latent_merge_kernel<<<S * H, 128, 0, st>>>(part, stat, static_cast<__nv_bfloat16*>(out), splits, c);
  LT_LAUNCH_CHECK();
  return 0;
}

}  // extern "C"
