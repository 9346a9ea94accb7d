// Attention of absorbed queries over a paged pool of latents (include/tlaloc_b200.h, tlaloc_b200_latent_attention).
//
// LatentAttentionGeneric: any sizes, f32 or bf16, plain FMA.  A CTA serves one (row, head): tiles of 128 positions, a warp
// per position for the scores (lanes over the channels), an online softmax in f32, then a thread per latent channel.
//
// LatentAttentionTc (bf16, pages of a multiple of 64 positions): all heads share a position's row, so a CTA takes 16 to 64 heads of one
// row of the batch and a slice of its positions, and the cached row leaves HBM once for all of them.  Tiles of 64 positions arrive as boxes of a
// tensor map over the pool (atoms of 64 positions x 64 channels, 128-byte swizzle) in a ring of two to four stages.
//   producer lane   boxes of the tiles, and an L2 prefetch two tiles ahead of them: the ring is full of tiles at work, so the way from
//                   HBM is hidden in front of it
//   MMA lane        scores: tcgen05.mma with the query as A out of TMEM (heads are its lanes, put there once) and the tile as B,
//                   into one of two accumulators of 64 columns
//   2 - 4 warps     softmax: two threads own a head's row of 64 scores and exchange its maximum; the weights go to shared memory as
//                   bf16.  The running maximum is raised lazily (the exponentials stay below 2^8), so the values' accumulators are rarely rescaled
//   sixteen warps   values: mma.sync m16n8k16 over the tile as it lies, the latent channels split over the warps, accumulators
//                   in registers (a TMEM accumulator of 512 channels would leave no room for the query)
// Each of the four works on a tile of its own.  Slices leave {max, sum, acc[kv_rank]} records in f32 that LatentCombine merges in slice
// order.  Every mbarrier wait is bounded.
#include <cuda.h>

#include <algorithm>

#include "common.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

struct LatentParams {
  const void* query;
  const void* pool;
  const int* tables;
  const int* row_tables;
  const int* seq_lens;
  void* out;
  int64_t pool_ld;
  int T, H, kv_rank, row, num_blocks, block_size, block_shift, max_blocks, num_tables, window;  // block_shift: log2 of block_size, or -1
  float scale;
};

constexpr int kGenericThreads = 128, kGenericTile = 128, kGenericChannels = 16;  // up to 16 * 128 latent channels

// The live positions of a row: [first, end).
__device__ __forceinline__ int2 LiveRange(const LatentParams& p, int t)
{
  const int end = min(max(__ldg(p.seq_lens + t), 0), p.max_blocks * p.block_size);
  return make_int2(p.window > 0 ? max(0, end - p.window) : 0, end);
}
__device__ __forceinline__ const int* TableOf(const LatentParams& p, int t)
{
  const int r = p.row_tables != nullptr ? __ldg(p.row_tables + t) : t;
  return p.tables + static_cast<size_t>(min(max(r, 0), p.num_tables - 1)) * p.max_blocks;
}
__device__ __forceinline__ size_t PoolRow(const LatentParams& p, const int* table, int pos)
{
  const int block = p.block_shift >= 0 ? pos >> p.block_shift : pos / p.block_size;
  const int page = min(max(__ldg(table + block), 0), p.num_blocks - 1);
  return (static_cast<size_t>(page) * p.block_size + (pos - block * p.block_size)) * p.pool_ld;
}

template <typename T>
__global__ void __launch_bounds__(kGenericThreads) LatentAttentionGeneric(LatentParams p)
{
  GridDependencySync();
  extern __shared__ float s_q[];  // the scaled query
  __shared__ float s_w[kGenericTile];
  __shared__ size_t s_row[kGenericTile];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const T* q = static_cast<const T*>(p.query) + (static_cast<size_t>(t) * p.H + h) * p.row;
  const T* pool = static_cast<const T*>(p.pool);
  const int* table = TableOf(p, t);
  const int2 live = LiveRange(p, t);
  for (int j = tid; j < p.row; j += kGenericThreads) s_q[j] = ToF32(q[j]);
  float acc[kGenericChannels];
#pragma unroll
  for (int i = 0; i < kGenericChannels; ++i) acc[i] = 0.f;
  float top = -INFINITY, sum = 0.f;
  for (int c0 = live.x; c0 < live.y; c0 += kGenericTile) {
    const int n = min(kGenericTile, live.y - c0);
    __syncthreads();
    if (tid < n) s_row[tid] = PoolRow(p, table, c0 + tid);
    __syncthreads();
    for (int i = warp; i < n; i += kGenericThreads / 32) {
      const T* k = pool + s_row[i];
      float d = 0.f;
      for (int j = lane; j < p.row; j += 32) d = fmaf(s_q[j], ToF32(k[j]), d);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
      if (lane == 0) s_w[i] = d * p.scale;
    }
    __syncthreads();
    float tile_top = -INFINITY;
    for (int i = 0; i < n; ++i) tile_top = fmaxf(tile_top, s_w[i]);
    const float new_top = fmaxf(top, tile_top), keep = expf(top - new_top);
    __syncthreads();
    if (tid < n) s_w[tid] = expf(s_w[tid] - new_top);
    __syncthreads();
    top = new_top;
    sum *= keep;
    for (int i = 0; i < n; ++i) sum += s_w[i];
#pragma unroll
    for (int c = 0; c < kGenericChannels; ++c) {
      const int j = tid + c * kGenericThreads;
      if (j >= p.kv_rank) break;
      float a = acc[c] * keep;
      for (int i = 0; i < n; ++i) a = fmaf(s_w[i], ToF32(pool[s_row[i] + j]), a);
      acc[c] = a;
    }
  }
  T* out = static_cast<T*>(p.out) + (static_cast<size_t>(t) * p.H + h) * p.kv_rank;
  const float inv = sum > 0.f ? 1.f / sum : 0.f;
#pragma unroll
  for (int c = 0; c < kGenericChannels; ++c) {
    const int j = tid + c * kGenericThreads;
    if (j >= p.kv_rank) break;
    out[j] = FromF32<T>(acc[c] * inv);
  }
}

// ---- the tensor-core form ---------------------------------------------------------------------------------------------
using namespace tc;

constexpr int kAtomBytes = 64 * 128;
constexpr int kMmaTile = 64, kValueWarps = 16, kProducerWarp = 18, kMmaWarp = 19;
// Warps 16, 17 and 20, 21 are the softmax: a warp reads the TMEM lanes of its number modulo 4, so both of a pair see the same heads.
constexpr int kMmaThreads = 22 * 32;
constexpr int kPStride = kMmaTile + 8, kMaxStages = 4;

__device__ __forceinline__ void LdMatrixX4(uint32_t (&r)[4], uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void LdMatrixX4Trans(uint32_t (&r)[4], uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
// Not volatile: the next fragments' loads may move ahead of it.
__device__ __forceinline__ void MmaBf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float Exp2(float x)
{
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t Pack(float a, float b)
{
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

struct SliceParams {
  float* records;  // [slices][T][H][kv_rank + 2], or null: one slice, straight to out
  int slices, slice_tiles, atoms, stages;  // atoms: 64-channel atoms of a tile
};

__device__ int g_latent_status = 0;  // nonzero after a wait timed out (sticky until read)

// A 16-byte word of a tile: 128-byte rows, the words of a row permuted by the row's place in its group of eight.
__device__ __forceinline__ uint32_t TileWord(int position, int word)
{
  return (word >> 3) * kAtomBytes + position * 128 + (((word & 7) ^ (position & 7)) << 4);
}
constexpr float kLazy = 8.f;  // how far (log2) a head's maximum may grow past the reference in use

// MT: 16-head tiles of the CTA; NP: 16-channel pairs of values per warp.
template <int MT, int NP>
__global__ void __launch_bounds__(kMmaThreads, 1)
    LatentAttentionTc(const __grid_constant__ CUtensorMap map, const __grid_constant__ LatentParams p, const __grid_constant__ SliceParams sp)
{
  constexpr int HT = MT * 16;
  GridDependencySync();
  extern __shared__ unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[2 * kMaxStages + 5];
  __shared__ uint32_t slot_store[2];
  __shared__ float s_keep[2][HT], s_row[2][2][(HT + 31) / 32 * 32];  // s_row: [tile parity][half of the positions][head]
  __shared__ alignas(16) __nv_bfloat16 s_p[2][HT * kPStride];
  const uint32_t base = (SmemAddr(smem_raw) + 1023u) & ~1023u;  // the swizzle is a function of address bits 4..9
  unsigned char* smem = smem_raw + (base - SmemAddr(smem_raw));
  const int tile_bytes = sp.atoms * kAtomBytes, stages = sp.stages;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t = blockIdx.z, h0 = blockIdx.y * HT, slice = blockIdx.x;
  const int2 live = LiveRange(p, t);
  const int tile0 = live.x / kMmaTile + slice * sp.slice_tiles;
  const int n = min((live.y + kMmaTile - 1) / kMmaTile, tile0 + sp.slice_tiles) - tile0;  // tiles of this CTA
  if (n <= 0) {  // an empty slice writes nothing; an empty row writes zeros
    if (slice == 0 && sp.records == nullptr) {
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (static_cast<size_t>(t) * p.H + h0) * p.kv_rank;
      for (int i = tid; i < min(HT, p.H - h0) * p.kv_rank; i += kMmaThreads) out[i] = __float2bfloat16_rn(0.f);
    }
    return;
  }
  const uint32_t full = SmemAddr(bars), free0 = full + 8 * kMaxStages, sfull = free0 + 8 * kMaxStages, sempty = sfull + 16;
  const uint32_t qready = sempty + 16;
  // The weights change hands at named barriers (4, 5: there; 6, 7: read), where a waiting warp costs no issue slots: sixteen warps
  // polling an mbarrier slowed the softmax down.  Trip counts are fixed, so every arrival has its wait.
  constexpr int kHandOver = (kValueWarps + 2 * ((HT + 31) / 32)) * 32;
  volatile uint32_t* abort_word = slot_store + 1;
  if (tid == 0) {
    slot_store[1] = 0u;
    for (int i = 0; i < kMaxStages; ++i) {
      MbarInit(full + 8 * i, 1);
      MbarInit(free0 + 8 * i, kValueWarps);
    }
    for (int i = 0; i < 2; ++i) {
      MbarInit(sfull + 8 * i, 1);
      MbarInit(sempty + 8 * i, 2 * ((HT + 31) / 32));
    }
    MbarInit(qready, kValueWarps);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(SmemAddr(slot_store)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *static_cast<volatile uint32_t*>(slot_store), tmem_q = tmem + 2 * kMmaTile;  // two score accumulators, then the query
  bool ok = true;

  if (warp == kProducerWarp) {
    if (ElectOne()) {
      const int* table = TableOf(p, t);
      int stage = 0;
      uint32_t phase = 1;  // a fresh barrier passes a wait for the phase before its first
      auto pool_row = [&](int j) {
        const int pos = (tile0 + j) * kMmaTile, block = pos >> p.block_shift;  // the tile's 64 rows lie in one page
        return min(max(__ldg(table + block), 0), p.num_blocks - 1) * p.block_size + (pos - (block << p.block_shift));
      };
      int row = pool_row(0), row1 = n > 1 ? pool_row(1) : 0, row2 = n > 2 ? pool_row(2) : 0;
      for (int j = 0; j < n; ++j) {
        const int row3 = j + 3 < n ? pool_row(j + 3) : 0;
        if (j + 2 < n && j + 2 >= stages) {
          for (int c = 0; c < sp.atoms; ++c) {
            asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global [%0, {%1, %2}];\n" ::"l"(reinterpret_cast<uint64_t>(&map)), "r"(c * 64), "r"(row2) : "memory");
          }
        }
        const uint32_t bar = full + 8 * stage, dst = base + stage * tile_bytes;
        ok = MbarWait(free0 + 8 * stage, phase, abort_word) && ok;
        MbarExpectTx(bar, tile_bytes);
        for (int c = 0; c < sp.atoms; ++c) {  // x = 64 c elements: a multiple of 128 bytes
          asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n" ::"r"(dst + c * kAtomBytes),
                       "l"(reinterpret_cast<uint64_t>(&map)), "r"(c * 64), "r"(row), "r"(bar)
                       : "memory");
        }
        row = row1;
        row1 = row2;
        row2 = row3;
        if (++stage == stages) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (!ok) {  // given up: let the copies in flight land before the CTA's shared memory goes away
        volatile uint32_t never = 0;
        for (int s = 0; s < stages; ++s)
          if (n > s) MbarWait(full + 8 * s, ((n - 1 - s) / stages) & 1, &never);
      }
    }
    __syncwarp();
  } else if (warp == kMmaWarp) {
    if (ElectOne()) {
      // f32 accumulator, bf16, both K-major, M = 128 (the lanes past the heads hold zeros), N = 64
      constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kMmaTile >> 3) << 17) | (8u << 24);
      const uint64_t d0 = SmemDesc(base, 16, 1024);
      const int steps = (p.row + 15) >> 4;
      ok = MbarWait(qready, 0, abort_word) && ok;
      int stage = 0;
      uint32_t phase = 0;
      for (int j = 0; j < n; ++j) {
        const uint32_t b = j & 1, acc = tmem + b * kMmaTile;
        ok = MbarWait(full + 8 * stage, phase, abort_word) && ok;
        ok = MbarWait(sempty + 8 * b, ((j >> 1) & 1) ^ 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint64_t d = d0 + static_cast<uint64_t>((stage * tile_bytes) >> 4);
        uint32_t q = tmem_q;
        for (int c = 0; c < sp.atoms; ++c, d += kAtomBytes >> 4, q += 32) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (4 * c + k < steps) TcMmaTmemA(acc, q + 8 * k, d + 2 * k, idesc, c > 0 || k > 0 ? 1u : 0u);
        }
        TcCommit(sfull + 8 * b);
        if (++stage == stages) {
          stage = 0;
          phase ^= 1;
        }
      }
    }
    __syncwarp();
  } else if (warp >= kValueWarps) {  // softmax
    const int quad = warp & 3, half = warp >= kMmaWarp ? 1 : 0, head = quad * 32 + lane;  // TMEM lane; positions [32 half, 32 half + 32)
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    constexpr int kHalf = kMmaTile / 2;
    // The other half of the row: the two warps of a quad meet at a named barrier of 64 threads.
    auto other = [&](int b, float mine) {
      s_row[b][half][head] = mine;
      asm volatile("bar.sync %0, 64;\n" ::"r"(2 + quad) : "memory");
      return s_row[b][half ^ 1][head];
    };
    if (quad * 32 < HT) {
      const float scale = p.scale * 1.4426950408889634f;
      float top = -INFINITY, sum = 0.f;
      for (int j = 0; j < n; ++j) {
        const int b = j & 1, tile_pos = (tile0 + j) * kMmaTile, pos = tile_pos + half * kHalf;
        ok = MbarWaitWarp(sfull + 8 * b, (j >> 1) & 1, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint32_t s[kHalf];
        TcLd32(tmem + lanes + b * kMmaTile + half * kHalf, s);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(sempty + 8 * b);
        float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        const bool edge = tile_pos < live.x || tile_pos + kMmaTile > live.y;
#pragma unroll
        for (int e = 0; e < kHalf; ++e) {
          float v = __uint_as_float(s[e]) * scale;
          if (edge && (pos + e < live.x || pos + e >= live.y)) v = -INFINITY;
          s[e] = __float_as_uint(v);
          t4[e & 3] = fmaxf(t4[e & 3], v);
        }
        const float mine = fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3]));
        const float tile_top = fmaxf(mine, other(b, mine));  // finite: a tile holds at least one live position
        float keep = 1.f;
        if (tile_top > top + kLazy || top == -INFINITY) {
          const float next = fmaxf(top, tile_top);
          keep = Exp2(top - next);
          sum *= keep;
          top = next;
        }
        float add[2] = {0.f, 0.f};
#pragma unroll
        for (int e = 0; e < kHalf; e += 2) {
          const float p0 = Exp2(__uint_as_float(s[e]) - top), p1 = Exp2(__uint_as_float(s[e + 1]) - top);
          add[0] += p0;
          add[1] += p1;
          s[e / 2] = Pack(p0, p1);
        }
        sum += add[0] + add[1];
        const float total = j == n - 1 ? sum + other(b ^ 1, sum) : 0.f;
        if (j >= 2) asm volatile("bar.sync %0, %1;\n" ::"r"(6 + b), "n"(kHandOver) : "memory");
        if (head < HT) {
          uint4* dst = reinterpret_cast<uint4*>(s_p[b] + head * kPStride + half * kHalf);
#pragma unroll
          for (int c = 0; c < 4; ++c) dst[c] = make_uint4(s[4 * c], s[4 * c + 1], s[4 * c + 2], s[4 * c + 3]);
          if (half == 0) {
            s_keep[b][head] = keep;
            if (j == n - 1) {
              s_row[b][0][head] = total;  // both maxima of this tile have been read
              if (sp.records != nullptr && h0 + head < p.H) {
                float* rec = sp.records + ((static_cast<size_t>(slice) * p.T + t) * p.H + h0 + head) * (p.kv_rank + 2);
                rec[0] = top;
                rec[1] = total;
              }
            }
          }
        }
        asm volatile("bar.arrive %0, %1;\n" ::"r"(4 + b), "n"(kHandOver) : "memory");
      }
    }
  } else {
    {  // the query into TMEM, zeros in the lanes past the heads: a warp takes the lanes of its quadrant and every fourth atom
      const int quad = warp & 3, head = quad * 32 + lane;
      const bool there = head < HT && h0 + head < p.H;
      const uint4* q = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.query) + (static_cast<size_t>(t) * p.H + h0 + head) * p.row);
      const int words = p.row >> 3;
      for (int c = warp >> 2; c < sp.atoms; c += kValueWarps / 4) {
        uint32_t w[32];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const uint4 v = there && c * 8 + e < words ? __ldg(q + c * 8 + e) : make_uint4(0, 0, 0, 0);
          w[4 * e] = v.x; w[4 * e + 1] = v.y; w[4 * e + 2] = v.z; w[4 * e + 3] = v.w;
        }
        TcSt32(tmem_q + (static_cast<uint32_t>(quad * 32) << 16) + c * 32, w);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
      __syncwarp();
      if (lane == 0) MbarArrive(qready);
    }
    const int gid = lane >> 2, tig = lane & 3;
    const int pairs = (p.kv_rank + 15) >> 4;
    float acc[MT][2 * NP][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int c = 0; c < 2 * NP; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[m][c][e] = 0.f;
    int stage = 0;
    uint32_t phase = 0;
    for (int j = 0; j < n; ++j) {
      const int b = j & 1, pos = (tile0 + j) * kMmaTile;
      asm volatile("bar.sync %0, %1;\n" ::"r"(4 + b), "n"(kHandOver) : "memory");
      if (lane == 0) ok = MbarWait(full + 8 * stage, phase, abort_word) && ok;  // the scores are there, so the tile is
      __syncwarp();
      const uint32_t tile_addr = base + stage * tile_bytes;
      // Rows of the page outside the live range may hold anything: 0 times it must stay 0.
      const int live_lo = live.x - pos, live_hi = live.y - pos;
      if (live_lo > 0 || live_hi < kMmaTile) {
        for (int i = tid; i < kMmaTile * sp.atoms * 8; i += kValueWarps * 32) {
          const int r = i & (kMmaTile - 1);
          if (r < live_lo || r >= live_hi) *reinterpret_cast<uint4*>(smem + stage * tile_bytes + TileWord(r, i / kMmaTile)) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");  // before the stage is fetched into again
        asm volatile("bar.sync 1, %0;\n" ::"n"(kValueWarps * 32) : "memory");
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float k0 = s_keep[b][m * 16 + gid], k1 = s_keep[b][m * 16 + gid + 8];
        if (__any_sync(0xffffffffu, k0 != 1.f || k1 != 1.f)) {
#pragma unroll
          for (int c = 0; c < 2 * NP; ++c) {
            acc[m][c][0] *= k0; acc[m][c][1] *= k0;
            acc[m][c][2] *= k1; acc[m][c][3] *= k1;
          }
        }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t pf[MT][4];  // matrices (heads 0-7, positions 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
#pragma unroll
        for (int m = 0; m < MT; ++m) LdMatrixX4(pf[m], SmemAddr(s_p[b] + (m * 16 + (lane & 15)) * kPStride + k * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int pair = warp + kValueWarps * i;
          if (pair < pairs) {
            uint32_t v[4];  // (positions 0-7, channels 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15), transposed
            LdMatrixX4Trans(v, tile_addr + TileWord(k * 16 + (lane & 15), 2 * pair + (lane >> 4)));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              MmaBf16(acc[m][2 * i], pf[m], v[0], v[1]);
              MmaBf16(acc[m][2 * i + 1], pf[m], v[2], v[3]);
            }
          }
        }
      }
      if (j + 2 < n) asm volatile("bar.arrive %0, %1;\n" ::"r"(6 + b), "n"(kHandOver) : "memory");
      __syncwarp();
      if (lane == 0) MbarArrive(free0 + 8 * stage);
      if (++stage == stages) {
        stage = 0;
        phase ^= 1;
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int hl = m * 16 + gid + half * 8, h = h0 + hl;
        if (h >= p.H) continue;
        const float total = s_row[(n - 1) & 1][0][hl], inv = total > 0.f ? 1.f / total : 0.f;
#pragma unroll
        for (int c2 = 0; c2 < 2 * NP; ++c2) {
          const int c = (warp + kValueWarps * (c2 >> 1)) * 16 + (c2 & 1) * 8 + tig * 2;
          if (c >= p.kv_rank) continue;
          const float x = acc[m][c2][2 * half], y = acc[m][c2][2 * half + 1];
          if (sp.records != nullptr) {
            *reinterpret_cast<float2*>(sp.records + ((static_cast<size_t>(slice) * p.T + t) * p.H + h) * (p.kv_rank + 2) + 2 + c) = make_float2(x, y);
          } else {
            *reinterpret_cast<__nv_bfloat162*>(static_cast<__nv_bfloat16*>(p.out) + (static_cast<size_t>(t) * p.H + h) * p.kv_rank + c) =
                __floats2bfloat162_rn(x * inv, y * inv);
          }
        }
      }
    }
  }
  if (!ok) atomicExch(&g_latent_status, 1);
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  if (warp == 0) {
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512u) : "memory");
  }
}

// Merges the slices of one (row, head): a thread per two latent channels.
__global__ void __launch_bounds__(128) LatentCombine(LatentParams p, SliceParams sp)
{
  GridDependencySync();
  const int h = blockIdx.x, t = blockIdx.y;
  const int2 live = LiveRange(p, t);
  const int tiles = live.y > live.x ? (live.y + kMmaTile - 1) / kMmaTile - live.x / kMmaTile : 0;
  const int n = (tiles + sp.slice_tiles - 1) / sp.slice_tiles;
  const float* rec = sp.records + (static_cast<size_t>(t) * p.H + h) * (p.kv_rank + 2);
  const size_t step = static_cast<size_t>(p.T) * p.H * (p.kv_rank + 2);
  float top = -INFINITY;
  for (int s = 0; s < n; ++s) top = fmaxf(top, rec[s * step]);
  float sum = 0.f;
  for (int s = 0; s < n; ++s) sum += Exp2(rec[s * step] - top) * rec[s * step + 1];
  const float inv = sum > 0.f ? 1.f / sum : 0.f;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (static_cast<size_t>(t) * p.H + h) * p.kv_rank;
  for (int c = threadIdx.x * 2; c < p.kv_rank; c += 256) {
    float a = 0.f, b = 0.f;
    for (int s = 0; s < n; ++s) {
      const float w = Exp2(rec[s * step] - top);
      const float2 v = *reinterpret_cast<const float2*>(rec + s * step + 2 + c);
      a = fmaf(w, v.x, a);
      b = fmaf(w, v.y, b);
    }
    *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(a * inv, b * inv);
  }
}

constexpr int kMmaMaxSmem = 227 * 1024;

int Atoms(int row) { return (row + 63) / 64; }
// Stages beside the static shared memory (weights of up to 64 heads, barriers: under 20 KB).
int Stages(int row) { return std::min(kMaxStages, (kMmaMaxSmem - 1024 - (Atoms(row) > 8 ? 10 : 20) * 1024) / (Atoms(row) * kAtomBytes)); }
size_t MmaSmem(int row) { return 1024 + static_cast<size_t>(Stages(row)) * Atoms(row) * kAtomBytes; }

// 16-head tiles of a CTA: enough for all heads where registers allow (two for latents wider than 256 channels, four up to that),
// else the count that leaves the fewest absent heads.
int HeadTiles(int heads, int kv_rank)
{
  const int most = kv_rank > 256 ? 2 : 4, need = (heads + 15) / 16;
  int best = 1;
  for (int mt = 1; mt <= most; ++mt) {
    const int ctas = (need + mt - 1) / mt, best_ctas = (need + best - 1) / best;
    if (ctas < best_ctas || (ctas == best_ctas && mt * ctas < best * best_ctas)) best = mt;
  }
  return best;
}

bool MmaApplies(int kv_rank, int rot_dim)
{
  const int row = kv_rank + rot_dim;
  return kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank <= 512 && Atoms(row) * 32 + 2 * kMmaTile <= 512 && Stages(row) >= 2;
}

// Slices of the positions: the fewest waves of CTAs times the tiles a CTA walks, for the longest live range a row may have.
int ChooseLatentSlices(int rows, int heads, int kv_rank, int max_live, int* slice_tiles)
{
  const int tiles = (max_live + kMmaTile - 1) / kMmaTile + 1;
  const int mt = HeadTiles(heads, kv_rank);
  const int ctas = rows * ((heads + 16 * mt - 1) / (16 * mt));
  const int slots = 148;  // a CTA's TMEM and shared memory fill its SM
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= std::min(tiles, 32); ++s) {
    const int per = (tiles + s - 1) / s;
    const double waves = std::max(1.0, static_cast<double>(ctas) * s / slots);
    const double cost = (waves <= 4 ? (ctas * s + slots - 1) / slots : waves) * (per + 2.5) + (s > 1 ? 2.0 + 0.2 * s * ctas / slots : 0.0);
    if (cost < best_cost * 0.98) {
      best_cost = cost;
      best = s;
    }
  }
  *slice_tiles = (tiles + best - 1) / best;
  return (tiles + *slice_tiles - 1) / *slice_tiles;
}

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// The pool as rows of `row` bf16 channels, boxes of 64 channels x 64 rows; channels past the row arrive as zeros.
bool EncodePool(CUtensorMap* map, const LatentParams& p)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  if (encode == nullptr || p.block_shift < 6) return false;
  const cuuint64_t dims[2] = {static_cast<cuuint64_t>(p.row), static_cast<cuuint64_t>(p.num_blocks) * p.block_size};
  const cuuint64_t strides[1] = {static_cast<cuuint64_t>(p.pool_ld) * 2};
  const cuuint32_t box[2] = {64, kMmaTile};
  const cuuint32_t elem[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p.pool), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int MT, int NP>
cudaError_t LaunchTc(const CUtensorMap& map, const LatentParams& p, const SliceParams& sp, cudaStream_t st)
{
  const dim3 grid(sp.slices, (p.H + 16 * MT - 1) / (16 * MT), p.T);
  return LaunchChained(LatentAttentionTc<MT, NP>, grid, kMmaThreads, MmaSmem(p.row), st, map, p, sp);
}

#define TLALOC_LATENT_FORMS(X) X(1, 1) X(2, 1) X(3, 1) X(4, 1) X(1, 2) X(2, 2)

cudaError_t PrepareLatentAttention()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
    const int most = static_cast<int>(std::max({MmaSmem(640), MmaSmem(576), MmaSmem(512), MmaSmem(448), MmaSmem(384), MmaSmem(320), MmaSmem(256), MmaSmem(192)}));
#define TLALOC_OPT_IN(MT, NP) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(LatentAttentionTc<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, std::min(most, kMmaMaxSmem - (MT > 2 ? 20 : 10) * 1024));
    TLALOC_LATENT_FORMS(TLALOC_OPT_IN)
#undef TLALOC_OPT_IN
    return e;
  });
}
int ReadLatentStatus()
{
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_latent_status, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_latent_status, &zero, sizeof(int));
  }
  return v;
}
KernelSetup g_setup(PrepareLatentAttention, ReadLatentStatus);

cudaError_t LaunchTcForm(const CUtensorMap& map, const LatentParams& p, const SliceParams& sp, cudaStream_t st)
{
  const int mt = HeadTiles(p.H, p.kv_rank), np = ((p.kv_rank + 15) / 16 + kValueWarps - 1) / kValueWarps;
#define TLALOC_TRY(MT, NP) \
  if (mt == MT && np <= NP) return LaunchTc<MT, NP>(map, p, sp, st);
  TLALOC_LATENT_FORMS(TLALOC_TRY)
#undef TLALOC_TRY
  return cudaErrorInvalidValue;
}

int MaxLive(int max_live, int window, int64_t table_positions)
{
  int64_t live = table_positions;
  if (window > 0 && window < live) live = window;
  if (max_live > 0 && max_live < live) live = max_live;
  return static_cast<int>(live);
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" size_t tlaloc_b200_latent_attention_scratch_bytes(int32_t num_tokens, int32_t num_heads, int32_t kv_rank, int32_t rot_dim,
                                                             int32_t max_live)
{
  if (num_tokens < 1 || num_heads < 1 || max_live < 1 || !MmaApplies(kv_rank, rot_dim)) return 0;
  // fewer rows may take more slices: the largest need over the row counts up to num_tokens
  size_t most = 0;
  for (int rows = 1;; rows = std::min(2 * rows, num_tokens)) {
    int tiles = 0;
    const int s = ChooseLatentSlices(rows, num_heads, kv_rank, max_live, &tiles);
    if (s > 1) most = std::max(most, static_cast<size_t>(s) * std::min(2 * rows, num_tokens) * num_heads * (kv_rank + 2) * sizeof(float));
    if (rows == num_tokens) break;
  }
  return most;
}

extern "C" int tlaloc_b200_latent_attention(const void* query, const void* pool, int64_t pool_ld, int32_t dtype,
                                            const int32_t* block_tables, const int32_t* row_tables, const int32_t* seq_lens, void* out,
                                            void* scratch, size_t scratch_bytes, int32_t num_tokens, int32_t num_heads, int32_t kv_rank,
                                            int32_t rot_dim, int32_t num_blocks, int32_t block_size, int32_t max_blocks,
                                            int32_t num_tables, int32_t window, int32_t max_live, float scale, void* stream)
{
  const char* op = "LATENT_ATTENTION";
  if (!query || !pool || !block_tables || !seq_lens || !out) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (num_tokens < 0 || num_heads < 1 || kv_rank < 1 || rot_dim < 0 || num_blocks < 1 || block_size < 1 || max_blocks < 1 ||
      num_tables < 1 || window < 0 || max_live < 0) {
    return Fail(kInvalid, "%s: bad sizes", op);
  }
  if (pool_ld < static_cast<int64_t>(kv_rank) + rot_dim) return Fail(kInvalid, "%s: a pool row is shorter than kv_rank + rot_dim", op);
  if (!row_tables && num_tables < num_tokens) return Fail(kInvalid, "%s: %d tables for %d rows", op, num_tables, num_tokens);
  if (num_tokens > 65535) return Fail(kInvalid, "%s: at most 65535 rows", op);
  if (kv_rank > kGenericChannels * kGenericThreads || kv_rank + rot_dim > 8192) {
    return Fail(kUnsupported, "%s: kv_rank up to %d", op, kGenericChannels * kGenericThreads);
  }
  if (num_tokens == 0) return kOk;
  LatentParams p;
  p.query = query;
  p.pool = pool;
  p.tables = block_tables;
  p.row_tables = row_tables;
  p.seq_lens = seq_lens;
  p.out = out;
  p.pool_ld = pool_ld;
  p.T = num_tokens;
  p.H = num_heads;
  p.kv_rank = kv_rank;
  p.row = kv_rank + rot_dim;
  p.num_blocks = num_blocks;
  p.block_size = block_size;
  p.block_shift = -1;
  for (int k = 0; k < 31; ++k)
    if (block_size == 1 << k) p.block_shift = k;
  p.max_blocks = max_blocks;
  p.num_tables = num_tables;
  p.window = window;
  p.scale = scale;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  CUtensorMap map;
  if (dtype == TLALOC_B200_BF16 && !OrderFaithful() && MmaApplies(kv_rank, rot_dim) && pool_ld % 8 == 0 && Aligned16(query) && Aligned16(pool) &&
      Aligned16(out) && (scratch == nullptr || Aligned16(scratch)) && EncodePool(&map, p)) {
    cudaError_t e = PrepareLatentAttention();
    if (e != cudaSuccess) return CudaFail("LATENT_ATTENTION set-up", e);
    SliceParams sp;
    const int live = MaxLive(max_live, window, static_cast<int64_t>(max_blocks) * block_size);
    sp.slices = ChooseLatentSlices(num_tokens, num_heads, kv_rank, live, &sp.slice_tiles);
    const size_t need = static_cast<size_t>(sp.slices) * num_tokens * num_heads * (kv_rank + 2) * sizeof(float);
    if (sp.slices > 1 && (scratch == nullptr || scratch_bytes < need)) {
      sp.slices = 1;
      sp.slice_tiles = 0x3fffffff;
    }
    if (sp.slices == 1) sp.slice_tiles = 0x3fffffff;
    sp.records = sp.slices > 1 ? static_cast<float*>(scratch) : nullptr;
    sp.atoms = Atoms(p.row);
    sp.stages = Stages(p.row);
    e = LaunchTcForm(map, p, sp, st);
    if (e == cudaSuccess && sp.slices > 1) e = LaunchChained(LatentCombine, dim3(num_heads, num_tokens), 128, 0, st, p, sp);
    if (e != cudaSuccess) return CudaFail("LATENT_ATTENTION launch", e);
    CountLaunches(sp.slices > 1 ? 2 : 1);
    return kOk;
  }
  const dim3 grid(num_heads, num_tokens);
  const size_t smem = sizeof(float) * static_cast<size_t>(p.row);
  const cudaError_t e = dtype == TLALOC_B200_F32 ? LaunchChained(LatentAttentionGeneric<float>, grid, kGenericThreads, smem, st, p)
                                                 : LaunchChained(LatentAttentionGeneric<__nv_bfloat16>, grid, kGenericThreads, smem, st, p);
  if (e != cudaSuccess) return CudaFail("LATENT_ATTENTION launch", e);
  CountLaunches(1);
  return kOk;
}
