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
//   MMA lane        scores S = Q C^T: the query is the A operand out of TMEM (heads are its lanes, put there once), the tile is B;
//                   then O^T += C^T P^T: the same tile, its channels now the M rows (an MN-major A operand, 128 channels at a time), the
//                   weights B, accumulators of 128 channel lanes x heads in TMEM
//   4 - 8 warps     softmax: four threads own a head's row of 64 scores and exchange its maximum; the weights go to shared memory as
//                   bf16.  The running maximum is raised lazily (the exponentials stay below 2^8), so O is rarely rescaled
//   four warps      rescale O when a maximum was raised, blank the dead rows of the edge tiles, and write the result
// Slices leave {max, sum, acc[kv_rank]} records in f32 that LatentCombine merges in slice
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
constexpr int kMmaTile = 64, kMaxStages = 4;
// Warps 0 - 3 write the output; 4, 8, 12, 16 (heads 0 - 31) and 5, 9, 13, 17 (32 - 63) are the softmax: a warp reads the TMEM lanes of
// its number modulo 4.  10, 11, 14, 15 have no work.
constexpr int kOutWarps = 4, kProducerWarp = 6, kMmaWarp = 7, kParts = 4, kMmaThreads = 18 * 32;

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
  int slices, slice_tiles, atoms, stages, score_buffers;  // atoms: 64-channel atoms of a tile
};

__device__ int g_latent_status = 0;  // nonzero after a wait timed out (sticky until read)

// A 16-byte word of a tile: 128-byte rows, the words of a row permuted by the row's place in its group of eight.
__device__ __forceinline__ uint32_t TileWord(int position, int word)
{
  return (word >> 3) * kAtomBytes + position * 128 + (((word & 7) ^ (position & 7)) << 4);
}
constexpr float kLazy = 8.f;  // how far (log2) a head's maximum may grow past the reference in use

// HT: heads of the CTA, a multiple of 16.
template <int HT>
__global__ void __launch_bounds__(kMmaThreads, 1)
    LatentAttentionTc(const __grid_constant__ CUtensorMap map, const __grid_constant__ LatentParams p, const __grid_constant__ SliceParams sp)
{
  constexpr int kQuads = (HT + 31) / 32;   // TMEM lane quadrants with heads in them
  constexpr int kOCols = kQuads * 32;      // columns of one O^T accumulator
  constexpr int kPBytes = HT * 128;        // one tile's weights: [heads][64 positions] bf16, 128-byte swizzle
  constexpr int kHandOver = (kOutWarps + kParts * kQuads) * 32;
  extern __shared__ unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[2 * kMaxStages + 9];
  __shared__ uint32_t slot_store[2];
  __shared__ float s_keep[2][kOCols], s_row[2][kParts][kOCols];  // s_row: [tile parity][quarter of the positions][head]
  const uint32_t base = (SmemAddr(smem_raw) + 1023u) & ~1023u;  // the swizzle is a function of address bits 4..9
  unsigned char* smem = smem_raw + (base - SmemAddr(smem_raw));
  const int tile_bytes = sp.atoms * kAtomBytes, stages = sp.stages;
  const uint32_t ring = base + 2 * kPBytes;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // full: a tile has landed; free: its products are done; sfull, sempty: scores there, read; pready: weights there and O in their
  // scale; odone: O has the tile in it.
  const uint32_t full = SmemAddr(bars), free0 = full + 8 * kMaxStages, sfull = free0 + 8 * kMaxStages, sempty = sfull + 16;
  const uint32_t pready = sempty + 16, odone = pready + 16, qready = odone + 16;
  volatile uint32_t* abort_word = slot_store + 1;
  if (tid == 0) {
    slot_store[1] = 0u;
    for (int i = 0; i < kMaxStages; ++i) {
      MbarInit(full + 8 * i, 1);
      MbarInit(free0 + 8 * i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      MbarInit(sfull + 8 * i, 1);
      MbarInit(sempty + 8 * i, kParts * kQuads);
      MbarInit(pready + 8 * i, kOutWarps);
      MbarInit(odone + 8 * i, 1);
    }
    MbarInit(qready, 12);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(SmemAddr(slot_store)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *static_cast<volatile uint32_t*>(slot_store);
  // Only with its TMEM in hand may the CTA let the next kernel's start (which may want some of it and waits for this one).
  GridDependencySync();
  const int t = blockIdx.z, h0 = blockIdx.y * HT, slice = blockIdx.x;
  const int2 live = LiveRange(p, t);
  const int tile0 = live.x / kMmaTile + slice * sp.slice_tiles;
  const int n = min((live.y + kMmaTile - 1) / kMmaTile, tile0 + sp.slice_tiles) - tile0;  // tiles of this CTA
  if (n <= 0) {  // an empty slice writes nothing; an empty row writes zeros
    if (slice == 0 && sp.records == nullptr) {
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (static_cast<size_t>(t) * p.H + h0) * p.kv_rank;
      for (int i = tid; i < min(HT, p.H - h0) * p.kv_rank; i += kMmaThreads) out[i] = __float2bfloat16_rn(0.f);
    }
    __syncthreads();
    if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512u) : "memory");
    return;
  }
  const int o_tiles = (p.kv_rank + 127) >> 7;
  const uint32_t tmem_q = tmem + sp.score_buffers * kMmaTile, tmem_o = tmem_q + sp.atoms * 32;
  bool ok = true;

  if ((warp & 3) < 2 ? warp < 18 : warp < kOutWarps) {
    // The query into TMEM, zeros in the lanes past the heads; the warps of a quadrant share its atoms.
    const int quad = warp & 3, head = quad * 32 + lane;
    const bool there = head < HT && h0 + head < p.H;
    const uint4* q = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.query) + (static_cast<size_t>(t) * p.H + h0 + head) * p.row);
    const int words = p.row >> 3;
    for (int c = warp >> 2; c < sp.atoms; c += quad < 2 ? 5 : 1) {
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
        const uint32_t bar = full + 8 * stage, dst = ring + stage * tile_bytes;
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
      // f32 accumulators, bf16, M = 128.  Scores: both K-major (the lanes past the heads hold zeros), N = 64 positions.  Output: the
      // tile's channels MN-major, N = heads.
      constexpr uint32_t s_idesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kMmaTile >> 3) << 17) | (8u << 24);
      constexpr uint32_t o_idesc = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 15) | (static_cast<uint32_t>(HT >> 3) << 17) | (8u << 24);
      const uint64_t sd = SmemDesc(ring, 16, 1024), cd = SmemDesc(ring, kAtomBytes, 1024), pd = SmemDesc(base, 16, 1024);
      const int steps = (p.row + 15) >> 4, buffers = sp.score_buffers;
      ok = MbarWait(qready, 0, abort_word) && ok;
      int s_stage = 0;
      uint32_t s_phase = 0;
      auto scores = [&](int j) {
        const uint32_t acc = tmem + (buffers == 2 ? (j & 1) * kMmaTile : 0);
        const int read = j - buffers;  // the scores whose place these take
        ok = MbarWait(full + 8 * s_stage, s_phase, abort_word) && ok;
        if (read >= 0) ok = MbarWait(sempty + 8 * (read & 1), (read >> 1) & 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint64_t d = sd + static_cast<uint64_t>((s_stage * tile_bytes) >> 4);
        uint32_t q = tmem_q;
        for (int c = 0; c < sp.atoms; ++c, d += kAtomBytes >> 4, q += 32) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (4 * c + k < steps) TcMmaTmemA(acc, q + 8 * k, d + 2 * k, s_idesc, c > 0 || k > 0 ? 1u : 0u);
        }
        TcCommit(sfull + 8 * (j & 1));
        if (++s_stage == stages) {
          s_stage = 0;
          s_phase ^= 1;
        }
      };
      scores(0);
      int stage = 0;
      for (int j = 0; j < n; ++j) {
        if (j + 1 < n) scores(j + 1);
        const int b = j & 1;
        ok = MbarWait(pready + 8 * b, (j >> 1) & 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint64_t d = cd + static_cast<uint64_t>((stage * tile_bytes) >> 4);
        const uint64_t w = pd + static_cast<uint64_t>((b * kPBytes) >> 4);
        uint32_t acc = tmem_o;
        for (int i = 0; i < o_tiles; ++i, d += (2 * kAtomBytes) >> 4, acc += kOCols) {
#pragma unroll
          for (int k = 0; k < 4; ++k) TcMmaBf16(acc, d + ((k * 16 * 128) >> 4), w + 2 * k, o_idesc, j > 0 || k > 0 ? 1u : 0u);
        }
        TcCommit(free0 + 8 * stage);
        TcCommit(odone + 8 * b);
        if (++stage == stages) stage = 0;
      }
    }
    __syncwarp();
  } else if (warp >= kOutWarps) {  // softmax, or nothing
    const int quad = warp & 3, part = (warp >> 2) - 1, head = quad * 32 + lane;  // TMEM lane; positions [16 part, 16 part + 16)
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    constexpr int kPart = kMmaTile / kParts;
    // Every part's value: the four warps of a quad meet at a named barrier of 128 threads.
    auto share = [&](int b, float mine) {
      s_row[b][part][head] = mine;
      asm volatile("bar.sync %0, 128;\n" ::"r"(2 + quad) : "memory");
      return make_float4(s_row[b][0][head], s_row[b][1][head], s_row[b][2][head], s_row[b][3][head]);
    };
    if (quad < kQuads) {
      const float scale = p.scale * 1.4426950408889634f;
      float top = -INFINITY, sum = 0.f;
      for (int j = 0; j < n; ++j) {
        const int b = j & 1, tile_pos = (tile0 + j) * kMmaTile, pos = tile_pos + part * kPart;
        ok = MbarWaitWarp(sfull + 8 * b, (j >> 1) & 1, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint32_t s[kPart];
        TcLd16(tmem + lanes + (sp.score_buffers == 2 ? b * kMmaTile : 0) + part * kPart, s);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(sempty + 8 * b);
        float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        const bool edge = tile_pos < live.x || tile_pos + kMmaTile > live.y;
#pragma unroll
        for (int e = 0; e < kPart; ++e) {
          float v = __uint_as_float(s[e]) * scale;
          if (edge && (pos + e < live.x || pos + e >= live.y)) v = -INFINITY;
          s[e] = __float_as_uint(v);
          t4[e & 3] = fmaxf(t4[e & 3], v);
        }
        const float4 tops = share(b, fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])));
        const float tile_top = fmaxf(fmaxf(tops.x, tops.y), fmaxf(tops.z, tops.w));  // finite: a tile holds at least one live position
        float keep = 1.f;
        if (tile_top > top + kLazy || top == -INFINITY) {
          const float next = fmaxf(top, tile_top);
          keep = Exp2(top - next);
          sum *= keep;
          top = next;
        }
        float add[2] = {0.f, 0.f};
#pragma unroll
        for (int e = 0; e < kPart; e += 2) {
          const float p0 = Exp2(__uint_as_float(s[e]) - top), p1 = Exp2(__uint_as_float(s[e + 1]) - top);
          add[0] += p0;
          add[1] += p1;
          s[e / 2] = Pack(p0, p1);
        }
        sum += add[0] + add[1];
        float total = 0.f;
        if (j == n - 1) {
          const float4 sums = share(b ^ 1, sum);
          total = (sums.x + sums.y) + (sums.z + sums.w);
        }
        if (j >= 2) ok = MbarWaitWarp(odone + 8 * b, ((j >> 1) - 1) & 1, lane, abort_word) && ok;  // the weights of tile j - 2 have been read
        if (head < HT) {
          unsigned char* dst = smem + b * kPBytes + head * 128;
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            *reinterpret_cast<uint4*>(dst + (((part * 2 + c) ^ (head & 7)) << 4)) = make_uint4(s[4 * c], s[4 * c + 1], s[4 * c + 2], s[4 * c + 3]);
          }
        }
        if (part == 0) {
          s_keep[b][head] = keep;
          if (j == n - 1) {
            s_row[b][0][head] = total;  // every maximum of this tile has been read
            if (sp.records != nullptr && head < HT && h0 + head < p.H) {
              float* rec = sp.records + ((static_cast<size_t>(slice) * p.T + t) * p.H + h0 + head) * (p.kv_rank + 2);
              rec[0] = top;
              rec[1] = total;
            }
          }
        }
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        __syncwarp();
        // A named barrier: waiting there costs no issue slots.  Trip counts are fixed, so every arrival has its wait.
        asm volatile("bar.arrive %0, %1;\n" ::"r"(4 + b), "n"(kHandOver) : "memory");
      }
    }
  } else {  // output: this thread's TMEM lane is channel 128 i + tid of accumulator i
    const uint32_t lanes = static_cast<uint32_t>(warp * 32) << 16;
    int stage = 0;
    for (int j = 0; j < n; ++j) {
      const int b = j & 1, pos = (tile0 + j) * kMmaTile;
      asm volatile("bar.sync %0, %1;\n" ::"r"(4 + b), "n"(kHandOver) : "memory");
      // Rows of the page outside the live range may hold anything: 0 times it must stay 0.
      const int live_lo = live.x - pos, live_hi = live.y - pos;
      if (live_lo > 0 || live_hi < kMmaTile) {
        for (int i = tid; i < kMmaTile * sp.atoms * 8; i += kOutWarps * 32) {
          const int r = i & (kMmaTile - 1);
          if (r < live_lo || r >= live_hi) *reinterpret_cast<uint4*>(smem + 2 * kPBytes + stage * tile_bytes + TileWord(r, i / kMmaTile)) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
      }
      if (j > 0) {
        bool raised = false;
#pragma unroll
        for (int k = 0; k < kQuads; ++k) raised = raised || s_keep[b][k * 32 + lane] != 1.f;
        if (__any_sync(0xffffffffu, raised)) {
          ok = MbarWaitWarp(odone + 8 * (b ^ 1), ((j - 1) >> 1) & 1, lane, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int c = 0; c < o_tiles * kOCols; c += 32) {
            uint32_t o[32];
            TcLd32(tmem_o + lanes + c, o);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            const float* keep = s_keep[b] + c % kOCols;
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * keep[e]);
            TcSt32(tmem_o + lanes + c, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
      __syncwarp();
      if (lane == 0) MbarArrive(pready + 8 * b);
      if (++stage == stages) stage = 0;
    }
    ok = MbarWaitWarp(odone + 8 * ((n - 1) & 1), ((n - 1) >> 1) & 1, lane, abort_word) && ok;
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const float* totals = s_row[(n - 1) & 1][0];
    for (int i = 0; i < o_tiles; ++i) {
      const int channel = i * 128 + tid;
#pragma unroll 1
      for (int g = 0; g < HT; g += 16) {
        uint32_t o[16];
        TcLd16(tmem_o + lanes + i * kOCols + g, o);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        if (channel < p.kv_rank) {
          const size_t at = static_cast<size_t>(t) * p.H + h0 + g;
          float* rec = sp.records + (static_cast<size_t>(slice) * p.T * p.H + at) * (p.kv_rank + 2) + 2 + channel;
          __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + at * p.kv_rank + channel;
          const int heads = p.H - h0 - g;
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            if (e >= heads) break;
            if (sp.records != nullptr) rec[e * (p.kv_rank + 2)] = __uint_as_float(o[e]);
            else out[e * p.kv_rank] = __float2bfloat16_rn(__uint_as_float(o[e]) / totals[g + e]);
          }
        }
      }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  }
  if (!ok) atomicExch(&g_latent_status, 1);
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
constexpr int StaticSmem(int mt) { return mt > 2 ? 3072 : 2048; }  // at least what the kernel declares

int Atoms(int row) { return (row + 63) / 64; }
// 16-head tiles of a CTA: enough for all heads where TMEM allows (two for latents wider than 256 channels, four up to that), else
// the count that leaves the fewest absent heads.
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
// TMEM columns beside the scores: the query, and O^T in accumulators of 128 channels.
int FixedColumns(int mt, int kv_rank, int row) { return Atoms(row) * 32 + (kv_rank + 127) / 128 * ((mt + 1) / 2 * 32); }
// What the last 128-channel operand of a tile may reach past its atoms.
int Slack(int kv_rank, int row) { return std::max(0, (kv_rank + 127) / 128 * 2 - Atoms(row)) * kAtomBytes; }
int Stages(int mt, int kv_rank, int row)
{
  return std::min(kMaxStages, (kMmaMaxSmem - StaticSmem(mt) - 1024 - 2 * mt * 16 * 128 - Slack(kv_rank, row)) / (Atoms(row) * kAtomBytes));
}
size_t MmaSmem(int mt, int kv_rank, int row)
{
  return 1024 + 2 * mt * 16 * 128 + static_cast<size_t>(Stages(mt, kv_rank, row)) * Atoms(row) * kAtomBytes + Slack(kv_rank, row);
}
bool MmaApplies(int heads, int kv_rank, int rot_dim)
{
  const int row = kv_rank + rot_dim, mt = HeadTiles(heads, kv_rank);
  return kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank <= 512 && FixedColumns(mt, kv_rank, row) + kMmaTile <= 512 && Stages(mt, kv_rank, row) >= 2;
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

template <int MT>
cudaError_t LaunchTc(const CUtensorMap& map, const LatentParams& p, const SliceParams& sp, cudaStream_t st)
{
  const dim3 grid(sp.slices, (p.H + 16 * MT - 1) / (16 * MT), p.T);
  return LaunchChained(LatentAttentionTc<16 * MT>, grid, kMmaThreads, MmaSmem(MT, p.kv_rank, p.row), st, map, p, sp);
}

cudaError_t PrepareLatentAttention()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(MT) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(LatentAttentionTc<16 * MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMmaMaxSmem - StaticSmem(MT))
    TLALOC_OPT_IN(1);
    TLALOC_OPT_IN(2);
    TLALOC_OPT_IN(3);
    TLALOC_OPT_IN(4);
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

cudaError_t LaunchTcForm(const CUtensorMap& map, const LatentParams& p, SliceParams sp, cudaStream_t st)
{
  const int mt = HeadTiles(p.H, p.kv_rank);
  sp.atoms = Atoms(p.row);
  sp.stages = Stages(mt, p.kv_rank, p.row);
  sp.score_buffers = FixedColumns(mt, p.kv_rank, p.row) + 2 * kMmaTile <= 512 ? 2 : 1;
  switch (mt) {
    case 1: return LaunchTc<1>(map, p, sp, st);
    case 2: return LaunchTc<2>(map, p, sp, st);
    case 3: return LaunchTc<3>(map, p, sp, st);
    default: return LaunchTc<4>(map, p, sp, st);
  }
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
  if (num_tokens < 1 || num_heads < 1 || max_live < 1 || !MmaApplies(num_heads, kv_rank, rot_dim)) return 0;
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
  if (dtype == TLALOC_B200_BF16 && !OrderFaithful() && MmaApplies(num_heads, kv_rank, rot_dim) && pool_ld % 8 == 0 && Aligned16(query) && Aligned16(pool) &&
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
