// Attention of absorbed queries over a paged pool of latents (include/tlaloc_b200.h, tlaloc_b200_latent_attention).
//
// LatentAttentionGeneric: any sizes, f32 or bf16, plain FMA.  A CTA serves one (row, head): tiles of 128 positions, a warp
// per position for the scores (lanes over the channels), an online softmax in f32, then a thread per latent channel.
//
// LatentAttentionMma (bf16): all heads share a position's row, so a CTA takes 16 to 64 heads of one row and a slice of its
// positions, and the row leaves HBM once for all of them.  Tiles of 64 positions arrive by 16-byte cp.async copies, two tiles in shared
// memory; both products run on mma.sync m16n8k16 (heads are the M rows) with f32 accumulators:
//   scores   the channels are split over eight warps (and the positions over two), so that a warp's share of the query stays in
//            registers for the whole slice; the eight partial sums meet in shared memory, where the softmax adds them
//   values   the latent channels are split over the sixteen warps; the tile is read again, transposed, as it lies
// Slices leave {max, sum, acc[kv_rank]} records in f32 that LatentCombine merges in slice order.
#include <algorithm>

#include "common.cuh"

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
constexpr int kMmaTile = 64, kMmaThreads = 512, kGroups = 8, kPStride = kMmaTile + 8, kPartStride = kMmaTile + 2;

__device__ __forceinline__ uint32_t SmemAddr(const void* ptr) { return static_cast<uint32_t>(__cvta_generic_to_shared(ptr)); }
__device__ __forceinline__ void CpAsync16(uint32_t dst, const void* src, int src_bytes)
{
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}
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
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float Exp2(float x)
{
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

struct SliceParams {
  float* records;  // [slices][T][H][kv_rank + 2], or null: one slice, straight to out
  int slices, slice_tiles, row_bytes;  // row_bytes: a tile row in shared memory, an odd number of 16-byte words
};

// kGroups warps split the channels of the scores.  MT: 16-head tiles of the CTA; KSG: 16-channel steps of the scores per warp; NP: 16-channel pairs of values per warp.
template <int MT, int KSG, int NP>
__global__ void __launch_bounds__(kMmaThreads, 1) LatentAttentionMma(LatentParams p, SliceParams sp)
{
  constexpr int HT = MT * 16;
  constexpr int kPerHead = HT <= 16 ? 32 : HT <= 32 ? 16 : 8, kPos = kMmaTile / kPerHead;  // softmax: threads of a head, positions of a thread
  GridDependencySync();
  extern __shared__ __align__(16) unsigned char smem[];
  const int tile_bytes = kMmaTile * sp.row_bytes;
  float* part = reinterpret_cast<float*>(smem + 2 * tile_bytes);                        // [kGroups][HT][kPartStride]
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(part + kGroups * HT * kPartStride);   // [HT][kPStride]
  float* s_keep = reinterpret_cast<float*>(s_p + HT * kPStride);                        // [HT]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
  const int t = blockIdx.z, h0 = blockIdx.y * HT, slice = blockIdx.x;
  const int2 live = LiveRange(p, t);
  const int tile0 = live.x / kMmaTile + slice * sp.slice_tiles;
  const int tile_end = min((live.y + kMmaTile - 1) / kMmaTile, tile0 + sp.slice_tiles);
  if (tile0 >= tile_end && !(slice == 0 && sp.records == nullptr)) return;  // an empty slice writes nothing; an empty row writes zeros
  const int* table = TableOf(p, t);
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(p.pool);
  const int words = p.row >> 3;  // 16-byte words of a row
  const int steps = (p.row + 15) >> 4;

  // Eight threads copy a position's row; positions outside the live range become zeros.  The row's place is looked up a tile
  // ahead, so that its latency is not in front of the copies.
  const int my_row = tid >> 3;
  auto place = [&](int tile) {
    const int pos = tile * kMmaTile + my_row;
    return pos >= live.x && pos < live.y ? pool + PoolRow(p, table, pos) : nullptr;
  };
  auto load = [&](const __nv_bfloat16* src, int stage) {
    const uint32_t dst = SmemAddr(smem) + stage * tile_bytes + my_row * sp.row_bytes;
    const int bytes = src != nullptr ? 16 : 0;
    if (src == nullptr) src = pool;
#pragma unroll 4
    for (int w = tid & 7; w < words; w += 8) CpAsync16(dst + w * 16, src + w * 8, bytes);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  const __nv_bfloat16* next_row = nullptr;
  if (tile0 < tile_end) {
    load(place(tile0), 0);
    if (tile0 + 1 < tile_end) next_row = place(tile0 + 1);
  }
  if (p.row & 8) {  // the last step's upper channels
    for (int i = tid; i < 2 * kMmaTile; i += kMmaThreads) {
      *reinterpret_cast<uint4*>(smem + (i / kMmaTile) * tile_bytes + (i % kMmaTile) * sp.row_bytes + words * 16) = make_uint4(0, 0, 0, 0);
    }
  }
  // The warp's share of the query: steps kg, kg + kGroups, ... of the channels, as A fragments.
  const int kg = warp % kGroups, ph = warp / kGroups;
  uint32_t q[KSG][MT][4];
  const __nv_bfloat16* query = static_cast<const __nv_bfloat16*>(p.query) + static_cast<size_t>(t) * p.H * p.row;
#pragma unroll
  for (int i = 0; i < KSG; ++i) {
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = h0 + m * 16 + gid + (e & 1) * 8, k = (kg + kGroups * i) * 16 + tig * 2 + (e >> 1) * 8;
        q[i][m][e] = h < p.H && k < p.row ? *reinterpret_cast<const uint32_t*>(query + static_cast<size_t>(h) * p.row + k) : 0u;
      }
    }
  }
  float acc[MT][2 * NP][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 2 * NP; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  const int sh = tid / kPerHead, s0 = (tid % kPerHead) * 2;  // softmax: this thread's head and first pair of positions
  const float scale = p.scale * 1.4426950408889634f;
  float top = -INFINITY, sum = 0.f;
  const int pairs = (p.kv_rank + 15) >> 4;

  for (int tile = tile0; tile < tile_end; ++tile) {
    const int stage = (tile - tile0) & 1;
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();  // the tile has landed and the tile before it has been read
    if (tile + 1 < tile_end) {
      load(next_row, stage ^ 1);
      if (tile + 2 < tile_end) next_row = place(tile + 2);
    }
    const uint32_t tile_addr = SmemAddr(smem) + stage * tile_bytes;
    // B fragments: matrices (positions 0-7, channels 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15) of a 16-position group
    const uint32_t row_addr = tile_addr + (ph * 32 + (lane & 7) + ((lane >> 4) << 3)) * sp.row_bytes + ((lane >> 3) & 1) * 16;
    float* dst = part + kg * HT * kPartStride + ph * 32 + tig * 2;
#pragma unroll
    for (int g = 0; g < 2; ++g) {
      float s[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[m][n][e] = 0.f;
#pragma unroll
      for (int i = 0; i < KSG; ++i) {
        const int step = kg + kGroups * i;
        if (step < steps) {
          uint32_t b[4];
          LdMatrixX4(b, row_addr + g * 16 * sp.row_bytes + step * 32);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            MmaBf16(s[m][0], q[i][m], b[0], b[1]);
            MmaBf16(s[m][1], q[i][m], b[2], b[3]);
          }
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          *reinterpret_cast<float2*>(dst + (m * 16 + gid) * kPartStride + g * 16 + n * 8) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(dst + (m * 16 + gid + 8) * kPartStride + g * 16 + n * 8) = make_float2(s[m][n][2], s[m][n][3]);
        }
    }
    __syncthreads();
    if (sh < HT) {  // whole warps
      float v[kPos], tile_top = -INFINITY;  // positions s0, s0 + 1, s0 + 2 kPerHead, ...
#pragma unroll
      for (int e = 0; e < kPos; e += 2) {
        const int at = s0 + e * kPerHead, pos = tile * kMmaTile + at;
        const float* src = part + sh * kPartStride + at;
        float2 d = *reinterpret_cast<const float2*>(src);
#pragma unroll
        for (int k = 1; k < kGroups; ++k) {
          const float2 more = *reinterpret_cast<const float2*>(src + k * HT * kPartStride);
          d.x += more.x;
          d.y += more.y;
        }
        v[e] = pos >= live.x && pos < live.y ? d.x * scale : -INFINITY;
        v[e + 1] = pos + 1 >= live.x && pos + 1 < live.y ? d.y * scale : -INFINITY;
        tile_top = fmaxf(tile_top, fmaxf(v[e], v[e + 1]));
      }
#pragma unroll
      for (int o = kPerHead / 2; o > 0; o >>= 1) tile_top = fmaxf(tile_top, __shfl_xor_sync(0xffffffffu, tile_top, o));
      const float next = fmaxf(top, tile_top);  // finite: a tile holds at least one live position
      const float keep = Exp2(top - next);
      float add = 0.f;
#pragma unroll
      for (int e = 0; e < kPos; e += 2) {
        const float p0 = Exp2(v[e] - next), p1 = Exp2(v[e + 1] - next);
        add += p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(s_p + sh * kPStride + s0 + e * kPerHead) = __floats2bfloat162_rn(p0, p1);
      }
      sum = sum * keep + add;
      top = next;
      if (tid % kPerHead == 0) s_keep[sh] = keep;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float k0 = s_keep[m * 16 + gid], k1 = s_keep[m * 16 + gid + 8];
      if (__any_sync(0xffffffffu, k0 != 1.f || k1 != 1.f)) {
#pragma unroll
        for (int n = 0; n < 2 * NP; ++n) {
          acc[m][n][0] *= k0; acc[m][n][1] *= k0;
          acc[m][n][2] *= k1; acc[m][n][3] *= k1;
        }
      }
    }
    const uint32_t v_addr = tile_addr + (lane & 15) * sp.row_bytes + (lane >> 4) * 16;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t pf[MT][4];  // matrices (heads 0-7, positions 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
#pragma unroll
      for (int m = 0; m < MT; ++m) LdMatrixX4(pf[m], SmemAddr(s_p + (m * 16 + (lane & 15)) * kPStride + k * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int pair = warp + 16 * i;
        if (pair < pairs) {
          uint32_t b[4];  // (positions 0-7, channels 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15), transposed
          LdMatrixX4Trans(b, v_addr + k * 16 * sp.row_bytes + pair * 32);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            MmaBf16(acc[m][2 * i], pf[m], b[0], b[1]);
            MmaBf16(acc[m][2 * i + 1], pf[m], b[2], b[3]);
          }
        }
      }
    }
  }
  // Sums of a head's threads, and its maximum, to everybody.
#pragma unroll
  for (int o = kPerHead / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  __syncthreads();
  if (sh < HT && tid % kPerHead == 0) {
    s_keep[sh] = sum;
    if (sp.records != nullptr && h0 + sh < p.H) {
      float* rec = sp.records + ((static_cast<size_t>(slice) * p.T + t) * p.H + h0 + sh) * (p.kv_rank + 2);
      rec[0] = top;
      rec[1] = sum;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int h = h0 + m * 16 + gid + half * 8;
      if (h >= p.H) continue;
      const float total = s_keep[m * 16 + gid + half * 8], inv = total > 0.f ? 1.f / total : 0.f;
#pragma unroll
      for (int n = 0; n < 2 * NP; ++n) {
        const int c = (warp + 16 * (n >> 1)) * 16 + (n & 1) * 8 + tig * 2;
        if (c >= p.kv_rank) continue;
        const float a = acc[m][n][2 * half], b = acc[m][n][2 * half + 1];
        if (sp.records != nullptr) {
          *reinterpret_cast<float2*>(sp.records + ((static_cast<size_t>(slice) * p.T + t) * p.H + h) * (p.kv_rank + 2) + 2 + c) = make_float2(a, b);
        } else {
          *reinterpret_cast<__nv_bfloat162*>(static_cast<__nv_bfloat16*>(p.out) + (static_cast<size_t>(t) * p.H + h) * p.kv_rank + c) =
              __floats2bfloat162_rn(a * inv, b * inv);
        }
      }
    }
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

int RowBytes(int row) { return ((2 * ((row + 15) / 16)) | 1) * 16; }
size_t MmaSmem(int mt, int row)
{
  return 2 * static_cast<size_t>(kMmaTile) * RowBytes(row) + mt * 16 * (kGroups * kPartStride * sizeof(float) + kPStride * 2 + sizeof(float));
}
constexpr size_t kMmaMaxSmem = 227 * 1024;

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
  return kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank <= 512 && (kv_rank + rot_dim + 15) / 16 <= 36 && (kv_rank > 256 || kv_rank + rot_dim <= 320);
}

// Slices of the positions: the fewest waves of CTAs times the tiles a CTA walks, for the longest live range a row may have.
int ChooseLatentSlices(int rows, int heads, int kv_rank, int row, int max_live, int* slice_tiles)
{
  const int tiles = (max_live + kMmaTile - 1) / kMmaTile + 1;
  const int mt = HeadTiles(heads, kv_rank);
  const int ctas = rows * ((heads + 16 * mt - 1) / (16 * mt));
  const int slots = 148 * std::max(1, std::min<int>(4, static_cast<int>(kMmaMaxSmem / MmaSmem(mt, row))));
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

template <int MT, int KSG, int NP>
cudaError_t LaunchMma(const LatentParams& p, const SliceParams& sp, cudaStream_t st)
{
  const dim3 grid(sp.slices, (p.H + 16 * MT - 1) / (16 * MT), p.T);
  return LaunchChained(LatentAttentionMma<MT, KSG, NP>, grid, kMmaThreads, MmaSmem(MT, p.row), st, p, sp);
}

#define TLALOC_LATENT_FORMS(X) \
  X(1, 3, 1) X(2, 3, 1) X(3, 3, 1) X(4, 3, 1) X(1, 5, 2) X(2, 5, 2)

cudaError_t PrepareLatentAttention()
{
  static OncePerDevice once;
  return once.Run([](int) {
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(MT, KSG, NP) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(LatentAttentionMma<MT, KSG, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kMmaMaxSmem));
    TLALOC_LATENT_FORMS(TLALOC_OPT_IN)
#undef TLALOC_OPT_IN
    return e;
  });
}
KernelSetup g_setup(PrepareLatentAttention, nullptr);

cudaError_t LaunchMmaForm(const LatentParams& p, const SliceParams& sp, cudaStream_t st)
{
  const int mt = HeadTiles(p.H, p.kv_rank), ksg = ((p.row + 15) / 16 + kGroups - 1) / kGroups, np = ((p.kv_rank + 15) / 16 + 15) / 16;
#define TLALOC_TRY(MT, KSG, NP) \
  if (mt == MT && ksg <= KSG && np <= NP) return LaunchMma<MT, KSG, NP>(p, sp, st);
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
    const int s = ChooseLatentSlices(rows, num_heads, kv_rank, kv_rank + rot_dim, max_live, &tiles);
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
  if (dtype == TLALOC_B200_BF16 && !OrderFaithful() && MmaApplies(kv_rank, rot_dim) && pool_ld % 8 == 0 && Aligned16(query) && Aligned16(pool) &&
      Aligned16(out) && (scratch == nullptr || Aligned16(scratch))) {
    cudaError_t e = PrepareLatentAttention();
    if (e != cudaSuccess) return CudaFail("LATENT_ATTENTION set-up", e);
    SliceParams sp;
    const int live = MaxLive(max_live, window, static_cast<int64_t>(max_blocks) * block_size);
    sp.slices = ChooseLatentSlices(num_tokens, num_heads, kv_rank, p.row, live, &sp.slice_tiles);
    const size_t need = static_cast<size_t>(sp.slices) * num_tokens * num_heads * (kv_rank + 2) * sizeof(float);
    if (sp.slices > 1 && (scratch == nullptr || scratch_bytes < need)) {
      sp.slices = 1;
      sp.slice_tiles = 0x3fffffff;
    }
    if (sp.slices == 1) sp.slice_tiles = 0x3fffffff;
    sp.records = sp.slices > 1 ? static_cast<float*>(scratch) : nullptr;
    sp.row_bytes = RowBytes(p.row);
    e = LaunchMmaForm(p, sp, st);
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
