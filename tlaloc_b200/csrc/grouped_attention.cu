// Attention of single tokens over a paged pool of grouped key and value heads, with a sliding window and kept first tokens, one or two
// maps of scores per query head over the same values (include/tlaloc_b200.h, tlaloc_b200_grouped_attention).
//
// The positions are taken in groups of 16, aligned, so that a group lies in one page: those of the kept tokens, then those of the window; what a
// row does not see of a group is masked.  With few rows the groups are cut into slices; each slice leaves a record per query head
// ({largest score (log2), sum, weighted values}), and the operator that consumes the result merges them.
//   GroupedAttentionMma      bf16, pages of a multiple of 16.  A CTA has one value head, up to 16 of its query heads (8 of two maps each) and one
//                            slice, so every cached byte of the slice is read once for all of them.  Four warps, each with groups and a
//                            ring of its own: one lane looks up the page and requests the group's boxes (64 channels x 16 rows, 128-byte
//                            swizzle) by TMA; no CTA-wide barrier in the loop.  Query heads are the rows of mma.m16n8k16; with two maps the
//                            rows 0-7 are the heads' first map and 8-15 the second, each multiplied with its own keys, so that one
//                            product with the values serves both.  The weights enter that product as two bf16 parts (f32 up to rounding).
//   GroupedAttentionGeneric  any size and type, plain FMA: the f32 path.
#include <cuda.h>

#include "common.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

using tc::ElectOne;
using tc::MbarExpectTx;
using tc::MbarInit;
using tc::MbarWait;
using tc::MbarWaitWarp;
using tc::SmemAddr;

constexpr int kGroup = 16, kWarps = 4, kMaxStages = 4;
constexpr int kAtom = kGroup * 128;  // 16 rows x 64 channels
constexpr int kMaxSmem = 227 * 1024;

__device__ int g_grouped_status = 0;

struct GroupedArgs {
  const void* q;
  const void* pool;
  const int *tables, *row_tables, *lens;
  float* records;
  int64_t pool_ld;
  int T, heads, v_heads, maps, dim, vdim, v_first, num_blocks, block_size, max_blocks, num_tables, window, keep, slices, qtiles, stages;
  float scale_log2;
};

// What row t sees: positions [0, kept) and [lo, lo + count - kept).
struct Seen {
  const int* table;
  int lo, kept, count;
};
__device__ __forceinline__ Seen SeenBy(const GroupedArgs& a, int t)
{
  Seen s;
  const int len = min(max(__ldg(a.lens + t), 0), a.max_blocks * a.block_size);
  const int tab = a.row_tables != nullptr ? __ldg(a.row_tables + t) : t;
  s.table = a.tables + static_cast<size_t>(min(max(tab, 0), a.num_tables - 1)) * a.max_blocks;
  s.lo = a.window > 0 ? max(0, len - a.window) : 0;
  s.kept = min(a.keep, s.lo);
  s.count = s.kept + len - s.lo;
  return s;
}
// Pool row of the i-th position seen.
__device__ __forceinline__ int64_t PoolRow(const GroupedArgs& a, const Seen& s, int i)
{
  const int pos = i < s.kept ? i : s.lo + i - s.kept, b = pos / a.block_size;
  const int page = min(max(__ldg(s.table + b), 0), a.num_blocks - 1);
  return static_cast<int64_t>(page) * a.block_size + (pos - b * a.block_size);
}

__device__ __forceinline__ void Mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1)
{
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void Ldm4(uint32_t* r, uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void Ldm4T(uint32_t* r, uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ float Exp2(float x)
{
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
// Two f32 as a pair of bf16 and the pair of what is left of them.
__device__ __forceinline__ void Split(float a, float b, uint32_t& hi, uint32_t& lo)
{
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// DK, NV: 16-channel steps of a key and a value head, in whole atoms of four.  What an atom holds past its head is multiplied with zero
// queries (keys) or left out of the result (values).
template <int DK, int NV>
__global__ void __launch_bounds__(kWarps * 32) GroupedAttentionMma(const __grid_constant__ CUtensorMap map, const __grid_constant__ GroupedArgs a)
{
  extern __shared__ unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[kWarps * kMaxStages];
  __shared__ uint32_t abort_store;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t base = (SmemAddr(smem_raw) + 1023u) & ~1023u;
  unsigned char* smem = smem_raw + (base - SmemAddr(smem_raw));
  const uint32_t bar = SmemAddr(bars + warp * kMaxStages);
  volatile uint32_t* abort_word = &abort_store;
  if (tid == 0) {
    abort_store = 0u;
    for (int i = 0; i < kWarps * kMaxStages; ++i) MbarInit(SmemAddr(bars + i), 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  __syncthreads();
  GridDependencySync();
  const int slice = blockIdx.x, vh = blockIdx.y / a.qtiles, qt = blockIdx.y % a.qtiles, t = blockIdx.z;
  const int group = a.heads / a.v_heads, per_map = group / a.maps;  // query heads (with maps counted) and without
  const int rows_per_map = 16 / a.maps;
  const int dk = a.dim >> 4;
  const int len = min(max(__ldg(a.lens + t), 0), a.max_blocks * a.block_size);
  const int tab = a.row_tables != nullptr ? __ldg(a.row_tables + t) : t;
  const int* table = a.tables + static_cast<size_t>(min(max(tab, 0), a.num_tables - 1)) * a.max_blocks;
  // Visible: lo <= position < len, or position < keep.  Groups [0, kept) and [first, ..).
  const int lo = a.window > 0 ? max(0, len - a.window) : 0, keep = min(a.keep, lo);
  const int kept = (keep + kGroup - 1) / kGroup, first = max(lo / kGroup, kept);
  const int groups = kept + (len + kGroup - 1) / kGroup - first, share = (groups + a.slices - 1) / a.slices;
  const int g0 = slice * share, g1 = min(groups, g0 + share);
  auto position = [&](int g) { return (g < kept ? g : first + g - kept) * kGroup; };
  // The query head of MMA row r: (place in the group, map).
  auto query_head = [&](int r) {
    const int place = qt * rows_per_map + r % rows_per_map, m = r / rows_per_map;
    return place < per_map ? (vh * per_map + place) * a.maps + m : -1;
  };
  const int rec = a.vdim + 2;
  float* records = a.records + (static_cast<size_t>(slice) * a.T + t) * a.heads * rec;
  if (g0 >= g1) {
    if (tid < 16) {
      const int h = query_head(tid);
      if (h >= 0) {
        records[static_cast<size_t>(h) * rec] = -INFINITY;
        records[static_cast<size_t>(h) * rec + 1] = 0.f;
      }
    }
    return;
  }

  // A stage: the atoms of every map's keys, then those of the values.  x is a multiple of 16 channels: a 16-byte boundary.
  constexpr int k_atoms = DK / 4, v_atoms = NV / 4;
  const int stage_bytes = (a.maps * k_atoms + v_atoms) * kAtom, stages = a.stages;
  const uint32_t ring = base + warp * stages * stage_bytes;
  const int k_col = vh * a.maps * a.dim, v_col = a.v_first + vh * a.vdim;
  const int steps = (g1 - g0 - warp + kWarps - 1) / kWarps;  // this warp's groups: g0 + warp, + kWarps, ..
  auto pool_row = [&](int i) {  // of the i-th group
    const int pos = position(g0 + warp + min(i, steps - 1) * kWarps), b = pos / a.block_size;
    return min(max(__ldg(table + b), 0), a.num_blocks - 1) * a.block_size + (pos - b * a.block_size);
  };
  auto load = [&](int row, int stage) {
    const uint32_t bar_s = bar + 8 * stage;
    uint32_t dst = ring + stage * stage_bytes;
    MbarExpectTx(bar_s, stage_bytes);
    auto box = [&](int x) {
      asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n" ::"r"(dst),
                   "l"(reinterpret_cast<uint64_t>(&map)), "r"(x), "r"(row), "r"(bar_s)
                   : "memory");
      dst += kAtom;
    };
    for (int m = 0; m < a.maps; ++m)
#pragma unroll
      for (int c = 0; c < k_atoms; ++c) box(k_col + m * a.dim + c * 64);
#pragma unroll
    for (int c = 0; c < v_atoms; ++c) box(v_col + c * 64);
  };
  if (steps > 0) {
    for (int i = 0; i < min(steps, stages); ++i) {
      const int row = pool_row(i);
      if (lane == 0) load(row, i);
      __syncwarp();
    }
  }
  int next_row = steps > 0 ? pool_row(stages) : 0;  // looked up ahead of its request

  // Queries as A fragments: rows lane / 4 and lane / 4 + 8.
  uint32_t qa[DK][2], qb[DK][2];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(t) * a.heads * a.dim;
    const int h0 = query_head(lane >> 2), h1 = query_head((lane >> 2) + 8);
#pragma unroll
    for (int k = 0; k < DK; ++k) {
      qa[k][0] = qa[k][1] = qb[k][0] = qb[k][1] = 0u;
      if (k < dk) {
        const int c = k * 16 + (lane & 3) * 2;
        if (h0 >= 0) {
          qa[k][0] = *reinterpret_cast<const uint32_t*>(q + static_cast<size_t>(h0) * a.dim + c);
          qa[k][1] = *reinterpret_cast<const uint32_t*>(q + static_cast<size_t>(h0) * a.dim + c + 8);
        }
        if (h1 >= 0) {
          qb[k][0] = *reinterpret_cast<const uint32_t*>(q + static_cast<size_t>(h1) * a.dim + c);
          qb[k][1] = *reinterpret_cast<const uint32_t*>(q + static_cast<size_t>(h1) * a.dim + c + 8);
        }
      }
    }
  }

  bool ok = true;
  float o[2 * NV][4], top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int mat = lane >> 3, r8 = lane & 7;
  // Offset of 16-byte word c of row r of a tile of atoms; of the words 2 k + mat this lane reads, those of k = 0..3 (an atom has eight).
  auto word = [](int r, int c) { return static_cast<uint32_t>((c >> 3) * kAtom + r * 128 + (((c & 7) ^ (r & 7)) << 4)); };
  uint32_t k_off[4], v_off[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    k_off[k] = word((mat >> 1) * 8 + r8, 2 * k + (mat & 1));
    v_off[k] = word((mat & 1) * 8 + r8, 2 * k + (mat >> 1));
  }
  int stage = 0, phase = 0;
  for (int i = 0; i < steps; ++i) {
    const int pos = position(g0 + warp + i * kWarps);
    const uint32_t kt = ring + stage * stage_bytes, vt = kt + a.maps * k_atoms * kAtom;
    ok = MbarWaitWarp(bar + 8 * stage, phase, lane, abort_word) && ok;
    if (pos + kGroup > len) {  // rows past the end hold whatever the page did: 0 times it must stay 0
      for (int r = len - pos; r < kGroup; ++r)
        for (int c = lane; c < v_atoms * 8; c += 32) {
          asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};\n" ::"r"(vt + word(r, c)), "r"(0u) : "memory");
        }
      asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
      __syncwarp();
    }
    float s[2][4] = {}, u[2][4] = {};
    {
      uint32_t at[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) at[k] = kt + k_off[k];
      if (a.maps == 2) {
#pragma unroll
        for (int k = 0; k < DK; ++k) {
          uint32_t b[4], d[4];
          Ldm4(b, at[k & 3] + (k >> 2) * kAtom);
          Ldm4(d, at[k & 3] + (k_atoms + (k >> 2)) * kAtom);
          Mma(s[0], qa[k][0], 0u, qa[k][1], 0u, b[0], b[1]);
          Mma(s[1], qa[k][0], 0u, qa[k][1], 0u, b[2], b[3]);
          Mma(u[0], 0u, qb[k][0], 0u, qb[k][1], d[0], d[1]);
          Mma(u[1], 0u, qb[k][0], 0u, qb[k][1], d[2], d[3]);
        }
      } else {
#pragma unroll
        for (int k = 0; k < DK; ++k) {
          uint32_t b[4];
          Ldm4(b, at[k & 3] + (k >> 2) * kAtom);
          float(*acc)[4] = (k & 1) ? u : s;
          Mma(acc[0], qa[k][0], qb[k][0], qa[k][1], qb[k][1], b[0], b[1]);
          Mma(acc[1], qa[k][0], qb[k][0], qa[k][1], qb[k][1], b[2], b[3]);
        }
      }
    }
    const int p0 = pos + (lane & 3) * 2;
    if (pos + kGroup > len || (pos < lo && pos + kGroup > keep)) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int p = p0 + n * 8 + (e & 1);
          s[n][e] = p < len && (p >= lo || p < keep) ? (s[n][e] + u[n][e]) * a.scale_log2 : -INFINITY;
        }
    } else {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = (s[n][e] + u[n][e]) * a.scale_log2;
    }
    float p[2][4];
    bool raise = false;
    float next[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float m = fmaxf(fmaxf(s[0][2 * r], s[0][2 * r + 1]), fmaxf(s[1][2 * r], s[1][2 * r + 1]));
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
      next[r] = fmaxf(top[r], m);  // some position of every group is visible: finite from here on
      raise = raise || next[r] > top[r];
    }
    if (__any_sync(0xffffffffu, raise)) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float f = Exp2(top[r] - next[r]);
        top[r] = next[r];
        sum[r] *= f;
#pragma unroll
        for (int n = 0; n < 2 * NV; ++n) {
          o[n][2 * r] *= f;
          o[n][2 * r + 1] *= f;
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        p[n][e] = Exp2(s[n][e] - top[e >> 1]);
        sum[e >> 1] += p[n][e];
      }
    uint32_t hi[4], low[4];  // as A: (row, k 0-7), (row + 8, k 0-7), (row, k 8-15), (row + 8, k 8-15)
    Split(p[0][0], p[0][1], hi[0], low[0]);
    Split(p[0][2], p[0][3], hi[1], low[1]);
    Split(p[1][0], p[1][1], hi[2], low[2]);
    Split(p[1][2], p[1][3], hi[3], low[3]);
    uint32_t at[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) at[k] = vt + v_off[k];
#pragma unroll
    for (int j = 0; j < NV; j += 2) {
      uint32_t b[4], d[4];
      Ldm4T(b, at[j & 3] + (j >> 2) * kAtom);
      Ldm4T(d, at[(j + 1) & 3] + (j >> 2) * kAtom);
      Mma(o[2 * j], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
      Mma(o[2 * j + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
      Mma(o[2 * j + 2], hi[0], hi[1], hi[2], hi[3], d[0], d[1]);
      Mma(o[2 * j + 3], hi[0], hi[1], hi[2], hi[3], d[2], d[3]);
      Mma(o[2 * j], low[0], low[1], low[2], low[3], b[0], b[1]);
      Mma(o[2 * j + 1], low[0], low[1], low[2], low[3], b[2], b[3]);
      Mma(o[2 * j + 2], low[0], low[1], low[2], low[3], d[0], d[1]);
      Mma(o[2 * j + 3], low[0], low[1], low[2], low[3], d[2], d[3]);
    }
    __syncwarp();  // the stage is read before it is filled again
    if (i + stages < steps) {
      if (lane == 0) load(next_row, stage);
      next_row = pool_row(i + stages + 1);
    }
    if (++stage == stages) {
      stage = 0;
      phase ^= 1;
    }
  }
  if (!ok) {
    // Given up: let the copies in flight land before the CTA's shared memory goes away.
    if (lane == 0) {
      volatile uint32_t never = 0;
      for (int s = 0; s < stages; ++s)
        if (steps > s) MbarWait(bar + 8 * s, ((steps - 1 - s) / stages) & 1, &never);
      atomicExch(&g_grouped_status, 1);
    }
    __syncwarp();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
  }

  // The warps' partial results meet in shared memory.
  __syncthreads();
  float* st = reinterpret_cast<float*>(smem);             // [warp][16 rows][2]
  float* acc = st + kWarps * 32;                          // [warp][16 rows][vdim + 4]
  const int acc_ld = a.vdim + 4;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = (lane >> 2) + 8 * r;
    if ((lane & 3) == 0) {
      st[(warp * 16 + row) * 2] = top[r];
      st[(warp * 16 + row) * 2 + 1] = sum[r];
    }
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) {
      if (i * 8 < a.vdim) {
        float* d = acc + static_cast<size_t>(warp * 16 + row) * acc_ld + i * 8 + (lane & 3) * 2;
        d[0] = o[i][2 * r];
        d[1] = o[i][2 * r + 1];
      }
    }
  }
  __syncthreads();
  for (int row = warp; row < 16; row += kWarps) {
    const int h = query_head(row);
    if (h < 0) continue;
    float m = -INFINITY, l = 0.f, f[kWarps];
#pragma unroll
    for (int w = 0; w < kWarps; ++w) m = fmaxf(m, st[(w * 16 + row) * 2]);
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float mw = st[(w * 16 + row) * 2];
      f[w] = mw > -INFINITY ? Exp2(mw - m) : 0.f;
      l = fmaf(st[(w * 16 + row) * 2 + 1], f[w], l);
    }
    float* d = records + static_cast<size_t>(h) * rec;
    if (lane == 0) {
      d[0] = m;
      d[1] = l;
    }
    for (int c = lane; c < a.vdim; c += 32) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) v = fmaf(acc[static_cast<size_t>(w * 16 + row) * acc_ld + c], f[w], v);
      d[2 + c] = v;
    }
  }
}

constexpr int kGenericThreads = 128, kGenericCols = 8;  // up to 1024 value columns

// One CTA per (row, query head): 128 positions at a time.
template <typename T>
__global__ void __launch_bounds__(kGenericThreads) GroupedAttentionGeneric(const __grid_constant__ GroupedArgs a)
{
  GridDependencySync();
  extern __shared__ __align__(16) unsigned char smem[];
  float* q = reinterpret_cast<float*>(smem);
  __shared__ float p[kGenericThreads], red[4];
  __shared__ long long at[kGenericThreads];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  const int vh = h / (a.heads / a.v_heads), kh = vh * a.maps + h % a.maps;
  const T* qr = static_cast<const T*>(a.q) + (static_cast<size_t>(t) * a.heads + h) * a.dim;
  for (int c = tid; c < a.dim; c += kGenericThreads) q[c] = ToF32(qr[c]);
  const Seen seen = SeenBy(a, t);
  const T* pool = static_cast<const T*>(a.pool);
  float top = -INFINITY, sum = 0.f, acc[kGenericCols] = {};
  for (int i0 = 0; i0 < seen.count; i0 += kGenericThreads) {
    const int n = min(kGenericThreads, seen.count - i0);
    __syncthreads();
    float s = -INFINITY;
    if (tid < n) {
      const long long row = PoolRow(a, seen, i0 + tid) * a.pool_ld;
      at[tid] = row + a.v_first + static_cast<long long>(vh) * a.vdim;
      const T* k = pool + row + static_cast<long long>(kh) * a.dim;
      float d = 0.f;
      for (int c = 0; c < a.dim; ++c) d = fmaf(q[c], ToF32(k[c]), d);
      s = d * a.scale_log2;
    }
    float m = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    if ((tid & 31) == 0) red[tid >> 5] = m;
    __syncthreads();
    m = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), top);
    const float keep = exp2f(top - m);  // top starts at -inf: 0
    top = m;
    const float w = tid < n ? exp2f(s - m) : 0.f;
    p[tid] = w;
    sum = sum * keep + w;  // this thread's share
    __syncthreads();
#pragma unroll
    for (int j = 0; j < kGenericCols; ++j) {
      const int c = tid + j * kGenericThreads;
      if (c >= a.vdim) break;
      float v = acc[j] * keep;
      for (int i = 0; i < n; ++i) v = fmaf(p[i], ToF32(pool[at[i] + c]), v);
      acc[j] = v;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  __syncthreads();
  if ((tid & 31) == 0) red[tid >> 5] = sum;
  __syncthreads();
  const int rec = a.vdim + 2;
  float* d = a.records + (static_cast<size_t>(t) * a.heads + h) * rec;
  if (tid == 0) {
    d[0] = top;
    d[1] = red[0] + red[1] + red[2] + red[3];
  }
#pragma unroll
  for (int j = 0; j < kGenericCols; ++j) {
    const int c = tid + j * kGenericThreads;
    if (c < a.vdim) d[2 + c] = acc[j];
  }
}

// Stages of a warp's ring that fit beside the alignment slack; 0: none.
int Stages(int maps, int dim, int vdim, size_t* smem)
{
  const size_t stage = static_cast<size_t>(maps * ((dim + 63) / 64) + (vdim + 63) / 64) * kAtom;
  const size_t merge = sizeof(float) * (kWarps * 32 + static_cast<size_t>(kWarps) * 16 * (vdim + 4));
  int n = stage <= 8192 ? 3 : kMaxStages;  // small stages: two CTAs per SM
  while (n > 0 && kWarps * n * stage + 1024 > kMaxSmem - 1024) --n;
  if (smem != nullptr) *smem = (kWarps * n * stage > merge ? kWarps * n * stage : merge) + 1024;
  return n;
}
bool MmaApplies(int maps, int dim, int vdim, int block_size, int dtype)
{
  return dtype == TLALOC_B200_BF16 && (maps == 1 || maps == 2) && dim % 16 == 0 && vdim % 16 == 0 && dim <= 128 && vdim <= 256 && block_size % kGroup == 0 &&
         Stages(maps, dim, vdim, nullptr) >= 2 && !OrderFaithful() && TensorMapEncoder() != nullptr;
}
using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// The pool as rows of pool_ld channels, boxes of 64 channels x 16 rows.
bool EncodePool(CUtensorMap* map, const void* pool, int64_t pool_ld, int64_t rows)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  const cuuint64_t dims[2] = {static_cast<cuuint64_t>(pool_ld), static_cast<cuuint64_t>(rows)};
  const cuuint64_t strides[1] = {static_cast<cuuint64_t>(pool_ld) * 2};
  const cuuint32_t box[2] = {64, kGroup}, elem[2] = {1, 1};
  return encode != nullptr &&
         encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(pool), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
int QueryTiles(int heads, int v_heads, int maps)
{
  const int per_map = heads / v_heads / maps, rows = 16 / maps;
  return (per_map + rows - 1) / rows;
}

// (channels of a key head, of a value head) / 16, in whole atoms
#define TLALOC_GROUPED_SIZES(F) F(4, 4) F(4, 8) F(4, 12) F(4, 16) F(8, 4) F(8, 8) F(8, 12) F(8, 16)

cudaError_t PrepareGrouped()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(DK, NV) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(GroupedAttentionMma<DK, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024);
    TLALOC_GROUPED_SIZES(TLALOC_OPT_IN)
#undef TLALOC_OPT_IN
    return e;
  });
}
int ReadGroupedStatus()
{
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_grouped_status, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_grouped_status, &zero, sizeof(int));
  }
  return v;
}
KernelSetup g_setup(PrepareGrouped, ReadGroupedStatus);

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_grouped_attention_slices(int32_t num_tokens, int32_t num_heads, int32_t v_heads, int32_t maps, int32_t dim, int32_t vdim,
                                                    int32_t block_size, int32_t dtype, int32_t max_live)
{
  if (num_tokens < 1 || v_heads < 1 || maps < 1 || num_heads < 1 || block_size < 1 || !MmaApplies(maps, dim, vdim, block_size, dtype)) return 1;
  // Enough CTAs for several waves, but no slice under 256 positions: each warp should have a few groups.
  const long long ctas = static_cast<long long>(num_tokens) * v_heads * QueryTiles(num_heads, v_heads, maps);
  long long s = (768 + ctas - 1) / ctas;
  const long long most = (max_live + 255) / 256;
  if (s > most) s = most;
  return s < 1 ? 1 : s > 512 ? 512 : static_cast<int>(s);
}

extern "C" int tlaloc_b200_grouped_attention(const void* q, const void* pool, int64_t pool_ld, int32_t dtype, const int32_t* block_tables,
                                             const int32_t* row_tables, const int32_t* seq_lens, float* records, int32_t slices, int32_t num_tokens,
                                             int32_t num_heads, int32_t v_heads, int32_t maps, int32_t dim, int32_t vdim, int32_t v_first,
                                             int32_t num_blocks, int32_t block_size, int32_t max_blocks, int32_t num_tables, int32_t window,
                                             int32_t keep_first, float scale, void* stream)
{
  const char* op = "GROUPED_ATTENTION";
  if (!q || !pool || !block_tables || !seq_lens || !records) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (num_tokens < 0 || num_tokens > 65535 || v_heads < 1 || maps < 1 || num_heads < 1 || num_heads % (v_heads * maps) || dim < 1 || vdim < 1 ||
      num_blocks < 1 || block_size < 1 || max_blocks < 1 || num_tables < 1 || window < 0 || keep_first < 0 || slices < 1) {
    return Fail(kInvalid, "%s: bad sizes", op);
  }
  if (v_first < v_heads * maps * dim || pool_ld < static_cast<int64_t>(v_first) + static_cast<int64_t>(v_heads) * vdim) {
    return Fail(kInvalid, "%s: a pool row is shorter than its heads", op);
  }
  if (num_tokens == 0) return kOk;
  GroupedArgs a = {};
  a.q = q;
  a.pool = pool;
  a.tables = block_tables;
  a.row_tables = row_tables;
  a.lens = seq_lens;
  a.records = records;
  a.pool_ld = pool_ld;
  a.T = num_tokens;
  a.heads = num_heads;
  a.v_heads = v_heads;
  a.maps = maps;
  a.dim = dim;
  a.vdim = vdim;
  a.v_first = v_first;
  a.num_blocks = num_blocks;
  a.block_size = block_size;
  a.max_blocks = max_blocks;
  a.num_tables = num_tables;
  a.window = window;
  a.keep = window > 0 ? keep_first : 0;
  a.slices = slices;
  a.qtiles = QueryTiles(num_heads, v_heads, maps);
  a.scale_log2 = scale * 1.4426950408889634f;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (MmaApplies(maps, dim, vdim, block_size, dtype)) {
    if (pool_ld % 8 || v_first % 8 || !Aligned16(q) || !Aligned16(pool)) return Fail(kInvalid, "%s: addresses and strides must be multiples of 16 bytes", op);
    if (static_cast<long long>(v_heads) * a.qtiles > 65535) return Fail(kInvalid, "%s: too many heads", op);
    e = PrepareGrouped();
    if (e != cudaSuccess) return CudaFail("GROUPED_ATTENTION set-up", e);
    CUtensorMap map;
    if (static_cast<int64_t>(num_blocks) * block_size > INT32_MAX || !EncodePool(&map, pool, pool_ld, static_cast<int64_t>(num_blocks) * block_size)) {
      return Fail(kInternal, "%s: the tensor map could not be encoded", op);
    }
    size_t smem = 0;
    a.stages = Stages(maps, dim, vdim, &smem);
    const dim3 grid(slices, v_heads * a.qtiles, num_tokens);
    const int dk = (dim + 63) / 64 * 4, nv = (vdim + 63) / 64 * 4;
    e = cudaErrorInvalidValue;
#define TLALOC_LAUNCH(DK, NV) \
  if (dk == DK && nv == NV) e = LaunchChained(GroupedAttentionMma<DK, NV>, grid, kWarps * 32, smem, st, map, a);
    TLALOC_GROUPED_SIZES(TLALOC_LAUNCH)
#undef TLALOC_LAUNCH
  } else {
    if (slices != 1) return Fail(kInvalid, "%s: one slice at these sizes", op);
    if (vdim > kGenericThreads * kGenericCols || dim > 8192) return Fail(kUnsupported, "%s: vdim up to %d", op, kGenericThreads * kGenericCols);
    const dim3 grid(num_heads, num_tokens);
    const size_t smem = sizeof(float) * dim;
    e = dtype == TLALOC_B200_F32 ? LaunchChained(GroupedAttentionGeneric<float>, grid, kGenericThreads, smem, st, a)
                                 : LaunchChained(GroupedAttentionGeneric<__nv_bfloat16>, grid, kGenericThreads, smem, st, a);
  }
  if (e != cudaSuccess) return CudaFail("GROUPED_ATTENTION launch", e);
  CountLaunches(1);
  return kOk;
}
