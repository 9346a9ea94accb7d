// Attention of single tokens over a paged pool of grouped key and value heads, with a sliding window and kept first tokens, one or two
// maps of scores per query head over the same values (include/tlaloc_b200.h, tlaloc_b200_grouped_attention).
//
// The positions a row sees are counted through: the kept ones, then those of the window.  They are cut into groups of 16 and, when there
// are few rows, into slices; each slice leaves a record per query head ({largest score (log2), sum, weighted values}), and the operator
// that consumes the result merges them.
//   GroupedAttentionMma      bf16.  A CTA has one value head, up to 16 of its query heads (8 of two maps each) and one slice, so every cached
//                            byte of the slice is read once for all of them.  Four warps, each with groups and a three-stage ring of its own,
//                            fed by 16-byte cp.async copies through the block table: no barrier in the loop.  Query heads are the rows of
//                            mma.m16n8k16; with two maps the rows 0-7 are the heads' first map and 8-15 the second, each multiplied with its
//                            own keys, so that one product with the values serves both.  The weights enter that product as two bf16
//                            parts (f32 up to rounding).
//   GroupedAttentionGeneric  any size and type, plain FMA: the f32 path.
#include "common.cuh"

namespace tlaloc_b200 {
namespace {

constexpr int kGroup = 16, kWarps = 4, kStages = 3;
constexpr int kMaxSmem = 227 * 1024;

struct GroupedArgs {
  const void* q;
  const void* pool;
  const int *tables, *row_tables, *lens;
  float* records;
  int64_t pool_ld;
  int T, heads, v_heads, maps, dim, vdim, v_first, num_blocks, block_size, max_blocks, num_tables, window, keep, slices, qtiles;
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

// DK: 16-channel steps of a key head at most, NV: 16-channel steps of a value head at most.
template <int DK, int NV>
__global__ void __launch_bounds__(kWarps * 32) GroupedAttentionMma(const __grid_constant__ GroupedArgs a)
{
  GridDependencySync();
  extern __shared__ __align__(16) unsigned char smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slice = blockIdx.x, vh = blockIdx.y / a.qtiles, qt = blockIdx.y % a.qtiles, t = blockIdx.z;
  const int group = a.heads / a.v_heads, per_map = group / a.maps;  // query heads (with maps counted) and without
  const int rows_per_map = 16 / a.maps;
  const int dk = a.dim >> 4, nv = a.vdim >> 4;
  const Seen seen = SeenBy(a, t);
  const int groups = (seen.count + kGroup - 1) / kGroup, share = (groups + a.slices - 1) / a.slices;
  const int g0 = slice * share, g1 = min(groups, g0 + share);
  // The query head of MMA row r: (place in the group, map).
  auto query_head = [&](int r) {
    const int place = qt * rows_per_map + r % rows_per_map, map = r / rows_per_map;
    return place < per_map ? (vh * per_map + place) * a.maps + map : -1;
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

  // A stage: 16 rows of [maps x dim] keys, then 16 rows of values; rows 16 bytes longer than their content (ldmatrix without conflicts).
  const int k_bytes = a.maps * a.dim * 2, k_ld = k_bytes + 16, v_ld = a.vdim * 2 + 16, stage_bytes = kGroup * (k_ld + v_ld);
  const uint32_t ring = static_cast<uint32_t>(__cvta_generic_to_shared(smem)) + warp * kStages * stage_bytes;
  const int k_chunks = k_bytes >> 4, chunks = k_chunks + (a.vdim >> 3);
  int span = 2;  // lanes of a row of chunks: a power of two
  while (span < chunks && span < 32) span <<= 1;
  const int c_lane = lane & (span - 1), r_lane = lane / span, r_step = 32 / span;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(a.pool);
  const int k_col = vh * a.maps * a.dim, v_col = a.v_first + vh * a.vdim;
  auto load = [&](int g, int stage) {
    if (g < g1) {
      const int i = g * kGroup + (lane & 15);
      long long off = -1;
      if (i < seen.count) off = PoolRow(a, seen, i) * a.pool_ld;
      const uint32_t base = ring + stage * stage_bytes;
      for (int r = r_lane; r < kGroup; r += r_step) {
        const long long o = __shfl_sync(0xffffffffu, off, r);
        for (int c = c_lane; c < chunks; c += span) {
          const bool key = c < k_chunks;
          const __nv_bfloat16* src = pool + (o < 0 ? 0 : o) + (key ? k_col + c * 8 : v_col + (c - k_chunks) * 8);
          const uint32_t dst = base + (key ? r * k_ld + c * 16 : kGroup * k_ld + r * v_ld + (c - k_chunks) * 16);
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(o < 0 ? 0 : 16) : "memory");  // dead rows: zeros
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };

  float o[2 * NV][4], top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (int s = 0; s < kStages - 1; ++s) load(g0 + warp + s * kWarps, s);
  int stage = 0;
  for (int g = g0 + warp; g < g1; g += kWarps) {
    {
      int ahead = stage + kStages - 1;
      if (ahead >= kStages) ahead -= kStages;
      load(g + (kStages - 1) * kWarps, ahead);
    }
    asm volatile("cp.async.wait_group %0;\n" ::"n"(kStages - 1) : "memory");
    __syncwarp();
    const uint32_t kt = ring + stage * stage_bytes, vt = kt + kGroup * k_ld;
    float s[2][4] = {};
    {
      const int m = lane >> 3;
      const uint32_t at = kt + ((m >> 1) * 8 + (lane & 7)) * k_ld + (m & 1) * 16;
      if (a.maps == 2) {
        const uint32_t at2 = at + a.dim * 2;
#pragma unroll
        for (int k = 0; k < DK; ++k) {
          if (k < dk) {
            uint32_t b[4];
            Ldm4(b, at + k * 32);
            Mma(s[0], qa[k][0], 0u, qa[k][1], 0u, b[0], b[1]);
            Mma(s[1], qa[k][0], 0u, qa[k][1], 0u, b[2], b[3]);
            Ldm4(b, at2 + k * 32);
            Mma(s[0], 0u, qb[k][0], 0u, qb[k][1], b[0], b[1]);
            Mma(s[1], 0u, qb[k][0], 0u, qb[k][1], b[2], b[3]);
          }
        }
      } else {
#pragma unroll
        for (int k = 0; k < DK; ++k) {
          if (k < dk) {
            uint32_t b[4];
            Ldm4(b, at + k * 32);
            Mma(s[0], qa[k][0], qb[k][0], qa[k][1], qb[k][1], b[0], b[1]);
            Mma(s[1], qa[k][0], qb[k][0], qa[k][1], qb[k][1], b[2], b[3]);
          }
        }
      }
    }
    const int i0 = g * kGroup + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = i0 + n * 8 + (e & 1) < seen.count ? s[n][e] * a.scale_log2 : -INFINITY;
    float p[2][4];
    bool raise = false;
    float next[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float m = fmaxf(fmaxf(s[0][2 * r], s[0][2 * r + 1]), fmaxf(s[1][2 * r], s[1][2 * r + 1]));
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
      next[r] = fmaxf(top[r], m);  // the group's first position is live: finite from here on
      raise = raise || next[r] > top[r];
    }
    if (__any_sync(0xffffffffu, raise)) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float keep = Exp2(top[r] - next[r]);
        top[r] = next[r];
        sum[r] *= keep;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) {
          o[i][2 * r] *= keep;
          o[i][2 * r + 1] *= keep;
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
    uint32_t hi[4], lo[4];  // as A: (row, k 0-7), (row + 8, k 0-7), (row, k 8-15), (row + 8, k 8-15)
    Split(p[0][0], p[0][1], hi[0], lo[0]);
    Split(p[0][2], p[0][3], hi[1], lo[1]);
    Split(p[1][0], p[1][1], hi[2], lo[2]);
    Split(p[1][2], p[1][3], hi[3], lo[3]);
    const int m = lane >> 3;
    const uint32_t at = vt + ((m & 1) * 8 + (lane & 7)) * v_ld + (m >> 1) * 16;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      if (j < nv) {
        uint32_t b[4];
        Ldm4T(b, at + j * 32);
        Mma(o[2 * j], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
        Mma(o[2 * j + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
        Mma(o[2 * j], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
        Mma(o[2 * j + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
      }
    }
    __syncwarp();  // the stage is read before it is filled again
    if (++stage == kStages) stage = 0;
  }
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
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
      if (i < 2 * nv) {
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

size_t MmaSmem(int maps, int dim, int vdim)
{
  const size_t ring = static_cast<size_t>(kWarps) * kStages * kGroup * (maps * dim * 2 + 16 + vdim * 2 + 16);
  const size_t merge = sizeof(float) * (kWarps * 32 + static_cast<size_t>(kWarps) * 16 * (vdim + 4));
  return ring > merge ? ring : merge;
}
bool MmaApplies(int maps, int dim, int vdim, int dtype)
{
  return dtype == TLALOC_B200_BF16 && (maps == 1 || maps == 2) && dim % 16 == 0 && vdim % 16 == 0 && dim <= 128 && vdim <= 256 &&
         MmaSmem(maps, dim, vdim) <= kMaxSmem && !OrderFaithful();
}
int QueryTiles(int heads, int v_heads, int maps)
{
  const int per_map = heads / v_heads / maps, rows = 16 / maps;
  return (per_map + rows - 1) / rows;
}

#define TLALOC_GROUPED_SIZES(F) F(4, 4) F(4, 8) F(4, 16) F(8, 4) F(8, 8) F(8, 16)

cudaError_t PrepareGrouped()
{
  static OncePerDevice once;
  return once.Run([](int) {
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(DK, NV) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(GroupedAttentionMma<DK, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
    TLALOC_GROUPED_SIZES(TLALOC_OPT_IN)
#undef TLALOC_OPT_IN
    return e;
  });
}
KernelSetup g_setup(PrepareGrouped, nullptr);

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_grouped_attention_slices(int32_t num_tokens, int32_t num_heads, int32_t v_heads, int32_t maps, int32_t dim, int32_t vdim,
                                                    int32_t dtype, int32_t max_live)
{
  if (num_tokens < 1 || v_heads < 1 || maps < 1 || num_heads < 1 || !MmaApplies(maps, dim, vdim, dtype)) return 1;
  // Enough CTAs for several waves, but no slice under 256 positions: each warp should have a few groups.
  const long long ctas = static_cast<long long>(num_tokens) * v_heads * QueryTiles(num_heads, v_heads, maps);
  long long s = (2048 + ctas - 1) / ctas;
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
  if (MmaApplies(maps, dim, vdim, dtype)) {
    if (pool_ld % 8 || v_first % 8 || !Aligned16(q) || !Aligned16(pool)) return Fail(kInvalid, "%s: addresses and strides must be multiples of 16 bytes", op);
    if (static_cast<long long>(v_heads) * a.qtiles > 65535) return Fail(kInvalid, "%s: too many heads", op);
    e = PrepareGrouped();
    if (e != cudaSuccess) return CudaFail("GROUPED_ATTENTION set-up", e);
    const dim3 grid(slices, v_heads * a.qtiles, num_tokens);
    const size_t smem = MmaSmem(maps, dim, vdim);
    const int dk = dim <= 64 ? 4 : 8, nv = vdim <= 64 ? 4 : vdim <= 128 ? 8 : 16;
    e = cudaErrorInvalidValue;
#define TLALOC_LAUNCH(DK, NV) \
  if (dk == DK && nv == NV) e = LaunchChained(GroupedAttentionMma<DK, NV>, grid, kWarps * 32, smem, st, a);
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
