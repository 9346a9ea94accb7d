// The bf16 projection on the tensor cores (include/tlaloc_b200.h, tlaloc_b200_dense_gemm): tcgen05.mma kind::f16 with f32
// accumulators in TMEM, both operands by TMA.
//
// Formulation: D[n, m] = sum_k W[n, k] X[m, k]: 128 WEIGHT rows are the MMA's M (TMEM lanes), a tile of 32 to 256 activation
// rows its N (TMEM columns).  So a decode step of a few rows wastes no lane on absent rows (the weights, which are all of its
// traffic, fill every tile), and a lane owns one output column: the 32 lanes of a warp store 32 consecutive outputs of
// a row without a detour through shared memory, and a bias is one register.
//
// A CTA has a producer lane (per block of 64 k: one box of weights, one of activations, 128-byte swizzle, onto the stage's mbarrier),
// an MMA lane (4 K-steps of 16, then a commit that hands the stage back), and eight epilogue warps.  Two forms:
//   persistent (many tiles)  a CTA walks tiles with two accumulators: the epilogue of one tile runs under the MMAs of the next;
//   K slices (few tiles)     the slices of one tile are a cluster; each leaves its partial tile in shared memory and the ranks
//                            finish every ks-th activation row, summing in rank order through distributed shared memory.
// Rows, columns and k past the ends are outside the tensor maps and arrive as zeros.  Every mbarrier wait is bounded.
//
// Grouped problems (experts): the weights are a batch, the activations one matrix whose rows are sorted by weight.  How many tiles
// a weight has is known on the device alone: each CTA counts them from the row offsets, and a tile that passes the end of its
// weight's rows computes rows of the next one too and leaves them out.  Gated activations: gate and other factor are sixteen
// lanes apart; two activation rows at a time, the half warps exchange one value each and both evaluate one output.
#include <cuda.h>

#include "common.cuh"
#include "dense_gemm.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

using namespace tc;

constexpr int kBN = 128, kBK = 64;  // weight rows and k of one block
constexpr int kWBytes = kBN * kBK * 2;
constexpr int kEpiWarps = 8;
constexpr int kThreads = kEpiWarps * 32 + 64;

template <int BT>
struct Layout {
  static constexpr int kXBytes = BT * kBK * 2;
  static constexpr int kStage = kWBytes + kXBytes;
  static constexpr int kStages = BT == 256 ? 4 : BT == 128 ? 6 : 8;
  static constexpr int kPipe = kStages * kStage;
  static constexpr int kTileStride = kBN + 4;  // the slice's partial tile [BT][kTileStride] f32, aliases the ring
  static_assert(kPipe >= BT * kTileStride * 4 || BT == 256, "the partial tile aliases the ring");
  static constexpr int kRows = BT / 2 < 32 ? BT / 2 : 32;          // activation rows an epilogue group takes at a time
  static constexpr int kOut = kPipe;                               // two groups' bf16 output rows [kRows][128]
  static constexpr int kBars = kOut + 2 * kRows * kBN * 2;
  static constexpr int kSlot = kBars + 8 * (2 * kStages + 4);
  static constexpr int kBytes = kSlot + 8 + 1024;  // slack to align to 1024
};

struct TcProblem {
  const float* bias;
  const float* residual;
  const int* offsets;  // grouped: [groups + 1]
  void* y;
  int64_t ld_res, ld_y, batch_y;
  int M, tiles_m;
  int k, n, act, y_f32, rows_bf16, tiles_n, swap_x, gated, groups;  // rows_bf16: y takes whole 16-byte words; swap_x: the activations' map has the batch before the rows
};
struct TcArgs {
  TcProblem p[2];
  int tiles0, tiles, ks, weights_const;  // a grouped problem's tiles are not counted here
};

__device__ int g_dense_status = 0;  // nonzero after an mbarrier wait timed out (sticky until read)

__host__ __device__ constexpr uint32_t InstrDescBf16(int n)  // f32 accumulator, bf16 A and B, both K-major, M = 128
{
  return (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(n >> 3) << 17) | (8u << 24);
}
// x (the k coordinate) is a multiple of 64 elements: always a 16-byte boundary.
__device__ __forceinline__ void TmaBox3d(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar, uint64_t policy)
{
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint [%0], [%1, {%2, %3, %4}], [%5], %6;\n" ::"r"(dst),
      "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(z), "r"(bar), "l"(policy)
      : "memory");
}
struct Tile {
  int pr, n0, m0, b, M;  // M: first row that is not the tile's to write
};
// start: of a grouped problem (the last one), the first tile of every group, counted from the problem's own first tile.
template <bool GROUPED>
__device__ __forceinline__ Tile TileAt(const TcArgs& a, int id, int BT, const int* start)
{
  Tile t;
  t.pr = id >= a.tiles0 ? 1 : 0;
  if (t.pr) id -= a.tiles0;
  const TcProblem& p = a.p[t.pr];
  if (GROUPED && p.offsets != nullptr) {
    int lo = 0, hi = p.groups;  // start[lo] <= id < start[hi]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (start[mid] <= id) lo = mid;
      else hi = mid;
    }
    id -= start[lo];
    t.b = lo;
    const int first = p.offsets[lo], tiles_m = (start[lo + 1] - start[lo]) / p.tiles_n;
    t.M = p.offsets[lo + 1];
    t.m0 = first + (id % tiles_m) * BT;
    t.n0 = (id / tiles_m) * kBN;
    return t;
  }
  t.M = p.M;
  t.m0 = (id % p.tiles_m) * BT;  // activation tiles of one weight tile run side by side: the weights leave HBM once
  id /= p.tiles_m;
  t.n0 = (id % p.tiles_n) * kBN;
  t.b = id / p.tiles_n;
  return t;
}

// v: CH rows of the warp's 32 columns, gate in the lower sixteen lanes -> CH / 2 outputs of column 16 quad + (lane & 15), of rows
// 2 i + (lane >> 4).
template <int CH>
__device__ __forceinline__ void Gate(int act, float* v, int lane)
{
  const bool upper = lane >= kGateBlock;
#pragma unroll
  for (int i = 0; i < CH / 2; ++i) {
    const float a = v[2 * i], b = v[2 * i + 1];
    const float got = __shfl_xor_sync(0xffffffffu, upper ? a : b, kGateBlock);
    v[i] = GatedValue(act, upper ? got : a, upper ? b : got);
  }
}
template <int CH>
__device__ __forceinline__ void StoreGated(const TcProblem& p, const Tile& t, int quad, int lane, int m, int M, const float* v)
{
  const int n = (t.n0 >> 1) + quad * kGateBlock + (lane & 15);
  if (n >= p.n / 2) return;
#pragma unroll
  for (int i = 0; i < CH / 2; ++i) {
    const int r = m + 2 * i + (lane >> 4);
    if (r >= M) return;
    const size_t at = t.b * p.batch_y + static_cast<size_t>(r) * p.ld_y + n;
    if (p.y_f32) static_cast<float*>(p.y)[at] = v[i];
    else static_cast<__nv_bfloat16*>(p.y)[at] = __float2bfloat16_rn(v[i]);
  }
}

// One output column n of CH consecutive rows from m: bias, activation, residual, store.
template <int CH, typename YT>
__device__ __forceinline__ void StoreColumnAs(const TcProblem& p, YT* y, const float* res, int rows, const float* v, float bias)
{
  const int64_t ld = p.ld_y, ld_res = p.ld_res;
  const int act = p.act;
  float r[CH];
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    r[c] = 0.f;
    if (res != nullptr && c < rows) {
      r[c] = *res;
      res += ld_res;
    }
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    if (c < rows) *y = FromF32<YT>(DenseActivation(act, v[c] + bias) + r[c]);
    y += ld;
  }
}
template <int CH>
__device__ __forceinline__ void StoreColumn(const TcProblem& p, const Tile& t, int n, int m, int M, const float* v, float bias)
{
  const int rows = min(CH, M - m);
  if (n >= p.n || rows <= 0) return;
  const float* res = p.residual != nullptr ? p.residual + static_cast<size_t>(m) * p.ld_res + n : nullptr;
  const size_t at = t.b * p.batch_y + static_cast<size_t>(m) * p.ld_y + n;
  if (p.y_f32) StoreColumnAs<CH>(p, static_cast<float*>(p.y) + at, res, rows, v, bias);
  else StoreColumnAs<CH>(p, static_cast<__nv_bfloat16*>(p.y) + at, res, rows, v, bias);
}

// The same for a whole 128-column bf16 tile of a group of four warps: the rows meet in shared memory and leave as 16-byte words.
template <int CH>
__device__ __forceinline__ void StoreRowsBf16(const TcProblem& p, const Tile& t, int m, int M, const float* v, float bias, __nv_bfloat16* stage,
                                              int tid, int group)
{
  const int col = tid & 127;
  if (p.act == TLALOC_B200_ACT_RELU2) {
#pragma unroll
    for (int c = 0; c < CH; ++c) stage[c * kBN + col] = __float2bfloat16_rn(DenseActivation(TLALOC_B200_ACT_RELU2, v[c] + bias));
  } else {
#pragma unroll
    for (int c = 0; c < CH; ++c) stage[c * kBN + col] = __float2bfloat16_rn(v[c] + bias);
  }
  asm volatile("bar.sync %0, 128;\n" ::"r"(1 + group) : "memory");
  const int64_t ld = p.ld_y;
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.y) + t.b * p.batch_y + static_cast<size_t>(m) * ld + t.n0 + (col & 15) * 8;
  const uint4* src = reinterpret_cast<const uint4*>(stage) + (col & 15);
#pragma unroll
  for (int i = 0; i < CH / 8; ++i) {
    const int r = i * 8 + (col >> 4);
    if (m + r < M) *reinterpret_cast<uint4*>(y + r * ld) = src[r * 16];
  }
  asm volatile("bar.sync %0, 128;\n" ::"r"(1 + group) : "memory");
}

// The same for the 64 outputs a row of a gated tile has.
template <int CH>
__device__ __forceinline__ void StoreRowsGatedBf16(const TcProblem& p, const Tile& t, int m, int M, const float* v, __nv_bfloat16* stage, int tid,
                                                   int group)
{
  const int col = tid & 127, lane = tid & 31, quad = col >> 5;
  constexpr int kW = kBN / 2;
#pragma unroll
  for (int i = 0; i < CH / 2; ++i) stage[(2 * i + (lane >> 4)) * kW + quad * kGateBlock + (lane & 15)] = __float2bfloat16_rn(v[i]);
  asm volatile("bar.sync %0, 128;\n" ::"r"(1 + group) : "memory");
  const int64_t ld = p.ld_y;
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.y) + t.b * p.batch_y + static_cast<size_t>(m) * ld + (t.n0 >> 1) + (col & 7) * 8;
  const uint4* src = reinterpret_cast<const uint4*>(stage) + (col & 7);
#pragma unroll
  for (int i = 0; i < CH / 16; ++i) {
    const int r = i * 16 + (col >> 3);
    if (m + r < M) *reinterpret_cast<uint4*>(y + r * ld) = src[r * 8];
  }
  asm volatile("bar.sync %0, 128;\n" ::"r"(1 + group) : "memory");
}

template <int BT, bool SPLIT, bool GROUPED = false>
__global__ void __launch_bounds__(kThreads, 1)
    DenseGemmTcKernel(const __grid_constant__ CUtensorMap w0, const __grid_constant__ CUtensorMap x0,
                      const __grid_constant__ CUtensorMap w1, const __grid_constant__ CUtensorMap x1, const __grid_constant__ TcArgs a)
{
  using L = Layout<BT>;
  constexpr int S = L::kStages;
  constexpr uint32_t kCols = SPLIT ? (BT < 32 ? 32 : BT) : 2 * BT;
  extern __shared__ unsigned char smem_raw[];
  const uint32_t base = (SmemAddr(smem_raw) + 1023u) & ~1023u;  // the swizzle is a function of address bits 4..9
  unsigned char* smem = smem_raw + (base - SmemAddr(smem_raw));
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t full = base + L::kBars, empty = full + 8 * S, tfull = empty + 8 * S, tempty = tfull + 16;
  volatile uint32_t* slot = reinterpret_cast<volatile uint32_t*>(smem + L::kSlot);
  volatile uint32_t* abort_word = slot + 1;
  if (tid == 0) {
    *abort_word = 0u;
    for (int i = 0; i < S; ++i) {
      MbarInit(full + 8 * i, 1);
      MbarInit(empty + 8 * i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      MbarInit(tfull + 8 * i, 1);
      MbarInit(tempty + 8 * i, kEpiWarps);
    }
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(base + L::kSlot), "r"(kCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *slot;
  __shared__ int s_start[GROUPED ? kMaxGroups + 1 : 1];
  int tiles = a.tiles;
  if constexpr (GROUPED) {
    GridDependencySync();
    const TcProblem& g = a.p[1].offsets != nullptr ? a.p[1] : a.p[0];
    if (warp == 0) {
      int total = 0;
      for (int e0 = 0; e0 < g.groups; e0 += 32) {
        const int e = e0 + lane;
        int v = e < g.groups ? (g.offsets[e + 1] - g.offsets[e] + BT - 1) / BT * g.tiles_n : 0;
        const int own = v;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const int u = __shfl_up_sync(0xffffffffu, v, o);
          if (lane >= o) v += u;
        }
        if (e < g.groups) s_start[e] = total + v - own;
        total += __shfl_sync(0xffffffffu, v, 31);
      }
      if (lane == 0) s_start[g.groups] = total;
    }
    __syncthreads();
    tiles += s_start[g.groups];
  }
  // The blocks of k of a tile this CTA sums: all of them, or the slice of its cluster rank.
  auto blocks = [&](const Tile& t, int& first) {
    const int nb = (a.p[t.pr].k + kBK - 1) / kBK;
    if (!SPLIT) {
      first = 0;
      return nb;
    }
    const int per = (nb + a.ks - 1) / a.ks;
    first = static_cast<int>(blockIdx.y) * per;
    return max(0, min(per, nb - first));
  };
  bool ok = true;

  if (warp == kEpiWarps) {
    if (ElectOne()) {
      uint64_t w_policy, x_policy;
      if (a.p[0].tiles_m == 1) asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;\n" : "=l"(w_policy));
      else asm volatile("createpolicy.fractional.L2::evict_normal.b64 %0, 1.0;\n" : "=l"(w_policy));
      asm volatile("createpolicy.fractional.L2::evict_last.b64 %0, 1.0;\n" : "=l"(x_policy));
      auto load_w = [&](const Tile& t, int kb, int s) {
        TmaBox3d(base + s * L::kStage, t.pr ? &w1 : &w0, kb * kBK, t.n0, t.b, full + 8 * s, w_policy);
      };
      auto load_x = [&](const Tile& t, int kb, int s) {
        const bool swap = a.p[t.pr].swap_x != 0;
        const int z = GROUPED && a.p[t.pr].offsets != nullptr ? 0 : t.b;
        TmaBox3d(base + s * L::kStage + kWBytes, t.pr ? &x1 : &x0, kb * kBK, swap ? z : t.m0, swap ? t.m0 : z, full + 8 * s, x_policy);
      };
      // Constant weights of the first stages travel before the dependency wait; activations only after it.
      Tile t;
      int first = 0, nb = 0;
      if (!GROUPED) {
        t = TileAt<GROUPED>(a, blockIdx.x, BT, s_start);
        nb = blocks(t, first);
      }
      const int ahead = !GROUPED && a.weights_const ? min(nb, S) : 0;
      for (int b = 0; b < ahead; ++b) {
        MbarExpectTx(full + 8 * b, L::kStage);
        load_w(t, first + b, b);
      }
      if (!GROUPED) GridDependencySync();
      for (int b = 0; b < ahead; ++b) load_x(t, first + b, b);
      int it = ahead, b = ahead;
      for (int id = blockIdx.x; id < tiles; id += gridDim.x) {
        if (GROUPED || id != static_cast<int>(blockIdx.x)) {
          t = TileAt<GROUPED>(a, id, BT, s_start);
          nb = blocks(t, first);
          b = 0;
        }
        for (; b < nb; ++b, ++it) {
          const int s = it % S;
          if (it >= S) ok = MbarWait(empty + 8 * s, ((it / S) - 1) & 1, abort_word) && ok;
          MbarExpectTx(full + 8 * s, L::kStage);
          load_w(t, first + b, s);
          load_x(t, first + b, s);
        }
      }
      if (!ok)  // given up: let the copies in flight land before the CTA's shared memory goes away
        for (int s = 0; s < S; ++s)
          if (it > s) {
            volatile uint32_t never = 0;
            MbarWait(full + 8 * s, (((it - 1 - s) / S)) & 1, &never);
          }
    }
    __syncwarp();
  } else if (warp == kEpiWarps + 1) {
    if (!GROUPED) GridDependencySync();  // nothing to read, but the time limit of its waits then starts with the work
    if (ElectOne()) {
      constexpr uint32_t idesc = InstrDescBf16(BT);
      const uint64_t wd0 = SmemDesc(base, 16, 1024), xd0 = SmemDesc(base + kWBytes, 16, 1024);
      int it = 0, lt = 0;
      for (int id = blockIdx.x; id < tiles; id += gridDim.x, ++lt) {
        const Tile t = TileAt<GROUPED>(a, id, BT, s_start);
        int first;
        const int nb = blocks(t, first);
        const uint32_t acc = tmem + (lt & 1) * BT;
        if (lt >= 2) {
          ok = MbarWait(tempty + 8 * (lt & 1), ((lt / 2) - 1) & 1, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        }
        for (int b = 0; b < nb; ++b, ++it) {
          const int s = it % S;
          ok = MbarWait(full + 8 * s, (it / S) & 1, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          const uint64_t at = static_cast<uint64_t>((s * L::kStage) >> 4);
#pragma unroll
          for (int ks = 0; ks < kBK / 16; ++ks) TcMmaBf16(acc, wd0 + at + 2 * ks, xd0 + at + 2 * ks, idesc, (b > 0 || ks > 0) ? 1u : 0u);
          TcCommit(empty + 8 * s);
        }
        TcCommit(tfull + 8 * (lt & 1));
      }
    }
    __syncwarp();
  } else {
    if (!GROUPED) GridDependencySync();
    const int quad = warp & 3, half = warp >> 2;
    constexpr int kHalf = BT / 2, CH = kHalf < 32 ? kHalf : 32;
    int lt = 0;
    for (int id = blockIdx.x; id < tiles; id += gridDim.x, ++lt) {
      const Tile t = TileAt<GROUPED>(a, id, BT, s_start);
      int first;
      const int nb = blocks(t, first);
      const TcProblem& p = a.p[t.pr];
      const int n = t.n0 + quad * 32 + lane;
      const float bias = p.bias != nullptr && n < p.n ? __ldg(p.bias + n) : 0.f;
      ok = MbarWaitWarp(tfull + 8 * (lt & 1), (lt / 2) & 1, lane, abort_word) && ok;
      asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll 1
      for (int c = half * kHalf; c < (half + 1) * kHalf; c += CH) {
        if (!SPLIT && t.m0 + c >= t.M) break;
        uint32_t r[CH];
        const uint32_t taddr = tmem + (static_cast<uint32_t>(quad * 32) << 16) + (lt & 1) * BT + c;
        if constexpr (CH == 32) TcLd32(taddr, r);
        else TcLd16(taddr, r);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        if constexpr (SPLIT) {
          float* tile = reinterpret_cast<float*>(smem);
#pragma unroll
          for (int e = 0; e < CH; ++e) tile[(c + e) * L::kTileStride + quad * 32 + lane] = nb > 0 ? __uint_as_float(r[e]) : 0.f;
        } else {
          float v[CH];
#pragma unroll
          for (int e = 0; e < CH; ++e) v[e] = __uint_as_float(r[e]);
          __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(smem + L::kOut) + half * CH * kBN;
          if (p.gated) {
            Gate<CH>(p.act, v, lane);
            if (p.rows_bf16 && t.n0 + kBN <= p.n) StoreRowsGatedBf16<CH>(p, t, t.m0 + c, t.M, v, stage, tid, half);
            else StoreGated<CH>(p, t, quad, lane, t.m0 + c, t.M, v);
          } else if (p.rows_bf16 && t.n0 + kBN <= p.n) {
            StoreRowsBf16<CH>(p, t, t.m0 + c, t.M, v, bias, stage, tid, half);
          } else {
            StoreColumn<CH>(p, t, n, t.m0 + c, t.M, v, bias);
          }
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
      __syncwarp();
      if (lane == 0) MbarArrive(tempty + 8 * (lt & 1));
    }
  }
  if (!ok) atomicExch(&g_dense_status, 1);
  if constexpr (SPLIT) {
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();  // every slice's tile is in its CTA's shared memory
    if (warp < kEpiWarps) {
      const Tile t = TileAt<false>(a, blockIdx.x, BT, s_start);
      const TcProblem& p = a.p[t.pr];
      const int nl = tid & 127, n = t.n0 + nl, nr = static_cast<int>(cluster.num_blocks());
      const float bias = p.bias != nullptr && n < p.n ? __ldg(p.bias + n) : 0.f;
      float* tile = reinterpret_cast<float*>(smem);
      const int rows = min(BT, t.M - t.m0), step = 2 * nr;
      constexpr int kU = 4;
      for (int c0 = static_cast<int>(cluster.block_rank()) + nr * (tid >> 7); c0 < rows; c0 += kU * step) {
        float v[kU] = {};
        for (int q = 0; q < nr; ++q) {
          const float* peer = cluster.map_shared_rank(tile, q) + nl;
          float u[kU];
#pragma unroll
          for (int e = 0; e < kU; ++e) u[e] = c0 + e * step < rows ? peer[(c0 + e * step) * L::kTileStride] : 0.f;
#pragma unroll
          for (int e = 0; e < kU; ++e) v[e] += u[e];
        }
        if (p.gated) {
          // rows c0 + 2 i step of the lower lanes' results, + step of the upper ones'
          Gate<kU>(p.act, v, lane);
          const int col = (t.n0 >> 1) + (nl >> 5) * kGateBlock + (lane & 15);
#pragma unroll
          for (int i = 0; i < kU / 2; ++i) {
            const int r = c0 + (2 * i + (lane >> 4)) * step;
            if (r >= rows || col >= p.n / 2) continue;
            const size_t at = t.b * p.batch_y + static_cast<size_t>(t.m0 + r) * p.ld_y + col;
            if (p.y_f32) static_cast<float*>(p.y)[at] = v[i];
            else static_cast<__nv_bfloat16*>(p.y)[at] = __float2bfloat16_rn(v[i]);
          }
          continue;
        }
#pragma unroll
        for (int e = 0; e < kU; ++e)
          if (c0 + e * step < rows) StoreColumn<1>(p, t, n, t.m0 + c0 + e * step, t.M, v + e, bias);
      }
    }
    cluster.sync();  // no CTA leaves while a peer may still read its tile
  } else {
    __syncthreads();
  }
  if (warp == 0) {
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(kCols) : "memory");
  }
}

// ---- host -----------------------------------------------------------------------------------------------------------
using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 [batch][rows][k] with strides in elements, boxes of 64 k x box_rows rows; the dimension with the smaller stride comes
// first (*swap: the batch).
bool EncodeMatrix(CUtensorMap* map, const void* ptr, int64_t k, int64_t rows, int64_t batch, int64_t ld, int64_t batch_stride,
                  uint32_t box_rows, int* swap)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  if (encode == nullptr) return false;
  *swap = batch > 1 && batch_stride < ld ? 1 : 0;
  if (batch == 1) batch_stride = ld;
  const cuuint64_t k_dim = static_cast<cuuint64_t>(k), r_dim = static_cast<cuuint64_t>(rows), b_dim = static_cast<cuuint64_t>(batch);
  const cuuint64_t r_str = static_cast<cuuint64_t>(ld) * 2, b_str = static_cast<cuuint64_t>(batch_stride) * 2;
  const cuuint64_t dims[3] = {k_dim, *swap ? b_dim : r_dim, *swap ? r_dim : b_dim};
  const cuuint64_t strides[2] = {*swap ? b_str : r_str, *swap ? r_str : b_str};
  const cuuint32_t box[3] = {kBK, *swap ? 1u : box_rows, *swap ? box_rows : 1u};
  const cuuint32_t elem[3] = {1, 1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

int g_slots[kMaxDevices][9];  // resident CTAs when launched as clusters of ks

cudaError_t PrepareDenseTc()
{
  static OncePerDevice once;
  return once.Run([](int device) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(BT, SPLIT) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(DenseGemmTcKernel<BT, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Layout<BT>::kBytes)
    TLALOC_OPT_IN(32, false);
    TLALOC_OPT_IN(64, false);
    TLALOC_OPT_IN(128, false);
    TLALOC_OPT_IN(256, false);
    TLALOC_OPT_IN(32, true);
    TLALOC_OPT_IN(64, true);
    TLALOC_OPT_IN(128, true);
#define TLALOC_OPT_IN_GROUPED(BT) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(DenseGemmTcKernel<BT, false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Layout<BT>::kBytes)
    TLALOC_OPT_IN_GROUPED(32);
    TLALOC_OPT_IN_GROUPED(64);
    TLALOC_OPT_IN_GROUPED(128);
    TLALOC_OPT_IN_GROUPED(256);
#undef TLALOC_OPT_IN_GROUPED
#undef TLALOC_OPT_IN
    if (e != cudaSuccess) return e;
    for (int ks = 1; ks <= 8; ++ks) {
      cudaLaunchConfig_t cfg = {};
      cfg.gridDim = dim3(148, ks, 1);
      cfg.blockDim = dim3(kThreads, 1, 1);
      cfg.dynamicSmemBytes = Layout<128>::kBytes;
      cudaLaunchAttribute attr[1];
      attr[0].id = cudaLaunchAttributeClusterDimension;
      attr[0].val.clusterDim.x = 1;
      attr[0].val.clusterDim.y = ks;
      attr[0].val.clusterDim.z = 1;
      cfg.attrs = attr;
      cfg.numAttrs = 1;
      int clusters = 0;
      if (cudaOccupancyMaxActiveClusters(&clusters, DenseGemmTcKernel<128, true>, &cfg) != cudaSuccess || clusters <= 0) {
        cudaGetLastError();
        clusters = (ks <= 2 ? 148 : ks <= 4 ? 128 : 112) / ks;
      }
      g_slots[device][ks] = clusters * ks;
    }
    return cudaSuccess;
  });
}

int ReadDenseStatus()
{
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_dense_status, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_dense_status, &zero, sizeof(int));
  }
  return v;
}
KernelSetup g_setup(PrepareDenseTc, ReadDenseStatus);

// K slices (1..8), in units of one 64-k block of one CTA: waves * (blocks per slice + fixed cost [+ cluster reduction]).
int ChooseSlices(int tiles, int nb)
{
  int device = 0;
  if (cudaGetDevice(&device) != cudaSuccess || device < 0 || device >= kMaxDevices) device = 0;
  int best = 1;
  double best_cost = 1e30;
  for (int ks = 1; ks <= 8; ++ks) {
    if (ks > 1 && nb / ks < 2) break;
    const int slots = g_slots[device][ks] > 0 ? g_slots[device][ks] : 148 / ks * ks;
    const int waves = (tiles * ks + slots - 1) / slots;
    const double cost = waves * ((nb + ks - 1) / ks + 8.0 + (ks > 1 ? 6.0 + ks : 0.0));
    if (cost < best_cost * 0.97) {
      best_cost = cost;
      best = ks;
    }
  }
  return best;
}

template <int BT, bool SPLIT, bool GROUPED = false>
cudaError_t Launch(const CUtensorMap* maps, const TcArgs& a, int ctas, cudaStream_t st)
{
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(ctas, SPLIT ? a.ks : 1, 1);
  cfg.blockDim = dim3(kThreads, 1, 1);
  cfg.dynamicSmemBytes = Layout<BT>::kBytes;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  cfg.numAttrs = ChainAttributes(attr, SPLIT ? a.ks : 0);
  cfg.attrs = attr;
  return cudaLaunchKernelEx(&cfg, DenseGemmTcKernel<BT, SPLIT, GROUPED>, maps[0], maps[1], maps[2], maps[3], a);
}

}  // namespace

bool DenseGemmTcApplies(const tlaloc_b200_dense_problem& p)
{
  return p.ld_x % 8 == 0 && p.k % 8 == 0 && Aligned16(p.x) && Aligned16(p.w) && (p.batch == 1 || p.batch_x % 8 == 0) &&
         TensorMapEncoder() != nullptr;
}

cudaError_t LaunchDenseGemmTc(const tlaloc_b200_dense_problem* problems, int count, int m, bool weights_const, cudaStream_t st)
{
  cudaError_t e = PrepareDenseTc();
  if (e != cudaSuccess) return e;
  // Rows of a tile: what the problem has, or what a group has on average (one that has more takes several tiles).
  int typical = 1;
  bool grouped = false;
  for (int i = 0; i < count; ++i) {
    const tlaloc_b200_dense_problem& s = problems[i];
    const int rows = s.rows > 0 ? s.rows : m;
    typical = max(typical, s.row_offsets != nullptr ? (rows + s.batch - 1) / s.batch : rows);
    grouped = grouped || s.row_offsets != nullptr;
  }
  int bt = typical <= 32 ? 32 : typical <= 64 ? 64 : typical <= 128 ? 128 : 256;
  if (bt == 256 && !grouped) {  // half the rows a tile where that fills the last wave of CTAs better by more than its own loss (about a seventh)
    int columns = 0;
    for (int i = 0; i < count; ++i) columns += (problems[i].n + kBN - 1) / kBN * problems[i].batch;
    auto waves = [&](int rows) { return (columns * ((typical + rows - 1) / rows) + 147) / 148; };
    if (waves(128) * 128 * 1.15 < waves(256) * 256) bt = 128;
  }
  CUtensorMap maps[4];
  TcArgs a = {};
  a.weights_const = weights_const ? 1 : 0;
  int nb = 1 << 30;
  for (int i = 0; i < count; ++i) {
    const tlaloc_b200_dense_problem& s = problems[i];
    TcProblem& p = a.p[i];
    int swap_w = 0;
    const bool groups = s.row_offsets != nullptr;
    p.M = s.rows > 0 ? s.rows : m;
    p.tiles_m = (p.M + bt - 1) / bt;
    p.offsets = s.row_offsets;
    p.groups = s.batch;
    p.gated = IsGated(s.act) ? 1 : 0;
    if (!EncodeMatrix(&maps[2 * i], s.w, s.k, s.n, s.batch, s.k, s.batch_w, kBN, &swap_w) || swap_w ||
        !EncodeMatrix(&maps[2 * i + 1], s.x, s.k, p.M, groups ? 1 : s.batch, s.ld_x, s.batch_x, bt, &p.swap_x)) {
      return cudaErrorInvalidValue;
    }
    p.bias = s.bias;
    p.residual = s.residual;
    p.y = s.y;
    p.ld_res = s.ld_res;
    p.ld_y = s.ld_y;
    p.batch_y = groups ? 0 : s.batch_y;
    p.k = s.k;
    p.n = s.n;
    p.act = s.act;
    p.y_f32 = s.y_dtype == TLALOC_B200_F32 ? 1 : 0;
    p.rows_bf16 = !p.y_f32 && !s.residual && s.ld_y % 8 == 0 && (s.batch == 1 || s.batch_y % 8 == 0) && Aligned16(s.y) ? 1 : 0;
    p.tiles_n = (s.n + kBN - 1) / kBN;
    if (!groups) a.tiles += p.tiles_n * p.tiles_m * s.batch;
    if (i == 0) a.tiles0 = groups ? 1 << 30 : a.tiles;
    nb = min(nb, (s.k + kBK - 1) / kBK);
  }
  if (count == 1) {
    maps[2] = maps[0];
    maps[3] = maps[1];
  }
  if (grouped) {
    a.ks = 1;
    switch (bt) {
      case 32: return Launch<32, false, true>(maps, a, 148, st);
      case 64: return Launch<64, false, true>(maps, a, 148, st);
      case 128: return Launch<128, false, true>(maps, a, 148, st);
      default: return Launch<256, false, true>(maps, a, 148, st);
    }
  }
  a.ks = bt <= 128 && a.p[0].tiles_m == 1 && (count == 1 || a.p[1].tiles_m == 1) ? ChooseSlices(a.tiles, nb) : 1;
  if (a.ks > 1) {
    switch (bt) {
      case 32: return Launch<32, true>(maps, a, a.tiles, st);
      case 64: return Launch<64, true>(maps, a, a.tiles, st);
      default: return Launch<128, true>(maps, a, a.tiles, st);
    }
  }
  const int ctas = min(a.tiles, 148);
  switch (bt) {
    case 32: return Launch<32, false>(maps, a, ctas, st);
    case 64: return Launch<64, false>(maps, a, ctas, st);
    case 128: return Launch<128, false>(maps, a, ctas, st);
    default: return Launch<256, false>(maps, a, ctas, st);
  }
}

}  // namespace tlaloc_b200
