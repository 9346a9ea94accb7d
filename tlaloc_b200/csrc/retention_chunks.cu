// Retention over a prompt portion on the tensor cores (include/tlaloc_b200.h, tlaloc_b200_retention_chunks): bf16 operands by TMA,
// tcgen05.mma kind::f16 with f32 accumulators in TMEM.
//
// The portion is cut into chunks of 128 tokens and, for parallelism, into segments of whole chunks.  Within a chunk, with S the state ahead
// of it and w = decay:
//   o_i = w^(i+1) S^T q_i + sum_{j <= i} w^(i-j) (q_i . k_j) v_j        S <- w^n S + sum_j w^(n-1-j) k_j v_j^T
// A CTA has one head, a slice of its value columns and one segment; S stays in TMEM (rows: the key's channels, 128 at a time).  What was
// computed in f32 and enters a product as an operand (S, the decayed scores, the decayed values) enters as two bf16 parts, which is f32 up
// to rounding.  Every product has 128 columns, so that it reads both operands at the rate it multiplies them: a slice has 128 value columns
// and the two parts are two products, or it has 64 and the parts lie side by side, their sums added later.
//   producer lane   Q, K and V, each as soon as its space is free; the output rows back, by TMA too
//   MMA lane        scores Q K^T; O = Q S; O = P V (its first part is in registers by then); S += K^T V'
//   sixteen warps   S as an operand (shared memory) and decayed; scores times decay, in their place in TMEM as the A operand P; the
//                   decayed values V' (in the place of S's operand); the output rows (in the place of V)
// Two launches where there are several segments: the first computes what each segment adds to the state (decayed to the segment's end, so
// that nothing in it is rescaled), the second starts every segment from the sum of those before it, writes the outputs and, in the last
// segment, the new state.  Every mbarrier wait is bounded.
#include <cuda.h>

#include "common.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

using namespace tc;

constexpr int kChunk = 128;
constexpr int kWorkers = 16, kWorkerThreads = kWorkers * 32, kParts = kWorkers / 4, kThreads = kWorkerThreads + 64;
constexpr int kAtom = kChunk * 128;  // 128 tokens x 64 channels
constexpr int kMaxSmem = 227 * 1024;

struct ChunkArgs {
  const int *positions, *row_states;
  const float* decay;
  float *state, *o, *sums;  // sums [segments][heads][slices][..]: what a segment adds; the last one's place holds the state before the portion
  int tokens, heads, dim, vdim, dp, num_slots, segment, segments, store_rows;  // store_rows: the output's rows can leave by TMA
};

__device__ int g_retention_status = 0;

// f32 accumulator, bf16 operands, M = 128.
__host__ __device__ constexpr uint32_t InstrDesc(int n, bool a_mn, bool b_mn)
{
  return (1u << 4) | (1u << 7) | (1u << 10) | (a_mn ? 1u << 15 : 0u) | (b_mn ? 1u << 16 : 0u) | (static_cast<uint32_t>(n >> 3) << 17) | (8u << 24);
}
// x is a multiple of 64 channels: a 16-byte boundary.
__device__ __forceinline__ void TmaBox(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar)
{
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(dst),
               "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(z), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void Split(float a, float b, uint32_t& hi, uint32_t& lo)
{
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float Low(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float High(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ void StoreShared16(uint32_t at, const uint32_t* v)
{
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};\n" ::"r"(at), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]) : "memory");
}

// Shared memory: Q | K (one or two buffers) | V, later the output rows | S as an operand, later V'.  For the state alone: two buffers of
// K from Q's place on, two of V, and V' (one or two).
struct Places {
  uint32_t q, k, v, s, bytes;
  int k_buffers, vd_buffers;
};
__host__ __device__ inline Places PlaceAll(int dp, int vs)
{
  Places p;
  const uint32_t tile = (dp + 63) / 64 * kAtom, v_tile = vs / 64 * kAtom;
  const uint32_t s_bytes = 2 * (vs / 64) * dp * 128, vd_bytes = 2 * v_tile, o_bytes = 2 * v_tile, rest = o_bytes + (s_bytes > vd_bytes ? s_bytes : vd_bytes);
  p.k_buffers = 3 * tile + rest <= kMaxSmem - 1024 ? 2 : 1;
  p.q = 0;
  p.k = tile;
  p.v = p.k + p.k_buffers * tile;
  p.s = p.v + o_bytes;
  p.vd_buffers = s_bytes >= 2 * vd_bytes ? 2 : 1;
  p.bytes = p.v + rest;
  return p;
}

template <int N>
__device__ __forceinline__ void LoadTmem(uint32_t taddr, uint32_t* r)
{
  if constexpr (N == 32) TcLd32(taddr, r);
  else TcLd16(taddr, r);
}
template <int N>
__device__ __forceinline__ void StoreTmem(uint32_t taddr, const uint32_t* r)
{
  if constexpr (N == 32) TcSt32(taddr, r);
  else TcSt16(taddr, r);
}

// BLOCKS: 128-channel blocks of S.  VS: value columns of a slice, 128 or 64.
template <int BLOCKS, int VS, bool OUT>
__global__ void __launch_bounds__(kThreads, 1) RetentionChunkTc(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                                const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_o,
                                                                const __grid_constant__ ChunkArgs a)
{
  constexpr bool kSideBySide = VS == 64;
  constexpr int VC = VS / kParts, kVAtoms = VS / 64;  // value columns of a worker thread
  constexpr uint32_t kCols = 512;                     // scores, O and each block of S: 128 columns
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[15];
  __shared__ uint32_t slot_store[2];
  __shared__ float pw_store[31 + kChunk + 1];  // 31 zeros, then w^0 .. w^128
  float* pw = pw_store + 31;
  const uint32_t base = SmemAddr(smem_raw);
  if ((base & 1023u) != 0u) {
    if (threadIdx.x == 0) atomicExch(&g_retention_status, 1);
    return;
  }
  const Places at = PlaceAll(a.dp, VS);
  const uint32_t at_q = base + at.q, at_k = base + (OUT ? at.k : at.q), at_v = base + at.v, at_s = base + at.s;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t full_q = SmemAddr(bars), full_k = full_q + 8, full_v = full_k + 16, sc_done = full_v + 16, s_ready = sc_done + 8, o_done = s_ready + 8,
                 p_ready = o_done + 8, pv_done = p_ready + 8, vd_ready = pv_done + 8, st_done = vd_ready + 16, o_ready = st_done + 16;
  volatile uint32_t* abort_word = slot_store + 1;
  if (tid == 0) {
    slot_store[1] = 0u;
    for (int i = 0; i < 15; ++i) {
      const uint32_t bar = SmemAddr(bars + i);
      MbarInit(bar, bar == s_ready || bar == p_ready || bar == vd_ready || bar == vd_ready + 8 || bar == o_ready ? kWorkers : 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(SmemAddr(slot_store)), "r"(kCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(slot_store), t_p = tmem, t_o = tmem + 128, t_s = tmem + 256;
  GridDependencySync();

  const int head = blockIdx.x, slice = blockIdx.y, seg = blockIdx.z, slices = gridDim.y;
  const int t_begin = seg * a.segment, t_end = min(a.tokens, t_begin + a.segment), chunks = (t_end - t_begin + kChunk - 1) / kChunk;
  const bool last = seg + 1 == a.segments;
  // Whether the state behind chunk c is wanted.
  auto carries = [&](int c) { return !OUT || last || c + 1 < chunks; };
  const int atoms = (a.dp + 63) / 64, steps = a.dp / 16, kb = OUT ? at.k_buffers : 2;
  const uint32_t k_tile = atoms * kAtom;
  // Barriers of K's buffers, of V' and of the state's products alternate with the chunk (one that is two phases ahead of a wait looks like one
  // that has not come).
  auto k_buf = [&](int c) { return kb == 2 ? c & 1 : 0; };
  auto k_par = [&](int c) { return static_cast<uint32_t>((kb == 2 ? c >> 1 : c) & 1); };
  auto st_bar = [&](int c) { return st_done + 8 * (c & 1); };
  auto vd_bar = [&](int c) { return vd_ready + 8 * (c & 1); };
  // The state alone: buffers of V alternate too, and those of V' if there are two.
  auto v_buf = [&](int c) { return OUT ? 0 : c & 1; };
  auto v_par = [&](int c) { return static_cast<uint32_t>((OUT ? c : c >> 1) & 1); };
  const int vdb = OUT ? 1 : at.vd_buffers;
  auto vd_at = [&](int c) { return static_cast<uint32_t>(vdb == 2 && (c & 1) ? 2 * kVAtoms * kAtom : 0); };
  bool ok = true;

  if (warp == kWorkers) {
    if (ElectOne()) {
      auto store_rows = [&](int c) {
        ok = MbarWait(o_ready, c & 1, abort_word) && ok;
        if (a.store_rows) {
          for (int x = 0; x < VS / 32; ++x) {
            if (slice * VS + x * 32 >= a.vdim) break;
            asm volatile("cp.async.bulk.tensor.3d.global.shared::cta.bulk_group [%0, {%2, %3, %4}], [%1];\n" ::"l"(reinterpret_cast<uint64_t>(&map_o)),
                         "r"(at_v + x * kAtom), "r"(slice * VS + x * 32), "r"(head), "r"(t_begin + c * kChunk)
                         : "memory");
          }
          asm volatile("cp.async.bulk.commit_group;\n" ::: "memory");
          asm volatile("cp.async.bulk.wait_group.read 0;\n" ::: "memory");
        }
      };
      for (int c = 0; c < chunks; ++c) {
        const int t0 = t_begin + c * kChunk;
        if (c >= kb) ok = MbarWait(st_bar(c - kb), ((c - kb) >> 1) & 1, abort_word) && ok;
        const uint32_t bar_k = full_k + 8 * k_buf(c), dst = at_k + k_buf(c) * k_tile;
        MbarExpectTx(bar_k, k_tile);
        for (int x = 0; x < atoms; ++x) TmaBox(dst + x * kAtom, &map_k, x * 64, head, t0, bar_k);
        if (OUT) {
          if (c > 0) ok = MbarWait(o_done, (c - 1) & 1, abort_word) && ok;
          MbarExpectTx(full_q, k_tile);
          for (int x = 0; x < atoms; ++x) TmaBox(at_q + x * kAtom, &map_q, x * 64, head, t0, full_q);
        }
        if (OUT && c > 0) store_rows(c - 1);  // V has been multiplied with and read, and the output rows in its place have left
        const uint32_t bar_v = full_v + 8 * v_buf(c), v_dst = at_v + v_buf(c) * kVAtoms * kAtom;
        MbarExpectTx(bar_v, kVAtoms * kAtom);
        for (int x = 0; x < kVAtoms; ++x) TmaBox(v_dst + x * kAtom, &map_v, slice * VS + x * 64, head, t0, bar_v);
      }
      if (OUT) {
        store_rows(chunks - 1);
        asm volatile("cp.async.bulk.wait_group 0;\n" ::: "memory");
      }
      if (!ok) {  // given up: let the copies in flight land before the CTA's shared memory goes away
        volatile uint32_t never = 0;
        for (int c = max(0, chunks - kb); c < chunks; ++c) MbarWait(full_k + 8 * k_buf(c), k_par(c), &never);
        if (OUT) MbarWait(full_q, (chunks - 1) & 1, &never);
        for (int c = max(0, chunks - (OUT ? 1 : 2)); c < chunks; ++c) MbarWait(full_v + 8 * v_buf(c), v_par(c), &never);
      }
    }
    __syncwarp();
  } else if (warp == kWorkers + 1) {
    if (ElectOne()) {
      constexpr uint32_t scores_desc = InstrDesc(kChunk, false, false), wide_desc = InstrDesc(128, false, true), out_desc = InstrDesc(VS, false, true),
                         state_desc = InstrDesc(128, true, true);
      const uint32_t s_atom = a.dp * 128;
      const uint64_t qd = SmemDesc(at_q, 16, 1024), kd = SmemDesc(at_k, 16, 1024), kt = SmemDesc(at_k, kAtom, 1024), vd = SmemDesc(at_v, kAtom, 1024);
      const uint64_t sh = SmemDesc(at_s, s_atom, 1024), sl = SmemDesc(at_s + kVAtoms * s_atom, s_atom, 1024);
      const uint64_t dh = SmemDesc(at_s, kAtom, 1024), dl = SmemDesc(at_s + kVAtoms * kAtom, kAtom, 1024);
      constexpr uint64_t kRows = (16 * 128) >> 4;  // sixteen rows of a tile further
      auto scores = [&](int c) {
        ok = MbarWait(full_k + 8 * k_buf(c), k_par(c), abort_word) && ok;
        ok = MbarWait(full_q, c & 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        const uint64_t ka = kd + static_cast<uint64_t>((k_buf(c) * k_tile) >> 4);
        for (int k = 0; k < steps; ++k) {
          const uint64_t off = static_cast<uint64_t>((k >> 2) * (kAtom >> 4) + 2 * (k & 3));
          TcMmaBf16(t_p, qd + off, ka + off, scores_desc, k > 0 ? 1u : 0u);
        }
        TcCommit(sc_done);
      };
      if (OUT) scores(0);
      for (int c = 0; c < chunks; ++c) {
        const uint32_t par = c & 1;
        if (OUT) {
          ok = MbarWait(s_ready, par, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int k = 0; k < steps; ++k) {
            const uint64_t off = static_cast<uint64_t>((k >> 2) * (kAtom >> 4) + 2 * (k & 3));
            TcMmaBf16(t_o, qd + off, sh + k * kRows, wide_desc, k > 0 ? 1u : 0u);
            if (!kSideBySide) TcMmaBf16(t_o, qd + off, sl + k * kRows, wide_desc, 1u);
          }
          TcCommit(o_done);
          ok = MbarWait(full_v, par, abort_word) && ok;
          ok = MbarWait(p_ready, par, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int k = 0; k < kChunk / 16; ++k) {
            const uint32_t pa = t_p + 32 * (k >> 1) + 8 * (k & 1);
            TcMmaTmemA(t_o, pa, vd + k * kRows, out_desc, k > 0 ? 1u : 0u);
            TcMmaTmemA(t_o, pa + 16, vd + k * kRows, out_desc, 1u);
          }
          TcCommit(pv_done);
          if (kb == 2 && c + 1 < chunks) scores(c + 1);  // P is used up; with one buffer K is still wanted for the state
        } else {
          ok = MbarWait(full_k + 8 * k_buf(c), k_par(c), abort_word) && ok;
        }
        if (carries(c)) {
          ok = MbarWait(vd_bar(c), (c >> 1) & 1, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll
          for (int b = 0; b < BLOCKS; ++b) {
            const uint64_t ka = kt + static_cast<uint64_t>((k_buf(c) * k_tile + b * 2 * kAtom) >> 4);
            const uint64_t off = vd_at(c) >> 4;
            for (int k = 0; k < kChunk / 16; ++k) {
              TcMmaBf16(t_s + b * 128, ka + k * kRows, dh + off + k * kRows, state_desc, 1u);
              if (!kSideBySide) TcMmaBf16(t_s + b * 128, ka + k * kRows, dl + off + k * kRows, state_desc, 1u);
            }
          }
          TcCommit(st_bar(c));
        }
        if (OUT && kb == 1 && c + 1 < chunks) scores(c + 1);
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3, part = warp >> 2, row = quad * 32 + lane;  // row: TMEM lane
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    const float w = __ldg(a.decay + head);
    for (int i = tid - 31; i <= kChunk; i += kWorkerThreads) pw[i] = i < 0 ? 0.f : powf(w, static_cast<float>(i));
    asm volatile("bar.sync 5, %0;\n" ::"n"(kWorkerThreads) : "memory");
    // This thread's columns of O or of a block of S: of 64-column slices the parts' halves are added, and stored with an empty second one.
    auto load_columns = [&](uint32_t t, float* v) {
      uint32_t* u = reinterpret_cast<uint32_t*>(v);
      LoadTmem<VC>(t + lanes + part * VC, u);
      if constexpr (kSideBySide) {
        uint32_t x[VC];
        LoadTmem<VC>(t + lanes + 64 + part * VC, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
        for (int e = 0; e < VC; ++e) v[e] += __uint_as_float(x[e]);
      } else {
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
      }
    };
    auto store_columns = [&](uint32_t t, const float* v) {
      StoreTmem<VC>(t + lanes + part * VC, reinterpret_cast<const uint32_t*>(v));
      if constexpr (kSideBySide) {
        uint32_t x[VC];
#pragma unroll
        for (int e = 0; e < VC; ++e) x[e] = 0u;
        StoreTmem<VC>(t + lanes + 64 + part * VC, x);
      }
    };

    // The state ahead of the segment.
    const int vp = (a.vdim + 3) & ~3, v0 = slice * VS + part * VC;
    const int slot = min(max(__ldg(a.row_states), 0), a.num_slots - 1);
    float* state = a.state + (static_cast<size_t>(slot) * a.heads + head) * a.dim * vp;
    auto sums = [&](int g) {
      return a.sums + ((static_cast<size_t>(g) * a.heads + head) * slices + slice) * (static_cast<size_t>(BLOCKS) * VC * kWorkerThreads) + tid;
    };
    const bool own = seg == 0 && !(OUT && a.segments > 1);
    const bool fresh = __ldg(a.positions) == 0;
    const float ws = powf(w, static_cast<float>(a.segment));  // over a whole segment
    const int g_lo = seg == 0 ? a.segments - 1 : 0, g_hi = seg == 0 ? a.segments : seg;
#pragma unroll 1
    for (int b = 0; b < BLOCKS; ++b) {
      const int d = b * 128 + row;
      float s[VC];
#pragma unroll
      for (int e = 0; e < VC; ++e) s[e] = 0.f;
      if (own) {
        if (!fresh && d < a.dim) {
          const float* p = state + static_cast<size_t>(d) * vp + v0;
#pragma unroll
          for (int e = 0; e < VC; e += 4) {
            if (v0 + e < vp) {
              const float4 x = *reinterpret_cast<const float4*>(p + e);
              s[e] = x.x; s[e + 1] = x.y; s[e + 2] = x.z; s[e + 3] = x.w;
            }
          }
        }
        if (!OUT) {
          float* p = sums(a.segments - 1) + b * VC * kWorkerThreads;
#pragma unroll
          for (int e = 0; e < VC; ++e) {
            p[e * kWorkerThreads] = s[e];
            s[e] *= ws;
          }
        }
      } else if (OUT) {
#pragma unroll 2
        for (int g = g_lo; g < g_hi; ++g) {
          const float* p = sums(g) + b * VC * kWorkerThreads;
#pragma unroll
          for (int e = 0; e < VC; ++e) s[e] = fmaf(ws, s[e], p[e * kWorkerThreads]);
        }
      }
      store_columns(t_s + b * 128, s);
    }
    asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");

    float w_ahead = 1.f;
    for (int c = 0; c < chunks; ++c) {
      const uint32_t par = c & 1;
      const int t0 = t_begin + c * kChunk, n = min(kChunk, t_end - t0);
      if (c >= vdb) {
        ok = MbarWaitWarp(st_bar(c - vdb), ((c - vdb) >> 1) & 1, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
      }
      float o[VC];
      if (OUT) {
        // S as an operand, and decayed for what the chunk adds.
        const float wn = pw[n];
#pragma unroll 1
        for (int b = 0; b < BLOCKS; ++b) {
          const int d = b * 128 + row;
          if (b * 128 + quad * 32 >= a.dp) break;  // nothing but padding in this warp's rows
          float s[VC];
          load_columns(t_s + b * 128, s);
          if (d < a.dp) {
#pragma unroll
            for (int i = 0; i < VC / 8; ++i) {
              uint32_t hi[4], lo[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) Split(s[8 * i + 2 * e], s[8 * i + 2 * e + 1], hi[e], lo[e]);
              const int col = part * VC + 8 * i;
              const uint32_t off = at_s + (col >> 6) * (a.dp * 128) + d * 128 + ((((col & 63) >> 3) ^ (d & 7)) << 4);
              StoreShared16(off, hi);
              StoreShared16(off + kVAtoms * a.dp * 128, lo);
            }
          }
#pragma unroll
          for (int e = 0; e < VC; ++e) s[e] *= wn;
          store_columns(t_s + b * 128, s);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(s_ready);

        // Scores times decay, 32 columns a warp: their first parts go to the first 16 of the columns, the second parts to the others.
        ok = MbarWaitWarp(sc_done, par, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        {
          const int j0 = part * 32;
          uint32_t hi[16], lo[16];
          if (part > quad) {  // all of it in the future
#pragma unroll
            for (int e = 0; e < 16; ++e) hi[e] = lo[e] = 0u;
          } else {
            uint32_t s[32];
            TcLd32(t_p + lanes + j0, s);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            const float* wr = pw + (row - j0);  // zeros for the future
#pragma unroll
            for (int e = 0; e < 32; e += 2) Split(__uint_as_float(s[e]) * wr[-e], __uint_as_float(s[e + 1]) * wr[-e - 1], hi[e / 2], lo[e / 2]);
          }
          TcSt16(t_p + lanes + j0, hi);
          TcSt16(t_p + lanes + j0 + 16, lo);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
        ok = MbarWaitWarp(o_done, par, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        load_columns(t_o, o);
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(p_ready);
        const float wi = pw[row + 1];
#pragma unroll
        for (int e = 0; e < VC; ++e) o[e] *= wi;
      }

      // Decayed values, in the place of S's operand (its products, or those with the values before, are done).
      if (carries(c)) {
        ok = MbarWaitWarp(full_v + 8 * v_buf(c), v_par(c), lane, abort_word) && ok;
        const uint32_t v_src = at_v + v_buf(c) * kVAtoms * kAtom, vd_dst = at_s + vd_at(c);
        float wc = 1.f;
        if (!OUT) {  // from the chunk's end to the segment's: one power a lane for 32 chunks
          if ((c & 31) == 0) w_ahead = powf(w, static_cast<float>(max(chunks - 1 - c - lane, 0) * kChunk));
          wc = __shfl_sync(0xffffffffu, w_ahead, c & 31);
        }
#pragma unroll
        for (int i = 0; i < kVAtoms * kAtom / 16 / kWorkerThreads; ++i) {
          const int idx = i * kWorkerThreads + tid, j = (idx & (kAtom / 16 - 1)) >> 3;
          uint32_t v[4], hi[4], lo[4];
          asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];\n" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(v_src + idx * 16) : "memory");
          const float wj = j < n ? pw[max(n - 1 - j, 0)] * wc : 0.f;
#pragma unroll
          for (int e = 0; e < 4; ++e) Split(Low(v[e]) * wj, High(v[e]) * wj, hi[e], lo[e]);
          StoreShared16(vd_dst + idx * 16, hi);
          StoreShared16(vd_dst + kVAtoms * kAtom + idx * 16, lo);
        }
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(vd_bar(c));
      }

      if (OUT) {
        ok = MbarWaitWarp(pv_done, par, lane, abort_word) && ok;
        if (carries(c)) ok = MbarWaitWarp(vd_bar(c), (c >> 1) & 1, lane, abort_word) && ok;  // all warps have read V
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint32_t x[VC];
        LoadTmem<VC>(t_o + lanes + part * VC, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        if (a.store_rows) {  // boxes of 32 columns
#pragma unroll
          for (int e = 0; e < VC; e += 4) {
            const int col = part * VC + e;
            const uint32_t u[4] = {__float_as_uint(o[e] + __uint_as_float(x[e])), __float_as_uint(o[e + 1] + __uint_as_float(x[e + 1])),
                                   __float_as_uint(o[e + 2] + __uint_as_float(x[e + 2])), __float_as_uint(o[e + 3] + __uint_as_float(x[e + 3]))};
            StoreShared16(at_v + (col >> 5) * kAtom + row * 128 + ((((col & 31) >> 2) ^ (row & 7)) << 4), u);
          }
          asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        } else if (row < n) {
          float* p = a.o + (static_cast<size_t>(t0 + row) * a.heads + head) * a.vdim + v0;
#pragma unroll
          for (int e = 0; e < VC; ++e)
            if (v0 + e < a.vdim) p[e] = o[e] + __uint_as_float(x[e]);
        }
        __syncwarp();
        if (lane == 0) MbarArrive(o_ready);
      }
    }

    if (!OUT || last) {
      ok = MbarWaitWarp(st_bar(chunks - 1), ((chunks - 1) >> 1) & 1, lane, abort_word) && ok;
      asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll 1
      for (int b = 0; b < BLOCKS; ++b) {
        const int d = b * 128 + row;
        float s[VC];
        load_columns(t_s + b * 128, s);
        if (!OUT) {
          float* p = sums(seg) + b * VC * kWorkerThreads;
#pragma unroll
          for (int e = 0; e < VC; ++e) p[e * kWorkerThreads] = d < a.dp ? s[e] : 0.f;
        } else if (d < a.dim) {
          float* p = state + static_cast<size_t>(d) * vp + v0;
#pragma unroll
          for (int e = 0; e < VC; e += 4) {
            if (v0 + e < vp) *reinterpret_cast<float4*>(p + e) = make_float4(s[e], s[e + 1], s[e + 2], s[e + 3]);
          }
        }
      }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  }
  if (!ok) atomicExch(&g_retention_status, 1);
  __syncthreads();
  if (warp == 0) {
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(kCols) : "memory");
  }
}

// What a call is cut into.
struct Plan {
  int dp, blocks, vs, slices, segment, segments;
  size_t sums_bytes;
};
Plan PlanFor(int tokens, int heads, int dim, int vdim)
{
  Plan p;
  p.dp = (dim + 15) / 16 * 16;
  p.blocks = (p.dp + 127) / 128;
  p.vs = p.blocks == 1 && vdim > 64 ? 128 : 64;
  p.slices = (vdim + p.vs - 1) / p.vs;
  const int chunks = (tokens + kChunk - 1) / kChunk, ctas = heads * p.slices, slots = 148;
  // Rounds of CTAs times chunks of a segment, in chunks of the second launch: the state alone at two fifths, a CTA's start at one, a launch at one
  // half, the sums of an earlier segment at an eighth per block of S.
  double best = 1e30;
  p.segments = 1;
  int per = chunks;
  for (int n = 1; n <= chunks && n <= 32; ++n) {
    const int len = (chunks + n - 1) / n, used = (chunks + len - 1) / len;
    const int rounds = (ctas * used + slots - 1) / slots, before = (ctas * (used - 1) + slots - 1) / slots;
    double cost = rounds * (len + 1.0);
    if (used > 1) cost += before * (0.4 * len + 1.0) + 0.5 + 0.125 * p.blocks * (used - 1) * rounds;
    if (cost < best * 0.97) {
      best = cost;
      p.segments = used;
      per = len;
    }
  }
  p.segment = per * kChunk;
  p.sums_bytes = p.segments > 1 ? static_cast<size_t>(p.segments) * ctas * p.blocks * kChunk * p.vs * sizeof(float) : 0;
  return p;
}

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// [tokens][heads][ld] of bf16 or f32, boxes of 128 bytes of one head x 128 tokens.
bool Encode(CUtensorMap* map, const void* ptr, int ld, int heads, int tokens, bool f32 = false)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  const cuuint64_t dims[3] = {static_cast<cuuint64_t>(ld), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(tokens)};
  const cuuint64_t size = f32 ? 4 : 2, strides[2] = {static_cast<cuuint64_t>(ld) * size, static_cast<cuuint64_t>(ld) * size * heads};
  const cuuint32_t box[3] = {f32 ? 32u : 64u, 1, kChunk}, elem[3] = {1, 1, 1};
  return encode != nullptr &&
         encode(map, f32 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT32 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

cudaError_t PrepareChunks()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(BLOCKS, VS)                                                                                                                      \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(RetentionChunkTc<BLOCKS, VS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024); \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(RetentionChunkTc<BLOCKS, VS, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024);
    TLALOC_OPT_IN(1, 64)
    TLALOC_OPT_IN(1, 128)
    TLALOC_OPT_IN(2, 64)
#undef TLALOC_OPT_IN
    return e;
  });
}
int ReadRetentionStatus()
{
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_retention_status, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_retention_status, &zero, sizeof(int));
  }
  return v;
}
KernelSetup g_setup(PrepareChunks, ReadRetentionStatus);

template <bool OUT>
cudaError_t Launch(const Plan& p, const CUtensorMap* maps, const ChunkArgs& a, int segments, cudaStream_t st)
{
  const dim3 grid(a.heads, p.slices, segments);
  const size_t smem = PlaceAll(a.dp, p.vs).bytes;
  if (p.blocks == 2) return LaunchChained(RetentionChunkTc<2, 64, OUT>, grid, kThreads, smem, st, maps[0], maps[1], maps[2], maps[3], a);
  if (p.vs == 64) return LaunchChained(RetentionChunkTc<1, 64, OUT>, grid, kThreads, smem, st, maps[0], maps[1], maps[2], maps[3], a);
  return LaunchChained(RetentionChunkTc<1, 128, OUT>, grid, kThreads, smem, st, maps[0], maps[1], maps[2], maps[3], a);
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_retention_chunks_applies(int32_t dim, int32_t vdim) { return dim >= 1 && dim <= 256 && vdim >= 1 && !OrderFaithful() ? 1 : 0; }

extern "C" size_t tlaloc_b200_retention_chunks_scratch_bytes(int32_t tokens, int32_t heads, int32_t dim, int32_t vdim)
{
  if (tokens < 1 || heads < 1 || !tlaloc_b200_retention_chunks_applies(dim, vdim)) return 0;
  return PlanFor(tokens, heads, dim, vdim).sums_bytes;
}

extern "C" int tlaloc_b200_retention_chunks(const void* q, const void* k, int32_t dim_ld, const void* v, int32_t v_ld, const int32_t* positions,
                                            const float* decay, const int32_t* row_states, float* state, float* o, void* scratch, size_t scratch_bytes,
                                            int32_t tokens, int32_t heads, int32_t dim, int32_t vdim, int32_t num_slots, void* stream)
{
  const char* op = "RETENTION_CHUNKS";
  if (!q || !k || !v || !positions || !decay || !row_states || !state || !o) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (tokens < 0 || heads < 1 || heads > 65535 || dim < 1 || vdim < 1 || num_slots < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (!tlaloc_b200_retention_chunks_applies(dim, vdim)) return Fail(kUnsupported, "%s: dim up to 256", op);
  if (dim_ld != (dim + 15) / 16 * 16 || v_ld < vdim || v_ld % 8 || !Aligned16(q) || !Aligned16(k) || !Aligned16(v) || !Aligned16(state) || !Aligned16(o)) {
    return Fail(kInvalid, "%s: rows of dim rounded up to 16 and of a multiple of 8 values, 16-byte aligned", op);
  }
  if (tokens == 0) return kOk;
  const Plan p = PlanFor(tokens, heads, dim, vdim);
  if (p.slices > 65535) return Fail(kInvalid, "%s: bad sizes", op);
  if (p.sums_bytes > 0 && (!scratch || scratch_bytes < p.sums_bytes)) return Fail(kInvalid, "%s: %zu bytes of scratch are needed", op, p.sums_bytes);
  cudaError_t e = PrepareChunks();
  if (e != cudaSuccess) return CudaFail("RETENTION_CHUNKS set-up", e);
  CUtensorMap maps[4];
  const bool store_rows = vdim % 4 == 0;
  if ((store_rows && !Encode(&maps[3], o, vdim, heads, tokens, true)) || !Encode(&maps[0], q, dim_ld, heads, tokens) || !Encode(&maps[1], k, dim_ld, heads, tokens) || !Encode(&maps[2], v, v_ld, heads, tokens)) {
    return Fail(kInternal, "%s: the tensor maps could not be encoded", op);
  }
  if (!store_rows) maps[3] = maps[2];
  ChunkArgs a = {};
  a.store_rows = store_rows ? 1 : 0;
  a.positions = positions;
  a.row_states = row_states;
  a.decay = decay;
  a.state = state;
  a.o = o;
  a.sums = static_cast<float*>(scratch);
  a.tokens = tokens;
  a.heads = heads;
  a.dim = dim;
  a.vdim = vdim;
  a.dp = p.dp;
  a.num_slots = num_slots;
  a.segment = p.segment;
  a.segments = p.segments;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (p.segments > 1) {
    e = Launch<false>(p, maps, a, p.segments - 1, st);
    if (e == cudaSuccess) CountLaunches(1);
  }
  if (e == cudaSuccess) e = Launch<true>(p, maps, a, p.segments, st);
  if (e != cudaSuccess) return CudaFail("RETENTION_CHUNKS launch", e);
  CountLaunches(1);
  return kOk;
}
