// Retention over a prompt portion on the tensor cores (include/tlaloc_b200.h, tlaloc_b200_retention_chunks): bf16 operands by TMA,
// tcgen05.mma kind::f16 with f32 accumulators in TMEM.
//
// The portion is cut into chunks of 128 tokens and, for parallelism, into segments of whole chunks.  Within a chunk, with S the state ahead
// of it and w = decay:
//   o_i = w^(i+1) S^T q_i + sum_{j <= i} w^(i-j) (q_i . k_j) v_j        S <- w^n S + sum_j w^(n-1-j) k_j v_j^T
// A CTA has one head, 64 value columns and one segment; S stays in TMEM (rows: the key's channels, 128 at a time).  What was computed in f32
// and enters a product as an operand (S, the decayed scores, the decayed values) enters as two bf16 parts, which is f32 up to rounding.
//   producer lane   Q, K and V of the next chunk
//   MMA lane        scores Q K^T; O = Q S; O = P V (its first part is in registers by then); S += K^T V'
//   worker warps    S as an operand (shared memory) and decayed; scores times decay, in their place in TMEM as the A operand P; the
//                   decayed values V' (in the place of Q); the output rows.  Eight, and two CTAs per SM, up to 128 channels; else sixteen
// Two launches where there are several segments: the first computes what each segment adds to the state, the second starts every
// segment from the sum of those before it, writes the outputs and, in the last segment, the new state.  Every mbarrier wait is bounded.
#include <cuda.h>

#include "common.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

using namespace tc;

constexpr int kChunk = 128, kVS = 64;
constexpr int kAtom = kChunk * 128;  // 128 tokens x 64 channels
constexpr int kMaxSmem = 227 * 1024;

struct ChunkArgs {
  const int *positions, *row_states;
  const float* decay;
  float *state, *o, *sums;  // sums [segments][heads][slices][..]: what a segment adds; the last one's place holds the state before the portion
  int tokens, heads, dim, vdim, dp, num_slots, segment, segments;
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

// Shared memory: Q | K | V | S (two parts) and, where Q is a single atom, the second part of V'; the first (two) atoms of Q hold V' when
// Q has been used.
struct Places {
  uint32_t q, k, v, s_hi, s_lo, vd_hi, vd_lo;
};
__host__ __device__ inline uint32_t PlaceAll(int dp, uint32_t base, Places* p)
{
  const uint32_t atoms = (dp + 63) / 64;
  p->q = base;
  p->k = p->q + atoms * kAtom;
  p->v = p->k + atoms * kAtom;
  p->s_hi = p->v + kAtom;
  p->s_lo = p->s_hi + dp * 128;
  p->vd_hi = p->q;
  uint32_t end = p->s_lo + dp * 128;
  if (atoms >= 2) {
    p->vd_lo = p->q + kAtom;
  } else {
    p->vd_lo = end;
    end += kAtom;
  }
  return end - base;
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

constexpr int WorkersFor(int blocks) { return blocks == 1 ? 8 : 16; }

// BLOCKS: 128-channel blocks of S.
template <int BLOCKS, bool OUT>
__global__ void __launch_bounds__(WorkersFor(BLOCKS) * 32 + 64, BLOCKS == 1 ? 2 : 1) RetentionChunkTc(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                             const __grid_constant__ CUtensorMap map_v, const __grid_constant__ ChunkArgs a)
{
  constexpr int kWorkers = WorkersFor(BLOCKS), kWorkerThreads = kWorkers * 32, kParts = kWorkers / 4;
  constexpr int VC = kVS / kParts, PC = kChunk / kParts;  // columns of O and S, and of the scores, of a worker warp
  constexpr uint32_t kCols = BLOCKS == 1 ? 256u : 512u;  // scores 128, O 64, S 64 per block
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[8];
  __shared__ uint32_t slot_store[2];
  __shared__ float pw[kChunk + 1];
  __shared__ __align__(16) float pw_down[32];  // w^31 .. w^0
  const uint32_t base = SmemAddr(smem_raw);  // two CTAs of 128 channels fill an SM to the byte: no slack to align within
  if ((base & 1023u) != 0u) {
    if (threadIdx.x == 0) atomicExch(&g_retention_status, 1);
    return;
  }
  Places at;
  PlaceAll(a.dp, base, &at);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t full = SmemAddr(bars), sc_done = full + 8, s_ready = full + 16, o_done = full + 24, p_ready = full + 32, pv_done = full + 40, vd_ready = full + 48,
                 st_done = full + 56;
  volatile uint32_t* abort_word = slot_store + 1;
  if (tid == 0) {
    slot_store[1] = 0u;
    MbarInit(full, 1);
    MbarInit(sc_done, 1);
    MbarInit(s_ready, kWorkers);
    MbarInit(o_done, 1);
    MbarInit(p_ready, kWorkers);
    MbarInit(pv_done, 1);
    MbarInit(vd_ready, kWorkers);
    MbarInit(st_done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(SmemAddr(slot_store)), "r"(kCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(slot_store), t_p = tmem, t_o = tmem + 128, t_s = tmem + 192;
  GridDependencySync();

  const int head = blockIdx.x, slice = blockIdx.y, seg = blockIdx.z, slices = gridDim.y;
  const int t_begin = seg * a.segment, t_end = min(a.tokens, t_begin + a.segment), chunks = (t_end - t_begin + kChunk - 1) / kChunk;
  const bool last = seg + 1 == a.segments;
  // Whether the state behind chunk c is wanted.
  auto carries = [&](int c) { return !OUT || last || c + 1 < chunks; };
  const int atoms = (a.dp + 63) / 64, steps = a.dp / 16;
  bool ok = true;

  if (warp == kWorkers) {
    if (ElectOne()) {
      for (int c = 0; c < chunks; ++c) {
        // Everything of the chunk before has been used when its last product is done.
        if (c > 0) ok = MbarWait(st_done, (c - 1) & 1, abort_word) && ok;
        const int t0 = t_begin + c * kChunk;
        MbarExpectTx(full, ((OUT ? 2 : 1) * atoms + 1) * kAtom);
        if (OUT)
          for (int x = 0; x < atoms; ++x) TmaBox(at.q + x * kAtom, &map_q, x * 64, head, t0, full);
        for (int x = 0; x < atoms; ++x) TmaBox(at.k + x * kAtom, &map_k, x * 64, head, t0, full);
        TmaBox(at.v, &map_v, slice * kVS, head, t0, full);
      }
      if (!ok) {  // given up: let the copies in flight land before the CTA's shared memory goes away
        volatile uint32_t never = 0;
        MbarWait(full, (chunks - 1) & 1, &never);
      }
    }
    __syncwarp();
  } else if (warp == kWorkers + 1) {
    if (ElectOne()) {
      constexpr uint32_t scores_desc = InstrDesc(kChunk, false, false), out_desc = InstrDesc(kVS, false, true), state_desc = InstrDesc(kVS, true, true);
      const uint64_t qd = SmemDesc(at.q, 16, 1024), kd = SmemDesc(at.k, 16, 1024), kt = SmemDesc(at.k, kAtom, 1024), vd = SmemDesc(at.v, kAtom, 1024);
      const uint64_t sh = SmemDesc(at.s_hi, kAtom, 1024), sl = SmemDesc(at.s_lo, kAtom, 1024);
      const uint64_t dh = SmemDesc(at.vd_hi, kAtom, 1024), dl = SmemDesc(at.vd_lo, kAtom, 1024);
      constexpr uint64_t kRows = (16 * 128) >> 4;  // sixteen rows of a tile further
      for (int c = 0; c < chunks; ++c) {
        const uint32_t par = c & 1;
        ok = MbarWait(full, par, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        if (OUT) {
          for (int k = 0; k < steps; ++k) {
            const uint64_t off = static_cast<uint64_t>((k >> 2) * (kAtom >> 4) + 2 * (k & 3));
            TcMmaBf16(t_p, qd + off, kd + off, scores_desc, k > 0 ? 1u : 0u);
          }
          TcCommit(sc_done);
          ok = MbarWait(s_ready, par, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int k = 0; k < steps; ++k) {
            const uint64_t off = static_cast<uint64_t>((k >> 2) * (kAtom >> 4) + 2 * (k & 3));
            TcMmaBf16(t_o, qd + off, sh + k * kRows, out_desc, k > 0 ? 1u : 0u);
            TcMmaBf16(t_o, qd + off, sl + k * kRows, out_desc, 1u);
          }
          TcCommit(o_done);
          ok = MbarWait(p_ready, par, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int k = 0; k < kChunk / 16; ++k) {
            const uint32_t pa = t_p + 32 * (k >> 1) + 8 * (k & 1);
            TcMmaTmemA(t_o, pa, vd + k * kRows, out_desc, k > 0 ? 1u : 0u);
            TcMmaTmemA(t_o, pa + 16, vd + k * kRows, out_desc, 1u);
          }
          TcCommit(pv_done);
        }
        if (carries(c)) {
          ok = MbarWait(vd_ready, par, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll
          for (int b = 0; b < BLOCKS; ++b) {
            const uint64_t kb = kt + static_cast<uint64_t>(b * 2 * (kAtom >> 4));
            for (int k = 0; k < kChunk / 16; ++k) {
              TcMmaBf16(t_s + b * 64, kb + k * kRows, dh + k * kRows, state_desc, 1u);
              TcMmaBf16(t_s + b * 64, kb + k * kRows, dl + k * kRows, state_desc, 1u);
            }
          }
          TcCommit(st_done);
        }
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3, part = warp >> 2, row = quad * 32 + lane;  // row: TMEM lane
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    const float w = __ldg(a.decay + head);
    for (int i = tid; i <= kChunk; i += kWorkerThreads) pw[i] = powf(w, static_cast<float>(i));
    if (tid < 32) pw_down[tid] = powf(w, static_cast<float>(31 - tid));
    asm volatile("bar.sync 5, %0;\n" ::"n"(kWorkerThreads) : "memory");

    // The state ahead of the segment.
    const int vp = (a.vdim + 3) & ~3, v0 = slice * kVS + part * VC;
    const int slot = min(max(__ldg(a.row_states), 0), a.num_slots - 1);
    float* state = a.state + (static_cast<size_t>(slot) * a.heads + head) * a.dim * vp;
    auto sums = [&](int g) {
      return a.sums + ((static_cast<size_t>(g) * a.heads + head) * slices + slice) * (static_cast<size_t>(BLOCKS) * VC * kWorkerThreads) + tid;
    };
    const bool own = seg == 0 && !(OUT && a.segments > 1);
    const bool fresh = __ldg(a.positions) == 0;
    const float ws = powf(w, static_cast<float>(a.segment));
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
          for (int e = 0; e < VC; ++e) p[e * kWorkerThreads] = s[e];
        }
      } else if (OUT) {
        for (int g = g_lo; g < g_hi; ++g) {
          const float* p = sums(g) + b * VC * kWorkerThreads;
#pragma unroll
          for (int e = 0; e < VC; ++e) s[e] = fmaf(ws, s[e], p[e * kWorkerThreads]);
        }
      }
      StoreTmem<VC>(t_s + lanes + b * 64 + part * VC, reinterpret_cast<const uint32_t*>(s));
    }
    asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");

    for (int c = 0; c < chunks; ++c) {
      const uint32_t par = c & 1;
      const int t0 = t_begin + c * kChunk, n = min(kChunk, t_end - t0);
      // S as an operand, and decayed for what the chunk adds.
      if (c > 0) {
        ok = MbarWaitWarp(st_done, (c - 1) & 1, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
      }
      const float wn = pw[n];
#pragma unroll 1
      for (int b = 0; b < BLOCKS; ++b) {
        const int d = b * 128 + row;
        if (b * 128 + quad * 32 >= a.dp) break;  // nothing but padding in this warp's rows
        uint32_t s[VC];
        LoadTmem<VC>(t_s + lanes + b * 64 + part * VC, s);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        if (OUT && d < a.dp) {
#pragma unroll
          for (int i = 0; i < VC / 8; ++i) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) Split(__uint_as_float(s[8 * i + 2 * e]), __uint_as_float(s[8 * i + 2 * e + 1]), hi[e], lo[e]);
            const uint32_t off = d * 128 + (((part * (VC / 8) + i) ^ (d & 7)) << 4);
            StoreShared16(at.s_hi + off, hi);
            StoreShared16(at.s_lo + off, lo);
          }
        }
#pragma unroll
        for (int e = 0; e < VC; ++e) s[e] = __float_as_uint(__uint_as_float(s[e]) * wn);
        StoreTmem<VC>(t_s + lanes + b * 64 + part * VC, s);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
      float o[VC];
      if (OUT) {
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(s_ready);

        // Scores times decay, 32 columns at a time: their first parts go to the first 16 of the columns, the second parts to the others.
        ok = MbarWaitWarp(sc_done, par, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll
        for (int g = 0; g < PC / 32; ++g) {
          const int j0 = part * PC + g * 32;
          uint32_t hi[16], lo[16];
          if (j0 > quad * 32 + 31) {  // all of it in the future
#pragma unroll
            for (int e = 0; e < 16; ++e) hi[e] = lo[e] = 0u;
          } else {
            uint32_t s[32];
            TcLd32(t_p + lanes + j0, s);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            if (j0 < quad * 32) {  // all of it in the past: w^(row - j) = w^(row - j0 - 31) w^(31 - e), both exponents from 0 up
              const float wr = pw[row - j0 - 31];
#pragma unroll
              for (int e = 0; e < 32; e += 4) {
                const float4 we = *reinterpret_cast<const float4*>(pw_down + e);
                Split(__uint_as_float(s[e]) * we.x * wr, __uint_as_float(s[e + 1]) * we.y * wr, hi[e / 2], lo[e / 2]);
                Split(__uint_as_float(s[e + 2]) * we.z * wr, __uint_as_float(s[e + 3]) * we.w * wr, hi[e / 2 + 1], lo[e / 2 + 1]);
              }
            } else {
#pragma unroll
              for (int e = 0; e < 32; e += 2) {
                const int back = lane - e;
                const float x = back >= 0 ? __uint_as_float(s[e]) * pw[max(back, 0)] : 0.f;
                const float y = back >= 1 ? __uint_as_float(s[e + 1]) * pw[max(back - 1, 0)] : 0.f;
                Split(x, y, hi[e / 2], lo[e / 2]);
              }
            }
          }
          TcSt16(t_p + lanes + j0, hi);
          TcSt16(t_p + lanes + j0 + 16, lo);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
        ok = MbarWaitWarp(o_done, par, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        LoadTmem<VC>(t_o + lanes + part * VC, reinterpret_cast<uint32_t*>(o));
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(p_ready);
        const float wi = pw[row + 1];
#pragma unroll
        for (int e = 0; e < VC; ++e) o[e] *= wi;
      }

      // Decayed values, in the place of Q (its products are done).
      if (carries(c)) {
        ok = MbarWaitWarp(full, par, lane, abort_word) && ok;
#pragma unroll
        for (int i = 0; i < kAtom / 16 / kWorkerThreads; ++i) {
          const int idx = i * kWorkerThreads + tid, j = idx >> 3;
          uint32_t v[4], hi[4], lo[4];
          asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];\n" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(at.v + idx * 16) : "memory");
          const float wj = j < n ? pw[max(n - 1 - j, 0)] : 0.f;
#pragma unroll
          for (int e = 0; e < 4; ++e) Split(Low(v[e]) * wj, High(v[e]) * wj, hi[e], lo[e]);
          StoreShared16(at.vd_hi + idx * 16, hi);
          StoreShared16(at.vd_lo + idx * 16, lo);
        }
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        __syncwarp();
        if (lane == 0) MbarArrive(vd_ready);
      }

      if (OUT) {
        ok = MbarWaitWarp(pv_done, par, lane, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        uint32_t x[VC];
        LoadTmem<VC>(t_o + lanes + part * VC, x);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        if (row < n) {
          float* p = a.o + (static_cast<size_t>(t0 + row) * a.heads + head) * a.vdim + v0;
          if (a.vdim % 4 == 0) {
#pragma unroll
            for (int e = 0; e < VC; e += 4) {
              if (v0 + e < a.vdim) {
                *reinterpret_cast<float4*>(p + e) = make_float4(o[e] + __uint_as_float(x[e]), o[e + 1] + __uint_as_float(x[e + 1]),
                                                                o[e + 2] + __uint_as_float(x[e + 2]), o[e + 3] + __uint_as_float(x[e + 3]));
              }
            }
          } else {
#pragma unroll
            for (int e = 0; e < VC; ++e)
              if (v0 + e < a.vdim) p[e] = o[e] + __uint_as_float(x[e]);
          }
        }
      }
    }

    if (!OUT || last) {
      ok = MbarWaitWarp(st_done, (chunks - 1) & 1, lane, abort_word) && ok;
      asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll 1
      for (int b = 0; b < BLOCKS; ++b) {
        const int d = b * 128 + row;
        uint32_t s[VC];
        LoadTmem<VC>(t_s + lanes + b * 64 + part * VC, s);
        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        if (!OUT) {
          float* p = sums(seg) + b * VC * kWorkerThreads;
#pragma unroll
          for (int e = 0; e < VC; ++e) p[e * kWorkerThreads] = d < a.dp ? __uint_as_float(s[e]) : 0.f;
        } else if (d < a.dim) {
          float* p = state + static_cast<size_t>(d) * vp + v0;
#pragma unroll
          for (int e = 0; e < VC; e += 4) {
            if (v0 + e < vp) {
              *reinterpret_cast<float4*>(p + e) = make_float4(__uint_as_float(s[e]), __uint_as_float(s[e + 1]), __uint_as_float(s[e + 2]), __uint_as_float(s[e + 3]));
            }
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

size_t SmemBytes(int dp)
{
  Places p;
  return PlaceAll(dp, 0, &p);
}

// What a call is cut into.
struct Plan {
  int dp, blocks, slices, segment, segments;
  size_t sums_bytes;
};
Plan PlanFor(int tokens, int heads, int dim, int vdim)
{
  Plan p;
  p.dp = (dim + 15) / 16 * 16;
  p.blocks = (p.dp + 127) / 128;
  p.slices = (vdim + kVS - 1) / kVS;
  const int chunks = (tokens + kChunk - 1) / kChunk, ctas = heads * p.slices, slots = 148 * (2 * (SmemBytes(p.dp) + 2048) <= 228 * 1024 && p.blocks == 1 ? 2 : 1);
  // Rounds of CTAs times chunks of a segment, in chunks of the second launch: the state alone at two fifths, a launch at one half, the sums of
  // an earlier segment at a sixteenth per block of S.
  double best = 1e30;
  p.segments = 1;
  int per = chunks;
  for (int n = 1; n <= chunks && n <= 32; ++n) {
    const int len = (chunks + n - 1) / n, used = (chunks + len - 1) / len;
    double cost = static_cast<double>((ctas * used + slots - 1) / slots) * len;
    if (used > 1) {
      cost += 0.4 * ((ctas * (used - 1) + slots - 1) / slots) * len + 0.5 + 0.0625 * p.blocks * (used - 1) * ((ctas * used + slots - 1) / slots);
    }
    if (cost < best * 0.97) {
      best = cost;
      p.segments = used;
      per = len;
    }
  }
  p.segment = per * kChunk;
  p.sums_bytes = p.segments > 1 ? static_cast<size_t>(p.segments) * ctas * p.blocks * kChunk * kVS * sizeof(float) : 0;
  return p;
}

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// bf16 [tokens][heads][ld], boxes of 64 channels of one head x 128 tokens.
bool Encode(CUtensorMap* map, const void* ptr, int ld, int heads, int tokens)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  const cuuint64_t dims[3] = {static_cast<cuuint64_t>(ld), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(tokens)};
  const cuuint64_t strides[2] = {static_cast<cuuint64_t>(ld) * 2, static_cast<cuuint64_t>(ld) * 2 * heads};
  const cuuint32_t box[3] = {64, 1, kChunk}, elem[3] = {1, 1, 1};
  return encode != nullptr &&
         encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

cudaError_t PrepareChunks()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(BLOCKS, OUT) \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(RetentionChunkTc<BLOCKS, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024);
    TLALOC_OPT_IN(1, true)
    TLALOC_OPT_IN(1, false)
    TLALOC_OPT_IN(2, true)
    TLALOC_OPT_IN(2, false)
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
  const size_t smem = SmemBytes(a.dp);
  const int threads = WorkersFor(p.blocks) * 32 + 64;
  return p.blocks == 1 ? LaunchChained(RetentionChunkTc<1, OUT>, grid, threads, smem, st, maps[0], maps[1], maps[2], a)
                       : LaunchChained(RetentionChunkTc<2, OUT>, grid, threads, smem, st, maps[0], maps[1], maps[2], a);
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
  CUtensorMap maps[3];
  if (!Encode(&maps[0], q, dim_ld, heads, tokens) || !Encode(&maps[1], k, dim_ld, heads, tokens) || !Encode(&maps[2], v, v_ld, heads, tokens)) {
    return Fail(kInternal, "%s: the tensor maps could not be encoded", op);
  }
  ChunkArgs a = {};
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
