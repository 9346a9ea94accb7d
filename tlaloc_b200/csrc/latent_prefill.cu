// Attention of a prompt portion over expanded keys and values (include/tlaloc_b200.h, tlaloc_b200_window_attention), bf16,
// on the tensor cores: tcgen05.mma kind::f16 with f32 accumulators in TMEM, every operand by TMA.
//
// A CTA owns 128 queries of one head and walks the tiles of 128 keys that any of them sees.  Scores S = Q K^T: queries are the
// MMA's M (TMEM lanes), keys its N, so a row of scores belongs to two softmax threads (64 keys each) that exchange one maximum.  Two score
// accumulators: the MMAs of tile j + 1 run under the softmax of tile j.  The weights, as bf16, take the place of their scores in TMEM
// and are the A operand of O += P V, with O in TMEM too; shared memory holds nothing but Q and the rings of K and V (two tiles each
// at the common sizes, so that a whole tile of each is in flight).  The running maximum is raised lazily: only when a row's maximum grows by more than 2^8 over the
// reference in use is O rescaled (the exponentials stay below 2^8 in f32, and the result is divided by their f32 sum).
//   producer lane   Q once; then K atoms (128 keys x 64 channels: the per-head part, then the rotated part all heads share) and V
//                   tiles in the order the MMAs use them, each onto its own ring
//   MMA lane        S(0); then S(j + 1), O += P(j) V(j)
//   eight warps     softmax and, at the end, the output rows: warps w and w + 4 share 32 queries
// Channels past a part's end are outside its tensor map and arrive as zeros.  Every mbarrier wait is bounded.
//
// Grouped heads and several maps: a query head is (value head, place in its group, map) and takes the keys of (value head, map).  The
// first keep_first keys stay visible: their tiles come ahead of the window's.
#include <cuda.h>

#include "common.cuh"
#include "tc_common.cuh"

namespace tlaloc_b200 {
namespace {

using namespace tc;

constexpr int kQ = 128, kKeys = 128;           // queries of a CTA, keys of a tile
constexpr int kAtom = kQ * 64 * 2;             // 128 rows x 64 channels
constexpr int kSoftmaxWarps = 8;
constexpr int kThreads = kSoftmaxWarps * 32 + 64;
constexpr int kMaxSmem = 227 * 1024;

struct WindowArgs {
  void* out;
  int64_t out_ld;
  int T, L, q0, window;         // query i is key q0 + i; window 0: everything up to itself
  int keep, group, maps, out_f32;  // keys visible whatever the window; query heads of a value head; key heads of a value head
  int dim, rot, vdim;
  int qk_atoms, dim_atoms, v_atoms, k_stages, v_stages;
  float scale_log2;
};

__device__ int g_window_status = 0;

__host__ __device__ constexpr uint32_t InstrDesc(int n, bool b_mn_major)  // f32 accumulator, bf16, A K-major, M = 128
{
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn_major ? 1u << 16 : 0u) | (static_cast<uint32_t>(n >> 3) << 17) | (8u << 24);
}
__device__ __forceinline__ void TmaBox(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar)
{
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(dst),
               "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(z), "r"(bar)
               : "memory");
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
constexpr float kLazy = 8.f;  // how far (log2) a row's maximum may grow past the reference in use

__global__ void __launch_bounds__(kThreads, 1)
    WindowAttentionTc(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_rot, const __grid_constant__ CUtensorMap map_v, const __grid_constant__ WindowArgs a)
{
  extern __shared__ unsigned char smem_raw[];
  __shared__ alignas(8) uint64_t bars[2 + 2 + 1 + 2 + 2 + 2];
  __shared__ uint32_t slot_store[2];
  __shared__ float s_row[2][2][kQ];  // [tile parity][half of the keys][query]
  const uint32_t base = (SmemAddr(smem_raw) + 1023u) & ~1023u;
  unsigned char* smem = smem_raw + (base - SmemAddr(smem_raw));
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // Of the tiles in the rings: kfull, vfull "landed"; a K stage is free again when the scores of its tile are there (sfull), a V stage
  // when its product is (odone).  pfull: the weights are there; two barriers, because the softmax may be a tile ahead of the product (one
  // that is two phases ahead of a wait looks like one that has not come).
  const uint32_t kfull = SmemAddr(bars), vfull = kfull + 16, qfull = vfull + 16, sfull = qfull + 8, pfull = sfull + 16, odone = pfull + 16;
  volatile uint32_t* slot = slot_store;
  volatile uint32_t* abort_word = slot_store + 1;
  const uint32_t sk = a.qk_atoms * kAtom, sv = sk + a.k_stages * a.qk_atoms * kAtom;  // offsets of the K and V rings, behind Q
  const int qk_atoms = a.qk_atoms, dim_atoms = a.dim_atoms, v_atoms = a.v_atoms, k_stages = a.k_stages, v_stages = a.v_stages;
  const int v_tile = v_atoms * kAtom, k_tile = qk_atoms * kAtom;
  const int m0 = blockIdx.x * kQ, head = blockIdx.y;
  const int q_last = min(m0 + kQ, a.T) - 1;
  const int v_head = head / a.group, k_head = v_head * a.maps + head % a.maps;
  // The tiles of kept keys, then those from the first one the window of any query reaches.
  const int tile_hi = min(a.q0 + q_last, a.L - 1) / kKeys;
  const int tile_lo = a.window > 0 ? max(0, a.q0 + m0 - a.window + 1) / kKeys : 0;
  const int kept = min((a.keep + kKeys - 1) / kKeys, tile_lo), tiles = tile_hi - tile_lo + 1 + kept;
  auto first_key = [&](int j) { return (j < kept ? j : tile_lo + j - kept) * kKeys; };
  if (tid == 0) {
    *abort_word = 0u;
    for (int i = 0; i < 2; ++i) {
      MbarInit(kfull + 8 * i, 1);
      MbarInit(vfull + 8 * i, 1);
      MbarInit(sfull + 8 * i, 1);
      MbarInit(pfull + 8 * i, kSoftmaxWarps);
      MbarInit(odone + 8 * i, 1);
    }
    MbarInit(qfull, 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(SmemAddr(slot_store)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  const uint32_t tmem = *slot, tmem_o = tmem + 256;  // S0, S1 at columns 0 and 128; O from column 256
  GridDependencySync();
  bool ok = true;

  if (warp == kSoftmaxWarps) {
    if (ElectOne()) {
      // Stages are one or two per ring; everything is counted along (a division per box would take longer than the box).
      auto load_k = [&](int j) {
        const int key = first_key(j), stage = k_stages == 2 ? j & 1 : 0, before = j - k_stages;
        const uint32_t bar = kfull + 8 * stage;
        uint32_t dst = base + sk + stage * k_tile;
        if (before >= 0) ok = MbarWait(sfull + 8 * (before & 1), (before >> 1) & 1, abort_word) && ok;
        MbarExpectTx(bar, k_tile);
        for (int c = 0; c < dim_atoms; ++c, dst += kAtom) TmaBox(dst, &map_k, c * 64, k_head, key, bar);
        for (int c = dim_atoms; c < qk_atoms; ++c, dst += kAtom) TmaBox(dst, &map_rot, (c - dim_atoms) * 64, 0, key, bar);
      };
      MbarExpectTx(qfull, qk_atoms * kAtom);
      for (int c = 0; c < qk_atoms; ++c) {
        TmaBox(base + c * kAtom, &map_q, c < dim_atoms ? c * 64 : a.dim + (c - dim_atoms) * 64, head, m0, qfull);
      }
      load_k(0);
      for (int j = 0; j < tiles; ++j) {
        if (j + 1 < tiles) load_k(j + 1);
        const int stage = v_stages == 2 ? j & 1 : 0, before = j - v_stages;
        const uint32_t bar = vfull + 8 * stage;
        if (before >= 0) ok = MbarWait(odone + 8 * (before & 1), (before >> 1) & 1, abort_word) && ok;
        MbarExpectTx(bar, v_tile);
        for (int c = 0; c < v_atoms; ++c) TmaBox(base + sv + stage * v_tile + c * kAtom, &map_v, c * 64, v_head, first_key(j), bar);
      }
      if (!ok) {  // given up: let the copies in flight land before the CTA's shared memory goes away
        volatile uint32_t never = 0;
        for (int s = 0; s < k_stages; ++s)
          if (tiles > s) MbarWait(kfull + 8 * s, ((tiles - 1 - s) / k_stages) & 1, &never);
        for (int s = 0; s < v_stages; ++s)
          if (tiles > s) MbarWait(vfull + 8 * s, ((tiles - 1 - s) / v_stages) & 1, &never);
      }
    }
    __syncwarp();
  } else if (warp == kSoftmaxWarps + 1) {
    if (ElectOne()) {
      const uint32_t s_idesc = InstrDesc(kKeys, false), o_idesc = InstrDesc((a.vdim + 15) / 16 * 16, true);
      const uint64_t qd = SmemDesc(base, 16, 1024), kd = SmemDesc(base + sk, 16, 1024);
      const uint64_t vd = SmemDesc(base + sv, kAtom, 1024);
      ok = MbarWait(qfull, 0, abort_word) && ok;
      auto scores = [&](int j) {
        const uint32_t b = j & 1, acc = tmem + b * 128;
        // The buffer held P(j - 2), whose product is in front of these MMAs in the same queue.
        const int stage = k_stages == 2 ? j & 1 : 0;
        uint64_t qa = qd, ka = kd + static_cast<uint64_t>((stage * k_tile) >> 4);
        ok = MbarWait(kfull + 8 * stage, (k_stages == 2 ? j >> 1 : j) & 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        for (int c = 0; c < qk_atoms; ++c, qa += kAtom >> 4, ka += kAtom >> 4) {
          const int width = c < dim_atoms ? a.dim - 64 * c : a.rot - 64 * (c - dim_atoms);
          if (width > 48) {
#pragma unroll
            for (int k = 0; k < 4; ++k) TcMmaBf16(acc, qa + 2 * k, ka + 2 * k, s_idesc, c > 0 || k > 0 ? 1u : 0u);
          } else {
            for (int k = 0; 16 * k < width; ++k) TcMmaBf16(acc, qa + 2 * k, ka + 2 * k, s_idesc, c > 0 || k > 0 ? 1u : 0u);
          }
        }
        TcCommit(sfull + 8 * b);
      };
      scores(0);
      for (int j = 0; j < tiles; ++j) {
        if (j + 1 < tiles) scores(j + 1);
        const int stage = v_stages == 2 ? j & 1 : 0;
        const uint64_t va = vd + static_cast<uint64_t>((stage * v_tile) >> 4);
        const uint32_t pa = tmem + (j & 1) * 128;
        ok = MbarWait(vfull + 8 * stage, (v_stages == 2 ? j >> 1 : j) & 1, abort_word) && ok;
        ok = MbarWait(pfull + 8 * (j & 1), (j >> 1) & 1, abort_word) && ok;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        // P: eight columns per 16 keys; V: keys are its rows, 16 of them per step
        TcMmaTmemA(tmem_o, pa, va, o_idesc, j > 0 ? 1u : 0u);
#pragma unroll
        for (int k = 1; k < kKeys / 16; ++k) TcMmaTmemA(tmem_o, pa + 8 * k, va + ((k * 16 * 128) >> 4), o_idesc, 1u);
        TcCommit(odone + 8 * (j & 1));
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3, half = warp >> 2, row = quad * 32 + lane;  // this thread's query: TMEM lane `row`, keys [64 half, 64 half + 64)
    const int qpos = a.q0 + m0 + row;
    const int first = a.window > 0 ? qpos - a.window + 1 : 0;
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    constexpr int kHalf = kKeys / 2;
    // The other half of the row: the two warps of a quad meet at a named barrier of 64 threads.
    auto other = [&](int b, float mine) {
      s_row[b][half][row] = mine;
      asm volatile("bar.sync %0, 64;\n" ::"r"(1 + quad) : "memory");
      return s_row[b][half ^ 1][row];
    };
    // The keys every query of the CTA sees need no mask: not past the first query, not before the last one's window.
    const int safe_hi = a.q0 + m0, safe_lo = a.window > 0 ? a.q0 + m0 + kQ - 1 - a.window + 1 : 0;
    const int o_lo = half * 32;  // O's columns in blocks of 32, every second one
    float top = -INFINITY, sum = 0.f;
    for (int j = 0; j < tiles; ++j) {
      const int key0 = first_key(j) + half * kHalf, b = j & 1;
      ok = MbarWaitWarp(sfull + 8 * b, (j >> 1) & 1, lane, abort_word) && ok;
      asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
      uint32_t s[kHalf];
      TcLd32(tmem + lanes + b * 128 + half * kHalf, s);
      TcLd32(tmem + lanes + b * 128 + half * kHalf + 32, s + 32);
      asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
      float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (key0 + kHalf - 1 > safe_hi || (key0 < safe_lo && key0 + kHalf > a.keep)) {
#pragma unroll
        for (int e = 0; e < kHalf; ++e) {
          const int key = key0 + e;
          if (key > qpos || (key < first && key >= a.keep)) s[e] = __float_as_uint(-INFINITY);
        }
      }
#pragma unroll
      for (int e = 0; e < kHalf; ++e) t4[e & 3] = fmaxf(t4[e & 3], __uint_as_float(s[e]));
      float tile_top = fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])) * a.scale_log2;  // the scale is positive
      tile_top = fmaxf(tile_top, other(b, tile_top));  // both halves of the scores are in registers from here on
      // O has tile j - 2 in it (its product was ahead of S(j)); each of the two barriers is never more than one phase ahead of a wait.
      if (j >= 2) ok = MbarWaitWarp(odone + 8 * b, ((j >> 1) - 1) & 1, lane, abort_word) && ok;
      // Both warps of a quad see the same maxima, so they take the same turn here.
      if (__any_sync(0xffffffffu, tile_top > top + kLazy || (top == -INFINITY && tile_top > -INFINITY))) {
        const float next = fmaxf(top, tile_top);
        const float keep = top == -INFINITY ? 0.f : Exp2(top - next);
        if (j > 0) {
          ok = MbarWaitWarp(odone + 8 * (b ^ 1), ((j - 1) >> 1) & 1, lane, abort_word) && ok;
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          for (int c = o_lo; c < a.vdim; c += 64) {
            uint32_t o[32];
            TcLd32(tmem_o + lanes + c, o);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * keep);
            TcSt32(tmem_o + lanes + c, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
        }
        sum *= keep;
        top = next;
      }
      const float ref = top == -INFINITY ? 0.f : top;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int e = 0; e < kHalf; e += 2) {
        const float p0 = Exp2(fmaf(__uint_as_float(s[e]), a.scale_log2, -ref)), p1 = Exp2(fmaf(__uint_as_float(s[e + 1]), a.scale_log2, -ref));
        s0 += p0;
        s1 += p1;
        s[e / 2] = Pack(p0, p1);
      }
      sum += s0 + s1;
      TcSt32(tmem + lanes + b * 128 + half * 32, s);
      asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
      __syncwarp();
      if (lane == 0) MbarArrive(pfull + 8 * b);
    }
    sum += other(tiles & 1, sum);
    ok = MbarWaitWarp(odone + 8 * ((tiles - 1) & 1), ((tiles - 1) >> 1) & 1, lane, abort_word) && ok;
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const float inv = sum > 0.f ? 1.f / sum : 0.f;
    const size_t out_at = static_cast<size_t>(m0 + row) * a.out_ld + static_cast<size_t>(head) * a.vdim;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + out_at;
    float* out32 = static_cast<float*>(a.out) + out_at;
    const bool live = m0 + row < a.T;
    for (int c = o_lo; c < a.vdim; c += 64) {
      uint32_t o[32];
      TcLd32(tmem_o + lanes + c, o);
      asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
      for (int e = 0; e < 32; e += 8) {
        if (live && c + e < a.vdim && a.out_f32) {
#pragma unroll
          for (int i = 0; i < 8; i += 4) {
            *reinterpret_cast<float4*>(out32 + c + e + i) = make_float4(__uint_as_float(o[e + i]) * inv, __uint_as_float(o[e + i + 1]) * inv,
                                                                        __uint_as_float(o[e + i + 2]) * inv, __uint_as_float(o[e + i + 3]) * inv);
          }
        } else if (live && c + e < a.vdim) {  // vdim is a multiple of 8
          uint32_t w[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) w[i] = Pack(__uint_as_float(o[e + 2 * i]) * inv, __uint_as_float(o[e + 2 * i + 1]) * inv);
          *reinterpret_cast<uint4*>(out + c + e) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  }
  if (!ok) atomicExch(&g_window_status, 1);
  __syncthreads();
  if (warp == 0) {
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512u) : "memory");
  }
}

// The rows [0, keep) and [first, first + count - keep) of one sequence out of its pages, 16 bytes a thread.
__global__ void __launch_bounds__(256) LatentGatherKernel(const uint4* pool, int64_t pool_ld16, const int* table, uint4* out, int64_t out_ld16,
                                                          int first, int keep, int count, int words, int block_size, int num_blocks,
                                                          int max_blocks)
{
  GridDependencySync();
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= static_cast<long long>(count) * words) return;
  const int r = static_cast<int>(i / words), w = static_cast<int>(i % words), pos = r < keep ? r : first + r - keep;
  const int page = min(max(__ldg(table + min(pos / block_size, max_blocks - 1)), 0), num_blocks - 1);
  out[r * out_ld16 + w] = pool[(static_cast<size_t>(page) * block_size + pos % block_size) * pool_ld16 + w];
}

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 [rows][heads][channels], boxes of 64 channels of one head x 128 rows.
bool Encode(CUtensorMap* map, const void* ptr, int channels, int heads, int rows, int64_t head_ld, int64_t row_ld)
{
  auto encode = reinterpret_cast<EncodeTiledFn>(TensorMapEncoder());
  if (encode == nullptr) return false;
  const cuuint64_t dims[3] = {static_cast<cuuint64_t>(channels), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows)};
  const cuuint64_t strides[2] = {static_cast<cuuint64_t>(head_ld) * 2, static_cast<cuuint64_t>(row_ld) * 2};
  const cuuint32_t box[3] = {64, 1, 128};
  const cuuint32_t elem[3] = {1, 1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

cudaError_t PrepareWindowAttention()
{
  static OncePerDevice once;
  return once.Run([](int) {
    TensorMapEncoder();
    return cudaFuncSetAttribute(WindowAttentionTc, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 3072);
  });
}
int ReadWindowStatus()
{
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_window_status, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_window_status, &zero, sizeof(int));
  }
  return v;
}
KernelSetup g_setup(PrepareWindowAttention, ReadWindowStatus);

// Shared-memory rings beside Q and P: false if the sizes do not fit.
bool Rings(int dim, int rot, int vdim, WindowArgs* a)
{
  a->dim_atoms = (dim + 63) / 64;
  a->qk_atoms = a->dim_atoms + (rot + 63) / 64;
  a->v_atoms = (vdim + 63) / 64;
  const int atoms = (kMaxSmem - 4096) / kAtom - a->qk_atoms;  // static shared memory and the alignment slack aside
  a->k_stages = atoms >= 2 * a->qk_atoms + a->v_atoms ? 2 : 1;
  a->v_stages = atoms - a->k_stages * a->qk_atoms >= 2 * a->v_atoms ? 2 : 1;
  return vdim <= 256 && atoms >= a->qk_atoms + a->v_atoms;
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_latent_gather(const void* pool, int64_t pool_ld, int32_t dtype, const int32_t* table, void* out, int64_t out_ld,
                                         int32_t first, int32_t keep, int32_t count, int32_t row, int32_t num_blocks, int32_t block_size,
                                         int32_t max_blocks, void* stream)
{
  const char* op = "LATENT_GATHER";
  if (!pool || !table || !out) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (first < keep || keep < 0 || keep > count || count < 0 || row < 1 || num_blocks < 1 || block_size < 1 || max_blocks < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (static_cast<int64_t>(first) + count - keep > static_cast<int64_t>(max_blocks) * block_size) return Fail(kInvalid, "%s: the rows pass the end of the table", op);
  const int per = 16 / static_cast<int>(DtypeBytes(dtype));
  const int words = (row + per - 1) / per;
  if (pool_ld % per || out_ld % per || pool_ld < words * per || out_ld < words * per || !Aligned16(pool) || !Aligned16(out)) {
    return Fail(kInvalid, "%s: rows must be whole 16-byte words on both sides", op);
  }
  if (count == 0) return kOk;
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(count) * words + 255) / 256);
  const cudaError_t e = LaunchChained(LatentGatherKernel, blocks, 256, 0, static_cast<cudaStream_t>(stream), static_cast<const uint4*>(pool),
                                      pool_ld / per, table, static_cast<uint4*>(out), out_ld / per, first, keep, count, words, block_size,
                                      num_blocks, max_blocks);
  if (e != cudaSuccess) return CudaFail("LATENT_GATHER launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_window_attention_applies(int32_t dim, int32_t rot_dim, int32_t vdim)
{
  WindowArgs a;
  return dim >= 8 && dim % 8 == 0 && rot_dim % 8 == 0 && rot_dim >= 0 && vdim >= 8 && vdim % 8 == 0 && Rings(dim, rot_dim, vdim, &a) ? 1 : 0;
}

extern "C" int tlaloc_b200_window_attention(const void* q, const void* k, int64_t k_head_ld, const void* k_rot, int64_t rot_ld, const void* v,
                                            int64_t v_head_ld, int64_t kv_ld, void* out, int64_t out_ld, int32_t out_dtype, int32_t num_queries,
                                            int32_t num_keys, int32_t first_query, int32_t num_heads, int32_t v_heads, int32_t maps, int32_t dim,
                                            int32_t rot_dim, int32_t vdim, int32_t window, int32_t keep_first, float scale, void* stream)
{
  const char* op = "WINDOW_ATTENTION";
  if (!q || !k || !v || !out || (rot_dim > 0 && !k_rot)) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (num_queries < 0 || num_keys < 1 || first_query < 0 || num_heads < 1 || window < 0 || num_heads > 65535) return Fail(kInvalid, "%s: bad sizes", op);
  if (v_heads < 1 || maps < 1 || num_heads % (v_heads * maps) || keep_first < 0 || !IsFloatType(out_dtype)) return Fail(kInvalid, "%s: bad heads", op);
  if (!(scale > 0.f)) return Fail(kUnsupported, "%s: the scale must be positive", op);
  if (first_query + num_queries > num_keys) return Fail(kInvalid, "%s: query %d has no key of its own", op, first_query + num_queries - 1);
  if (!tlaloc_b200_window_attention_applies(dim, rot_dim, vdim)) {
    return Fail(kUnsupported, "%s: dim, rot_dim and vdim are multiples of 8, vdim up to 256, and the tiles must fit shared memory", op);
  }
  if (rot_ld % 8 || kv_ld % 8 || k_head_ld % 8 || v_head_ld % 8 || out_ld % 8 || !Aligned16(q) || !Aligned16(k) || !Aligned16(k_rot) || !Aligned16(v) || !Aligned16(out)) {
    return Fail(kInvalid, "%s: addresses and strides must be multiples of 16 bytes", op);
  }
  if (num_queries == 0) return kOk;
  cudaError_t e = PrepareWindowAttention();
  if (e != cudaSuccess) return CudaFail("WINDOW_ATTENTION set-up", e);
  WindowArgs a = {};
  Rings(dim, rot_dim, vdim, &a);
  a.out = out;
  a.out_f32 = out_dtype == TLALOC_B200_F32 ? 1 : 0;
  a.keep = window > 0 ? keep_first : 0;
  a.maps = maps;
  a.group = num_heads / v_heads;
  a.out_ld = out_ld;
  a.T = num_queries;
  a.L = num_keys;
  a.q0 = first_query;
  a.window = window;
  a.dim = dim;
  a.rot = rot_dim;
  a.vdim = vdim;
  a.scale_log2 = scale * 1.4426950408889634f;
  CUtensorMap mq, mk, mr, mv;
  const int64_t q_row = dim + rot_dim;
  if (!Encode(&mq, q, dim + rot_dim, num_heads, num_queries, q_row, q_row * num_heads) || !Encode(&mk, k, dim, v_heads * maps, num_keys, k_head_ld, kv_ld) ||
      !Encode(&mv, v, vdim, v_heads, num_keys, v_head_ld, kv_ld) || (rot_dim > 0 && !Encode(&mr, k_rot, rot_dim, 1, num_keys, rot_ld, rot_ld))) {
    return Fail(kInternal, "%s: the tensor maps could not be encoded", op);
  }
  if (rot_dim == 0) mr = mk;
  const size_t smem = static_cast<size_t>(a.qk_atoms + a.k_stages * a.qk_atoms + a.v_stages * a.v_atoms) * kAtom + 1024;
  const dim3 grid((num_queries + kQ - 1) / kQ, num_heads);
  e = LaunchChained(WindowAttentionTc, grid, kThreads, smem, static_cast<cudaStream_t>(stream), mq, mk, mr, mv, a);
  if (e != cudaSuccess) return CudaFail("WINDOW_ATTENTION launch", e);
  CountLaunches(1);
  return kOk;
}
