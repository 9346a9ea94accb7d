// Attention of absorbed queries over a paged pool of latents (include/tlaloc_b200.h, tlaloc_b200_latent_attention).
//
// LatentAttentionGeneric: any sizes, f32 or bf16, plain FMA.  A CTA serves one (row, head): tiles of 128 positions, a warp
// per position for the scores (lanes over the channels), an online softmax in f32, then a thread per latent channel.
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
  int T, H, kv_rank, row, num_blocks, block_size, max_blocks, num_tables, window;
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
  const int page = min(max(__ldg(table + pos / p.block_size), 0), p.num_blocks - 1);
  return (static_cast<size_t>(page) * p.block_size + pos % p.block_size) * p.pool_ld;
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

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" size_t tlaloc_b200_latent_attention_scratch_bytes(int32_t, int32_t, int32_t, int32_t, int32_t) { return 0; }

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
  (void)scratch;
  (void)scratch_bytes;
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
  p.max_blocks = max_blocks;
  p.num_tables = num_tables;
  p.window = window;
  p.scale = scale;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid(num_heads, num_tokens);
  const size_t smem = sizeof(float) * static_cast<size_t>(p.row);
  const cudaError_t e = dtype == TLALOC_B200_F32 ? LaunchChained(LatentAttentionGeneric<float>, grid, kGenericThreads, smem, st, p)
                                                 : LaunchChained(LatentAttentionGeneric<__nv_bfloat16>, grid, kGenericThreads, smem, st, p);
  if (e != cudaSuccess) return CudaFail("LATENT_ATTENTION launch", e);
  CountLaunches(1);
  return kOk;
}
