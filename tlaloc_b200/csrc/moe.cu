// Routing of tokens to experts: the experts with the largest logits and the softmax of those, then the tokens sorted by expert, so that an
// expert's rows are consecutive and one grouped projection runs all experts.  Logits and weights are f32.
#include "common.cuh"
#include "dense_gemm.cuh"

namespace tlaloc_b200 {
namespace {

constexpr int kRouteThreads = 1024, kRouteWarps = kRouteThreads / 32;
constexpr int kSmallTokens = 128;  // up to here one CTA does both parts

// One token: `top` times the largest logit left (the first of equals); a lane holds the experts lane, lane + 32, ...
template <int PER>
__device__ __forceinline__ void PickTop(const float* z, int experts, int top, int* ids, float* weights, int lane)
{
  float v[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) v[i] = lane + 32 * i < experts ? z[lane + 32 * i] : -INFINITY;
  uint32_t taken = 0;
  float first = 0.f, sum = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + 32 * i;
      if (e < experts && !((taken >> i) & 1u) && (at == 0x7fffffff || v[i] > best)) {
        best = v[i];
        at = e;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (oa != 0x7fffffff && (at == 0x7fffffff || ob > best || (ob == best && oa < at))) {
        best = ob;
        at = oa;
      }
    }
    at = min(at, experts - 1);
    if (k == 0) first = best;
    const float w = expf(best - first);
    sum += w;
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    if (lane == 0) {
      ids[k] = at;
      weights[k] = w;
    }
  }
  __syncwarp();
  for (int k = lane; k < top; k += 32) weights[k] /= sum;
}

// PICK: each warp picks for its tokens.  SORT (one CTA): counts, row offsets of the experts, every entry's row.
template <int PER, bool PICK, bool SORT>
__global__ void __launch_bounds__(kRouteThreads) RouteKernel(const float* logits, int64_t ld, int* ids, float* weights, int* offsets, int* entry_rows,
                                                             int* row_tokens, int tokens, int experts, int top)
{
  GridDependencySync();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if constexpr (PICK) {
    for (int t = blockIdx.x * kRouteWarps + warp; t < tokens; t += gridDim.x * kRouteWarps) {
      PickTop<PER>(logits + t * ld, experts, top, ids + static_cast<size_t>(t) * top, weights + static_cast<size_t>(t) * top, lane);
    }
    if constexpr (SORT) __syncthreads();
  }
  if constexpr (SORT) {
    __shared__ int next[kMaxGroups];
    const int n = tokens * top;
    for (int e = tid; e < experts; e += kRouteThreads) next[e] = 0;
    __syncthreads();
    for (int i = tid; i < n; i += kRouteThreads) atomicAdd(&next[ids[i]], 1);
    __syncthreads();
    if (warp == 0) {
      int total = 0;
      for (int e0 = 0; e0 < experts; e0 += 32) {
        const int e = e0 + lane, own = e < experts ? next[e] : 0;
        int v = own;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const int u = __shfl_up_sync(0xffffffffu, v, o);
          if (lane >= o) v += u;
        }
        if (e < experts) {
          next[e] = total + v - own;
          offsets[e] = total + v - own;
        }
        total += __shfl_sync(0xffffffffu, v, 31);
      }
      if (lane == 0) offsets[experts] = total;
    }
    __syncthreads();
    for (int i = tid; i < n; i += kRouteThreads) {
      const int r = atomicAdd(&next[ids[i]], 1);  // which row of its expert an entry gets does not matter to its result
      entry_rows[i] = r;
      row_tokens[r] = i / top;
    }
  }
}

// out[r, :] = in[rows[r], :], 16 bytes a thread.
__global__ void __launch_bounds__(256) GatherRowsKernel(const uint4* in, const int* rows, uint4* out, long long total, int words)
{
  GridDependencySync();
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= total) return;
  const long long r = i / words;
  out[i] = in[static_cast<long long>(__ldg(rows + r)) * words + (i - r * words)];
}
__global__ void __launch_bounds__(256) GatherRows2Kernel(const uint16_t* in, const int* rows, uint16_t* out, long long total, int words)
{
  GridDependencySync();
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= total) return;
  const long long r = i / words;
  out[i] = in[static_cast<long long>(__ldg(rows + r)) * words + (i - r * words)];
}

template <int PER>
cudaError_t LaunchRoute(const float* logits, int64_t ld, int* ids, float* weights, int* offsets, int* entry_rows, int* row_tokens, int tokens,
                        int experts, int top, cudaStream_t st, int* launches)
{
  if (tokens <= kSmallTokens) {
    *launches = 1;
    return LaunchChained(RouteKernel<PER, true, true>, 1, kRouteThreads, 0, st, logits, ld, ids, weights, offsets, entry_rows, row_tokens, tokens, experts, top);
  }
  *launches = 2;
  const cudaError_t e = LaunchChained(RouteKernel<PER, true, false>, min((tokens + kRouteWarps - 1) / kRouteWarps, 148), kRouteThreads, 0, st, logits, ld, ids,
                                      weights, offsets, entry_rows, row_tokens, tokens, experts, top);
  if (e != cudaSuccess) return e;
  return LaunchChained(RouteKernel<PER, false, true>, 1, kRouteThreads, 0, st, logits, ld, ids, weights, offsets, entry_rows, row_tokens, tokens, experts, top);
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_moe_route(const float* logits, int64_t ld, int32_t* ids, float* weights, int32_t* offsets, int32_t* entry_rows,
                                     int32_t* row_tokens, int32_t tokens, int32_t experts, int32_t top, void* stream)
{
  const char* op = "MOE_ROUTE";
  if (!logits || !ids || !weights || !offsets || !entry_rows || !row_tokens) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (tokens < 0 || experts < 1 || top < 1 || top > experts || ld < experts) return Fail(kInvalid, "%s: bad sizes", op);
  if (experts > kMaxGroups) return Fail(kUnsupported, "%s: at most %d experts", op, kMaxGroups);
  if (static_cast<long long>(tokens) * top > (1 << 30)) return Fail(kInvalid, "%s: too many tokens", op);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int launches = 0;
  cudaError_t e;
  if (tokens == 0) return kOk;
#define TLALOC_ROUTE(PER) LaunchRoute<PER>(logits, ld, ids, weights, offsets, entry_rows, row_tokens, tokens, experts, top, st, &launches)
  if (experts <= 32) e = TLALOC_ROUTE(1);
  else if (experts <= 64) e = TLALOC_ROUTE(2);
  else if (experts <= 128) e = TLALOC_ROUTE(4);
  else if (experts <= 256) e = TLALOC_ROUTE(8);
  else e = TLALOC_ROUTE(32);
#undef TLALOC_ROUTE
  if (e != cudaSuccess) return CudaFail("MOE_ROUTE launch", e);
  CountLaunches(launches);
  return kOk;
}

extern "C" int tlaloc_b200_gather_rows(const void* in, const int32_t* rows, void* out, int32_t count, int64_t row_bytes, void* stream)
{
  const char* op = "GATHER_ROWS";
  if (!in || !rows || !out) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (count < 0 || row_bytes < 2 || row_bytes % 2) return Fail(kInvalid, "%s: bad sizes", op);
  if (count == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = row_bytes % 16 == 0 && Aligned16(in) && Aligned16(out);
  const int words = static_cast<int>(row_bytes / (vec ? 16 : 2));
  const long long total = static_cast<long long>(count) * words;
  const unsigned blocks = static_cast<unsigned>((total + 255) / 256);
  const cudaError_t e = vec ? LaunchChained(GatherRowsKernel, blocks, 256, 0, st, static_cast<const uint4*>(in), rows, static_cast<uint4*>(out), total, words)
                            : LaunchChained(GatherRows2Kernel, blocks, 256, 0, st, static_cast<const uint16_t*>(in), rows, static_cast<uint16_t*>(out), total, words);
  if (e != cudaSuccess) return CudaFail("GATHER_ROWS launch", e);
  CountLaunches(1);
  return kOk;
}
