// Token ids into rows and rows into token ids (ir/.../inference/HfDecoderGraph.kt: embedding :904-909; greedy next token): what every
// model of the framework begins and ends a step with.
#include "common.cuh"

namespace tlaloc_b200 {
namespace {

template <typename TT>
__global__ void EmbeddingKernel(const TT* table, const int* ids, float* out, int vocab, int dim)
{
  GridDependencySync();
  const int p = blockIdx.x;
  int v = __ldg(ids + p);
  v = v < 0 ? 0 : (v >= vocab ? vocab - 1 : v);
  const TT* src = table + static_cast<size_t>(v) * dim;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) out[static_cast<size_t>(p) * dim + d] = ToF32(src[d]);
}

// One CTA per row; the first index of the maximum wins (DxirInterpreter.kt:2414-2426).
__global__ void __launch_bounds__(256) ArgmaxKernel(const float* x, int* out, int n)
{
  GridDependencySync();
  __shared__ float bv[8];
  __shared__ int bi[8];
  const float* xr = x + static_cast<size_t>(blockIdx.x) * n;
  float best = -INFINITY;
  int idx = 0x7fffffff;
  for (int j = threadIdx.x; j < n; j += blockDim.x) {
    const float v = xr[j];
    if (v > best || (v == best && j < idx)) {
      best = v;
      idx = j;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
    if (ov > best || (ov == best && oi < idx)) {
      best = ov;
      idx = oi;
    }
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) {
    bv[warp] = best;
    bi[warp] = idx;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < static_cast<int>(blockDim.x >> 5); ++w) {
      if (bv[w] > best || (bv[w] == best && bi[w] < idx)) {
        best = bv[w];
        idx = bi[w];
      }
    }
    // A row of NaNs (or an empty comparison) leaves idx unset: the interpreter's answer is index 0.
    out[blockIdx.x] = idx == 0x7fffffff ? 0 : idx;
  }
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_embedding(const void* table, int32_t table_dtype, const int32_t* ids, float* out,
                                     int32_t positions, int32_t vocab, int32_t dim, void* stream)
{
  if (!table || !ids || !out) return Fail(kInvalid, "EMBEDDING: a required device pointer is null");
  if (!IsFloatType(table_dtype)) return Fail(kInvalid, "EMBEDDING: the table must be f32 or bf16");
  if (positions < 0 || vocab < 1 || dim < 1) return Fail(kInvalid, "EMBEDDING: bad sizes");
  if (positions == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (table_dtype == TLALOC_B200_F32) {
    e = LaunchChained(EmbeddingKernel<float>, positions, 256, 0, st, static_cast<const float*>(table), ids, out, vocab, dim);
  } else {
    e = LaunchChained(EmbeddingKernel<__nv_bfloat16>, positions, 256, 0, st, static_cast<const __nv_bfloat16*>(table), ids, out, vocab, dim);
  }
  if (e != cudaSuccess) return CudaFail("EMBEDDING launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_argmax(const float* logits, int32_t* out, int32_t rows, int32_t n, void* stream)
{
  if (!logits || !out) return Fail(kInvalid, "ARGMAX: a required device pointer is null");
  if (rows < 0 || n < 1) return Fail(kInvalid, "ARGMAX: bad sizes");
  if (rows == 0) return kOk;
  const cudaError_t e = LaunchChained(ArgmaxKernel, rows, 256, 0, static_cast<cudaStream_t>(stream), logits, out, n);
  if (e != cudaSuccess) return CudaFail("ARGMAX launch", e);
  CountLaunches(1);
  return kOk;
}
