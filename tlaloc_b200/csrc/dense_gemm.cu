// Projections over weights kept in f32 or bf16, [out, in] as a checkpoint stores them (include/tlaloc_b200.h,
// tlaloc_b200_dense_gemm): the entry point, and the kernel that takes any size and type.
//
// DenseGemmTiled: 64 x 64 output tiles, 256 threads with 4 x 4 outputs each, k in steps of 16 through shared memory as
// f32, plain FMA in k order.  It is the whole of the f32 path (true f32 products and sums) and the fallback of the bf16
// path for sizes and strides the tensor-core kernels do not take.
#include "common.cuh"
#include "dense_gemm.cuh"

namespace tlaloc_b200 {
namespace {

constexpr int kTile = 64, kStepK = 16;

template <typename T, typename YT>
__global__ void __launch_bounds__(256) DenseGemmTiled(tlaloc_b200_dense_problem p, int M)
{
  GridDependencySync();
  int first = 0;
  if (p.row_offsets != nullptr) {  // this weight's rows of the matrix
    first = __ldg(p.row_offsets + blockIdx.z);
    M = min(__ldg(p.row_offsets + blockIdx.z + 1), M);
    if (first + static_cast<int>(blockIdx.y) * kTile >= M) return;
  }
  __shared__ float xs[kStepK][kTile + 4], ws[kStepK][kTile + 4];
  const int tid = threadIdx.x, n0 = blockIdx.x * kTile, m0 = first + blockIdx.y * kTile;
  const T* x = static_cast<const T*>(p.x) + (p.row_offsets != nullptr ? 0 : p.batch_x * blockIdx.z);
  const T* w = static_cast<const T*>(p.w) + p.batch_w * blockIdx.z;
  YT* y = static_cast<YT*>(p.y) + (p.row_offsets != nullptr ? 0 : p.batch_y * blockIdx.z);
  const int tn = (tid & 15) * 4, tm = (tid >> 4) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kStepK) {
    for (int i = tid; i < kTile * kStepK; i += 256) {
      const int r = i / kStepK, c = i % kStepK, k = k0 + c;
      xs[c][r] = (m0 + r < M && k < p.k) ? ToF32(x[static_cast<size_t>(m0 + r) * p.ld_x + k]) : 0.f;
      ws[c][r] = (n0 + r < p.n && k < p.k) ? ToF32(w[static_cast<size_t>(n0 + r) * p.k + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kStepK; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[c][tm]), b = *reinterpret_cast<const float4*>(&ws[c][tn]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (IsGated(p.act)) {  // columns n and n + 16 of a block of 32 are four threads apart
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int m = m0 + tm + i;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float other = __shfl_xor_sync(0xffffffffu, acc[i][j], 4);
        const int n = n0 + tn + j;
        if (n < p.n && m < M && (n & kGateBlock) == 0) {
          y[static_cast<size_t>(m) * p.ld_y + (n >> 5) * kGateBlock + (n & 15)] = FromF32<YT>(GatedValue(p.act, acc[i][j], other));
        }
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + tm + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tn + j;
      if (n < p.n) y[static_cast<size_t>(m) * p.ld_y + n] = FromF32<YT>(DenseEpilogue(p, acc[i][j], m, n));
    }
  }
}

template <typename T>
cudaError_t LaunchTiled(const tlaloc_b200_dense_problem& p, int m, cudaStream_t st)
{
  if (p.rows > 0) m = p.rows;
  const dim3 grid((p.n + kTile - 1) / kTile, (m + kTile - 1) / kTile, p.batch);
  return p.y_dtype == TLALOC_B200_F32 ? LaunchChained(DenseGemmTiled<T, float>, grid, 256, 0, st, p, m)
                                      : LaunchChained(DenseGemmTiled<T, __nv_bfloat16>, grid, 256, 0, st, p, m);
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_dense_gemm(const tlaloc_b200_dense_problem* problems, int32_t count, int32_t dtype, int32_t m,
                                      int32_t flags, void* stream)
{
  const char* op = "DENSE_PROJ";
  if (!problems || count < 1 || count > 2) return Fail(kInvalid, "%s: one or two problems", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: x and w must be f32 or bf16", op);
  if (m < 0) return Fail(kInvalid, "%s: bad row count", op);
  for (int i = 0; i < count; ++i) {
    const tlaloc_b200_dense_problem& p = problems[i];
    if (!p.x || !p.w || !p.y) return Fail(kInvalid, "%s: a required device pointer is null", op);
    if (p.k < 1 || p.n < 1 || p.batch < 1 || p.batch > 65535) return Fail(kInvalid, "%s: bad sizes", op);
    if (!IsFloatType(p.y_dtype)) return Fail(kInvalid, "%s: y must be f32 or bf16", op);
    if (p.act != TLALOC_B200_ACT_NONE && p.act != TLALOC_B200_ACT_RELU2 && !IsGated(p.act)) return Fail(kInvalid, "%s: unknown activation %d", op, p.act);
    if (IsGated(p.act) && (p.n % (2 * kGateBlock) != 0 || p.bias || p.residual)) {
      return Fail(kInvalid, "%s: a gated projection has a multiple of %d rows, no bias and no residual", op, 2 * kGateBlock);
    }
    if (p.row_offsets && i + 1 < count) return Fail(kInvalid, "%s: a grouped projection is the last of a call", op);
    if (p.rows < 0 || (p.row_offsets && (p.residual || p.bias || p.batch > kMaxGroups))) return Fail(kInvalid, "%s: bad groups", op);
    if (((p.rows > 0 ? p.rows : m) + kTile - 1) / kTile > 65535) return Fail(kInvalid, "%s: too many rows", op);
    if (p.ld_x < p.k || p.ld_y < (IsGated(p.act) ? p.n / 2 : p.n) || (p.residual && p.ld_res < p.n)) return Fail(kInvalid, "%s: a row stride is shorter than its row", op);
    if (p.batch > 1 && (p.residual || p.bias)) return Fail(kInvalid, "%s: a batched projection takes no bias and no residual", op);
  }
  if (m == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int launches = 0;
  cudaError_t e = cudaSuccess;
  bool tc = dtype == TLALOC_B200_BF16 && !OrderFaithful();
  for (int i = 0; i < count; ++i) tc = tc && DenseGemmTcApplies(problems[i]);
  if (tc) {
    e = LaunchDenseGemmTc(problems, count, m, (flags & TLALOC_B200_GEMM_WEIGHTS_CONST) != 0, st);
    launches = 1;
  }
  for (int i = 0; i < count && e == cudaSuccess && !tc; ++i) {
    e = dtype == TLALOC_B200_F32 ? LaunchTiled<float>(problems[i], m, st) : LaunchTiled<__nv_bfloat16>(problems[i], m, st);
    ++launches;
  }
  if (e != cudaSuccess) return CudaFail("DENSE_PROJ launch", e);
  CountLaunches(launches);
  return kOk;
}
