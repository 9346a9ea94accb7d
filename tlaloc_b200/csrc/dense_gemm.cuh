// Shared by the kernels behind tlaloc_b200_dense_gemm.
#pragma once

#include "common.cuh"

namespace tlaloc_b200 {

// What happens to a finished sum before it is stored.
__device__ __forceinline__ float DenseActivation(int act, float v)
{
  if (act == TLALOC_B200_ACT_RELU2) {
    const float r = fmaxf(v, 0.f);
    return r * r;
  }
  return v;
}
__device__ __forceinline__ float DenseEpilogue(const tlaloc_b200_dense_problem& p, float v, int m, int n)
{
  if (p.bias != nullptr) v += __ldg(p.bias + n);
  v = DenseActivation(p.act, v);
  if (p.residual != nullptr) v += p.residual[static_cast<size_t>(m) * p.ld_res + n];
  return v;
}

// The tensor-core kernel (dense_gemm_tc.cu): bf16 x and w whose addresses, row and batch strides are multiples of 16 bytes.
bool DenseGemmTcApplies(const tlaloc_b200_dense_problem& p);
cudaError_t LaunchDenseGemmTc(const tlaloc_b200_dense_problem* problems, int count, int m, bool weights_const, cudaStream_t st);

}  // namespace tlaloc_b200
