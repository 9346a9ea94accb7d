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
// Gated activations: rows of w in blocks of 32, 16 of the gate and the 16 that it multiplies.
constexpr int kGateBlock = 16, kMaxGroups = 1024;
__host__ __device__ __forceinline__ bool IsGated(int act) { return act == TLALOC_B200_ACT_SILU_MUL || act == TLALOC_B200_ACT_GELU_TANH_MUL; }
__device__ __forceinline__ float GatedValue(int act, float gate, float other)
{
  if (act == TLALOC_B200_ACT_SILU_MUL) return gate / (1.f + expf(-gate)) * other;
  const float t = tanhf(0.7978845608028654f * (gate + 0.044715f * gate * gate * gate));
  return 0.5f * gate * (1.f + t) * other;
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
