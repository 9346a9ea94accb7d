// The row operations of a latent-attention layer: the pair of RMS norms in front of parallel mixer and feed-forward
// branches, the norms / rotation / cache write between the down- and up-projections, and interleaved RoPE.  Everything
// is evaluated in f32; only results are narrowed.
#include "common.cuh"

namespace tlaloc_b200 {
namespace {

// Sum over the CTA (blockDim.x a multiple of 32, at most 256); every thread gets it.
__device__ __forceinline__ float CtaSum(float v, float* red)
{
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) r += red[w];
  return r;
}

__device__ __forceinline__ float InvRms(float sum_sq, int n, float eps)
{
  return 1.f / sqrtf(sum_sq / static_cast<float>(n) + eps);
}

__device__ __forceinline__ void Store4(float* o, float a, float b, float c, float d) { *reinterpret_cast<float4*>(o) = make_float4(a, b, c, d); }
__device__ __forceinline__ void Store4(__nv_bfloat16* o, float a, float b, float c, float d)
{
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&lo);
  u.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(o) = u;
}

// One CTA per row.  VEC: rows of up to 8192 values, a multiple of 4, 16-byte aligned: read once, kept in registers.
template <typename OT, bool VEC>
__global__ void __launch_bounds__(256) RmsNormPairKernel(const float* x, const float* gain_a, OT* out_a, const float* gain_b,
                                                         OT* out_b, int n, float eps)
{
  GridDependencySync();
  __shared__ float red[8];
  const size_t row = static_cast<size_t>(blockIdx.x) * n;
  const float* xr = x + row;
  if constexpr (VEC) {
    const int n4 = n >> 2;
    float4 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int j = threadIdx.x + i * 256;
      v[i] = j < n4 ? reinterpret_cast<const float4*>(xr)[j] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
    const float inv = InvRms(CtaSum(ss, red), n, eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int j = threadIdx.x + i * 256;
      if (j >= n4) break;
      const float a = v[i].x * inv, b = v[i].y * inv, c = v[i].z * inv, d = v[i].w * inv;
      const float4 g = reinterpret_cast<const float4*>(gain_a)[j];
      Store4(out_a + row + 4 * j, a * g.x, b * g.y, c * g.z, d * g.w);
      if (out_b != nullptr) {
        const float4 h = reinterpret_cast<const float4*>(gain_b)[j];
        Store4(out_b + row + 4 * j, a * h.x, b * h.y, c * h.z, d * h.w);
      }
    }
  } else {
    float ss = 0.f;
    for (int j = threadIdx.x; j < n; j += 256) ss = fmaf(xr[j], xr[j], ss);
    const float inv = InvRms(CtaSum(ss, red), n, eps);
    for (int j = threadIdx.x; j < n; j += 256) {
      const float v = xr[j] * inv;
      out_a[row + j] = FromF32<OT>(v * gain_a[j]);
      if (out_b != nullptr) out_b[row + j] = FromF32<OT>(v * gain_b[j]);
    }
  }
}

// The pair (u, v) at an angle whose cosine and sine (with the design's magnitude already in them) are c and s.
__device__ __forceinline__ float2 Rotate(float u, float v, float c, float s)
{
  return make_float2(u * c - v * s, v * c + u * s);
}

// One CTA per token: two norms, one rotation, one cache row.
template <typename T>
__global__ void __launch_bounds__(256) LatentKvWriteKernel(const float* in, int64_t ld, const float* q_gain, const float* kv_gain, float eps,
                                                           const int* positions, const float* cos_t, const float* sin_t, const int* slots,
                                                           T* cq, T* pool, int64_t pool_ld, int q_rank, int kv_rank, int rot_dim,
                                                           int rot_dims, int num_slots, int max_pos)
{
  GridDependencySync();
  __shared__ float red[8], red2[8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const float* row = in + static_cast<size_t>(t) * ld;
  const float* kv = row + q_rank;
  float sq = 0.f, sk = 0.f;
  for (int j = tid; j < q_rank; j += 256) sq = fmaf(row[j], row[j], sq);
  for (int j = tid; j < kv_rank; j += 256) sk = fmaf(kv[j], kv[j], sk);
  sq = CtaSum(sq, red);
  sk = CtaSum(sk, red2);
  if (q_rank > 0) {
    const float inv = InvRms(sq, q_rank, eps);
    for (int j = tid; j < q_rank; j += 256) cq[static_cast<size_t>(t) * q_rank + j] = FromF32<T>(row[j] * inv * q_gain[j]);
  }
  const int slot = __ldg(slots + t);
  if (slot < 0 || slot >= num_slots) return;
  T* out = pool + static_cast<size_t>(slot) * pool_ld;
  const float inv = InvRms(sk, kv_rank, eps);
  for (int j = tid; j < kv_rank; j += 256) out[j] = FromF32<T>(kv[j] * inv * kv_gain[j]);
  const float* rot = kv + kv_rank;
  const int pos = min(max(__ldg(positions + t), 0), max_pos - 1), pairs = rot_dims >> 1;
  for (int i = tid; i < pairs; i += 256) {
    const float2 r = Rotate(rot[2 * i], rot[2 * i + 1], cos_t[static_cast<size_t>(pos) * pairs + i], sin_t[static_cast<size_t>(pos) * pairs + i]);
    out[kv_rank + 2 * i] = FromF32<T>(r.x);
    out[kv_rank + 2 * i + 1] = FromF32<T>(r.y);
  }
  for (int j = rot_dims + tid; j < rot_dim; j += 256) out[kv_rank + j] = FromF32<T>(rot[j]);
}

// A thread per pair (or, past rot_dims, per two copied elements).
template <typename T>
__global__ void __launch_bounds__(256) RopeInterleavedKernel(const T* in, int64_t in_t, int64_t in_h, T* out, int64_t out_t, int64_t out_h,
                                                             const int* positions, const float* cos_t, const float* sin_t, long long total,
                                                             int heads, int width, int rot_dims, int max_pos)
{
  GridDependencySync();
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= total) return;
  const int half = (width + 1) >> 1, pairs = rot_dims >> 1;
  const int p = static_cast<int>(i % half);
  const long long th = i / half;
  const int h = static_cast<int>(th % heads);
  const long long t = th / heads;
  const T* src = in + t * in_t + h * in_h + 2 * p;
  T* dst = out + t * out_t + h * out_h + 2 * p;
  if (p < pairs) {
    const int pos = min(max(__ldg(positions + t), 0), max_pos - 1);
    const float2 r = Rotate(ToF32(src[0]), ToF32(src[1]), cos_t[static_cast<size_t>(pos) * pairs + p], sin_t[static_cast<size_t>(pos) * pairs + p]);
    dst[0] = FromF32<T>(r.x);
    dst[1] = FromF32<T>(r.y);
  } else {
    dst[0] = src[0];
    if (2 * p + 1 < width) dst[1] = src[1];
  }
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_rmsnorm_pair(const float* x, const float* gain_a, void* out_a, const float* gain_b, void* out_b,
                                        int32_t out_dtype, int32_t rows, int32_t n, float eps, void* stream)
{
  const char* op = "RMSNORM_PAIR";
  if (!x || !gain_a || !out_a || (out_b && !gain_b)) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(out_dtype)) return Fail(kInvalid, "%s: out must be f32 or bf16", op);
  if (rows < 0 || n < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = n % 4 == 0 && n <= 8192 && Aligned16(x) && Aligned16(gain_a) && Aligned16(gain_b) && Aligned16(out_a) && Aligned16(out_b);
  cudaError_t e;
#define TLALOC_LAUNCH(OT, VEC) \
  e = LaunchChained(RmsNormPairKernel<OT, VEC>, rows, 256, 0, st, x, gain_a, static_cast<OT*>(out_a), gain_b, static_cast<OT*>(out_b), n, eps)
  if (out_dtype == TLALOC_B200_F32) {
    if (vec) TLALOC_LAUNCH(float, true);
    else TLALOC_LAUNCH(float, false);
  } else {
    if (vec) TLALOC_LAUNCH(__nv_bfloat16, true);
    else TLALOC_LAUNCH(__nv_bfloat16, false);
  }
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("RMSNORM_PAIR launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_latent_kv_write(const float* in, int64_t ld, const float* q_gain, const float* kv_gain, float eps,
                                           const int32_t* positions, const float* cos_table, const float* sin_table,
                                           const int32_t* slot_mapping, void* cq, void* pool, int32_t dtype, int64_t pool_ld,
                                           int32_t num_tokens, int32_t q_rank, int32_t kv_rank, int32_t rot_dim, int32_t rot_dims,
                                           int32_t num_slots, int32_t max_pos, void* stream)
{
  const char* op = "LATENT_KV_WRITE";
  if (!in || !kv_gain || !positions || !cos_table || !sin_table || !slot_mapping || !pool || (q_rank > 0 && (!q_gain || !cq))) {
    return Fail(kInvalid, "%s: a required device pointer is null", op);
  }
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: the pool must be f32 or bf16", op);
  if (num_tokens < 0 || q_rank < 0 || kv_rank < 1 || rot_dim < 0 || num_slots < 1 || max_pos < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > rot_dim) {
    return Fail(kInvalid, "%s: %d rotated dimensions; an even number up to %d", op, rot_dims, rot_dim);
  }
  if (ld < static_cast<int64_t>(q_rank) + kv_rank + rot_dim || pool_ld < static_cast<int64_t>(kv_rank) + rot_dim) {
    return Fail(kInvalid, "%s: a row stride is shorter than its row", op);
  }
  if (num_tokens == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
#define TLALOC_LAUNCH(T)                                                                                                              \
  e = LaunchChained(LatentKvWriteKernel<T>, num_tokens, 256, 0, st, in, ld, q_gain, kv_gain, eps, positions, cos_table, sin_table,     \
                    slot_mapping, static_cast<T*>(cq), static_cast<T*>(pool), pool_ld, q_rank, kv_rank, rot_dim, rot_dims, num_slots, max_pos)
  if (dtype == TLALOC_B200_F32) TLALOC_LAUNCH(float);
  else TLALOC_LAUNCH(__nv_bfloat16);
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("LATENT_KV_WRITE launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_rope_interleaved(const void* in, int64_t in_ld_token, int64_t in_ld_head, void* out, int64_t out_ld_token,
                                            int64_t out_ld_head, int32_t dtype, const int32_t* positions, const float* cos_table,
                                            const float* sin_table, int32_t num_tokens, int32_t num_heads, int32_t width,
                                            int32_t rot_dims, int32_t max_pos, void* stream)
{
  const char* op = "ROPE_INTERLEAVED";
  if (!in || !out || !positions || !cos_table || !sin_table) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (num_tokens < 0 || num_heads < 1 || width < 1 || max_pos < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > width) return Fail(kInvalid, "%s: %d rotated dimensions; an even number up to %d", op, rot_dims, width);
  if (num_tokens == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long total = static_cast<long long>(num_tokens) * num_heads * ((width + 1) / 2);
  const unsigned blocks = static_cast<unsigned>((total + 255) / 256);
  cudaError_t e;
#define TLALOC_LAUNCH(T)                                                                                                           \
  e = LaunchChained(RopeInterleavedKernel<T>, blocks, 256, 0, st, static_cast<const T*>(in), in_ld_token, in_ld_head,              \
                    static_cast<T*>(out), out_ld_token, out_ld_head, positions, cos_table, sin_table, total, num_heads, width, rot_dims, max_pos)
  if (dtype == TLALOC_B200_F32) TLALOC_LAUNCH(float);
  else TLALOC_LAUNCH(__nv_bfloat16);
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("ROPE_INTERLEAVED launch", e);
  CountLaunches(1);
  return kOk;
}
