// Retention: linear attention with a fixed decay per head (include/tlaloc_b200.h).  The state is f32 throughout.
//   RetentionStepKernel   one token per row, fused: rotation, state update, output, its norm and gate.  A CTA has one head of one
//                         row and streams its state through registers once: the kernel is bound by those bytes.
//   RetentionScanKernel   a portion token by token with the state in registers, 32 value columns a CTA: any size and type.
#include "common.cuh"

namespace tlaloc_b200 {
namespace {

constexpr int kThreads = 256, kAhead = 8;

__device__ __forceinline__ float WarpSum(float v)
{
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Thread (r, c): state rows r, r + R, ... and the four columns from 4 c.
template <typename T>
__global__ void __launch_bounds__(kThreads) RetentionStepKernel(const float* in, int64_t ld, const int* positions, const float* cos_t, const float* sin_t,
                                                                const float* decay, const int* row_states, float* state, T* out, int64_t out_ld, int heads,
                                                                int dim, int vdim, int rot_dims, int num_slots, int max_pos, float k_scale, float eps)
{
  GridDependencySync();
  extern __shared__ float smem[];
  __shared__ float red[8];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  const int vp = (vdim + 3) & ~3, cols = vp >> 2, R = min(kThreads / cols, dim), c = tid % cols, r = tid / cols;
  const int dp = (dim + 3) & ~3;
  float *qs = smem, *ks = smem + dp, *part = smem + 2 * dp;  // part [R][vp], 16-byte aligned
  const float* row = in + t * ld;
  const float *q = row + h * dim, *k = row + (heads + h) * dim, *v = row + 2 * heads * dim + h * vdim, *g = v + heads * vdim;
  const int pos = min(max(__ldg(positions + t), 0), max_pos - 1), half = rot_dims >> 1;
  const bool fresh = pos == 0;
  for (int i = tid; i < dim; i += kThreads) {
    float a = q[i], b = k[i];
    if (i < rot_dims) {
      const bool upper = i >= half;
      const int f = upper ? i - half : i, o = upper ? f : i + half;
      const float cs = cos_t[static_cast<size_t>(pos) * half + f], sn = sin_t[static_cast<size_t>(pos) * half + f];
      a = upper ? a * cs + q[o] * sn : a * cs - q[o] * sn;
      b = upper ? b * cs + k[o] * sn : b * cs - k[o] * sn;
    }
    qs[i] = a;
    ks[i] = b * k_scale;
  }
  float4 vv = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool live = r < R;
  if (live) {
    vv.x = v[4 * c];
    if (4 * c + 1 < vdim) vv.y = v[4 * c + 1];
    if (4 * c + 2 < vdim) vv.z = v[4 * c + 2];
    if (4 * c + 3 < vdim) vv.w = v[4 * c + 3];
  }
  const int slot = min(max(__ldg(row_states + t), 0), num_slots - 1);
  const float d = __ldg(decay + h);
  float* s = state + (static_cast<size_t>(slot) * heads + h) * dim * vp + 4 * c;
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (live) {
    for (int i0 = r; i0 < dim; i0 += R * kAhead) {
      float4 x[kAhead];
#pragma unroll
      for (int e = 0; e < kAhead; ++e) {
        const int i = i0 + e * R;
        x[e] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < dim && !fresh) x[e] = *reinterpret_cast<const float4*>(s + static_cast<size_t>(i) * vp);
      }
#pragma unroll
      for (int e = 0; e < kAhead; ++e) {
        const int i = i0 + e * R;
        if (i >= dim) break;
        const float kk = ks[i], qq = qs[i];
        x[e] = make_float4(fmaf(d, x[e].x, kk * vv.x), fmaf(d, x[e].y, kk * vv.y), fmaf(d, x[e].z, kk * vv.z), fmaf(d, x[e].w, kk * vv.w));
        *reinterpret_cast<float4*>(s + static_cast<size_t>(i) * vp) = x[e];
        o = make_float4(fmaf(qq, x[e].x, o.x), fmaf(qq, x[e].y, o.y), fmaf(qq, x[e].z, o.z), fmaf(qq, x[e].w, o.w));
      }
    }
    *reinterpret_cast<float4*>(part + r * vp + 4 * c) = o;
  }
  __syncthreads();
  float sum[4], ss = 0.f;  // vdim <= 1024: up to four columns a thread
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int j = tid + e * kThreads;
    sum[e] = 0.f;
    if (j < vdim) {
      for (int i = 0; i < R; ++i) sum[e] += part[i * vp + j];
    }
    ss = fmaf(sum[e], sum[e], ss);
  }
  ss = WarpSum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(vdim) + eps);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int j = tid + e * kThreads;
    if (j < vdim) out[t * out_ld + h * vdim + j] = FromF32<T>(sum[e] * inv * (g[j] / (1.f + expf(-g[j]))));
  }
}

constexpr int kBatch = 8;  // tokens staged at a time

// Warp w holds state rows w, w + 8, ..., a lane one column.
template <typename T, int ROWS>
__global__ void __launch_bounds__(256) RetentionScanKernel(const T* q, const T* k, int dim_ld, const T* v, int v_ld, const int* positions, const float* decay,
                                                           const int* row_states, float* state, float* o, int tokens, int heads, int dim, int vdim,
                                                           int num_slots)
{
  GridDependencySync();
  extern __shared__ float smem[];
  float *qs = smem, *ks = qs + kBatch * dim, *vs = ks + kBatch * dim, *part = vs + kBatch * 32;  // part [8 warps][kBatch][32]
  const int h = blockIdx.x, c0 = blockIdx.y * 32, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, col = c0 + lane;
  const int vp = (vdim + 3) & ~3;
  const int slot = min(max(__ldg(row_states), 0), num_slots - 1);
  const bool fresh = __ldg(positions) == 0;
  const float d = __ldg(decay + h);
  float* st = state + (static_cast<size_t>(slot) * heads + h) * dim * vp + col;
  float s[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = warp + 8 * i;
    s[i] = !fresh && r < dim && col < vp ? st[static_cast<size_t>(r) * vp] : 0.f;
  }
  for (int t0 = 0; t0 < tokens; t0 += kBatch) {
    const int n = min(kBatch, tokens - t0);
    __syncthreads();
    for (int i = tid; i < n * dim; i += 256) {
      const size_t at = (static_cast<size_t>(t0 + i / dim) * heads + h) * dim_ld + i % dim;
      qs[i] = ToF32(q[at]);
      ks[i] = ToF32(k[at]);
    }
    if (warp < n) vs[tid] = col < vdim ? ToF32(v[(static_cast<size_t>(t0 + warp) * heads + h) * v_ld + col]) : 0.f;
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float vv = vs[t * 32 + lane];
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int r = warp + 8 * i;
        if (r < dim) {
          s[i] = fmaf(d, s[i], ks[t * dim + r] * vv);
          acc = fmaf(qs[t * dim + r], s[i], acc);
        }
      }
      part[(warp * kBatch + t) * 32 + lane] = acc;
    }
    __syncthreads();
    if (warp < n && col < vdim) {
      float acc = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) acc += part[(w * kBatch + warp) * 32 + lane];
      o[(static_cast<size_t>(t0 + warp) * heads + h) * vdim + col] = acc;
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = warp + 8 * i;
    if (r < dim && col < vp) st[static_cast<size_t>(r) * vp] = s[i];
  }
}

template <typename T>
cudaError_t LaunchScan(const void* q, const void* k, int dim_ld, const void* v, int v_ld, const int* positions, const float* decay, const int* row_states,
                       float* state, float* o, int tokens, int heads, int dim, int vdim, int num_slots, cudaStream_t st)
{
  const dim3 grid(heads, (vdim + 31) / 32);
  const size_t smem = sizeof(float) * (2 * kBatch * dim + kBatch * 32 + 8 * kBatch * 32);
#define TLALOC_SCAN(ROWS)                                                                                                                          \
  LaunchChained(RetentionScanKernel<T, ROWS>, grid, 256, smem, st, static_cast<const T*>(q), static_cast<const T*>(k), dim_ld, static_cast<const T*>(v), \
                v_ld, positions, decay, row_states, state, o, tokens, heads, dim, vdim, num_slots)
  if (dim <= 64) return TLALOC_SCAN(8);
  if (dim <= 128) return TLALOC_SCAN(16);
  if (dim <= 256) return TLALOC_SCAN(32);
  return TLALOC_SCAN(64);
#undef TLALOC_SCAN
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_retention_step(const float* in, int64_t ld, const int32_t* positions, const float* cos_table, const float* sin_table,
                                          const float* decay, const int32_t* row_states, float* state, void* out, int64_t out_ld, int32_t dtype,
                                          int32_t rows, int32_t heads, int32_t dim, int32_t vdim, int32_t rot_dims, int32_t num_slots, int32_t max_pos,
                                          float k_scale, float eps, void* stream)
{
  const char* op = "RETENTION_STEP";
  if (!in || !positions || !decay || !row_states || !state || !out || (rot_dims > 0 && (!cos_table || !sin_table))) {
    return Fail(kInvalid, "%s: a required device pointer is null", op);
  }
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: out must be f32 or bf16", op);
  if (rows < 0 || rows > 65535 || heads < 1 || dim < 1 || vdim < 1 || num_slots < 1 || max_pos < 1 || rot_dims < 0 || rot_dims % 2 || rot_dims > dim ||
      ld < 2ll * heads * (dim + vdim) || out_ld < static_cast<int64_t>(heads) * vdim || !Aligned16(state)) {
    return Fail(kInvalid, "%s: bad sizes", op);
  }
  if (dim > 512 || vdim > 1024) return Fail(kUnsupported, "%s: dim up to 512, vdim up to 1024", op);
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vp = (vdim + 3) / 4 * 4, lanes = kThreads / (vp / 4);
  const size_t smem = sizeof(float) * (2 * ((dim + 3) / 4 * 4) + static_cast<size_t>(lanes < dim ? lanes : dim) * vp);
  const dim3 grid(heads, rows);
  cudaError_t e;
#define TLALOC_LAUNCH(T)                                                                                                                         \
  e = LaunchChained(RetentionStepKernel<T>, grid, kThreads, smem, st, in, ld, positions, cos_table, sin_table, decay, row_states, state,          \
                    static_cast<T*>(out), out_ld, heads, dim, vdim, rot_dims, num_slots, max_pos, k_scale, eps)
  if (dtype == TLALOC_B200_F32) TLALOC_LAUNCH(float);
  else TLALOC_LAUNCH(__nv_bfloat16);
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("RETENTION_STEP launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_retention_scan(const void* q, const void* k, int32_t dim_ld, const void* v, int32_t v_ld, int32_t dtype,
                                          const int32_t* positions, const float* decay, const int32_t* row_states, float* state, float* o, int32_t tokens,
                                          int32_t heads, int32_t dim, int32_t vdim, int32_t num_slots, void* stream)
{
  const char* op = "RETENTION_SCAN";
  if (!q || !k || !v || !positions || !decay || !row_states || !state || !o) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (tokens < 0 || heads < 1 || dim < 1 || vdim < 1 || num_slots < 1 || dim_ld < dim || v_ld < vdim) return Fail(kInvalid, "%s: bad sizes", op);
  if (dim > 512 || vdim > 1024) return Fail(kUnsupported, "%s: dim up to 512, vdim up to 1024", op);
  if (tokens == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const cudaError_t e =
      dtype == TLALOC_B200_F32
          ? LaunchScan<float>(q, k, dim_ld, v, v_ld, positions, decay, row_states, state, o, tokens, heads, dim, vdim, num_slots, st)
          : LaunchScan<__nv_bfloat16>(q, k, dim_ld, v, v_ld, positions, decay, row_states, state, o, tokens, heads, dim, vdim, num_slots, st);
  if (e != cudaSuccess) return CudaFail("RETENTION_SCAN launch", e);
  CountLaunches(1);
  return kOk;
}
