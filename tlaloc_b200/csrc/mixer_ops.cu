// The row operations of decoders with a norm on both sides of every branch and mixers of several kinds: the branch's output norm, the
// residual sum and the next branch's input norm in one pass (also over the weighted outputs of a token's experts); rotate-half
// positions on the way from a projection into cache and query rows; the difference of two attention maps; the norm and gate of
// a recurrence's heads.  Everything is evaluated in f32; only results are narrowed.
#include "common.cuh"
#include "dense_gemm.cuh"

namespace tlaloc_b200 {
namespace {

__device__ __forceinline__ float WarpSum(float v)
{
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over 256 threads; every thread gets it.
__device__ __forceinline__ float CtaSum(float v, float* red)
{
  v = WarpSum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) r += red[w];
  return r;
}
__device__ __forceinline__ float InvRms(float sum_sq, int n, float eps) { return 1.f / sqrtf(sum_sq / static_cast<float>(n) + eps); }
__device__ __forceinline__ float Sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float Silu(float z) { return z / (1.f + expf(-z)); }

__device__ __forceinline__ float4 Load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 Load4(const __nv_bfloat16* p)
{
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void Store4(float* o, float4 v) { *reinterpret_cast<float4*>(o) = v; }
__device__ __forceinline__ void Store4(__nv_bfloat16* o, float4 v)
{
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&lo);
  u.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(o) = u;
}
__device__ __forceinline__ void StorePair(float* o, float a, float b) { *reinterpret_cast<float2*>(o) = make_float2(a, b); }
__device__ __forceinline__ void StorePair(__nv_bfloat16* o, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(o) = __floats2bfloat162_rn(a, b); }
__device__ __forceinline__ float4 Fma4(float a, float4 v, float4 c)
{
  return make_float4(fmaf(a, v.x, c.x), fmaf(a, v.y, c.y), fmaf(a, v.z, c.z), fmaf(a, v.w, c.w));
}
__device__ __forceinline__ float Dot4(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }

struct Branch {
  const float* y;              // [rows, n], the branch itself or its shared expert; may be null with experts
  const float* gate;           // logit of the shared expert's gate, gate_ld apart; null: none
  int64_t gate_ld;
  const void* parts;           // experts: rows of n values in the results' type; null: none
  const int* part_rows;        // [rows, top]
  const float* part_weights;   // [rows, top]
  int top;
};

// One CTA per row.  VEC: up to 8192 values, a multiple of 4, 16-byte aligned, kept in registers; else the row is read several times.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ResidualNormKernel(Branch b, float* x, const float* gain_post, const float* gain_next, T* out, int n, float eps)
{
  GridDependencySync();
  __shared__ float red[8];
  const int row = blockIdx.x;
  const T* parts = static_cast<const T*>(b.parts);
  const float shared = b.gate != nullptr ? Sigmoid(b.gate[row * b.gate_ld]) : 1.f;
  const size_t at = static_cast<size_t>(row) * n;
  if constexpr (VEC) {
    const int n4 = n >> 2;
    float4 v[8];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int j = threadIdx.x + i * 256;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < n4) {
        if (b.y != nullptr) {
          v[i] = Load4(b.y + at + 4 * j);
          if (b.gate != nullptr) v[i] = Fma4(shared, v[i], make_float4(0.f, 0.f, 0.f, 0.f));
        }
        for (int k = 0; k < b.top; ++k) {
          v[i] = Fma4(b.part_weights[row * b.top + k], Load4(parts + static_cast<size_t>(b.part_rows[row * b.top + k]) * n + 4 * j), v[i]);
        }
        ss += Dot4(v[i]);
      }
    }
    const float inv = InvRms(CtaSum(ss, red), n, eps);
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int j = threadIdx.x + i * 256;
      if (j < n4) {
        const float4 g = Load4(gain_post + 4 * j), r = Load4(x + at + 4 * j);
        v[i] = make_float4(r.x + v[i].x * inv * g.x, r.y + v[i].y * inv * g.y, r.z + v[i].z * inv * g.z, r.w + v[i].w * inv * g.w);
        Store4(x + at + 4 * j, v[i]);
        ss += Dot4(v[i]);
      }
    }
    if (out == nullptr) return;
    const float inv2 = InvRms(CtaSum(ss, red), n, eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int j = threadIdx.x + i * 256;
      if (j < n4) {
        const float4 g = Load4(gain_next + 4 * j);
        Store4(out + at + 4 * j, make_float4(v[i].x * inv2 * g.x, v[i].y * inv2 * g.y, v[i].z * inv2 * g.z, v[i].w * inv2 * g.w));
      }
    }
  } else {
    auto value = [&](int j) {
      float v = b.y != nullptr ? b.y[at + j] * shared : 0.f;
      for (int k = 0; k < b.top; ++k) {
        v = fmaf(b.part_weights[row * b.top + k], ToF32(parts[static_cast<size_t>(b.part_rows[row * b.top + k]) * n + j]), v);
      }
      return v;
    };
    float ss = 0.f;
    for (int j = threadIdx.x; j < n; j += 256) {
      const float v = value(j);
      ss = fmaf(v, v, ss);
    }
    const float inv = InvRms(CtaSum(ss, red), n, eps);
    ss = 0.f;
    for (int j = threadIdx.x; j < n; j += 256) {
      const float v = x[at + j] + value(j) * inv * gain_post[j];
      x[at + j] = v;  // read again by the same thread
      ss = fmaf(v, v, ss);
    }
    if (out == nullptr) return;
    const float inv2 = InvRms(CtaSum(ss, red), n, eps);
    for (int j = threadIdx.x; j < n; j += 256) out[at + j] = FromF32<T>(x[at + j] * inv2 * gain_next[j]);
  }
}

struct RotateArgs {
  tlaloc_b200_rotate_part part[3];
  int count;
};

// One CTA per token, W elements a thread at a time (W 4: sizes, offsets and the halves of the rotation are multiples of 4).
template <typename T, int W>
__global__ void __launch_bounds__(256) RotateRowsKernel(const float* in, int64_t ld, const __grid_constant__ RotateArgs a, const int* positions,
                                                        const float* cos_t, const float* sin_t, const int* slots, int rot_dims, int num_slots, int max_pos)
{
  GridDependencySync();
  const int t = blockIdx.x, half = rot_dims >> 1;
  const float* row = in + static_cast<size_t>(t) * ld;
  const int pos = min(max(__ldg(positions + t), 0), max_pos - 1);
  const float *c_row = cos_t + static_cast<size_t>(pos) * half, *s_row = sin_t + static_cast<size_t>(pos) * half;
  const int slot = slots != nullptr ? __ldg(slots + t) : 0;
  for (int p = 0; p < a.count; ++p) {
    const tlaloc_b200_rotate_part& s = a.part[p];
    if (s.by_slot && (slot < 0 || slot >= num_slots)) continue;
    T* dst = static_cast<T*>(s.out) + static_cast<size_t>(s.by_slot ? slot : t) * s.out_ld;
    const int per = s.padded / W, total = s.heads * per;
    for (int i = threadIdx.x; i < total; i += 256) {
      const int h = i / per, c = (i - h * per) * W;
      const float* src = row + s.first + h * s.dim;
      float v[W];
#pragma unroll
      for (int e = 0; e < W; ++e) v[e] = 0.f;
      if (c < s.dim) {
        if constexpr (W == 4) {
          const float4 u = Load4(src + c);
          v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
        } else {
          v[0] = src[c];
        }
        if (s.rotate && c < rot_dims) {
          const bool upper = c >= half;
          const int f = upper ? c - half : c;
          float o[W], cs[W], sn[W];
          if constexpr (W == 4) {
            const float4 u = Load4(src + (upper ? f : c + half)), cc = Load4(c_row + f), ss = Load4(s_row + f);
            o[0] = u.x; o[1] = u.y; o[2] = u.z; o[3] = u.w;
            cs[0] = cc.x; cs[1] = cc.y; cs[2] = cc.z; cs[3] = cc.w;
            sn[0] = ss.x; sn[1] = ss.y; sn[2] = ss.z; sn[3] = ss.w;
          } else {
            o[0] = src[upper ? f : c + half];
            cs[0] = c_row[f];
            sn[0] = s_row[f];
          }
#pragma unroll
          for (int e = 0; e < W; ++e) v[e] = upper ? v[e] * cs[e] + o[e] * sn[e] : v[e] * cs[e] - o[e] * sn[e];
        }
      }
      T* d = dst + h * s.out_head_ld + c;
      if constexpr (W == 4) {
        Store4(d, make_float4(v[0] * s.scale, v[1] * s.scale, v[2] * s.scale, v[3] * s.scale));
      } else {
        *d = FromF32<T>(v[0] * s.scale);
      }
    }
  }
}

// One warp per (token, head): the two maps' outputs out of the slices' records ({maximum (log2), sum, acc[in_ld]}; slices > 0) or as
// they are (slices 0); their difference, its norm, the head's gate.  PAIRS: even sizes up to 512 values, two a lane at a time, kept in
// registers; else the values are computed twice.
template <typename T, bool PAIRS>
__global__ void __launch_bounds__(128) MapDifferenceKernel(const float* in, int slices, const float* gate, int64_t gate_ld, T* out, int64_t out_ld, int rows,
                                                           int heads, int vdim, int in_ld, float lambda, float keep, float eps)
{
  GridDependencySync();
  const int w = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= rows * heads) return;
  const int t = w / heads, h = w - t * heads;
  const int rec = slices > 0 ? in_ld + 2 : in_ld;
  const float* a = in + (static_cast<size_t>(t) * heads + h) * 2 * rec;
  const size_t slice_ld = static_cast<size_t>(rows) * heads * 2 * rec;
  float top[2] = {0.f, 0.f}, scale[2] = {1.f, -lambda};  // of each map's values in the difference
  if (slices > 0) {
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      float m = -INFINITY;
      for (int s = 0; s < slices; ++s) m = fmaxf(m, a[s * slice_ld + p * rec]);
      float sum = 0.f;
      for (int s = 0; s < slices; ++s) {
        const float ms = a[s * slice_ld + p * rec];
        if (ms > -INFINITY) sum += a[s * slice_ld + p * rec + 1] * exp2f(ms - m);
      }
      top[p] = m;
      scale[p] = sum > 0.f ? scale[p] / sum : 0.f;
    }
  }
  const float g = keep * (gate != nullptr ? Sigmoid(gate[t * gate_ld + h]) : 1.f);
  T* dst = out + t * out_ld + static_cast<size_t>(h) * vdim;
  if constexpr (PAIRS) {
    const int pairs = vdim >> 1;
    float2 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = make_float2(0.f, 0.f);
    for (int s = 0; s < max(slices, 1); ++s) {
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const float* r = a + s * slice_ld + p * rec;
        float f = scale[p];
        if (slices > 0) {
          if (!(r[0] > -INFINITY)) continue;  // nothing of the row is in this slice
          f *= exp2f(r[0] - top[p]);
          r += 2;
        }
        float2 x[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (lane + 32 * i < pairs) x[i] = *reinterpret_cast<const float2*>(r + 2 * (lane + 32 * i));
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (lane + 32 * i < pairs) v[i] = make_float2(fmaf(f, x[i].x, v[i].x), fmaf(f, x[i].y, v[i].y));
        }
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
    const float f = InvRms(WarpSum(ss), vdim, eps) * g;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (lane + 32 * i < pairs) StorePair(dst + 2 * (lane + 32 * i), v[i].x * f, v[i].y * f);
    }
  } else {
    auto value = [&](int c) {
      float v = 0.f;
      for (int s = 0; s < max(slices, 1); ++s) {
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const float* r = a + s * slice_ld + p * rec;
          if (slices == 0) v = fmaf(scale[p], r[c], v);
          else if (r[0] > -INFINITY) v = fmaf(scale[p] * exp2f(r[0] - top[p]), r[2 + c], v);
        }
      }
      return v;
    };
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) {
      const float u = value(c);
      ss = fmaf(u, u, ss);
    }
    const float f = InvRms(WarpSum(ss), vdim, eps) * g;
    for (int c = lane; c < vdim; c += 32) dst[c] = FromF32<T>(value(c) * f);
  }
}

// One warp per (token, head): a recurrence's output over its root mean square, times silu of the gate.  PAIRS as above.
template <typename T, bool PAIRS>
__global__ void __launch_bounds__(128) HeadNormGateKernel(const float* in, const float* gate, int64_t gate_ld, T* out, int64_t out_ld, int rows, int heads,
                                                          int vdim, float eps)
{
  GridDependencySync();
  const int w = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= rows * heads) return;
  const int t = w / heads, h = w - t * heads;
  const float* a = in + (static_cast<size_t>(t) * heads + h) * vdim;
  const float* g = gate + t * gate_ld + static_cast<size_t>(h) * vdim;
  T* dst = out + t * out_ld + static_cast<size_t>(h) * vdim;
  float ss = 0.f;
  if constexpr (PAIRS) {
    const int pairs = vdim >> 1;
    float2 v[8], z[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      v[i] = z[i] = make_float2(0.f, 0.f);
      if (lane + 32 * i < pairs) {
        v[i] = *reinterpret_cast<const float2*>(a + 2 * (lane + 32 * i));
        z[i] = *reinterpret_cast<const float2*>(g + 2 * (lane + 32 * i));
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
    const float inv = InvRms(WarpSum(ss), vdim, eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (lane + 32 * i < pairs) StorePair(dst + 2 * (lane + 32 * i), v[i].x * inv * Silu(z[i].x), v[i].y * inv * Silu(z[i].y));
    }
  } else {
    for (int c = lane; c < vdim; c += 32) ss = fmaf(a[c], a[c], ss);
    const float inv = InvRms(WarpSum(ss), vdim, eps);
    for (int c = lane; c < vdim; c += 32) dst[c] = FromF32<T>(a[c] * inv * Silu(g[c]));
  }
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_residual_norm(const float* y, const float* gate, int64_t gate_ld, const void* parts, const int32_t* part_rows,
                                         const float* part_weights, int32_t top, float* x, const float* gain_post, const float* gain_next, void* out,
                                         int32_t dtype, int32_t rows, int32_t n, float eps, void* stream)
{
  const char* op = "RESIDUAL_NORM";
  if (!x || !gain_post || (!y && !parts) || (gate && !y) || (parts && (!part_rows || !part_weights)) || (out && !gain_next)) {
    return Fail(kInvalid, "%s: a required device pointer is null", op);
  }
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (rows < 0 || n < 1 || top < 0 || (parts != nullptr) != (top > 0)) return Fail(kInvalid, "%s: bad sizes", op);
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Branch b = {y, gate, gate_ld, parts, part_rows, part_weights, top};
  const bool vec = n % 4 == 0 && n <= 8192 && Aligned16(y) && Aligned16(parts) && Aligned16(x) && Aligned16(gain_post) && Aligned16(gain_next) && Aligned16(out);
  cudaError_t e;
#define TLALOC_LAUNCH(T, VEC) e = LaunchChained(ResidualNormKernel<T, VEC>, rows, 256, 0, st, b, x, gain_post, gain_next, static_cast<T*>(out), n, eps)
  if (dtype == TLALOC_B200_F32) {
    if (vec) TLALOC_LAUNCH(float, true);
    else TLALOC_LAUNCH(float, false);
  } else {
    if (vec) TLALOC_LAUNCH(__nv_bfloat16, true);
    else TLALOC_LAUNCH(__nv_bfloat16, false);
  }
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("RESIDUAL_NORM launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_rotate_rows(const float* in, int64_t ld, const tlaloc_b200_rotate_part* parts, int32_t count, int32_t dtype,
                                       const int32_t* positions, const float* cos_table, const float* sin_table, const int32_t* slot_mapping,
                                       int32_t num_tokens, int32_t rot_dims, int32_t num_slots, int32_t max_pos, void* stream)
{
  const char* op = "ROTATE_ROWS";
  if (!in || !parts || !positions || (rot_dims > 0 && (!cos_table || !sin_table))) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (count < 1 || count > 3 || num_tokens < 0 || max_pos < 1 || rot_dims < 0 || rot_dims % 2) return Fail(kInvalid, "%s: bad sizes", op);
  RotateArgs a = {};
  a.count = count;
  const int64_t es = static_cast<int64_t>(DtypeBytes(dtype));
  bool vec = ld % 4 == 0 && Aligned16(in) && rot_dims % 8 == 0 && Aligned16(cos_table) && Aligned16(sin_table);
  for (int i = 0; i < count; ++i) {
    const tlaloc_b200_rotate_part& p = parts[i];
    if (!p.out) return Fail(kInvalid, "%s: a required device pointer is null", op);
    if (p.heads < 1 || p.dim < 1 || p.padded < p.dim || p.first < 0 || p.first + static_cast<int64_t>(p.heads) * p.dim > ld ||
        p.out_head_ld < p.padded || (p.rotate && rot_dims > p.dim)) {
      return Fail(kInvalid, "%s: part %d does not fit its row", op, i);
    }
    if (p.by_slot && (!slot_mapping || num_slots < 1)) return Fail(kInvalid, "%s: a part goes by slots and there are none", op);
    vec = vec && p.first % 4 == 0 && p.dim % 4 == 0 && p.padded % 4 == 0 && p.out_ld % 4 == 0 && p.out_head_ld % 4 == 0 &&
          reinterpret_cast<uintptr_t>(p.out) % (4 * es) == 0;
    a.part[i] = p;
  }
  if (num_tokens == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
#define TLALOC_LAUNCH(T, W) \
  e = LaunchChained(RotateRowsKernel<T, W>, num_tokens, 256, 0, st, in, ld, a, positions, cos_table, sin_table, slot_mapping, rot_dims, num_slots, max_pos)
  if (dtype == TLALOC_B200_F32) {
    if (vec) TLALOC_LAUNCH(float, 4);
    else TLALOC_LAUNCH(float, 1);
  } else {
    if (vec) TLALOC_LAUNCH(__nv_bfloat16, 4);
    else TLALOC_LAUNCH(__nv_bfloat16, 1);
  }
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("ROTATE_ROWS launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_map_difference(const float* in, int32_t slices, const float* gate, int64_t gate_ld, void* out, int64_t out_ld, int32_t dtype,
                                          int32_t rows, int32_t heads, int32_t vdim, int32_t in_ld, float lambda, float keep, float eps, void* stream)
{
  const char* op = "MAP_DIFFERENCE";
  if (!in || !out) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (slices < 0 || rows < 0 || heads < 1 || vdim < 1 || in_ld < vdim || out_ld < static_cast<int64_t>(heads) * vdim) return Fail(kInvalid, "%s: bad sizes", op);
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(rows) * heads + 3) / 4);
  cudaError_t e;
  const bool pairs = vdim % 2 == 0 && in_ld % 2 == 0 && vdim <= 512 && out_ld % 2 == 0 && reinterpret_cast<uintptr_t>(in) % 8 == 0 &&
                     reinterpret_cast<uintptr_t>(out) % 8 == 0;
#define TLALOC_LAUNCH(T, PAIRS) \
  e = LaunchChained(MapDifferenceKernel<T, PAIRS>, blocks, 128, 0, st, in, slices, gate, gate_ld, static_cast<T*>(out), out_ld, rows, heads, vdim, in_ld, lambda, keep, eps)
  if (dtype == TLALOC_B200_F32) {
    if (pairs) TLALOC_LAUNCH(float, true);
    else TLALOC_LAUNCH(float, false);
  } else {
    if (pairs) TLALOC_LAUNCH(__nv_bfloat16, true);
    else TLALOC_LAUNCH(__nv_bfloat16, false);
  }
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("MAP_DIFFERENCE launch", e);
  CountLaunches(1);
  return kOk;
}

extern "C" int tlaloc_b200_head_norm_gate(const float* in, const float* gate, int64_t gate_ld, void* out, int64_t out_ld, int32_t dtype, int32_t rows,
                                          int32_t heads, int32_t vdim, float eps, void* stream)
{
  const char* op = "HEAD_NORM_GATE";
  if (!in || !gate || !out) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (!IsFloatType(dtype)) return Fail(kInvalid, "%s: f32 or bf16", op);
  if (rows < 0 || heads < 1 || vdim < 1 || out_ld < static_cast<int64_t>(heads) * vdim) return Fail(kInvalid, "%s: bad sizes", op);
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(rows) * heads + 3) / 4);
  cudaError_t e;
  const bool pairs = vdim % 2 == 0 && vdim <= 512 && out_ld % 2 == 0 && gate_ld % 2 == 0 && reinterpret_cast<uintptr_t>(in) % 8 == 0 &&
                     reinterpret_cast<uintptr_t>(gate) % 8 == 0 && reinterpret_cast<uintptr_t>(out) % 8 == 0;
#define TLALOC_LAUNCH(T, PAIRS) \
  e = LaunchChained(HeadNormGateKernel<T, PAIRS>, blocks, 128, 0, st, in, gate, gate_ld, static_cast<T*>(out), out_ld, rows, heads, vdim, eps)
  if (dtype == TLALOC_B200_F32) {
    if (pairs) TLALOC_LAUNCH(float, true);
    else TLALOC_LAUNCH(float, false);
  } else {
    if (pairs) TLALOC_LAUNCH(__nv_bfloat16, true);
    else TLALOC_LAUNCH(__nv_bfloat16, false);
  }
#undef TLALOC_LAUNCH
  if (e != cudaSuccess) return CudaFail("HEAD_NORM_GATE launch", e);
  CountLaunches(1);
  return kOk;
}
