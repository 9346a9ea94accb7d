// Retention over a prompt portion on the tensor cores, bf16 operands (include/tlaloc_b200.h, tlaloc_b200_retention_chunks).
//
// The portion is cut into chunks of 64 tokens and, for parallelism, into segments of whole chunks.  Within a chunk, with S the state ahead
// of it and w = decay:
//   o_i = w^(i+1) S^T q_i + sum_{j <= i} w^(i-j) (q_i . k_j) v_j        S <- w^n S + sum_j w^(n-1-j) k_j v_j^T
// A CTA has one head, a slice of its value columns and one segment; S stays in its registers as f32 accumulators of the transposed product
// (value columns as the rows of mma.m16n8k16, so that an accumulator is also the operand layout of S^T q).  What was computed in f32 and
// enters a product as an operand (S, the decayed scores, the decayed values) enters as two bf16 parts, which is f32 up to rounding.
// Two launches where there are several segments: the first computes what each segment adds to the state, the second starts every
// segment from the sum of those before it, writes the outputs and, in the last segment, the new state.
#include "common.cuh"

namespace tlaloc_b200 {
namespace {

constexpr int kChunk = 64, kWarps = 4, kThreads = kWarps * 32;
constexpr int kMaxSmem = 227 * 1024;

struct ChunkArgs {
  const __nv_bfloat16 *q, *k, *v;
  const int *positions, *row_states;
  const float* decay;
  float *state, *o, *sums;  // sums [segments][heads][slices][..]: what a segment adds; the last one's place holds the state before the portion
  int tokens, heads, dim, vdim, dim_ld, v_ld, num_slots, segment, segments;
};

__device__ __forceinline__ void Mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1)
{
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void Ldm4(uint32_t* r, uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void Ldm4T(uint32_t* r, uint32_t addr)
{
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void Split(float a, float b, uint32_t& hi, uint32_t& lo)
{
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float Low(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float High(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// DK: 16-channel steps of a key at most; VS: value columns of a slice.  The warps share S as VS / 16 groups of value columns by
// 64 / VS parts of the channels.
template <int DK, int VS, bool OUT>
__global__ void __launch_bounds__(kThreads) RetentionChunkKernel(const __grid_constant__ ChunkArgs a)
{
  GridDependencySync();
  constexpr int kParts = 64 / VS, kTiles = 2 * DK / kParts;  // 8-channel tiles of S a warp holds
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float pw[kChunk + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.x, slice = blockIdx.y, seg = blockIdx.z, slices = gridDim.y;
  const int dk = a.dim_ld >> 4, k_ld = a.dim_ld * 2 + 16, v_ld = VS * 2 + 16;
  const uint32_t base = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  const int q_bytes = OUT ? kChunk * k_ld : 0, k_bytes = kChunk * k_ld, buf_bytes = q_bytes + k_bytes + kChunk * v_ld;
  const uint32_t s_hi = base + 2 * buf_bytes, s_lo = s_hi + VS * k_ld;
  const float w = __ldg(a.decay + head);
  for (int i = tid; i <= kChunk; i += kThreads) pw[i] = powf(w, static_cast<float>(i));

  const int t_begin = seg * a.segment, t_end = min(a.tokens, t_begin + a.segment);
  auto load = [&](int t0, int buf) {
    const uint32_t dst = base + buf * buf_bytes;
    const int kc = a.dim_ld >> 3, rows = t_end - t0;
    for (int i = tid; i < kChunk * kc; i += kThreads) {
      const int r = i / kc, c = i - r * kc;
      const size_t at = (static_cast<size_t>(t0 + min(r, rows - 1)) * a.heads + head) * a.dim_ld + c * 8;
      const int bytes = r < rows ? 16 : 0;
      if (OUT) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst + r * k_ld + c * 16), "l"(a.q + at), "r"(bytes) : "memory");
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst + q_bytes + r * k_ld + c * 16), "l"(a.k + at), "r"(bytes) : "memory");
    }
    for (int i = tid; i < kChunk * (VS / 8); i += kThreads) {
      const int r = i / (VS / 8), c = i % (VS / 8), col = slice * VS + c * 8;
      const size_t at = (static_cast<size_t>(t0 + min(r, rows - 1)) * a.heads + head) * a.v_ld + min(col, a.v_ld - 8);
      const int bytes = r < rows && col < a.v_ld ? 16 : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst + q_bytes + k_bytes + r * v_ld + c * 16), "l"(a.v + at), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  load(t_begin, 0);

  // S: rows v0 + lane / 4 (+ 8), channels d0 + 8 n + 2 (lane % 4) (+ 1).
  const int v0 = (warp / kParts) * 16, d0 = (warp % kParts) * (kTiles * 8);
  float s[kTiles][4];
  const int vp = (a.vdim + 3) & ~3;
  const int slot = min(max(__ldg(a.row_states), 0), a.num_slots - 1);
  float* state = a.state + (static_cast<size_t>(slot) * a.heads + head) * a.dim * vp;
  const size_t frag = static_cast<size_t>(kTiles) * 4 * kThreads;
  auto sums = [&](int g) { return a.sums + ((static_cast<size_t>(g) * a.heads + head) * slices + slice) * frag + tid; };
#pragma unroll
  for (int n = 0; n < kTiles; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
  if (seg == 0 && !(OUT && a.segments > 1)) {
    if (__ldg(a.positions) != 0) {
#pragma unroll
      for (int n = 0; n < kTiles; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = d0 + n * 8 + (lane & 3) * 2 + (e & 1), v = slice * VS + v0 + (lane >> 2) + (e >> 1) * 8;
          if (d < a.dim && v < vp) s[n][e] = state[static_cast<size_t>(d) * vp + v];
        }
    }
    if (!OUT) {
      float* p = sums(a.segments - 1);
#pragma unroll
      for (int n = 0; n < kTiles; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) p[(n * 4 + e) * kThreads] = s[n][e];
    }
  } else if (OUT) {
    const float ws = powf(w, static_cast<float>(a.segment));
    for (int g = seg == 0 ? a.segments - 1 : 0; g < (seg == 0 ? a.segments : seg); ++g) {
      const float* p = sums(g);
#pragma unroll
      for (int n = 0; n < kTiles; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = fmaf(ws, s[n][e], p[(n * 4 + e) * kThreads]);
    }
  }

  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += kChunk, buf ^= 1) {
    const int count = min(kChunk, t_end - t0);
    const uint32_t qt = base + buf * buf_bytes, kt = qt + q_bytes, vt = kt + k_bytes;
    if (OUT) {  // the state ahead of the chunk, for all warps
#pragma unroll
      for (int n = 0; n < kTiles; ++n) {
        if (d0 + n * 8 < a.dim_ld) {
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            uint32_t hi, lo;
            Split(s[n][2 * r], s[n][2 * r + 1], hi, lo);
            const uint32_t at = (v0 + (lane >> 2) + 8 * r) * k_ld + (d0 + n * 8 + (lane & 3) * 2) * 2;
            asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(s_hi + at), "r"(hi) : "memory");
            asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(s_lo + at), "r"(lo) : "memory");
          }
        }
      }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    if (t0 + kChunk < t_end) load(t0 + kChunk, buf ^ 1);  // its last readers are behind the barrier at the end of the chunk before

    const int m = lane >> 3, r8 = lane & 7;
    if (OUT) {
      const int i0 = warp * 16 + (lane >> 2);
      uint32_t qa[DK][4];
#pragma unroll
      for (int k = 0; k < DK; ++k)
        if (k < dk) Ldm4(qa[k], qt + (warp * 16 + (m & 1) * 8 + r8) * k_ld + k * 32 + (m >> 1) * 16);
      float o[VS / 8][4];
#pragma unroll
      for (int n = 0; n < VS / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
#pragma unroll
      for (int k = 0; k < DK; ++k) {
        if (k < dk) {
#pragma unroll
          for (int n = 0; n < VS / 16; ++n) {
            uint32_t b[4];
            const uint32_t at = (n * 16 + (m >> 1) * 8 + r8) * k_ld + k * 32 + (m & 1) * 16;
            Ldm4(b, s_hi + at);
            Mma(o[2 * n], qa[k], b[0], b[1]);
            Mma(o[2 * n + 1], qa[k], b[2], b[3]);
            Ldm4(b, s_lo + at);
            Mma(o[2 * n], qa[k], b[0], b[1]);
            Mma(o[2 * n + 1], qa[k], b[2], b[3]);
          }
        }
      }
      const float w0 = pw[i0 + 1], w1 = pw[i0 + 9];
#pragma unroll
      for (int n = 0; n < VS / 8; ++n) {
        o[n][0] *= w0;
        o[n][1] *= w0;
        o[n][2] *= w1;
        o[n][3] *= w1;
      }
#pragma unroll 1
      for (int j = 0; j <= warp; ++j) {  // 16 keys at a time, none past the queries
        float c[2][4] = {};
#pragma unroll
        for (int k = 0; k < DK; ++k) {
          if (k < dk) {
            uint32_t b[4];
            Ldm4(b, kt + (j * 16 + (m >> 1) * 8 + r8) * k_ld + k * 32 + (m & 1) * 16);
            Mma(c[0], qa[k], b[0], b[1]);
            Mma(c[1], qa[k], b[2], b[3]);
          }
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int back = i0 + (e >> 1) * 8 - (j * 16 + n * 8 + (lane & 3) * 2 + (e & 1));
            c[n][e] = back >= 0 ? c[n][e] * pw[max(back, 0)] : 0.f;
          }
        uint32_t hi[4], lo[4];
        Split(c[0][0], c[0][1], hi[0], lo[0]);
        Split(c[0][2], c[0][3], hi[1], lo[1]);
        Split(c[1][0], c[1][1], hi[2], lo[2]);
        Split(c[1][2], c[1][3], hi[3], lo[3]);
#pragma unroll
        for (int n = 0; n < VS / 16; ++n) {
          uint32_t b[4];
          Ldm4T(b, vt + (j * 16 + (m & 1) * 8 + r8) * v_ld + n * 32 + (m >> 1) * 16);
          Mma(o[2 * n], hi, b[0], b[1]);
          Mma(o[2 * n + 1], hi, b[2], b[3]);
          Mma(o[2 * n], lo, b[0], b[1]);
          Mma(o[2 * n + 1], lo, b[2], b[3]);
        }
      }
      float* out = a.o + (static_cast<size_t>(t0) * a.heads + head) * a.vdim;
      const bool pairs = a.vdim % 2 == 0;
#pragma unroll
      for (int n = 0; n < VS / 8; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = i0 + 8 * r, col = slice * VS + n * 8 + (lane & 3) * 2;
          float* p = out + static_cast<size_t>(i) * a.heads * a.vdim + col;
          if (i < count && col + 1 < a.vdim && pairs) {
            *reinterpret_cast<float2*>(p) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
          } else if (i < count) {
            if (col < a.vdim) p[0] = o[n][2 * r];
            if (col + 1 < a.vdim) p[1] = o[n][2 * r + 1];
          }
        }
    }

    // the state behind the chunk
    if (!OUT || seg + 1 == a.segments || t0 + kChunk < t_end) {
      const float wn = pw[count];
#pragma unroll
      for (int n = 0; n < kTiles; ++n) {
        s[n][0] *= wn;
        s[n][1] *= wn;
        s[n][2] *= wn;
        s[n][3] *= wn;
      }
#pragma unroll 1
      for (int j = 0; j < kChunk / 16; ++j) {
        uint32_t va[4], hi[4], lo[4];
        Ldm4T(va, vt + (j * 16 + (m >> 1) * 8 + r8) * v_ld + (v0 + (m & 1) * 8) * 2);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int tok = count - 1 - (j * 16 + h * 8 + (lane & 3) * 2);
          const float wa = tok >= 0 ? pw[max(tok, 0)] : 0.f, wb = tok >= 1 ? pw[max(tok - 1, 0)] : 0.f;
          Split(Low(va[2 * h]) * wa, High(va[2 * h]) * wb, hi[2 * h], lo[2 * h]);
          Split(Low(va[2 * h + 1]) * wa, High(va[2 * h + 1]) * wb, hi[2 * h + 1], lo[2 * h + 1]);
        }
#pragma unroll
        for (int n = 0; n < kTiles / 2; ++n) {
          if (d0 + n * 16 < a.dim_ld) {
            uint32_t b[4];
            Ldm4T(b, kt + (j * 16 + (m & 1) * 8 + r8) * k_ld + (d0 + n * 16 + (m >> 1) * 8) * 2);
            Mma(s[2 * n], hi, b[0], b[1]);
            Mma(s[2 * n + 1], hi, b[2], b[3]);
            Mma(s[2 * n], lo, b[0], b[1]);
            Mma(s[2 * n + 1], lo, b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();
  }

  if (!OUT) {
    float* p = sums(seg);
#pragma unroll
    for (int n = 0; n < kTiles; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) p[(n * 4 + e) * kThreads] = s[n][e];
  } else if (seg + 1 == a.segments) {
#pragma unroll
    for (int n = 0; n < kTiles; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = d0 + n * 8 + (lane & 3) * 2 + (e & 1), v = slice * VS + v0 + (lane >> 2) + (e >> 1) * 8;
        if (d < a.dim && v < vp) state[static_cast<size_t>(d) * vp + v] = s[n][e];
      }
  }
}

// What a call is cut into.
struct Plan {
  int dk, vs, slices, segment, segments;
  size_t sums_bytes;
};
Plan PlanFor(int tokens, int heads, int dim, int vdim)
{
  Plan p;
  const int dp = (dim + 15) / 16 * 16;
  p.dk = dp <= 64 ? 4 : dp <= 128 ? 8 : 16;
  p.vs = p.dk == 16 ? 32 : 64;
  p.slices = (vdim + p.vs - 1) / p.vs;
  const int chunks = (tokens + kChunk - 1) / kChunk;
  int want = (3 * 148 + heads * p.slices - 1) / (heads * p.slices);  // a few CTAs per SM
  want = want < 1 ? 1 : want > 32 ? 32 : want;
  const int per = (chunks + want - 1) / want;
  p.segment = per * kChunk;
  p.segments = (chunks + per - 1) / per;
  p.sums_bytes = p.segments > 1 ? static_cast<size_t>(p.segments) * heads * p.slices * p.vs * p.dk * 16 * sizeof(float) : 0;
  return p;
}
size_t SmemBytes(int dk, int vs, int dim_ld, bool out)
{
  const size_t k_ld = dim_ld * 2 + 16, v_ld = vs * 2 + 16;
  (void)dk;
  return 2 * ((out ? 2 : 1) * kChunk * k_ld + kChunk * v_ld) + (out ? 2 * vs * k_ld : 0);
}

cudaError_t PrepareChunks()
{
  static OncePerDevice once;
  return once.Run([](int) {
    cudaError_t e = cudaSuccess;
#define TLALOC_OPT_IN(DK, VS)                                                                                                                    \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(RetentionChunkKernel<DK, VS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024); \
  if (e == cudaSuccess) e = cudaFuncSetAttribute(RetentionChunkKernel<DK, VS, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem - 1024);
    TLALOC_OPT_IN(4, 64)
    TLALOC_OPT_IN(8, 64)
    TLALOC_OPT_IN(16, 32)
#undef TLALOC_OPT_IN
    return e;
  });
}
KernelSetup g_setup(PrepareChunks, nullptr);

template <bool OUT>
cudaError_t Launch(const Plan& p, const ChunkArgs& a, int segments, cudaStream_t st)
{
  const dim3 grid(a.heads, p.slices, segments);
  const size_t smem = SmemBytes(p.dk, p.vs, a.dim_ld, OUT);
  if (p.dk == 4) return LaunchChained(RetentionChunkKernel<4, 64, OUT>, grid, kThreads, smem, st, a);
  if (p.dk == 8) return LaunchChained(RetentionChunkKernel<8, 64, OUT>, grid, kThreads, smem, st, a);
  return LaunchChained(RetentionChunkKernel<16, 32, OUT>, grid, kThreads, smem, st, a);
}

}  // namespace
}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_retention_chunks_applies(int32_t dim, int32_t vdim) { return dim >= 1 && dim <= 256 && vdim >= 1 && !OrderFaithful() ? 1 : 0; }

extern "C" size_t tlaloc_b200_retention_chunks_scratch_bytes(int32_t tokens, int32_t heads, int32_t dim, int32_t vdim)
{
  if (tokens < 1 || heads < 1 || !tlaloc_b200_retention_chunks_applies(dim, vdim)) return 0;
  return PlanFor(tokens, heads, dim, vdim).sums_bytes;
}

extern "C" int tlaloc_b200_retention_chunks(const void* q, const void* k, int32_t dim_ld, const void* v, int32_t v_ld, const int32_t* positions,
                                            const float* decay, const int32_t* row_states, float* state, float* o, void* scratch, size_t scratch_bytes,
                                            int32_t tokens, int32_t heads, int32_t dim, int32_t vdim, int32_t num_slots, void* stream)
{
  const char* op = "RETENTION_CHUNKS";
  if (!q || !k || !v || !positions || !decay || !row_states || !state || !o) return Fail(kInvalid, "%s: a required device pointer is null", op);
  if (tokens < 0 || heads < 1 || heads > 65535 || dim < 1 || vdim < 1 || num_slots < 1) return Fail(kInvalid, "%s: bad sizes", op);
  if (!tlaloc_b200_retention_chunks_applies(dim, vdim)) return Fail(kUnsupported, "%s: dim up to 256", op);
  if (dim_ld != (dim + 15) / 16 * 16 || v_ld < vdim || v_ld % 8 || !Aligned16(q) || !Aligned16(k) || !Aligned16(v) || !Aligned16(state)) {
    return Fail(kInvalid, "%s: rows of dim rounded up to 16 and of a multiple of 8 values, 16-byte aligned", op);
  }
  if (tokens == 0) return kOk;
  const Plan p = PlanFor(tokens, heads, dim, vdim);
  if (p.sums_bytes > 0 && (!scratch || scratch_bytes < p.sums_bytes)) return Fail(kInvalid, "%s: %zu bytes of scratch are needed", op, p.sums_bytes);
  cudaError_t e = PrepareChunks();
  if (e != cudaSuccess) return CudaFail("RETENTION_CHUNKS set-up", e);
  ChunkArgs a = {};
  a.q = static_cast<const __nv_bfloat16*>(q);
  a.k = static_cast<const __nv_bfloat16*>(k);
  a.v = static_cast<const __nv_bfloat16*>(v);
  a.positions = positions;
  a.row_states = row_states;
  a.decay = decay;
  a.state = state;
  a.o = o;
  a.sums = static_cast<float*>(scratch);
  a.tokens = tokens;
  a.heads = heads;
  a.dim = dim;
  a.vdim = vdim;
  a.dim_ld = dim_ld;
  a.v_ld = v_ld;
  a.num_slots = num_slots;
  a.segment = p.segment;
  a.segments = p.segments;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (p.segments > 1) {
    e = Launch<false>(p, a, p.segments - 1, st);
    if (e == cudaSuccess) CountLaunches(1);
  }
  if (e == cudaSuccess) e = Launch<true>(p, a, p.segments, st);
  if (e != cudaSuccess) return CudaFail("RETENTION_CHUNKS launch", e);
  CountLaunches(1);
  return kOk;
}
