// K6 norm_residual: (x [+ x2] [+ residual]) -> new residual, LayerNorm / RMSNorm of it.
//
// Replaces the reference's separate ATen add + layer_norm launches (SURVEY.md G2, G13;
// gptj_modeling.py:296,310,496; gpt_bigcode_modeling.py:367,379,404,407) and provides the
// capability of the never-instantiated FastLayerNorm wrapper (layers.py:217-256, G18).
// One CTA per row, row held in registers (16-byte vector loads), fp32 statistics,
// two-pass variance.  Memory-bound: reads x(+res) once, writes normed(+res) once.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int kMaxVec = 4;  // 256 thr * 4 vec * 8 elem = H <= 8192

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (l < kThreads / 32) ? red[l] : 0.f;
  return warp_sum(t);
}

template <typename T>
__global__ void __launch_bounds__(kThreads) norm_residual_kernel(
    const T* __restrict__ x, const T* __restrict__ x2, const T* residual_in, T* residual_out,
    const T* __restrict__ weight, const T* __restrict__ bias, T* __restrict__ out, int H, int64_t ldx,
    int64_t ldx2, int64_t ldr, int64_t ldo, float eps, int kind) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[kThreads / 32];
  const int row = blockIdx.x;
  const int nvec = H >> 3;
  float v[kMaxVec][8];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxVec; ++i) {
    const int c = threadIdx.x + i * kThreads;
    if (c < nvec) {
      uint4 raw = *reinterpret_cast<const uint4*>(x + row * ldx + c * 8);
      unpack8<T>(raw, v[i]);
      if (x2 != nullptr) {
        float t[8];
        raw = *reinterpret_cast<const uint4*>(x2 + row * ldx2 + c * 8);
        unpack8<T>(raw, t);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] += t[j];
      }
      if (residual_in != nullptr) {
        float t[8];
        raw = *reinterpret_cast<const uint4*>(residual_in + row * ldr + c * 8);
        unpack8<T>(raw, t);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] += t[j];
      }
      if (residual_out != nullptr) {
        *reinterpret_cast<uint4*>(residual_out + row * ldr + c * 8) = pack8<T>(v[i]);
        // the normalisation sees the value as stored (same rounding as the unfused path)
        unpack8<T>(pack8<T>(v[i]), v[i]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) sum += (kind == LLMSS_NORM_RMS) ? v[i][j] * v[i][j] : v[i][j];
    }
  }
  float mean = 0.f, rstd;
  if (kind == LLMSS_NORM_RMS) {
    float ss = block_sum(sum, red);
    rstd = rsqrtf(ss / (float)H + eps);
  } else {
    mean = block_sum(sum, red) / (float)H;
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxVec; ++i) {
      const int c = threadIdx.x + i * kThreads;
      if (c < nvec) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          float d = v[i][j] - mean;
          sq += d * d;
        }
      }
    }
    float var = block_sum(sq, red) / (float)H;
    rstd = rsqrtf(var + eps);
  }
#pragma unroll
  for (int i = 0; i < kMaxVec; ++i) {
    const int c = threadIdx.x + i * kThreads;
    if (c < nvec) {
      float w[8], b[8], o[8];
      unpack8<T>(*reinterpret_cast<const uint4*>(weight + c * 8), w);
      if (bias != nullptr) unpack8<T>(*reinterpret_cast<const uint4*>(bias + c * 8), b);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        float y = (v[i][j] - mean) * rstd * w[j];
        o[j] = (bias != nullptr) ? y + b[j] : y;
      }
      *reinterpret_cast<uint4*>(out + row * ldo + c * 8) = pack8<T>(o);
    }
  }
}

// ------------------------------------------------------------------------------------------------ 32-bit residual stream
// r = resid + mult * y (y null: r = resid) ; h = LayerNorm / RMS norm of r times weight (+ bias), stored as TO.  One CTA per row, the
// row in registers (VEC = 4: 16-byte accesses; longer rows are read back from `out_r`), two-pass variance, 32-bit throughout.
struct RnArgs {
  const float* resid; int64_t ldr;
  const float* y; int64_t ldy;
  const float* w; const float* bias;
  float* out_r; void* out_h;         // [M, W] contiguous; out_r null: r is not stored (y null)
  int W; float eps; int kind;
  float mult;                        // factor on y
};
constexpr int kRnRegs = 4;

template <int VEC> __device__ __forceinline__ void rn_load(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  } else v[0] = p[0];
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(kThreads) residual_norm_kernel(RnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[kThreads / 32];
  const int64_t t = blockIdx.x;
  const int W = a.W;
  constexpr int STEP = kThreads * VEC;
  float keep[kRnRegs][VEC];
  float sum = 0.f;
  const bool rms = a.kind == LLMSS_NORM_RMS;
  auto fetch = [&](int c, float (&v)[VEC]) {
    rn_load<VEC>(a.resid + t * a.ldr + c, v);
    if (a.y != nullptr) {
      float u[VEC];
      rn_load<VEC>(a.y + t * a.ldy + c, u);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = fmaf(a.mult, u[e], v[e]);
    }
    if (a.out_r != nullptr) {
      float* o = a.out_r + t * (int64_t)W + c;
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]);
      else o[0] = v[0];
    }
  };
  const float* again = a.out_r != nullptr ? a.out_r + t * (int64_t)W : a.resid + t * a.ldr;   // this thread's own columns of r
#pragma unroll
  for (int i = 0; i < kRnRegs; ++i) {
    const int c = threadIdx.x * VEC + i * STEP;
    if (c < W) {
      fetch(c, keep[i]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum += rms ? keep[i][e] * keep[i][e] : keep[i][e];
    }
  }
  for (int c = threadIdx.x * VEC + kRnRegs * STEP; c < W; c += STEP) {
    float v[VEC];
    fetch(c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum += rms ? v[e] * v[e] : v[e];
  }
  float mean = 0.f, rstd;
  if (rms) {
    rstd = rsqrtf(block_sum(sum, red) / (float)W + a.eps);
  } else {
    mean = block_sum(sum, red) / (float)W;
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < kRnRegs; ++i) {
      const int c = threadIdx.x * VEC + i * STEP;
      if (c < W) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { const float d = keep[i][e] - mean; sq = fmaf(d, d, sq); }
      }
    }
    for (int c = threadIdx.x * VEC + kRnRegs * STEP; c < W; c += STEP) {
      float v[VEC];
      rn_load<VEC>(again + c, v);
#pragma unroll
      for (int e = 0; e < VEC; ++e) { const float d = v[e] - mean; sq = fmaf(d, d, sq); }
    }
    rstd = rsqrtf(block_sum(sq, red) / (float)W + a.eps);
  }
  auto emit = [&](int c, const float (&v)[VEC]) {
    float wv[VEC], bv[VEC];
    rn_load<VEC>(a.w + c, wv);
    if (a.bias != nullptr) rn_load<VEC>(a.bias + c, bv);
    TO* ho = reinterpret_cast<TO*>(a.out_h) + t * (int64_t)W + c;
    struct alignas(VEC * sizeof(TO)) Pack { TO v[VEC]; };
    Pack o;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const float h = (v[e] - mean) * rstd * wv[e];
      o.v[e] = from_f32<TO>(a.bias != nullptr ? h + bv[e] : h);
    }
    *reinterpret_cast<Pack*>(ho) = o;
  };
#pragma unroll
  for (int i = 0; i < kRnRegs; ++i) {
    const int c = threadIdx.x * VEC + i * STEP;
    if (c < W) emit(c, keep[i]);
  }
  for (int c = threadIdx.x * VEC + kRnRegs * STEP; c < W; c += STEP) {
    float v[VEC];
    rn_load<VEC>(again + c, v);
    emit(c, v);
  }
}

template <typename TO>
int residual_norm_launch(const RnArgs& a, int M, bool vec, cudaStream_t stream) {
  if (vec) LLMSS_CHECK_CUDA(launch_pdl(residual_norm_kernel<TO, 4>, dim3(M), dim3(kThreads), 0, stream, a));
  else LLMSS_CHECK_CUDA(launch_pdl(residual_norm_kernel<TO, 1>, dim3(M), dim3(kThreads), 0, stream, a));
  return 0;
}

}  // namespace

// The counterpart of llmss_norm_residual over a 32-bit residual stream: resid [M, W] (row stride ldr), y [M, W] or null, weight /
// bias 32-bit (bias may be null), out_r [M, W] contiguous (null with y null), out_h [M, W] contiguous in out_dtype.
// mult: factor on y.
LLMSS_API int llmss_residual_norm_ex(const float* resid, int64_t ldr, const float* y, int64_t ldy, float mult, const float* weight,
                                     const float* bias, float* out_r, void* out_h, int M, int W, float eps, int kind, int out_dtype,
                                     cudaStream_t stream) {
  LLMSS_REQUIRE(W > 0 && weight != nullptr && out_h != nullptr && (y == nullptr || out_r != nullptr), "residual_norm: bad arguments");
  LLMSS_REQUIRE(kind == LLMSS_NORM_LAYER || kind == LLMSS_NORM_RMS, "residual_norm: norm kind %d", kind);
  if (M <= 0) return 0;
  RnArgs a{resid, ldr, y, ldy, weight, bias, out_r, out_h, W, eps, kind, mult};
  const bool vec = W % 4 == 0 && ldr % 4 == 0 && ldy % 4 == 0 &&
                   ((((uintptr_t)resid) | ((uintptr_t)y) | ((uintptr_t)weight) | ((uintptr_t)bias) | ((uintptr_t)out_r) | ((uintptr_t)out_h)) & 15) == 0;
  LLMSS_BY_DTYPE(out_dtype, return (residual_norm_launch<T>(a, M, vec, stream)));
}

LLMSS_API int llmss_residual_norm(const float* resid, int64_t ldr, const float* y, int64_t ldy, const float* weight, const float* bias,
                                  float* out_r, void* out_h, int M, int W, float eps, int kind, int out_dtype, cudaStream_t stream) {
  return llmss_residual_norm_ex(resid, ldr, y, ldy, 1.f, weight, bias, out_r, out_h, M, W, eps, kind, out_dtype, stream);
}

LLMSS_API int llmss_norm_residual(const void* x, const void* x2, const void* residual_in, void* residual_out,
                                  const void* weight, const void* bias, void* out, int M, int H, int64_t ldx,
                                  int64_t ldx2, int64_t ldr, int64_t ldo, float eps, int kind, int dtype,
                                  cudaStream_t stream) {
  LLMSS_REQUIRE(H % 8 == 0 && H <= kThreads * kMaxVec * 8, "norm_residual: H=%d must be a multiple of 8 and <= %d", H,
                kThreads * kMaxVec * 8);
  LLMSS_REQUIRE(dtype == LLMSS_F16 || dtype == LLMSS_BF16, "norm_residual: dtype must be f16/bf16");
  LLMSS_REQUIRE(ldx % 8 == 0 && ldo % 8 == 0 && ldr % 8 == 0 && ldx2 % 8 == 0, "norm_residual: row strides must be multiples of 8");
  if (M == 0) return 0;
  if (dtype == LLMSS_F16)
    LLMSS_CHECK_CUDA(launch_pdl(norm_residual_kernel<__half>, dim3(M), dim3(kThreads), 0, stream, (const __half*)x, (const __half*)x2, (const __half*)residual_in, (__half*)residual_out, (const __half*)weight, (const __half*)bias, (__half*)out, H, ldx, ldx2, ldr, ldo, eps, kind));
  else
    LLMSS_CHECK_CUDA(launch_pdl(norm_residual_kernel<__nv_bfloat16>, dim3(M), dim3(kThreads), 0, stream, (const __nv_bfloat16*)x, (const __nv_bfloat16*)x2, (const __nv_bfloat16*)residual_in, (__nv_bfloat16*)residual_out, (const __nv_bfloat16*)weight, (const __nv_bfloat16*)bias, (__nv_bfloat16*)out, H, ldx, ldx2, ldr, ldo, eps, kind));
  LLMSS_CHECK_CUDA(cudaGetLastError());
  return 0;
}
