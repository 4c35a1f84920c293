// Linear attention with one constant decay per head, S <- a_h S + k v^T, y = S^T q (evo_decay_scan_fwd), and the norm over all heads
// with a sigmoid gate that closes it (evo_norm_gate).
#include "common.cuh"
#include "../../include/evo_b200.h"
#include <math.h>
#include <stdint.h>

using namespace evo;

namespace evo {
int decay_scan_recurrent(const evo_decay_scan_params* p, cudaStream_t st);      // matrix_state.cu
}

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

// ---- evo_norm_gate: one CTA per row; a thread keeps its first NG_KEEP groups of four values in registers between the two passes
constexpr int NG_T = 256, NG_KEEP = 4;

__device__ __forceinline__ float row_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < NG_T / 32; ++i) t += red[i];
  return t;
}
template <typename T> __device__ __forceinline__ float sigmoid_of(float z);
template <> __device__ __forceinline__ float sigmoid_of<float>(float z) { return 1.f / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float sigmoid_of<bf16>(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

template <typename T>
__global__ void __launch_bounds__(NG_T) norm_gate4_kernel(const float* __restrict__ y, const T* __restrict__ gate, int64_t ldg, const bf16* __restrict__ nw,
                                                          T* __restrict__ out, int64_t ldo, int width, float eps) {
  __shared__ float red[NG_T / 32];
  const int64_t r = blockIdx.x;
  const float* yr = y + r * width;
  const T* gr = gate + r * ldg;
  T* orow = out + r * ldo;
  float4 keep[NG_KEEP];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NG_KEEP; ++k) {
    const int c = (k * NG_T + threadIdx.x) * 4;
    keep[k] = c < width ? *reinterpret_cast<const float4*>(yr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss = fmaf(keep[k].x, keep[k].x, fmaf(keep[k].y, keep[k].y, fmaf(keep[k].z, keep[k].z, fmaf(keep[k].w, keep[k].w, ss))));
  }
  for (int c = (NG_KEEP * NG_T + threadIdx.x) * 4; c < width; c += NG_T * 4) {
    const float4 v = *reinterpret_cast<const float4*>(yr + c);
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
  }
  const float rs = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
  const auto put = [&](int c, float4 v) {
    float g[4], w[4];
    if (sizeof(T) == 4) {
      const float4 u = *reinterpret_cast<const float4*>(gr + c);
      g[0] = u.x; g[1] = u.y; g[2] = u.z; g[3] = u.w;
    } else {
      const uint2 u = *reinterpret_cast<const uint2*>(gr + c);
      g[0] = bf_lo(u.x); g[1] = bf_hi(u.x); g[2] = bf_lo(u.y); g[3] = bf_hi(u.y);
    }
    const uint2 u = *reinterpret_cast<const uint2*>(nw + c);
    w[0] = bf_lo(u.x); w[1] = bf_hi(u.x); w[2] = bf_lo(u.y); w[3] = bf_hi(u.y);
    const float o0 = v.x * rs * w[0] * sigmoid_of<T>(g[0]), o1 = v.y * rs * w[1] * sigmoid_of<T>(g[1]);
    const float o2 = v.z * rs * w[2] * sigmoid_of<T>(g[2]), o3 = v.w * rs * w[3] * sigmoid_of<T>(g[3]);
    if (sizeof(T) == 4) *reinterpret_cast<float4*>(orow + c) = make_float4(o0, o1, o2, o3);
    else *reinterpret_cast<uint2*>(orow + c) = make_uint2(pack_bf16(o0, o1), pack_bf16(o2, o3));
  };
#pragma unroll
  for (int k = 0; k < NG_KEEP; ++k) {
    const int c = (k * NG_T + threadIdx.x) * 4;
    if (c < width) put(c, keep[k]);
  }
  for (int c = (NG_KEEP * NG_T + threadIdx.x) * 4; c < width; c += NG_T * 4) put(c, *reinterpret_cast<const float4*>(yr + c));
  for (int64_t c = width + threadIdx.x; c < ldo; c += NG_T) stf(orow + c, 0.f);
}

template <typename T>
__global__ void __launch_bounds__(NG_T) norm_gate_kernel(const float* __restrict__ y, const T* __restrict__ gate, int64_t ldg, const bf16* __restrict__ nw,
                                                         T* __restrict__ out, int64_t ldo, int width, float eps) {
  __shared__ float red[NG_T / 32];
  const int64_t r = blockIdx.x;
  const float* yr = y + r * width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += NG_T) ss = fmaf(yr[c], yr[c], ss);
  const float rs = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
  for (int64_t c = threadIdx.x; c < ldo; c += NG_T)
    stf(out + r * ldo + c, c < width ? yr[c] * rs * __bfloat162float(nw[c]) * sigmoid_of<T>(ldf(gate + r * ldg + c)) : 0.f);
}

}  // namespace

extern "C" size_t evo_decay_scan_workspace(const evo_decay_scan_params* p) { return 0; }

extern "C" int evo_decay_scan_fwd(const evo_decay_scan_params* p, void* workspace, size_t workspace_bytes, void* stream) {
  EVO_REQUIRE(p->q && p->k && p->v && p->decay && p->y, "evo_decay_scan_fwd: null argument");
  EVO_REQUIRE(p->B >= 0 && p->L >= 0 && p->H > 0 && p->dk > 0 && p->dv > 0, "evo_decay_scan_fwd: bad shape");
  if (p->B == 0 || p->L == 0) return 0;
  return decay_scan_recurrent(p, (cudaStream_t)stream);
}

extern "C" int evo_norm_gate(const float* y, const void* gate, int64_t ldg, const void* norm_w, void* out, int64_t ldo, int64_t rows, int width, float eps, int dtype, void* stream) {
  EVO_REQUIRE(y && gate && norm_w && out && width > 0 && ldo >= width && ldg >= width && rows >= 0, "evo_norm_gate: bad arguments");
  if (rows == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const uintptr_t am = dtype ? 15 : 7;
  const bool vec = width % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)norm_w & 7) == 0 && (((uintptr_t)gate | (uintptr_t)out) & am) == 0;
  const unsigned grid = (unsigned)rows;
  if (dtype) {
    if (vec) norm_gate4_kernel<float><<<grid, NG_T, 0, st>>>(y, (const float*)gate, ldg, (const bf16*)norm_w, (float*)out, ldo, width, eps);
    else norm_gate_kernel<float><<<grid, NG_T, 0, st>>>(y, (const float*)gate, ldg, (const bf16*)norm_w, (float*)out, ldo, width, eps);
  } else {
    if (vec) norm_gate4_kernel<bf16><<<grid, NG_T, 0, st>>>(y, (const bf16*)gate, ldg, (const bf16*)norm_w, (bf16*)out, ldo, width, eps);
    else norm_gate_kernel<bf16><<<grid, NG_T, 0, st>>>(y, (const bf16*)gate, ldg, (const bf16*)norm_w, (bf16*)out, ldo, width, eps);
  }
  return check_launch("evo_norm_gate");
}
