// Softmax attention whose heads exchange scores before the softmax ("talking heads"), over a linear key/value cache:
//   a_g(i, j) = scale * temp_g * q_g(i) . k(j),   s_h(i, j) = sum_g talk[h, g] a_g(i, j),   p_h = softmax over the keys j that i sees
// with a chunked causal mask (i sees j <= i of its own chunk of positions, chunks counted from position 0; chunk 0: plain causal) and an
// optional sigmoid output gate of one number per head.  Scores, their mixture, softmax weights and sums are fp32 whatever the activation type.
// scale, temp and talk fold into one fp32 matrix, so the mixture costs H multiply-adds per score.
//
// mixed_attn_mma_kernel (bf16, 16 query rows or more): all heads of a query tile must be scored before any of them can run its softmax, so a
// cluster of ceil(H / 16) CTAs owns a tile of 16 queries and a CTA owns up to 16 heads, one per warp, as score heads AND as output heads.
// Per tile of keys: (1) every warp scores its head on the tensor cores (mma.sync m16n8k16, fp32 accumulation) and writes the fp32 scores to
// the score buffer of every CTA of the cluster (distributed shared memory); (2) a thread takes one or two (query, key) places, reads that
// place's score of all H heads and writes the mixed scores of the CTA's output heads over its own score slots; (3) every warp runs the online
// softmax of its head on mma fragments and accumulates P.V in registers, each weight as bf16 high part + bf16 remainder.  K of the next tile
// is on its way during (2) and (3), V during (1) and (2) (16-byte asynchronous copies), so one buffer of each is enough.  The score slots of a
// CTA's own heads are written by nobody else after (2), so the other CTAs may start the next tile as soon as this one has mixed.
//
// mixed_attn_split_kernel (any type, any row count; the step and the all-fp32 mode): one CTA per (query, sequence, range of keys) with all heads:
// K and V tiles are read once for all heads, staged in shared memory by 16-byte loads; ranges are merged by mixed_attn_merge_kernel.
#include "common.cuh"
#include "mma_sync.cuh"
#include "../../include/evo_b200.h"
#include <math.h>
#include <algorithm>

using namespace evo;

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

template <typename T> struct Row16;      // 16 bytes of a row as floats
template <> struct Row16<float> {
  static constexpr int EV = 4;
  static __device__ __forceinline__ void load(const float* p, float* o) { const float4 u = *reinterpret_cast<const float4*>(p); o[0] = u.x; o[1] = u.y; o[2] = u.z; o[3] = u.w; }
};
template <> struct Row16<bf16> {
  static constexpr int EV = 8;
  static __device__ __forceinline__ void load(const bf16* p, float* o) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    o[0] = bf_lo(u.x); o[1] = bf_hi(u.x); o[2] = bf_lo(u.y); o[3] = bf_hi(u.y); o[4] = bf_lo(u.z); o[5] = bf_hi(u.z); o[6] = bf_lo(u.w); o[7] = bf_hi(u.w);
  }
};

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// first key that position i sees
__device__ __forceinline__ int64_t first_key(int64_t i, int64_t chunk) { return chunk > 0 ? i / chunk * chunk : 0; }
// entry (output head h, score head g) of the folded mixture
__device__ __forceinline__ float mix_entry(const evo_mixed_attn_params& p, int h, int g) {
  const float t = p.talk ? __bfloat162float(((const bf16*)p.talk)[(int64_t)h * p.H + g]) : (h == g ? 1.f : 0.f);
  return t * (p.temp ? __bfloat162float(((const bf16*)p.temp)[g]) : 1.f) * p.scale;
}
template <typename T>
__device__ __forceinline__ float head_gate(const evo_mixed_attn_params& p, int64_t row, int h) {
  return p.gate ? 1.f / (1.f + expf(-ldf((const T*)p.gate + row * p.gate_tok_stride + h))) : 1.f;
}

// ================================================================ one CTA per (query, sequence, key range), all heads
constexpr int SK = 32;       // keys per tile (one per lane)

struct SplitPlan { int threads, nacc, kt, nsplit; int64_t keys; size_t smem; };

template <typename T, int NACC, bool VEC>
__global__ void __launch_bounds__(512) mixed_attn_split_kernel(evo_mixed_attn_params p, int kt, int64_t keys_per_split, int nsplit, float* __restrict__ ws) {
  extern __shared__ __align__(16) float smem[];
  const int H = p.H, G = p.G, dk = p.dk, dv = p.dv, rep = H / G;
  constexpr int EV = Row16<T>::EV;
  const int kst = (G * dk + EV - 1) / EV * EV + EV, vst = (G * dv + EV - 1) / EV * EV + EV;      // row strides: 16 bytes more than a multiple of 16
  T* Kt = reinterpret_cast<T*>(smem);                       // [kt][kst]
  T* Vt = Kt + kt * kst;                                     // [kt][vst]
  float* Pr = reinterpret_cast<float*>(Vt + kt * vst);       // [H][36] softmax weights of the tile
  float* Qs = Pr + H * 36;                                   // [H*dk] (+ padding to 4)
  float* Ts = Qs + (H * dk + 3) / 4 * 4;                     // [H][H] mixture
  float* Sr = Ts + H * H;                                    // [H][33] raw scores
  float* ms = Sr + H * 33;                                   // [H] running maximum, sum, correction
  float* ls = ms + H;
  float* cr = ls + H;
  const int b = blockIdx.z, split = blockIdx.x;
  const int tid = threadIdx.x, nthr = blockDim.x, w = tid >> 5, lane = tid & 31, nw = nthr >> 5;
  const int64_t pos = p.pos_dev ? *p.pos_dev : p.q_pos0;
  const int64_t rel = blockIdx.y, i = pos + rel, row = (int64_t)b * p.Lq + rel;
  const int64_t lo = first_key(i, p.chunk);
  const int64_t s0 = lo + split * keys_per_split, s1 = min(i + 1, s0 + keys_per_split);
  if (s0 >= s1) return;                                      // no keys in this range: the merge does not look at it
  const T* q = (const T*)p.q + row * p.q_tok_stride;
  for (int e = tid; e < H * dk; e += nthr) Qs[e] = ldf(q + e);
  for (int e = tid; e < H * H; e += nthr) Ts[e] = mix_entry(p, e / H, e % H);
  for (int h = tid; h < H; h += nthr) { ms[h] = -INFINITY; ls[h] = 0.f; }
  const T* kb = (const T*)p.k + (int64_t)b * p.k_batch_stride;
  const T* vb = (const T*)p.v + (int64_t)b * p.v_batch_stride;
  float acc[NACC];
#pragma unroll
  for (int a = 0; a < NACC; ++a) acc[a] = 0.f;
  for (int64_t k0 = s0; k0 < s1; k0 += kt) {
    const int nk = (int)min((int64_t)kt, s1 - k0), nk4 = (nk + 3) / 4 * 4;
    __syncthreads();                                         // the previous tile is no longer read
    if (VEC) {
      const int kc = G * dk / EV, vc = G * dv / EV;
      for (int idx = tid; idx < nk * kc; idx += nthr) {
        const int r = idx / kc, c = idx % kc;
        *reinterpret_cast<uint4*>(Kt + r * kst + c * EV) = *reinterpret_cast<const uint4*>(kb + (k0 + r) * p.k_tok_stride + c * EV);
      }
      for (int idx = tid; idx < nk4 * vc; idx += nthr) {
        const int r = idx / vc, c = idx % vc;
        uint4 u = make_uint4(0u, 0u, 0u, 0u);
        if (r < nk) u = *reinterpret_cast<const uint4*>(vb + (k0 + r) * p.v_tok_stride + c * EV);
        *reinterpret_cast<uint4*>(Vt + r * vst + c * EV) = u;
      }
    } else {
      for (int idx = tid; idx < nk * G * dk; idx += nthr) { const int r = idx / (G * dk), c = idx % (G * dk); Kt[r * kst + c] = kb[(k0 + r) * p.k_tok_stride + c]; }
      for (int idx = tid; idx < nk4 * G * dv; idx += nthr) {
        const int r = idx / (G * dv), c = idx % (G * dv);
        if (r < nk) Vt[r * vst + c] = vb[(k0 + r) * p.v_tok_stride + c]; else stf(Vt + r * vst + c, 0.f);
      }
    }
    __syncthreads();
    // raw scores: a warp per head, a lane per key
    for (int g = w; g < H; g += nw) {
      if (lane < nk) {
        const T* krow = Kt + lane * kst + (g / rep) * dk;
        const float* qh = Qs + g * dk;
        float d = 0.f;
        if (VEC) {
#pragma unroll 4
          for (int e = 0; e < dk; e += EV) {
            float kv[EV];
            Row16<T>::load(krow + e, kv);
#pragma unroll
            for (int u = 0; u < EV; u += 4) {
              const float4 q4 = *reinterpret_cast<const float4*>(qh + e + u);
              d = fmaf(q4.x, kv[u], fmaf(q4.y, kv[u + 1], fmaf(q4.z, kv[u + 2], fmaf(q4.w, kv[u + 3], d))));
            }
          }
        } else {
          for (int e = 0; e < dk; ++e) d = fmaf(qh[e], ldf(krow + e), d);
        }
        Sr[g * 33 + lane] = d;
      }
    }
    __syncthreads();
    // mixture and softmax: a warp per output head
    for (int h = w; h < H; h += nw) {
      float s = 0.f;
      const float* th = Ts + h * H;
      if (lane < nk) for (int g = 0; g < H; ++g) s = fmaf(th[g], Sr[g * 33 + lane], s);
      const float mo = ms[h], mn = fmaxf(mo, warp_max(lane < nk ? s : -INFINITY));
      const float pr = lane < nk ? expf(s - mn) : 0.f, c = expf(mo - mn), sum = warp_sum(pr);
      Pr[h * 36 + lane] = pr;
      __syncwarp();
      if (lane == 0) { ms[h] = mn; ls[h] = ls[h] * c + sum; cr[h] = c; }
    }
    __syncthreads();
    // P.V: a thread owns output columns tid, tid + nthr, ..
#pragma unroll
    for (int a = 0; a < NACC; ++a) {
      const int col = tid + a * nthr;
      if (col < H * dv) {
        const int h = col / dv, c = col - h * dv;
        const T* vcol = Vt + (h / rep) * dv + c;
        const float* ph = Pr + h * 36;
        float o = acc[a] * cr[h];
        for (int r = 0; r < nk4; r += 4) {
          const float4 p4 = *reinterpret_cast<const float4*>(ph + r);
          o = fmaf(p4.x, ldf(vcol + r * vst), fmaf(p4.y, ldf(vcol + (r + 1) * vst), fmaf(p4.z, ldf(vcol + (r + 2) * vst), fmaf(p4.w, ldf(vcol + (r + 3) * vst), o))));
        }
        acc[a] = o;
      }
    }
  }
  if (nsplit == 1) {
    T* orow = (T*)p.out + row * p.ldo;
#pragma unroll
    for (int a = 0; a < NACC; ++a) {
      const int col = tid + a * nthr;
      if (col < H * dv) { const int h = col / dv; stf(orow + col, acc[a] / ls[h] * head_gate<T>(p, row, h)); }
    }
    for (int64_t c = (int64_t)H * dv + tid; c < p.ldo; c += nthr) stf(orow + c, 0.f);
    return;
  }
  float* part = ws + (row * nsplit + split) * (int64_t)(2 * H + H * dv);      // maxima, sums, accumulators
  for (int h = tid; h < H; h += nthr) { part[h] = ms[h]; part[H + h] = ls[h]; }
#pragma unroll
  for (int a = 0; a < NACC; ++a) {
    const int col = tid + a * nthr;
    if (col < H * dv) part[2 * H + col] = acc[a];
  }
}

// grid (head, query row): the ranges' partial softmax states of one head
template <typename T>
__global__ void __launch_bounds__(128) mixed_attn_merge_kernel(evo_mixed_attn_params p, int64_t keys_per_split, int nsplit, const float* __restrict__ ws) {
  const int H = p.H, dv = p.dv, h = blockIdx.x;
  const int64_t row = blockIdx.y, rel = row % p.Lq;
  const int64_t i = (p.pos_dev ? *p.pos_dev : p.q_pos0) + rel;
  const int64_t n = i - first_key(i, p.chunk) + 1;
  const int used = (int)min((int64_t)nsplit, (n + keys_per_split - 1) / keys_per_split);
  const int64_t stride = 2 * H + H * (int64_t)dv;
  const float* part = ws + row * nsplit * stride;
  float mx = -INFINITY;
  for (int s = 0; s < used; ++s) mx = fmaxf(mx, part[s * stride + h]);
  float l = 0.f;
  for (int s = 0; s < used; ++s) l = fmaf(part[s * stride + H + h], expf(part[s * stride + h] - mx), l);
  const float mul = head_gate<T>(p, row, h) / l;
  T* orow = (T*)p.out + row * p.ldo;
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < used; ++s) o = fmaf(part[s * stride + 2 * H + h * dv + c], expf(part[s * stride + h] - mx), o);
    stf(orow + h * dv + c, o * mul);
  }
  if (h == H - 1)
    for (int64_t c = (int64_t)H * dv + threadIdx.x; c < p.ldo; c += blockDim.x) stf(orow + c, 0.f);
}

// keys that one query can see at most in this call
inline int64_t key_span(const evo_mixed_attn_params* p) {
  const int64_t end = p->pos_dev ? std::max<int64_t>(p->max_keys, 1) : p->q_pos0 + p->Lq;
  return p->chunk > 0 ? std::min(p->chunk, end) : end;
}

inline SplitPlan split_plan(const evo_mixed_attn_params* p) {
  SplitPlan s = {};
  const int ev = p->dtype ? 4 : 8, esz = p->dtype ? 4 : 2;
  const int cols = p->H * p->dv;
  s.threads = cols > 256 * 16 ? 512 : 256;
  s.nacc = (cols + s.threads - 1) / s.threads;
  const size_t row = (size_t)((p->G * p->dk + ev - 1) / ev * ev + ev + (p->G * p->dv + ev - 1) / ev * ev + ev) * esz;
  const size_t fixed = sizeof(float) * ((size_t)p->H * 36 + (p->H * p->dk + 3) / 4 * 4 + (size_t)p->H * p->H + p->H * 33 + 3 * p->H);
  for (s.kt = SK; s.kt >= 4; s.kt >>= 1)
    if (fixed + s.kt * row <= 110 * 1024 || (s.kt == 4 && fixed + s.kt * row <= 227 * 1024)) break;
  if (s.kt < 4 || s.nacc > 32) { s.kt = 0; return s; }
  s.smem = fixed + s.kt * row;
  // enough ranges that about two CTAs per SM are at work, none shorter than 64 keys
  const int64_t span = key_span(p), rows = std::max<int64_t>((int64_t)p->B * p->Lq, 1);
  const int64_t want = std::max<int64_t>(1, (2 * device_sm_count() + rows - 1) / rows);
  s.keys = std::max<int64_t>(64, (span + want - 1) / want);
  s.keys = (s.keys + SK - 1) / SK * SK;
  s.nsplit = (int)((span + s.keys - 1) / s.keys);
  return s;
}
inline size_t split_workspace(const evo_mixed_attn_params* p, const SplitPlan& s) {
  return s.nsplit > 1 ? sizeof(float) * (size_t)p->B * p->Lq * s.nsplit * (2 * (size_t)p->H + (size_t)p->H * p->dv) : 0;
}

template <typename T, int NACC>
int launch_split(const evo_mixed_attn_params* p, const SplitPlan& s, float* ws, cudaStream_t st) {
  constexpr int EV = Row16<T>::EV;
  auto a16 = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool vec = p->dk % EV == 0 && p->dv % EV == 0 && p->k_tok_stride % EV == 0 && p->v_tok_stride % EV == 0 && p->k_batch_stride % EV == 0 &&
                   p->v_batch_stride % EV == 0 && a16(p->k) && a16(p->v);
  auto kern = vec ? mixed_attn_split_kernel<T, NACC, true> : mixed_attn_split_kernel<T, NACC, false>;
  if (s.smem > 48 * 1024) EVO_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s.smem));
  for (int64_t r0 = 0; r0 < p->Lq; r0 += 32768) {            // a grid's y extent is limited to 65535
    evo_mixed_attn_params c = *p;
    const int64_t n = std::min<int64_t>(32768, p->Lq - r0);
    EVO_REQUIRE(p->Lq <= 32768 || (p->B == 1 && !p->pos_dev && s.nsplit == 1), "evo_mixed_attn_fwd: more than 32768 query rows of several sequences");
    const int64_t esz = sizeof(T);
    c.Lq = n; c.q_pos0 += r0;
    c.q = (const char*)p->q + r0 * p->q_tok_stride * esz; c.out = (char*)p->out + r0 * p->ldo * esz;
    if (p->gate) c.gate = (const char*)p->gate + r0 * p->gate_tok_stride * esz;
    kern<<<dim3(s.nsplit, (unsigned)n, p->B), s.threads, s.smem, st>>>(c, s.kt, s.keys, s.nsplit, ws);
    int rc = check_launch("evo_mixed_attn_fwd");
    if (rc) return rc;
  }
  if (s.nsplit > 1) {
    mixed_attn_merge_kernel<T><<<dim3(p->H, (unsigned)(p->B * p->Lq)), 128, 0, st>>>(*p, s.keys, s.nsplit, ws);
    return check_launch("evo_mixed_attn_fwd");
  }
  return 0;
}
template <typename T>
int dispatch_split(const evo_mixed_attn_params* p, const SplitPlan& s, float* ws, cudaStream_t st) {
  if (s.nacc <= 2) return launch_split<T, 2>(p, s, ws, st);
  if (s.nacc <= 4) return launch_split<T, 4>(p, s, ws, st);
  if (s.nacc <= 8) return launch_split<T, 8>(p, s, ws, st);
  if (s.nacc <= 16) return launch_split<T, 16>(p, s, ws, st);
  return launch_split<T, 32>(p, s, ws, st);
}

// ================================================================ tensor-core prompt kernel
constexpr int QROWS = 16, MIXN = 16;      // queries per tile, most heads per CTA

__device__ __forceinline__ void copy16_async(void* dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ void store_remote(uint32_t local_addr, uint32_t cta, float2 v) {
  asm volatile("{\n\t.reg .b32 ra;\n\tmapa.shared::cluster.u32 ra, %0, %1;\n\tst.shared::cluster.v2.f32 [ra], {%2, %3};\n\t}\n"
               ::"r"(local_addr), "r"(cta), "f"(v.x), "f"(v.y) : "memory");
}

// mixed scores of output heads [h0, h0 + nh) over their own slots of the score buffer S [H][QROWS][KT + 8], from the scores of all H heads; Ts [H][MIXN]
template <int NO, int KT>
__device__ __forceinline__ void mix_places(float* __restrict__ Ss, const float* __restrict__ Ts, int H, int h0, int nh) {
  constexpr int SST = KT + 8, PLANE = QROWS * SST;
  const int tid = threadIdx.x, nthr = blockDim.x;
  if (nthr > QROWS * KT / 2) {
    for (int t = tid; t < QROWS * KT; t += nthr) {
      float* at = Ss + (t / KT) * SST + t % KT;
      float acc[NO];
#pragma unroll
      for (int h = 0; h < NO; ++h) acc[h] = 0.f;
#pragma unroll 4
      for (int g = 0; g < H; ++g) {
        const float s = at[g * PLANE];
        const float4* t4 = reinterpret_cast<const float4*>(Ts + g * MIXN);
#pragma unroll
        for (int u = 0; u < NO / 4; ++u) {
          const float4 m = t4[u];
          acc[4 * u] = fmaf(m.x, s, acc[4 * u]); acc[4 * u + 1] = fmaf(m.y, s, acc[4 * u + 1]);
          acc[4 * u + 2] = fmaf(m.z, s, acc[4 * u + 2]); acc[4 * u + 3] = fmaf(m.w, s, acc[4 * u + 3]);
        }
      }
#pragma unroll
      for (int h = 0; h < NO; ++h) if (h < nh) at[(h0 + h) * PLANE] = acc[h];
    }
    return;
  }
  for (int t = tid; t < QROWS * KT / 2; t += nthr) {
    float* at = Ss + (t / (KT / 2)) * SST + t % (KT / 2) * 2;
    float2 acc[NO];
#pragma unroll
    for (int h = 0; h < NO; ++h) acc[h] = make_float2(0.f, 0.f);
#pragma unroll 2
    for (int g = 0; g < H; ++g) {
      const float2 s = *reinterpret_cast<const float2*>(at + g * PLANE);
      const float4* t4 = reinterpret_cast<const float4*>(Ts + g * MIXN);
#pragma unroll
      for (int u = 0; u < NO / 4; ++u) {
        const float4 m = t4[u];
        acc[4 * u].x = fmaf(m.x, s.x, acc[4 * u].x); acc[4 * u].y = fmaf(m.x, s.y, acc[4 * u].y);
        acc[4 * u + 1].x = fmaf(m.y, s.x, acc[4 * u + 1].x); acc[4 * u + 1].y = fmaf(m.y, s.y, acc[4 * u + 1].y);
        acc[4 * u + 2].x = fmaf(m.z, s.x, acc[4 * u + 2].x); acc[4 * u + 2].y = fmaf(m.z, s.y, acc[4 * u + 2].y);
        acc[4 * u + 3].x = fmaf(m.w, s.x, acc[4 * u + 3].x); acc[4 * u + 3].y = fmaf(m.w, s.y, acc[4 * u + 3].y);
      }
    }
#pragma unroll
    for (int h = 0; h < NO; ++h) if (h < nh) *reinterpret_cast<float2*>(at + (h0 + h) * PLANE) = acc[h];
  }
}

struct MmaShape { int dkp, qst, kst, vst, hb, ncta, gv, vec; };      // padded head size, row strides, heads per CTA, CTAs per cluster, most key heads per CTA

template <int NV8, int KT, bool CLUSTER>
__global__ void __launch_bounds__(MIXN * 32) mixed_attn_mma_kernel(evo_mixed_attn_params p, MmaShape sh) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int SST = KT + 8, DVP = NV8 * 8;
  const int H = p.H, dk = p.dk, dv = p.dv, rep = H / p.G;
  const int rank = CLUSTER ? (int)(blockIdx.x % sh.ncta) : 0;
  const int h0 = rank * sh.hb, nh = min(sh.hb, H - h0);                // this CTA's heads [h0, h0 + nh)
  const int g0 = h0 / rep, ng = (h0 + nh - 1) / rep - g0 + 1;          // their key heads [g0, g0 + ng)
  bf16* Qs = reinterpret_cast<bf16*>(smem_raw);                        // [hb][16][qst]
  bf16* Ks = Qs + sh.hb * QROWS * sh.qst;                              // [KT][kst]
  bf16* Vs = Ks + KT * sh.kst;                                         // [KT][vst]
  float* Ss = reinterpret_cast<float*>(Vs + KT * sh.vst);              // [H][16][SST] scores of all heads; mixed scores in the own heads' slots
  float* Ts = Ss + H * QROWS * SST;                                    // [H][MIXN] mixture (base-2), row = score head
  const int tid = threadIdx.x, nthr = blockDim.x, w = tid >> 5, lane = tid & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int b = blockIdx.y;
  const int64_t pos = p.pos_dev ? *p.pos_dev : p.q_pos0;
  const int64_t rel0 = (int64_t)(CLUSTER ? blockIdx.x / sh.ncta : blockIdx.x) * QROWS;
  const int64_t i_lo = pos + rel0, i_hi = pos + min(p.Lq - 1, rel0 + QROWS - 1);
  const int64_t key_lo = first_key(i_lo, p.chunk), key_hi = i_hi + 1;
  const bf16 zero = __float2bfloat16_rn(0.f);

  for (int e = tid; e < H * MIXN; e += nthr) {
    const int g = e / MIXN, hl = e % MIXN;
    Ts[e] = hl < nh ? mix_entry(p, h0 + hl, g) * 1.4426950408889634f : 0.f;
  }
  const int cpq = sh.dkp / 8;
  if (sh.vec) {
    for (int idx = tid; idx < nh * QROWS * cpq; idx += nthr) {
      const int hl = idx / (QROWS * cpq), rest = idx % (QROWS * cpq), r = rest / cpq, e = rest % cpq * 8;
      uint4 u = make_uint4(0u, 0u, 0u, 0u);
      if (rel0 + r < p.Lq && e < dk) u = *reinterpret_cast<const uint4*>((const bf16*)p.q + ((int64_t)b * p.Lq + rel0 + r) * p.q_tok_stride + (int64_t)(h0 + hl) * dk + e);
      *reinterpret_cast<uint4*>(Qs + (hl * QROWS + r) * sh.qst + e) = u;
    }
  } else {
    for (int idx = tid; idx < nh * QROWS * sh.dkp; idx += nthr) {
      const int hl = idx / (QROWS * sh.dkp), rest = idx % (QROWS * sh.dkp), r = rest / sh.dkp, e = rest % sh.dkp;
      bf16 u = zero;
      if (rel0 + r < p.Lq && e < dk) u = ((const bf16*)p.q)[((int64_t)b * p.Lq + rel0 + r) * p.q_tok_stride + (int64_t)(h0 + hl) * dk + e];
      Qs[(hl * QROWS + r) * sh.qst + e] = u;
    }
  }
  const bf16* kb = (const bf16*)p.k + (int64_t)b * p.k_batch_stride + (int64_t)g0 * dk;
  const bf16* vb = (const bf16*)p.v + (int64_t)b * p.v_batch_stride + (int64_t)g0 * dv;
  const auto fetch_k = [&](int64_t k0) {
    const int nk = (int)max((int64_t)0, min((int64_t)KT, key_hi - k0));
    if (sh.vec) {
      const int c8 = ng * cpq;
      if (nk > 0)
        for (int idx = tid; idx < KT * c8; idx += nthr) {
          const int r = idx / c8, c = idx - r * c8, g = c / cpq, e = (c - g * cpq) * 8;
          const bool live = r < nk && e < dk;
          copy16_async(Ks + r * sh.kst + c * 8, live ? kb + (k0 + r) * p.k_tok_stride + g * dk + e : kb, live);
        }
      copies_commit();
    } else if (nk > 0) {
      for (int idx = tid; idx < KT * ng * sh.dkp; idx += nthr) {
        const int r = idx / (ng * sh.dkp), c = idx % (ng * sh.dkp), g = c / sh.dkp, e = c % sh.dkp;
        Ks[r * sh.kst + c] = (r < nk && e < dk) ? kb[(k0 + r) * p.k_tok_stride + g * dk + e] : zero;
      }
    }
  };
  const auto fetch_v = [&](int64_t k0) {
    const int nk = (int)max((int64_t)0, min((int64_t)KT, key_hi - k0));
    if (sh.vec) {
      const int c8 = ng * NV8;
      if (nk > 0)
        for (int idx = tid; idx < KT * c8; idx += nthr) {
          const int r = idx / c8, c = idx - r * c8, g = c / NV8, e = (c - g * NV8) * 8;
          const bool live = r < nk && e < dv;
          copy16_async(Vs + r * sh.vst + c * 8, live ? vb + (k0 + r) * p.v_tok_stride + g * dv + e : vb, live);
        }
      copies_commit();
    } else if (nk > 0) {
      for (int idx = tid; idx < KT * ng * DVP; idx += nthr) {
        const int r = idx / (ng * DVP), c = idx % (ng * DVP), g = c / DVP, e = c % DVP;
        Vs[r * sh.vst + c] = (r < nk && e < dv) ? vb[(k0 + r) * p.v_tok_stride + g * dv + e] : zero;
      }
    }
  };

  const bool on = w < nh;                                              // this warp has a head
  const int kvl = on ? (h0 + w) / rep - g0 : 0;                        // its key head within the CTA
  const int64_t i0 = i_lo + qr, i1 = i0 + 8;                           // positions of the thread's two rows
  const int64_t f0 = first_key(i0, p.chunk), f1 = first_key(i1, p.chunk);
  float O[NV8][4], mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NV8; ++n) O[n][0] = O[n][1] = O[n][2] = O[n][3] = 0.f;

  fetch_k(key_lo);
  if (CLUSTER) cluster_arrive();                                       // matches the wait in front of the first tile's remote writes
  for (int64_t k0 = key_lo; k0 < key_hi; k0 += KT) {
    const int nk = (int)min((int64_t)KT, key_hi - k0);
    copies_wait<0>();
    __syncthreads();                                                   // K has landed; every warp has left the previous tile's V
    fetch_v(k0);
    if (CLUSTER) cluster_wait();                                       // every CTA has mixed the previous tile: its foreign score slots are free
    if (on) {
      float S[KT / 8][4];
#pragma unroll
      for (int n = 0; n < KT / 8; ++n) S[n][0] = S[n][1] = S[n][2] = S[n][3] = 0.f;
      const bf16* Qw = Qs + w * QROWS * sh.qst;
#pragma unroll 4
      for (int ks = 0; ks < sh.dkp / 16; ++ks) {
        uint32_t a[4];                                                 // rows 0-7 / 8-15 x features 0-7 / 8-15
        ldmatrix_x4(a, Qw + ((lane & 7) + ((lane >> 3) & 1) * 8) * sh.qst + ks * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < KT / 8; n += 2) {
          uint32_t kf[4];
          ldmatrix_x4(kf, Ks + ((n + (lane >> 4)) * 8 + (lane & 7)) * sh.kst + kvl * sh.dkp + ks * 16 + ((lane >> 3) & 1) * 8);
          mma_bf16(S[n], a, kf[0], kf[1]);
          mma_bf16(S[n + 1], a, kf[2], kf[3]);
        }
      }
      float* dst = Ss + ((h0 + w) * QROWS + qr) * SST + qc;
#pragma unroll
      for (int n = 0; n < KT / 8; ++n) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(S[n][0], S[n][1]);
        *reinterpret_cast<float2*>(dst + 8 * SST + n * 8) = make_float2(S[n][2], S[n][3]);
      }
      if (CLUSTER) {
        const uint32_t addr = smem_u32(dst);
        for (int c = 1; c < sh.ncta; ++c) {
          const uint32_t to = (rank + c) % sh.ncta;
#pragma unroll
          for (int n = 0; n < KT / 8; ++n) {
            store_remote(addr + n * 32, to, make_float2(S[n][0], S[n][1]));
            store_remote(addr + (8 * SST + n * 8) * 4, to, make_float2(S[n][2], S[n][3]));
          }
        }
      }
    }
    if (CLUSTER) { cluster_arrive(); cluster_wait(); } else __syncthreads();      // all heads' scores are in; K is no longer read
    fetch_k(k0 + KT);
    // mixture: a thread takes one place, or two neighbouring ones when there are fewer threads than places
    if (nh > 8) mix_places<16, KT>(Ss, Ts, H, h0, nh); else mix_places<8, KT>(Ss, Ts, H, h0, nh);
    __syncwarp();
    if (CLUSTER) cluster_arrive();                                     // this CTA's foreign score slots may be written again
    if (sh.vec) copies_wait<1>();                                      // V has landed (the group behind it is the next K)
    __syncthreads();
    if (on) {
      const float* src = Ss + ((h0 + w) * QROWS + qr) * SST + qc;
      float P[KT / 8][4];
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int n = 0; n < KT / 8; ++n) {
        const float2 u0 = *reinterpret_cast<const float2*>(src + n * 8), u1 = *reinterpret_cast<const float2*>(src + 8 * SST + n * 8);
        P[n][0] = u0.x; P[n][1] = u0.y; P[n][2] = u1.x; P[n][3] = u1.y;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int col = n * 8 + qc + (c & 1);
          const int64_t kj = k0 + col;
          const bool vis = col < nk && (c < 2 ? (kj <= i0 && kj >= f0) : (kj <= i1 && kj >= f1));
          if (!vis) P[n][c] = -INFINITY;
          if (c < 2) mx0 = fmaxf(mx0, P[n][c]); else mx1 = fmaxf(mx1, P[n][c]);
        }
      }
      mx0 = quad_max(mx0); mx1 = quad_max(mx1);
      const float mn0 = fmaxf(mrun[0], mx0), mn1 = fmaxf(mrun[1], mx1);
      const float r0 = mn0 == -INFINITY ? 0.f : mn0, r1 = mn1 == -INFINITY ? 0.f : mn1;      // a row that has seen no key yet
      const float c0 = ex2(mrun[0] - r0), c1 = ex2(mrun[1] - r1);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int n = 0; n < KT / 8; ++n) {
        P[n][0] = ex2(P[n][0] - r0); P[n][1] = ex2(P[n][1] - r0); P[n][2] = ex2(P[n][2] - r1); P[n][3] = ex2(P[n][3] - r1);
        s0 += P[n][0] + P[n][1]; s1 += P[n][2] + P[n][3];
      }
      lrun[0] = lrun[0] * c0 + quad_sum(s0); lrun[1] = lrun[1] * c1 + quad_sum(s1);
      const bool moved = !__all_sync(0xffffffffu, mn0 == mrun[0] && mn1 == mrun[1]);
      mrun[0] = mn0; mrun[1] = mn1;
      if (moved) {
#pragma unroll
        for (int n = 0; n < NV8; ++n) { O[n][0] *= c0; O[n][1] *= c0; O[n][2] *= c1; O[n][3] *= c1; }
      }
#pragma unroll
      for (int kk = 0; kk < KT / 16; ++kk) {
        uint32_t ah[4], al[4];
        split_pack(P[2 * kk][0], P[2 * kk][1], ah[0], al[0]);
        split_pack(P[2 * kk][2], P[2 * kk][3], ah[1], al[1]);
        split_pack(P[2 * kk + 1][0], P[2 * kk + 1][1], ah[2], al[2]);
        split_pack(P[2 * kk + 1][2], P[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
        for (int n = 0; n < NV8; n += 2) {
          uint32_t bv[4];
          ldmatrix_x4_trans(bv, Vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * sh.vst + kvl * DVP + (n + (lane >> 4)) * 8);
          mma_bf16(O[n], ah, bv[0], bv[1]); mma_bf16(O[n], al, bv[0], bv[1]);
          mma_bf16(O[n + 1], ah, bv[2], bv[3]); mma_bf16(O[n + 1], al, bv[2], bv[3]);
        }
      }
    }
  }
  if (CLUSTER) cluster_wait();                                         // nobody leaves while another CTA may still address its shared memory
  copies_wait<0>();
  if (!on) return;
  const int h = h0 + w;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int64_t rel = rel0 + qr + 8 * r;
    if (rel >= p.Lq) continue;
    const int64_t row = (int64_t)b * p.Lq + rel;
    bf16* orow = (bf16*)p.out + row * p.ldo + (int64_t)h * dv;
    const float mul = head_gate<bf16>(p, row, h) / lrun[r];
#pragma unroll
    for (int n = 0; n < NV8; ++n) {
      const int ch = n * 8 + qc;
      if (ch < dv) orow[ch] = __float2bfloat16_rn(O[n][2 * r] * mul);
      if (ch + 1 < dv) orow[ch + 1] = __float2bfloat16_rn(O[n][2 * r + 1] * mul);
    }
    if (h == H - 1)
      for (int64_t c = (int64_t)H * dv + (lane & 3); c < p.ldo; c += 4) ((bf16*)p.out)[row * p.ldo + c] = zero;
  }
}

template <int NV8, int KT, bool CLUSTER>
int launch_mma(const evo_mixed_attn_params* p, const MmaShape& sh, size_t smem, cudaStream_t st) {
  auto kern = mixed_attn_mma_kernel<NV8, KT, CLUSTER>;
  if (smem > 48 * 1024) EVO_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const unsigned tiles = (unsigned)((p->Lq + QROWS - 1) / QROWS);
  if (!CLUSTER) {
    kern<<<dim3(tiles, p->B), sh.hb * 32, smem, st>>>(*p, sh);
    return check_launch("evo_mixed_attn_fwd");
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles * sh.ncta, p->B); cfg.blockDim = dim3(sh.hb * 32); cfg.dynamicSmemBytes = smem; cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = sh.ncta; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  EVO_CUDA(cudaLaunchKernelEx(&cfg, kern, *p, sh));
  return check_launch("evo_mixed_attn_fwd");
}
template <int NV8>
int launch_nv(const evo_mixed_attn_params* p, const MmaShape& sh, int kt, size_t smem, cudaStream_t st) {
  if (sh.ncta > 1) return kt == 32 ? launch_mma<NV8, 32, true>(p, sh, smem, st) : launch_mma<NV8, 16, true>(p, sh, smem, st);
  return kt == 32 ? launch_mma<NV8, 32, false>(p, sh, smem, st) : launch_mma<NV8, 16, false>(p, sh, smem, st);
}

// 1: shape not covered
int mixed_attn_mma(const evo_mixed_attn_params* p, cudaStream_t st) {
  if (p->dtype != 0 || p->Lq < 16 || p->dv > 128 || p->H > 8 * MIXN) return 1;
  MmaShape sh = {};
  const int rep = p->H / p->G, nv8 = (p->dv + 15) / 16 * 2;
  sh.ncta = (p->H + MIXN - 1) / MIXN;
  sh.hb = (p->H + sh.ncta - 1) / sh.ncta;
  if ((sh.ncta - 1) * sh.hb >= p->H) return 1;
  for (int c = 0; c < sh.ncta; ++c) sh.gv = std::max(sh.gv, (std::min((c + 1) * sh.hb, p->H) - 1) / rep - c * sh.hb / rep + 1);
  sh.dkp = (p->dk + 15) / 16 * 16;
  sh.qst = sh.dkp + 8; sh.kst = sh.gv * sh.dkp + 8; sh.vst = sh.gv * nv8 * 8 + 8;
  auto a16 = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  sh.vec = p->dk % 8 == 0 && p->dv % 8 == 0 && p->q_tok_stride % 8 == 0 && p->k_tok_stride % 8 == 0 && p->v_tok_stride % 8 == 0 && p->k_batch_stride % 8 == 0 &&
           p->v_batch_stride % 8 == 0 && a16(p->q) && a16(p->k) && a16(p->v);
  int kt = 32;
  size_t smem = 0;
  for (; kt >= 16; kt >>= 1) {
    smem = sizeof(bf16) * ((size_t)sh.hb * QROWS * sh.qst + (size_t)kt * (sh.kst + sh.vst)) + sizeof(float) * ((size_t)p->H * QROWS * (kt + 8) + (size_t)p->H * MIXN);
    if (smem <= 227 * 1024) break;
  }
  if (kt < 16) return 1;
  switch (nv8) {
    case 2: return launch_nv<2>(p, sh, kt, smem, st);
    case 4: return launch_nv<4>(p, sh, kt, smem, st);
    case 6: return launch_nv<6>(p, sh, kt, smem, st);
    case 8: return launch_nv<8>(p, sh, kt, smem, st);
    case 10: return launch_nv<10>(p, sh, kt, smem, st);
    case 12: return launch_nv<12>(p, sh, kt, smem, st);
    case 14: return launch_nv<14>(p, sh, kt, smem, st);
    default: return launch_nv<16>(p, sh, kt, smem, st);
  }
}

}  // namespace

extern "C" size_t evo_mixed_attn_workspace(const evo_mixed_attn_params* p) { return split_workspace(p, split_plan(p)); }

extern "C" int evo_mixed_attn_fwd(const evo_mixed_attn_params* p, void* workspace, size_t workspace_bytes, void* stream) {
  EVO_REQUIRE(p->q && p->k && p->v && p->out, "evo_mixed_attn_fwd: null argument");
  EVO_REQUIRE(p->B >= 0 && p->Lq >= 0 && p->H > 0 && p->G > 0 && p->H % p->G == 0 && p->dk > 0 && p->dv > 0 && p->chunk >= 0, "evo_mixed_attn_fwd: bad shape");
  EVO_REQUIRE(p->ldo >= (int64_t)p->H * p->dv, "evo_mixed_attn_fwd: ldo too small");
  if (p->B == 0 || p->Lq == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  if (!p->cuda_cores) {
    const int rc = mixed_attn_mma(p, st);
    if (rc <= 0) return rc;
  }
  const SplitPlan s = split_plan(p);
  EVO_REQUIRE(s.kt > 0, "evo_mixed_attn_fwd: heads too many or too wide (%d heads of %d / %d)", p->H, p->dk, p->dv);
  const size_t need = split_workspace(p, s);
  EVO_REQUIRE(need == 0 || (workspace && workspace_bytes >= need), "evo_mixed_attn_fwd: workspace too small (%zu < %zu)", workspace_bytes, need);
  EVO_REQUIRE(s.nsplit == 1 || (int64_t)p->B * p->Lq <= 65535, "evo_mixed_attn_fwd: too many query rows");
  return p->dtype ? dispatch_split<float>(p, s, (float*)workspace, st) : dispatch_split<bf16>(p, s, (float*)workspace, st);
}
