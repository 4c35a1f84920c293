// Softmax attention whose heads exchange scores before the softmax ("talking heads"), over a linear key/value cache:
//   a_g(i, j) = scale * temp_g * q_g(i) . k(j),   s_h(i, j) = sum_g talk[h, g] a_g(i, j),   p_h = softmax over the keys j that i sees
// with a chunked causal mask (i sees j <= i of its own chunk of positions, chunks counted from position 0; chunk 0: plain causal) and an
// optional sigmoid output gate of one number per head.  Scores, their mixture, softmax weights and sums are fp32 whatever the activation type.
// scale, temp and talk fold into one fp32 matrix, so the mixture costs H multiply-adds per score.
//
// mixed_attn_mma_kernel (bf16, 16 query rows or more): all heads of a query tile must be scored before any of them can run its softmax, so a
// cluster of ceil(H / 16) CTAs owns a tile of 16 queries and a CTA owns up to 16 heads, one per warp, as score heads AND as output heads.
// Per tile of keys: (1) every warp scores its head on the tensor cores (mma.sync m16n8k16, fp32 accumulation) and puts the fp32 scores into the
// score buffer of every CTA of the cluster (bulk copies between the shared memories); (2) the mixture is a product (output heads x score heads)
// . (score heads x places), also on the tensor cores: matrix and scores enter as leading part + remainder in tf32 (three products, about 21
// mantissa bits, fp32 sums), and a warp writes the mixed scores of its places over the CTA's own score slots; (3) every warp runs the online
// softmax of its head on mma fragments, accumulates P.V in registers -- each weight as bf16 high part + bf16 remainder -- and goes on to the
// scores of the next tile without a barrier in between.  K and V rows arrive as bulk copies on mbarriers.  The score slots of a CTA's own heads
// are written by nobody else, so the other CTAs may send the next tile's scores as soon as this one has mixed.
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
  int ph[NACC], pv[NACC];                                    // where a column's weights and values are; columns past the last one read the first head's
#pragma unroll
  for (int a = 0; a < NACC; ++a) {
    const int col = tid + a * nthr, h = col < H * dv ? col / dv : 0;
    acc[a] = 0.f; ph[a] = h * 36; pv[a] = h / rep * dv + (col < H * dv ? col - h * dv : 0);
  }
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
    for (int a = 0; a < NACC; ++a) acc[a] *= cr[ph[a] / 36];
#pragma unroll 1
    for (int r = 0; r < nk4; r += 4) {
      const T* vr = Vt + r * vst;
#pragma unroll
      for (int a = 0; a < NACC; ++a) {
        const float4 p4 = *reinterpret_cast<const float4*>(Pr + ph[a] + r);
        const T* v = vr + pv[a];
        acc[a] = fmaf(p4.x, ldf(v), fmaf(p4.y, ldf(v + vst), fmaf(p4.z, ldf(v + 2 * vst), fmaf(p4.w, ldf(v + 3 * vst), acc[a]))));
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
  s.threads = cols > 256 * 8 ? 512 : 256;
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
  if (s.nacc <= 4) return launch_split<T, 4>(p, s, ws, st);
  if (s.nacc <= 8) return launch_split<T, 8>(p, s, ws, st);
  return launch_split<T, 32>(p, s, ws, st);
}

// ================================================================ tensor-core prompt kernel
constexpr int QROWS = 16, MAXH = 16;      // queries per tile, most heads per CTA

// waits that ran out (a copy that never completed): the kernel goes on, its result is wrong, the host can ask
__device__ unsigned int mixed_attn_lost_waits;

__device__ __forceinline__ void wait_bounded(uint64_t* bar, uint32_t parity) {
  for (int n = 0; n < (1 << 20); ++n)
    if (mbar_try_wait(bar, parity)) return;
  atomicAdd(&mixed_attn_lost_waits, 1u);
}
// untiled bulk copy global -> own shared memory; 16-byte aligned addresses and size
__device__ __forceinline__ void copy_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
// bulk copy own shared memory -> the same place of another CTA's, completion on that CTA's barrier
__device__ __forceinline__ void send_bulk(const void* from, uint32_t bytes, uint64_t* bar, uint32_t cta) {
  asm volatile("{\n\t.reg .b32 ra, rb;\n\tmapa.shared::cluster.u32 ra, %0, %3;\n\tmapa.shared::cluster.u32 rb, %2, %3;\n\t"
               "cp.async.bulk.shared::cluster.shared::cta.mbarrier::complete_tx::bytes [ra], [%0], %1, [rb];\n\t}\n"
               ::"r"(smem_u32(from)), "r"(bytes), "r"(smem_u32(bar)), "r"(cta) : "memory");
}
// fp32 x fp32 through tf32 tensor-core products: the leading part (10 mantissa bits, what the tensor core reads) and the remainder
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// bf16 leading part and bf16 remainder of two weights (16 mantissa bits together), both cut off: byte permutes and a subtraction
__device__ __forceinline__ void cut_pack(float x, float y, uint32_t& hi, uint32_t& lo) {
  const uint32_t ux = __float_as_uint(x), uy = __float_as_uint(y);
  hi = __byte_perm(ux, uy, 0x7632);
  lo = __byte_perm(__float_as_uint(x - __uint_as_float(ux & 0xffff0000u)), __float_as_uint(y - __uint_as_float(uy & 0xffff0000u)), 0x7632);
}

// padded head size, row strides (elements), heads per CTA, CTAs per cluster, most key heads per CTA, score slots (heads padded to 8), stride of the mixture's rows, V buffers, score buffers
// sw: K and V arrive as 128-byte-swizzled tiles of 64 columns (tensor maps) instead of rows
struct MmaShape { int dkp, qst, kst, vst, hb, ncta, gv, hk, tst, nvb, nsb, vec, sw; };

template <int NV8, int KT, bool CLUSTER, bool SW>
__global__ void __launch_bounds__(MAXH * 32) mixed_attn_mma_kernel(evo_mixed_attn_params p, MmaShape sh, const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int SST = KT + 8, PLANE = QROWS * SST + (KT == 32 ? 8 : 24), DVP = NV8 * 8;  // PLANE % 32 == 8: the score heads of a fragment lie in different banks
  const int H = p.H, dk = p.dk, dv = p.dv, rep = H / p.G;
  const int rank = CLUSTER ? (int)(blockIdx.x % sh.ncta) : 0;
  const int h0 = rank * sh.hb, nh = min(sh.hb, H - h0);                // this CTA's heads [h0, h0 + nh)
  const int g0 = h0 / rep, ng = (h0 + nh - 1) / rep - g0 + 1;          // their key heads [g0, g0 + ng)
  // swizzled tiles want 1024-byte alignment
  bf16* Ks = reinterpret_cast<bf16*>(smem_raw + (SW ? (1024u - (smem_u32(smem_raw) & 1023u)) & 1023u : 0u));      // [KT][kst]        SW: [key heads * dk / 64][KT][64]
  bf16* Vs = Ks + KT * sh.kst;                                         // [nvb][KT][vst]   SW: [nvb][key heads * dv / 64][KT][64]
  bf16* Qs = Vs + sh.nvb * KT * sh.vst;                                // [hb][16][qst]
  float* Ts = reinterpret_cast<float*>(Qs + sh.hb * QROWS * sh.qst);   // [2][16][tst] mixture (base-2): leading parts, remainders; row = the CTA's output head
  float* Ss = Ts + 2 * MAXH * sh.tst;                                  // [nsb][hk][PLANE] scores of all heads; mixed scores in the own heads' slots
  uint64_t* bar = reinterpret_cast<uint64_t*>(Ss + sh.nsb * sh.hk * PLANE);      // K, the other CTAs' scores, the other CTAs have this one's, V buffers
  const int tid = threadIdx.x, nthr = blockDim.x, w = tid >> 5, lane = tid & 31, nw = nthr >> 5, qr = lane >> 2, qc = (lane & 3) * 2;
  const int b = blockIdx.y;
  const int64_t pos = p.pos_dev ? *p.pos_dev : p.q_pos0;
  const int64_t rel0 = (int64_t)(CLUSTER ? blockIdx.x / sh.ncta : blockIdx.x) * QROWS;
  const int64_t i_lo = pos + rel0, i_hi = pos + min(p.Lq - 1, rel0 + QROWS - 1);
  const int64_t key_lo = first_key(i_lo, p.chunk);
  const int nkeys = (int)(i_hi + 1 - key_lo);                          // keys that some row of the tile sees; key positions below are relative to key_lo
  const bf16 zero = __float2bfloat16_rn(0.f);
  const bf16* kb = (const bf16*)p.k + (int64_t)b * p.k_batch_stride + (int64_t)g0 * dk + key_lo * p.k_tok_stride;
  const bf16* vb = (const bf16*)p.v + (int64_t)b * p.v_batch_stride + (int64_t)g0 * dv + key_lo * p.v_tok_stride;

  // rows [k0, k0 + KT) of one operand: swizzled tiles, K by the first warps and V by the last ones, one or two each (a thread is held up
  // until its copy is under way); bulk copies (one per row, or per row and head where heads are padded) spread over the warps; or element by element
  const auto fetch = [&](const CUtensorMap* map, const bf16* src, int64_t stride, bf16* dst, int dst_stride, int d, int dpad, int k0, uint64_t* br) {
    const int n = min(KT, nkeys - k0);
    if (SW) {
      const int boxes = ng * d / 64;
      if (tid == 0) mbar_arrive_expect_tx(br, (uint32_t)(boxes * KT * 128));
      if (lane == 0)
        for (int x = br == bar ? w : nw - 1 - w; x < boxes; x += nw) tma_load_3d(dst + x * KT * 64, map, br, g0 * d + x * 64, (int)key_lo + k0, b);
    } else if (sh.vec) {
      const int pieces = d == dpad ? 1 : ng, width = d == dpad ? ng * d : d;
      if (tid == 0) mbar_arrive_expect_tx(br, (uint32_t)(n * pieces * width * 2));
      for (int idx = lane * nw + w; idx < n * pieces; idx += nthr) {
        const int r = pieces == 1 ? idx : idx / pieces, g = pieces == 1 ? 0 : idx - r * pieces;
        copy_bulk(dst + r * dst_stride + g * dpad, src + (int64_t)(k0 + r) * stride + g * d, (uint32_t)(width * 2), br);
      }
    } else {
      for (int idx = tid; idx < KT * ng * dpad; idx += nthr) {
        const int r = idx / (ng * dpad), c = idx % (ng * dpad), g = c / dpad, e = c % dpad;
        dst[r * dst_stride + c] = (r < n && e < d) ? src[(int64_t)(k0 + r) * stride + g * d + e] : zero;
      }
    }
  };

  if (tid == 0) {
    mbar_init(bar, 1); mbar_init(bar + 1, 1); mbar_init(bar + 2, CLUSTER ? sh.ncta - 1 : 1); mbar_init(bar + 3, 1); mbar_init(bar + 4, 1);
    fence_barrier_init();
  }
  if (sh.vec) {                                                        // padding columns, and rows that no copy has reached yet, hold zeros
    if (!SW) for (int e = tid; e < KT * (sh.kst + sh.nvb * sh.vst) / 8; e += nthr) reinterpret_cast<uint4*>(Ks)[e] = make_uint4(0u, 0u, 0u, 0u);
    fence_proxy_async_smem();
    __syncthreads();
    fetch(&kmap, kb, p.k_tok_stride, Ks, sh.kst, dk, sh.dkp, 0, bar);
    fetch(&vmap, vb, p.v_tok_stride, Vs, sh.vst, dv, DVP, 0, bar + 3);
  } else {
    fetch(&kmap, kb, p.k_tok_stride, Ks, sh.kst, dk, sh.dkp, 0, bar);
  }
  for (int e = tid; e < MAXH * sh.tst; e += nthr) {
    const int hl = e / sh.tst, g = e % sh.tst;
    uint32_t hi, lo;
    split_tf32((hl < nh && g < H) ? mix_entry(p, h0 + hl, g) * 1.4426950408889634f : 0.f, hi, lo);
    Ts[e] = __uint_as_float(hi); Ts[MAXH * sh.tst + e] = __uint_as_float(lo);
  }
  const int sbuf = sh.nsb == 2 ? sh.hk * PLANE : 0;
  for (int e = tid; e < (sh.hk - H) * PLANE; e += nthr) Ss[H * PLANE + e] = Ss[sbuf + H * PLANE + e] = 0.f;
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

  const bool on = w < nh;                                              // this warp has a head
  const int kvl = on ? (h0 + w) / rep - g0 : 0;                        // its key head within the CTA
  const int slot = (h0 + (on ? w : 0)) * PLANE;                        // its score slot within a buffer
  // visible keys of the thread's two rows, and of all rows, relative to key_lo
  const int v0 = (int)(i_lo + qr - key_lo), v1 = v0 + 8;
  const int f0 = (int)(first_key(i_lo + qr, p.chunk) - key_lo), f1 = (int)(first_key(i_lo + qr + 8, p.chunk) - key_lo);
  const int v_all = (int)(i_lo - key_lo), f_all = (int)(first_key(i_hi, p.chunk) - key_lo);
  const uint32_t qaddr = smem_u32(Qs + ((on ? w : 0) * QROWS + (lane & 15)) * sh.qst + (lane >> 4) * 8);
  // fragment addresses; swizzled: 16-byte piece c of row r lies at piece c ^ (r & 7) of its 128 bytes
  const int hi = (lane >> 3) & 1;
  const uint32_t kaddr = SW ? smem_u32(Ks) + kvl * (dk / 64) * (KT * 128) + ((lane >> 4) * 8 + (lane & 7)) * 128
                            : smem_u32(Ks + ((lane >> 4) * 8 + (lane & 7)) * sh.kst + kvl * sh.dkp + hi * 8);
  const uint32_t kx = (uint32_t)(hi ^ (lane & 7)) << 4;
  const uint32_t vaddr = SW ? smem_u32(Vs) + kvl * (DVP / 64) * (KT * 128) + (lane & 15) * 128 : smem_u32(Vs + (lane & 15) * sh.vst + kvl * DVP + (lane >> 4) * 8);
  const uint32_t vx = (uint32_t)((lane >> 4) ^ (lane & 7)) << 4;
  float O[NV8][4], mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NV8; ++n) O[n][0] = O[n][1] = O[n][2] = O[n][3] = 0.f;

  if (CLUSTER) cluster_arrive();                                       // matches the wait in front of the first tile's sends
  __syncthreads();                                                     // Q and the mixture are in place
  // iteration `next`: mixture, softmax and P.V of tile next - 1 (from the second on), then the scores of tile `next` (but for the last)
  for (int next = 0; ; ++next) {
    const int k0 = (next - 1) * KT;
    const bool more = k0 + KT < nkeys;
    float* const Sj = Ss + ((next - 1) & 1) * sbuf;                    // buffer of tile next - 1
    float* const Sn = Ss + (next & 1) * sbuf;                          // and of tile next
    const int vbuf = sh.nvb == 2 ? (next - 1) & 1 : 0;
    if (next > 0) {
      // K of this tile and V of the previous one are no longer read
      if (sh.vec) {
        if (sh.nvb == 1 && next > 1) fetch(&vmap, vb, p.v_tok_stride, Vs, sh.vst, dv, DVP, k0, bar + 3);
        if (more) fetch(&kmap, kb, p.k_tok_stride, Ks, sh.kst, dk, sh.dkp, k0 + KT, bar);
        if (sh.nvb == 2) { if (more) fetch(&vmap, vb, p.v_tok_stride, Vs + (next & 1) * KT * sh.vst, sh.vst, dv, DVP, k0 + KT, bar + 3 + (next & 1)); }
      } else {
        fetch(&vmap, vb, p.v_tok_stride, Vs, sh.vst, dv, DVP, k0, bar);
        if (more) fetch(&kmap, kb, p.k_tok_stride, Ks, sh.kst, dk, sh.dkp, k0 + KT, bar);
      }
      // ---- mixture: a warp takes every nw-th run of eight neighbouring places, four runs at a time
      for (int nt0 = w; nt0 < QROWS * KT / 8; nt0 += 4 * nw) {
        float D[4][4] = {};
        uint32_t s[4];
#pragma unroll
        for (uint32_t u = 0; u < 4; ++u) {
          const uint32_t nt = min((uint32_t)nt0 + u * nw, QROWS * KT / 8 - 1u);          // past the end: computed, not stored
          s[u] = nt / (KT / 8) * SST + nt % (KT / 8) * 8;
        }
        const float* ta = Ts + qr * sh.tst + (lane & 3);
        for (int ks = 0; ks < sh.hk / 8; ++ks) {
          uint32_t th[4], tl[4];
          const float* t = ta + ks * 8;
          const float* sk = Sj + (ks * 8 + (lane & 3)) * PLANE + qr;
          th[0] = __float_as_uint(t[0]); th[1] = __float_as_uint(t[8 * sh.tst]); th[2] = __float_as_uint(t[4]); th[3] = __float_as_uint(t[8 * sh.tst + 4]);
          t += MAXH * sh.tst;
          tl[0] = __float_as_uint(t[0]); tl[1] = __float_as_uint(t[8 * sh.tst]); tl[2] = __float_as_uint(t[4]); tl[3] = __float_as_uint(t[8 * sh.tst + 4]);
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            uint32_t b0h, b0l, b1h, b1l;
            split_tf32(sk[s[u]], b0h, b0l);
            split_tf32(sk[s[u] + 4 * PLANE], b1h, b1l);
            mma_tf32(D[u], tl, b0h, b1h);
            mma_tf32(D[u], th, b0l, b1l);
            mma_tf32(D[u], th, b0h, b1h);
          }
        }
        __syncwarp();
        if (CLUSTER) wait_bounded(bar + 2, (next - 1) & 1);              // the own slots have been read by everyone
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (nt0 + u * nw >= QROWS * KT / 8) break;
          float* dst = Sj + (h0 + qr) * PLANE + qc + s[u];
          if (qr < nh) *reinterpret_cast<float2*>(dst) = make_float2(D[u][0], D[u][1]);
          if (qr + 8 < nh) *reinterpret_cast<float2*>(dst + 8 * PLANE) = make_float2(D[u][2], D[u][3]);
        }
      }
      __syncwarp();
      if (CLUSTER) cluster_arrive();                                     // this CTA's foreign score slots may be written again
      if (sh.vec) wait_bounded(bar + 3 + vbuf, sh.nvb == 2 ? ((next - 1) >> 1) & 1 : (next - 1) & 1);
      __syncthreads();
    }
    // ---- with two score buffers half of the warps of every scheduler score the next tile first, so that the stages use different pipes at the same time
#pragma unroll 1
    for (int stage = 0; stage < 2; ++stage) {
      if (stage == (sh.nsb == 2 ? (w >> 2) & 1 : 0)) {
        // ---- softmax of the warp's head and P.V
        if (on && next > 0) {
          const float* src = Sj + slot + qr * SST + qc;
          const uint32_t va = vaddr + vbuf * (KT * sh.vst * 2);
          float P[KT / 8][4];
          float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
          for (int n = 0; n < KT / 8; ++n) {
            const float2 u0 = *reinterpret_cast<const float2*>(src + n * 8), u1 = *reinterpret_cast<const float2*>(src + 8 * SST + n * 8);
            P[n][0] = u0.x; P[n][1] = u0.y; P[n][2] = u1.x; P[n][3] = u1.y;
          }
          if (k0 + KT - 1 > v_all || k0 < f_all) {                         // some row does not see the whole tile
#pragma unroll
            for (int n = 0; n < KT / 8; ++n)
#pragma unroll
              for (int c = 0; c < 4; ++c) {
                const int kj = k0 + n * 8 + qc + (c & 1);
                if (c < 2 ? (kj > v0 || kj < f0) : (kj > v1 || kj < f1)) P[n][c] = -INFINITY;
              }
          }
#pragma unroll
          for (int n = 0; n < KT / 8; ++n) { mx0 = fmaxf(mx0, fmaxf(P[n][0], P[n][1])); mx1 = fmaxf(mx1, fmaxf(P[n][2], P[n][3])); }
          mx0 = quad_max(mx0); mx1 = quad_max(mx1);
          // the reference of the exponentials follows the maximum only when that has moved by more than 2^8: weights stay below 2^8, and the
          // accumulators are seldom rescaled
          if (!__all_sync(0xffffffffu, mx0 <= mrun[0] + 8.f && mx1 <= mrun[1] + 8.f)) {
            const float mn0 = fmaxf(mrun[0], mx0), mn1 = fmaxf(mrun[1], mx1);
            const float c0 = mn0 == -INFINITY ? 1.f : ex2(mrun[0] - mn0), c1 = mn1 == -INFINITY ? 1.f : ex2(mrun[1] - mn1);
            lrun[0] *= c0; lrun[1] *= c1;
            mrun[0] = mn0; mrun[1] = mn1;
#pragma unroll
            for (int n = 0; n < NV8; ++n) { O[n][0] *= c0; O[n][1] *= c0; O[n][2] *= c1; O[n][3] *= c1; }
          }
          const float r0 = mrun[0] == -INFINITY ? 0.f : mrun[0], r1 = mrun[1] == -INFINITY ? 0.f : mrun[1];      // a row that has seen no key yet
#pragma unroll
          for (int kk = 0; kk < KT / 16; ++kk) {
#pragma unroll
            for (int n = 2 * kk; n < 2 * kk + 2; ++n) {
              P[n][0] = ex2(P[n][0] - r0); P[n][1] = ex2(P[n][1] - r0); P[n][2] = ex2(P[n][2] - r1); P[n][3] = ex2(P[n][3] - r1);
              lrun[0] += P[n][0] + P[n][1]; lrun[1] += P[n][2] + P[n][3];              // this thread's share, folded over its quad at the end
            }
            uint32_t ah[4], al[4];
            cut_pack(P[2 * kk][0], P[2 * kk][1], ah[0], al[0]);
            cut_pack(P[2 * kk][2], P[2 * kk][3], ah[1], al[1]);
            cut_pack(P[2 * kk + 1][0], P[2 * kk + 1][1], ah[2], al[2]);
            cut_pack(P[2 * kk + 1][2], P[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
            for (int n = 0; n < NV8; n += 4) {                             // four independent sums between a high part's product and the remainder's
              uint32_t bv[2][4];
#pragma unroll
              for (int x = 0; x < 2; ++x)
                ldmatrix_x4_trans_at(bv[x], SW ? va + (n >> 3) * (KT * 128) + kk * 2048 + (vx ^ (((n + 2 * x) & 6) << 4)) : va + kk * 32 * sh.vst + (n + 2 * x) * 16);
#pragma unroll
              for (int x = 0; x < 2; ++x) { mma_bf16(O[n + 2 * x], ah, bv[x][0], bv[x][1]); mma_bf16(O[n + 2 * x + 1], ah, bv[x][2], bv[x][3]); }
#pragma unroll
              for (int x = 0; x < 2; ++x) { mma_bf16(O[n + 2 * x], al, bv[x][0], bv[x][1]); mma_bf16(O[n + 2 * x + 1], al, bv[x][2], bv[x][3]); }
            }
          }
        }
      } else if (more) {
        if (sh.vec) wait_bounded(bar, next & 1);
        // ---- scores of the warp's head -> own slot, and a copy to the other CTAs
        if (on) {
          float S[KT / 8][4];
#pragma unroll
          for (int n = 0; n < KT / 8; ++n) S[n][0] = S[n][1] = S[n][2] = S[n][3] = 0.f;
#pragma unroll 2
          for (int ks = 0; ks < sh.dkp / 16; ++ks) {
            uint32_t a[4];                                                 // rows 0-7 / 8-15 x features 0-7 / 8-15
            ldmatrix_x4_at(a, qaddr + ks * 32);
            uint32_t kf[KT / 16][4];
#pragma unroll
            for (int n = 0; n < KT / 16; ++n)
              ldmatrix_x4_at(kf[n], SW ? kaddr + (ks >> 2) * (KT * 128) + n * 2048 + (kx ^ ((ks & 3) << 5)) : kaddr + n * 32 * sh.kst + ks * 32);
#pragma unroll
            for (int n = 0; n < KT / 16; ++n) { mma_bf16(S[2 * n], a, kf[n][0], kf[n][1]); mma_bf16(S[2 * n + 1], a, kf[n][2], kf[n][3]); }
          }
          float* dst = Sn + slot + qr * SST + qc;
#pragma unroll
          for (int n = 0; n < KT / 8; ++n) {
            *reinterpret_cast<float2*>(dst + n * 8) = make_float2(S[n][0], S[n][1]);
            *reinterpret_cast<float2*>(dst + 8 * SST + n * 8) = make_float2(S[n][2], S[n][3]);
          }
        }
      }
    }
    if (!more) break;
    if (CLUSTER) {
      fence_proxy_async_smem();                                        // the slots are read by the copies below
      if (tid == 0) mbar_arrive_expect_tx(bar + 1, (uint32_t)((H - nh) * PLANE * 4));
      __syncwarp();
      cluster_wait();                                                  // every CTA has mixed the previous tile: its foreign slots may be written
      if (on)
        for (int c = 1 + lane; c < sh.ncta; c += 32) send_bulk(Sn + slot, PLANE * 4, bar + 1, (rank + c) % sh.ncta);
    }
    __syncthreads();                                                   // the CTA's own heads are scored; K is no longer read
    if (CLUSTER) {
      wait_bounded(bar + 1, next & 1);                                   // all other heads' scores have arrived: tell their senders
      if (w == 0)
        for (int c = 1 + lane; c < sh.ncta; c += 32) mbar_arrive_cluster(bar + 2, (rank + c) % sh.ncta);
    }
  }
  if (CLUSTER) { __syncwarp(); cluster_wait(); }                       // nobody leaves while another CTA may still address its shared memory
  if (!on) return;
  const int h = h0 + w;
  lrun[0] = quad_sum(lrun[0]); lrun[1] = quad_sum(lrun[1]);
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

template <int NV8, int KT, bool CLUSTER, bool SW>
int launch_sw(const evo_mixed_attn_params* p, const MmaShape& sh, size_t smem, cudaStream_t st) {
  CUtensorMap kmap = {}, vmap = {};
  if (SW) {
    const uint64_t rows = (uint64_t)(p->q_pos0 + p->Lq);
    const uint32_t box[3] = {64, KT, 1};
    const uint64_t kd[3] = {(uint64_t)p->G * p->dk, rows, (uint64_t)p->B}, ks[2] = {(uint64_t)p->k_tok_stride * 2, (uint64_t)p->k_batch_stride * 2};
    const uint64_t vd[3] = {(uint64_t)p->G * p->dv, rows, (uint64_t)p->B}, vs[2] = {(uint64_t)p->v_tok_stride * 2, (uint64_t)p->v_batch_stride * 2};
    int rc = make_tmap_nd_bf16(&kmap, p->k, 3, kd, ks, box, true);
    if (rc == 0) rc = make_tmap_nd_bf16(&vmap, p->v, 3, vd, vs, box, true);
    if (rc) return rc;
  }
  auto kern = mixed_attn_mma_kernel<NV8, KT, CLUSTER, SW>;
  if (smem > 48 * 1024) EVO_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const unsigned tiles = (unsigned)((p->Lq + QROWS - 1) / QROWS);
  if (!CLUSTER) {
    kern<<<dim3(tiles, p->B), sh.hb * 32, smem, st>>>(*p, sh, kmap, vmap);
    return check_launch("evo_mixed_attn_fwd");
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles * sh.ncta, p->B); cfg.blockDim = dim3(sh.hb * 32); cfg.dynamicSmemBytes = smem; cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = sh.ncta; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  EVO_CUDA(cudaLaunchKernelEx(&cfg, kern, *p, sh, kmap, vmap));
  return check_launch("evo_mixed_attn_fwd");
}

template <int NV8, int KT, bool CLUSTER>
int launch_mma(const evo_mixed_attn_params* p, const MmaShape& sh, size_t smem, cudaStream_t st) {
  if constexpr (NV8 >= 8)
    if (sh.sw) return launch_sw<NV8, KT, CLUSTER, true>(p, sh, smem, st);
  return launch_sw<NV8, KT, CLUSTER, false>(p, sh, smem, st);
}

// 1: shape not covered
int mixed_attn_mma(const evo_mixed_attn_params* p, cudaStream_t st) {
  if (p->dtype != 0 || p->Lq < 16 || p->dv > 128 || p->H > 8 * MAXH || p->q_pos0 + p->Lq >= ((int64_t)1 << 31)) return 1;
  MmaShape sh = {};
  const int rep = p->H / p->G, nv8 = p->dv <= 32 ? 4 : (p->dv <= 64 ? 8 : 16);
  sh.ncta = (p->H + MAXH - 1) / MAXH;
  sh.hb = (p->H + sh.ncta - 1) / sh.ncta;
  if ((sh.ncta - 1) * sh.hb >= p->H) return 1;
  for (int c = 0; c < sh.ncta; ++c) sh.gv = std::max(sh.gv, (std::min((c + 1) * sh.hb, p->H) - 1) / rep - c * sh.hb / rep + 1);
  sh.dkp = (p->dk + 15) / 16 * 16;
  sh.hk = (p->H + 7) / 8 * 8; sh.tst = sh.hk % 16 == 0 ? sh.hk + 4 : sh.hk + 12;
  sh.qst = sh.dkp + 8; sh.kst = sh.gv * sh.dkp + 8; sh.vst = sh.gv * nv8 * 8 + 8;
  auto a16 = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  sh.vec = p->dk % 8 == 0 && p->dv % 8 == 0 && p->q_tok_stride % 8 == 0 && p->k_tok_stride % 8 == 0 && p->v_tok_stride % 8 == 0 && p->k_batch_stride % 8 == 0 &&
           p->v_batch_stride % 8 == 0 && a16(p->q) && a16(p->k) && a16(p->v);
  // whole tiles of 64 columns and positions known to the host: tensor maps (no padded rows)
  sh.sw = sh.vec && p->dk % 64 == 0 && p->dv == nv8 * 8 && nv8 >= 8 && !p->pos_dev;
  if (sh.sw) { sh.kst -= 8; sh.vst -= 8; }
  int kt = 32;
  size_t smem = 0;
  const auto bytes = [&](int nvb, int nsb) {
    return sizeof(bf16) * ((size_t)sh.hb * QROWS * sh.qst + (size_t)kt * (sh.kst + nvb * sh.vst)) +
           sizeof(float) * ((size_t)2 * MAXH * sh.tst + (size_t)nsb * sh.hk * (QROWS * (kt + 8) + (kt == 32 ? 8 : 24))) + 48 + (sh.sw ? 1024 : 0);
  };
  for (; kt >= (nv8 == 16 ? 16 : 32); kt >>= 1)
    if ((smem = bytes(1, 1)) <= 227 * 1024) break;
  // a second score buffer (not across a cluster) and a second V buffer where they cost no resident CTA
  sh.nvb = sh.nsb = 1;
  const auto resident = [&](size_t b) { return std::min<size_t>(228 * 1024 / (b + 1024), 16 / sh.hb); };
  for (int pick = 3; pick > 0; --pick) {
    const int nvb = 1 + (pick & 1), nsb = 1 + (pick >> 1);
    if ((nvb == 2 && !sh.vec) || (nsb == 2 && sh.ncta > 1)) continue;
    const size_t b = bytes(nvb, nsb);
    if (b > 227 * 1024 || resident(b) < resident(smem)) continue;
    sh.nvb = nvb; sh.nsb = nsb; smem = b;
    break;
  }
  if (smem > 227 * 1024) return 1;
  const bool cl = sh.ncta > 1;
  if (nv8 == 4) return cl ? launch_mma<4, 32, true>(p, sh, smem, st) : launch_mma<4, 32, false>(p, sh, smem, st);
  if (nv8 == 8) return cl ? launch_mma<8, 32, true>(p, sh, smem, st) : launch_mma<8, 32, false>(p, sh, smem, st);
  if (kt == 32) return cl ? launch_mma<16, 32, true>(p, sh, smem, st) : launch_mma<16, 32, false>(p, sh, smem, st);
  return cl ? launch_mma<16, 16, true>(p, sh, smem, st) : launch_mma<16, 16, false>(p, sh, smem, st);
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

extern "C" int evo_mixed_attn_lost_waits(unsigned int* count) {
  EVO_REQUIRE(count, "evo_mixed_attn_lost_waits: null argument");
  EVO_CUDA(cudaMemcpyFromSymbol(count, mixed_attn_lost_waits, sizeof(unsigned int)));
  return 0;
}
