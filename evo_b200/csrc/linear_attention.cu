// Linear attention with one constant decay per head, S <- a S + k v^T, y = S^T q (evo_decay_scan_fwd), and the norm over all heads
// with a sigmoid gate that closes it (evo_norm_gate).
//
// Prompts (bf16) run block by block on the tensor cores.  For the 64 tokens of a block behind state S (rows i, j in the block):
//   y_i = a^{i+1} S^T q_i + sum_{j <= i} a^{i-j} (q_i . k_j) v_j,      S <- a^{64} S + sum_j a^{63-j} k_j v_j^T
// A CTA of four or eight warps owns one head, 64 or 128 value channels and a run of consecutive blocks (a part); the next block's rows are
// on their way (asynchronous 16-byte copies into a second buffer) while one is in work.  Warp w of a group of four computes the outputs of rows 16 w .. and keeps the state rows of its share of the key channels in fp32 registers; the state is a product's operand as a bf16 high
// part and a bf16 remainder in shared memory.  Whatever carries a decay -- the masked products q.k, the keys of the update -- is
// multiplied in fp32 and enters its product as high part + remainder too, so that products and sums keep 16 mantissa bits or more of
// every fp32 factor.  Powers of a come from one table per CTA.
// Where (sequences x heads x channel slices) leave SMs idle, a sequence is cut into several parts: decay_part_kernel sums every part but
// the last from an empty state (all in parallel), decay_carry_kernel folds the sums into the state at each part's start, and the output kernel
// runs the parts in parallel.  fp32 activations, short calls and head sizes above 128 go token by token (matrix_state.cu).
#include "common.cuh"
#include "mma_sync.cuh"
#include "../../include/evo_b200.h"
#include <math.h>
#include <stdint.h>
#include <algorithm>

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

// ---- block-wise linear attention
constexpr int BT = 64;                         // tokens per block; a group of four warps owns 64 value channels

struct BlockPlan { int parts; int64_t part_len; };          // parts 0: token by token
inline int column_groups(const evo_decay_scan_params* p) { return p->dv > 64 ? 2 : 1; }
inline BlockPlan block_plan(const evo_decay_scan_params* p) {
  if (p->recurrent || p->dtype != 0 || p->dk > 128 || p->L < 32) return {0, 0};
  const int vc = 64 * column_groups(p);
  const int64_t blocks = (p->L + BT - 1) / BT, ctas = (int64_t)p->B * p->H * ((p->dv + vc - 1) / vc), sms = device_sm_count();
  int64_t per = blocks;                                     // blocks per part
  if (p->part_len > 0) {
    per = (p->part_len + BT - 1) / BT;
  } else if (ctas < sms) {                                  // one CTA per SM: the number of parts whose rounds of CTAs walk the fewest blocks
    // (a part costs its blocks, half of that again for its sum -- the last one needs none -- and about a block to start)
    double best = 1e30;
    for (int64_t n = 1; n <= blocks / 4 || n == 1; ++n) {
      const int64_t len = (blocks + n - 1) / n, parts = (blocks + len - 1) / len;
      double cost = (double)((ctas * parts + sms - 1) / sms) * (len + 1);
      if (parts > 1) cost += 0.5 * (double)((ctas * (parts - 1) + sms - 1) / sms) * (len + 1) + 2.0;
      if (cost < best) { best = cost; per = len; }
      if (ctas * n > 4 * sms) break;
    }
  }
  per = std::min(per, blocks);
  return {(int)((blocks + per - 1) / per), per * BT};
}

__device__ __forceinline__ void copy16(void* dst, const void* src, bool live) {       // 16 bytes global -> shared, asynchronous; !live: zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ uint32_t act_pair(uint32_t u, int act, float s) {
  float a = bf_lo(u), b = bf_hi(u);
  if (act) { a = silu_fast(a); b = silu_fast(b); }
  return pack_bf16(a * s, b * s);
}
// `cols` columns (a multiple of 8) of BT rows -> shared memory; rows >= nt and columns >= live are zero
template <int NT>
__device__ __forceinline__ void fetch(bf16* dst, int st, const bf16* src, int64_t ld, int nt, int cols, int live, bool vec) {
  const int cpr = cols / 8;
  for (int idx = threadIdx.x; idx < BT * cpr; idx += NT) {
    const int r = idx / cpr, c = (idx % cpr) * 8;
    const bf16* g = src + r * ld + c;
    if (vec) {
      const bool on = r < nt && c < live;
      copy16(dst + r * st + c, on ? g : src, on);
    } else {
      uint32_t e[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) e[k] = r < nt && c + k < live ? (uint32_t)__bfloat16_as_ushort(g[k]) : 0u;
      *reinterpret_cast<uint4*>(dst + r * st + c) = make_uint4(e[0] | e[1] << 16, e[2] | e[3] << 16, e[4] | e[5] << 16, e[6] | e[7] << 16);
    }
  }
}
// silu and the factor on the pieces that this very thread fetched
template <int NT>
__device__ __forceinline__ void activate(bf16* dst, int st, int cols, int act, float s) {
  if (!act && s == 1.f) return;
  const int cpr = cols / 8;
  for (int idx = threadIdx.x; idx < BT * cpr; idx += NT) {
    uint4* at = reinterpret_cast<uint4*>(dst + (idx / cpr) * st + (idx % cpr) * 8);
    uint4 u = *at;
    u.x = act_pair(u.x, act, s); u.y = act_pair(u.y, act, s); u.z = act_pair(u.z, act, s); u.w = act_pair(u.w, act, s);
    *at = u;
  }
}
__device__ __forceinline__ void fetched() { asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory"); }

// S += (a^{nt-1-j} k_j)^T v_j over the block's tokens: MT tiles of 16 state rows per warp (tiles w, w + 4), 64 columns
template <int MT>
__device__ __forceinline__ void update_state(float (&S)[MT][8][4], const bf16* Ks, int kst, const bf16* Vs, int vst, const float* pw, int nt, int w, int lane, int mtiles) {
  const int qc = (lane & 3) * 2, mi = lane >> 3;
#pragma unroll
  for (int kk = 0; kk < BT / 16; ++kk) {
    uint32_t bv[8][2];
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      uint32_t f[4];
      ldmatrix_x4_trans(f, Vs + (kk * 16 + (mi & 1) * 8 + (lane & 7)) * vst + (n + (mi >> 1)) * 8);
      bv[n][0] = f[0]; bv[n][1] = f[1]; bv[n + 1][0] = f[2]; bv[n + 1][1] = f[3];
    }
    const int t0 = nt - 1 - (kk * 16 + qc);
    const float p0 = pw[max(t0, 0)], p1 = pw[max(t0 - 1, 0)], p8 = pw[max(t0 - 8, 0)], p9 = pw[max(t0 - 9, 0)];     // tokens past nt are zero rows
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (w + 4 * m < mtiles) {
        uint32_t f[4], ah[4], al[4];
        ldmatrix_x4_trans(f, Ks + (kk * 16 + (mi >> 1) * 8 + (lane & 7)) * kst + (w + 4 * m) * 16 + (mi & 1) * 8);
        split_pack(bf_lo(f[0]) * p0, bf_hi(f[0]) * p1, ah[0], al[0]);
        split_pack(bf_lo(f[1]) * p0, bf_hi(f[1]) * p1, ah[1], al[1]);
        split_pack(bf_lo(f[2]) * p8, bf_hi(f[2]) * p9, ah[2], al[2]);
        split_pack(bf_lo(f[3]) * p8, bf_hi(f[3]) * p9, ah[3], al[3]);
#pragma unroll
        for (int n = 0; n < 8; ++n) mma_bf16(S[m][n], ah, bv[n][0], bv[n][1]);       // products into the same sums stay eight apart
#pragma unroll
        for (int n = 0; n < 8; ++n) mma_bf16(S[m][n], al, bv[n][0], bv[n][1]);
      }
    }
  }
}

// what the two block kernels share: grid (value slices, heads, sequences x parts)
struct BlockArgs {
  evo_decay_scan_params p;
  float* part_state;            // (parts, B, H, dk, dv): a part's sum (decay_part_kernel), then the state at its start; NULL: one part
  int parts; int64_t part_len;
  int dkp, kst, vec;
};

template <int MT>
__device__ __forceinline__ void move_state(float (&S)[MT][8][4], float* g, int dk, int dv, int j0, int w, int lane, bool load) {
  const int qr = lane >> 2, qc = (lane & 3) * 2;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int row = (w + 4 * m) * 16 + qr + (c >> 1) * 8, col = j0 + n * 8 + qc + (c & 1);
        const bool live = row < dk && col < dv;
        if (load) S[m][n][c] = live ? g[(int64_t)row * dv + col] : 0.f;
        else if (live) g[(int64_t)row * dv + col] = S[m][n][c];
      }
}
template <int MT>
__device__ __forceinline__ void scale_state(float (&S)[MT][8][4], float s) {
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) S[m][n][c] *= s;
}

template <int MT, int CG>
__global__ void __launch_bounds__(128 * CG) decay_part_kernel(BlockArgs a) {
  constexpr int NT = 128 * CG, VC = 64 * CG, VST = VC + 8;     // row strides with 16 bytes of padding: conflict-free fragment reads
  extern __shared__ __align__(16) unsigned char smraw[];
  __shared__ float pw[BT + 1];
  const evo_decay_scan_params& p = a.p;
  const int kbuf = BT * a.kst, stage = kbuf + BT * VST;    // [2] x ([BT][kst] keys, [BT][VST] values)
  bf16* sm = reinterpret_cast<bf16*>(smraw);
  const int h = blockIdx.y, j0 = blockIdx.x * VC, part = blockIdx.z % (a.parts - 1), b = blockIdx.z / (a.parts - 1);
  const int w = (threadIdx.x >> 5) & 3, cg = threadIdx.x >> 7, lane = threadIdx.x & 31, mtiles = a.dkp / 16;
  if (threadIdx.x <= BT) pw[threadIdx.x] = powf(p.decay[h], (float)threadIdx.x);
  const int64_t t_begin = part * a.part_len, t_end = min(p.L, t_begin + a.part_len);
  const bf16* kg = (const bf16*)p.k + (int64_t)h * p.dk;
  const bf16* vg = (const bf16*)p.v + (int64_t)h * p.dv + j0;
  const auto load = [&](int64_t t0, bf16* at) {
    const int64_t row0 = (int64_t)b * p.L + t0;
    const int nt = (int)min((int64_t)BT, t_end - t0);
    fetch<NT>(at, a.kst, kg + row0 * p.ld, p.ld, nt, a.dkp, p.dk, a.vec);
    fetch<NT>(at + kbuf, VST, vg + row0 * p.ld, p.ld, nt, VC, p.dv - j0, a.vec);
  };
  float S[MT][8][4] = {};
  load(t_begin, sm);
  int cur = 0;
  for (int64_t t0 = t_begin; t0 < t_end; t0 += BT) {
    const int nt = (int)min((int64_t)BT, t_end - t0);
    bf16* Ks = sm + cur * stage;
    fetched();
    activate<NT>(Ks, a.kst, a.dkp, p.act, 1.f);
    activate<NT>(Ks + kbuf, VST, VC, p.act, 1.f);
    __syncthreads();                                       // the block is complete, and every warp has left the other buffer
    if (t0 + BT < t_end) load(t0 + BT, sm + (cur ^ 1) * stage);
    scale_state<MT>(S, pw[nt]);
    update_state<MT>(S, Ks, a.kst, Ks + kbuf + cg * 64, VST, pw, nt, w, lane, mtiles);
    cur ^= 1;
  }
  move_state<MT>(S, a.part_state + (((int64_t)part * p.B + b) * p.H + h) * p.dk * (int64_t)p.dv, p.dk, p.dv, j0 + cg * 64, w, lane, false);
}

// part sums -> states at the parts' starts (the last part's slot holds no sum)
__global__ void __launch_bounds__(256) decay_carry_kernel(BlockArgs a) {
  const evo_decay_scan_params& p = a.p;
  const int64_t per_head = (int64_t)p.dk * p.dv, n = (int64_t)p.B * p.H * per_head;
  const int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= n) return;
  const float step = powf(p.decay[(e / per_head) % p.H], (float)a.part_len);
  float S = (p.state && !p.zero_start) ? p.state[e] : 0.f;
  for (int s = 0; s < a.parts; ++s) {
    const float u = s + 1 < a.parts ? a.part_state[s * n + e] : 0.f;
    a.part_state[s * n + e] = S;
    S = fmaf(step, S, u);
  }
}

template <int MT, int CG>
__global__ void __launch_bounds__(128 * CG) decay_block_kernel(BlockArgs a) {
  constexpr int NT = 128 * CG, VC = 64 * CG, VST = VC + 8;
  extern __shared__ __align__(16) unsigned char smraw[];
  __shared__ float pw[BT + 1];
  const evo_decay_scan_params& p = a.p;
  const int kbuf = BT * a.kst, stage = 2 * kbuf + BT * VST;      // [2] x ([BT][kst] queries, [BT][kst] keys, [BT][VST] values)
  bf16* sm = reinterpret_cast<bf16*>(smraw);
  bf16* Sh = sm + 2 * stage;                               // [dkp][VST] state, high part
  bf16* Sl = Sh + a.dkp * VST;                             // [dkp][VST] state, remainder
  const int h = blockIdx.y, j0 = blockIdx.x * VC, part = blockIdx.z % a.parts, b = blockIdx.z / a.parts;
  const int w = (threadIdx.x >> 5) & 3, cg = threadIdx.x >> 7, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2, mi = lane >> 3, mtiles = a.dkp / 16;
  if (threadIdx.x <= BT) pw[threadIdx.x] = powf(p.decay[h], (float)threadIdx.x);
  const int64_t t_begin = part * a.part_len, t_end = min(p.L, t_begin + a.part_len);
  const bf16* qg = (const bf16*)p.q + (int64_t)h * p.dk;
  const bf16* kg = (const bf16*)p.k + (int64_t)h * p.dk;
  const bf16* vg = (const bf16*)p.v + (int64_t)h * p.dv + j0;
  const auto load = [&](int64_t t0, bf16* at) {
    const int64_t row0 = (int64_t)b * p.L + t0;
    const int nt = (int)min((int64_t)BT, t_end - t0);
    fetch<NT>(at, a.kst, qg + row0 * p.ld, p.ld, nt, a.dkp, p.dk, a.vec);
    fetch<NT>(at + kbuf, a.kst, kg + row0 * p.ld, p.ld, nt, a.dkp, p.dk, a.vec);
    fetch<NT>(at + 2 * kbuf, VST, vg + row0 * p.ld, p.ld, nt, VC, p.dv - j0, a.vec);
  };
  load(t_begin, sm);
  const int64_t head_state = ((int64_t)b * p.H + h) * p.dk * (int64_t)p.dv;
  float* start = a.parts > 1 ? a.part_state + (int64_t)part * p.B * p.H * p.dk * p.dv + head_state : (p.state && !p.zero_start ? p.state + head_state : nullptr);
  const int jc = j0 + cg * 64;                             // first of the warp's value channels
  float S[MT][8][4] = {};
  if (start) move_state<MT>(S, start, p.dk, p.dv, jc, w, lane, true);
  bool empty = start == nullptr || (a.parts > 1 && part == 0 && (!p.state || p.zero_start));
  const int r0 = w * 16 + qr, nmax = 2 * w + 2;            // the thread's first row; key tiles of 8 that the warp's rows see
  int cur = 0;
  for (int64_t t0 = t_begin; t0 < t_end; t0 += BT) {
    const int nt = (int)min((int64_t)BT, t_end - t0);
    const int64_t row0 = (int64_t)b * p.L + t0;
    bf16* Qs = sm + cur * stage;
    bf16* Ks = Qs + kbuf;
    bf16* Vs = Ks + kbuf;
    // the state behind the previous block is put in place (its readers are past the barrier below the read-outs) while the block's rows arrive
    if (!empty) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
        if (w + 4 * m < mtiles)
#pragma unroll
          for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              uint32_t hi, lo;
              split_pack(S[m][n][2 * half], S[m][n][2 * half + 1], hi, lo);
              const int at = ((w + 4 * m) * 16 + qr + 8 * half) * VST + cg * 64 + n * 8 + qc;
              *reinterpret_cast<uint32_t*>(Sh + at) = hi;
              *reinterpret_cast<uint32_t*>(Sl + at) = lo;
            }
    }
    fetched();
    activate<NT>(Qs, a.kst, a.dkp, p.act, p.q_scale);
    activate<NT>(Ks, a.kst, a.dkp, p.act, 1.f);
    activate<NT>(Vs, VST, VC, p.act, 1.f);
    __syncthreads();                                       // rows and state are complete, and every warp has left the other buffer
    if (t0 + BT < t_end) load(t0 + BT, sm + (cur ^ 1) * stage);
    // O = a^{i+1} Q S and P = Q K^T share the query fragments
    float O[8][4] = {}, P[BT / 8][4] = {};
    for (int ks = 0; ks < mtiles; ++ks) {
      uint32_t q[4];
      ldmatrix_x4(q, Qs + (w * 16 + (mi & 1) * 8 + (lane & 7)) * a.kst + ks * 16 + (mi >> 1) * 8);
      if (!empty) {
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          uint32_t f[4];
          ldmatrix_x4_trans(f, Sh + (ks * 16 + (mi & 1) * 8 + (lane & 7)) * VST + cg * 64 + (n + (mi >> 1)) * 8);
          mma_bf16(O[n], q, f[0], f[1]); mma_bf16(O[n + 1], q, f[2], f[3]);
        }
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          uint32_t f[4];
          ldmatrix_x4_trans(f, Sl + (ks * 16 + (mi & 1) * 8 + (lane & 7)) * VST + cg * 64 + (n + (mi >> 1)) * 8);
          mma_bf16(O[n], q, f[0], f[1]); mma_bf16(O[n + 1], q, f[2], f[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < BT / 8; n += 2)
        if (n < nmax) {
          uint32_t f[4];
          ldmatrix_x4(f, Ks + ((n + (mi >> 1)) * 8 + (lane & 7)) * a.kst + ks * 16 + (mi & 1) * 8);
          mma_bf16(P[n], q, f[0], f[1]); mma_bf16(P[n + 1], q, f[2], f[3]);
        }
    }
    __syncthreads();                                       // the state in shared memory is no longer read
    const float s0 = pw[r0 + 1], s1 = pw[r0 + 9];
#pragma unroll
    for (int n = 0; n < 8; ++n) { O[n][0] *= s0; O[n][1] *= s0; O[n][2] *= s1; O[n][3] *= s1; }
#pragma unroll
    for (int n = 0; n < BT / 8; ++n)
      if (n < nmax) {
        const int d = r0 - (n * 8 + qc);                   // distance of the row from the tile's column qc
        P[n][0] = d >= 0 ? P[n][0] * pw[d] : 0.f;
        P[n][1] = d >= 1 ? P[n][1] * pw[d - 1] : 0.f;
        P[n][2] = d >= -8 ? P[n][2] * pw[d + 8] : 0.f;
        P[n][3] = d >= -7 ? P[n][3] * pw[d + 7] : 0.f;
      }
#pragma unroll
    for (int kk = 0; kk < BT / 16; ++kk)
      if (2 * kk < nmax) {
        uint32_t ah[4], al[4];
        split_pack(P[2 * kk][0], P[2 * kk][1], ah[0], al[0]);
        split_pack(P[2 * kk][2], P[2 * kk][3], ah[1], al[1]);
        split_pack(P[2 * kk + 1][0], P[2 * kk + 1][1], ah[2], al[2]);
        split_pack(P[2 * kk + 1][2], P[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
        for (int n = 0; n < 8; n += 4) {
          uint32_t f[4], e[4];
          ldmatrix_x4_trans(f, Vs + (kk * 16 + (mi & 1) * 8 + (lane & 7)) * VST + cg * 64 + (n + (mi >> 1)) * 8);
          ldmatrix_x4_trans(e, Vs + (kk * 16 + (mi & 1) * 8 + (lane & 7)) * VST + cg * 64 + (n + 2 + (mi >> 1)) * 8);
          mma_bf16(O[n], ah, f[0], f[1]); mma_bf16(O[n + 1], ah, f[2], f[3]); mma_bf16(O[n + 2], ah, e[0], e[1]); mma_bf16(O[n + 3], ah, e[2], e[3]);
          mma_bf16(O[n], al, f[0], f[1]); mma_bf16(O[n + 1], al, f[2], f[3]); mma_bf16(O[n + 2], al, e[0], e[1]); mma_bf16(O[n + 3], al, e[2], e[3]);
        }
      }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = r0 + 8 * half;
      if (r < nt) {
        float* y = p.y + ((row0 + r) * p.H + h) * p.dv + jc;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          const int c = n * 8 + qc;
          if (jc + c + 1 < p.dv && p.dv % 2 == 0) *reinterpret_cast<float2*>(y + c) = make_float2(O[n][2 * half], O[n][2 * half + 1]);
          else {
            if (jc + c < p.dv) y[c] = O[n][2 * half];
            if (jc + c + 1 < p.dv) y[c + 1] = O[n][2 * half + 1];
          }
        }
      }
    }
    if (t0 + BT >= t_end && (!p.state || part + 1 < a.parts)) break;          // nobody reads the state behind this part's last block
    scale_state<MT>(S, pw[nt]);
    update_state<MT>(S, Ks, a.kst, Vs + cg * 64, VST, pw, nt, w, lane, mtiles);
    empty = false;
    cur ^= 1;
  }
  if (p.state && part + 1 == a.parts) move_state<MT>(S, p.state + head_state, p.dk, p.dv, jc, w, lane, false);
}

template <int MT, int CG>
int launch_blocks(const evo_decay_scan_params* p, const BlockPlan& pl, float* ws, cudaStream_t st) {
  BlockArgs a;
  a.p = *p; a.part_state = pl.parts > 1 ? ws : nullptr; a.parts = pl.parts; a.part_len = pl.part_len;
  a.dkp = (p->dk + 15) / 16 * 16; a.kst = a.dkp + 8;
  auto a16 = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  a.vec = p->dk % 8 == 0 && p->dv % 8 == 0 && p->ld % 8 == 0 && a16(p->q) && a16(p->k) && a16(p->v);
  constexpr int VC = 64 * CG, VST = VC + 8;
  const unsigned slices = (unsigned)((p->dv + VC - 1) / VC);
  if (pl.parts > 1) {
    const size_t smem = sizeof(bf16) * 2 * (size_t)BT * (a.kst + VST);
    auto kern = decay_part_kernel<MT, CG>;                 // (the table of powers comes on top of the dynamic shared memory)
    if (smem > 47 * 1024) EVO_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<dim3(slices, (unsigned)p->H, (unsigned)(p->B * (pl.parts - 1))), 128 * CG, smem, st>>>(a);
    int rc = check_launch("evo_decay_scan_fwd");
    if (rc) return rc;
    const int64_t n = (int64_t)p->B * p->H * p->dk * p->dv;
    decay_carry_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(a);
    rc = check_launch("evo_decay_scan_fwd");
    if (rc) return rc;
  }
  const size_t smem = sizeof(bf16) * (2 * (size_t)BT * (2 * a.kst + VST) + 2 * (size_t)a.dkp * VST);
  auto kern = decay_block_kernel<MT, CG>;
  if (smem > 47 * 1024) EVO_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<dim3(slices, (unsigned)p->H, (unsigned)(p->B * pl.parts)), 128 * CG, smem, st>>>(a);
  return check_launch("evo_decay_scan_fwd");
}

}  // namespace

extern "C" size_t evo_decay_scan_workspace(const evo_decay_scan_params* p) {
  const BlockPlan pl = block_plan(p);
  return pl.parts > 1 ? sizeof(float) * (size_t)pl.parts * p->B * p->H * p->dk * p->dv : 0;
}

extern "C" int evo_decay_scan_fwd(const evo_decay_scan_params* p, void* workspace, size_t workspace_bytes, void* stream) {
  EVO_REQUIRE(p->q && p->k && p->v && p->decay && p->y, "evo_decay_scan_fwd: null argument");
  EVO_REQUIRE(p->B >= 0 && p->L >= 0 && p->H > 0 && p->dk > 0 && p->dv > 0, "evo_decay_scan_fwd: bad shape");
  if (p->B == 0 || p->L == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const BlockPlan pl = block_plan(p);
  if (pl.parts == 0) return decay_scan_recurrent(p, st);
  EVO_REQUIRE(pl.parts == 1 || (workspace && workspace_bytes >= evo_decay_scan_workspace(p)), "evo_decay_scan_fwd: workspace too small");
  EVO_REQUIRE(p->H <= 65535 && (int64_t)p->B * pl.parts <= 65535, "evo_decay_scan_fwd: grid too large");
  float* ws = (float*)workspace;
  if (column_groups(p) == 2) return p->dk > 64 ? launch_blocks<2, 2>(p, pl, ws, st) : launch_blocks<1, 2>(p, pl, ws, st);
  return p->dk > 64 ? launch_blocks<2, 1>(p, pl, ws, st) : launch_blocks<1, 1>(p, pl, ws, st);
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
