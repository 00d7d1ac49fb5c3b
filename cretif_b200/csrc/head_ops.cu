// Per-head work around an attention whose projections are normed head by head: bias, RMS norm
// of every query and key head with a weight shared by the heads, rotation of the first
// rot_dim channels of a head, the write into the block cache -- one kernel, 32-bit inside --
// and the per-head output gate.  Also the small row kernels of ungated feed-forwards and
// capped logits.
//
// headnorm_rope_kv_append: proj rows [q (nh hd) | k (nkv hd) | v (nkv vd) | ...] in float32 or
// bfloat16.  Per token and head (a warp each; a head's channels stay in the lanes' registers):
//   x = proj + bias                                    (bias may be null)
//   q, k:  x <- x / sqrt(mean(x^2) + eps) * w          (w of hd numbers, null: no norm)
//   q, k:  channels (i, partner(i)) of the first rot_dim are rotated by pos * f_j
//          (pairing 0: partner i + rot_dim/2; 1: i ^ 1), cos/sin from a 32-bit table
//   q -> q_out, k -> key cache, v -> value cache at the token's position.
//
// projnorm_rope_kv_append: the same with the norms over the WHOLE query and the whole key projection
// (a weight per channel), from float32 rows, a CTA per token; v is multiplied by v_scale before it is
// stored, so that a factor on the attention's output costs nothing.  Instead of a bias the projected
// rows may pass a short causal convolution over time, channel by channel, before norms and rotation:
//   x_t[c] = sum_j conv_w[j, c] u_(t - taps + 1 + j)[c]
// with u from this step's rows or, where the window reaches back before the step, from the sequence's
// saved last taps - 1 inputs (conv_state, [C, taps - 1] per slot, zeros at a sequence's start).  A
// step of one token a sequence also brings the saved inputs up to date (save_inputs): each channel is
// read and replaced by one thread.  After any other step delta_conv_state (delta_rule.cu) does.
//
// Pooled entries (PooledKeys in common.cuh): pool_kv writes the means of the blocks of tokens that
// the step completes; a step of one token a sequence does it at the end of
// projnorm_rope_kv_append instead.
#include "api.h"
#include "common.cuh"

namespace cretif {

namespace {
constexpr int kHnWarps = 8;
constexpr int kHnMaxD = 512;

template <typename TI, typename T, int NCH>
__global__ void __launch_bounds__(kHnWarps * 32)
headnorm_rope_kv_append_kernel(const TI* __restrict__ proj, int ldp,
                               const float* __restrict__ bias, const float* __restrict__ wq,
                               const float* __restrict__ wk, float eps,
                               const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                               int pairing, int rot_dim, const int* __restrict__ tok_pos,
                               const int* __restrict__ tok_seq, const int* __restrict__ seq_slot,
                               int nh, int nkv, int hd, int vd, T* __restrict__ q_out, int ldq,
                               const int* __restrict__ table, int table_stride,
                               T* __restrict__ kc, T* __restrict__ vc, int bt, int write_cache,
                               unsigned int* __restrict__ fault) {
  __shared__ float normed[kHnWarps][kHnMaxD];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int units = nh + 2 * nkv;
  const int pos = tok_pos[t];
  const TI* row = proj + (size_t)t * ldp;
  int blk = -1;
  if (write_cache) {
    const int slot = seq_slot[tok_seq[t]];
    blk = table[(size_t)slot * table_stride + pos / bt];
    if (blk < 0 && threadIdx.x == 0 && blockIdx.y == 0) atomicOr(fault, kFaultBlockTable);
  }
  const int half = rot_dim >> 1;
  const float* c = cos_t + (size_t)pos * half;
  const float* s = sin_t + (size_t)pos * half;
  float* mine = normed[warp];
  for (int unit = blockIdx.y * kHnWarps + warp; unit < units; unit += gridDim.y * kHnWarps) {
    const bool is_q = unit < nh, is_k = !is_q && unit < nh + nkv;
    const int n = (is_q || is_k) ? hd : vd;
    const int c0 = is_q ? unit * hd : is_k ? nh * hd + (unit - nh) * hd
                                           : (nh + nkv) * hd + (unit - nh - nkv) * vd;
    T* dst;
    if (is_q) {
      dst = q_out + (size_t)t * ldq + (size_t)unit * hd;
    } else {
      if (blk < 0) continue;
      const int kvh = is_k ? unit - nh : unit - nh - nkv;
      dst = (is_k ? kc : vc) + (((size_t)blk * nkv + kvh) * bt + (pos % bt)) * n;
    }
    float val[NCH];
    float ss = 0.f;
#pragma unroll
    for (int m = 0; m < NCH; ++m) {
      const int i = lane + 32 * m;
      val[m] = i < n ? to_float(row[c0 + i]) + (bias ? bias[c0 + i] : 0.f) : 0.f;
      ss += val[m] * val[m];
    }
    const float* w = is_q ? wq : wk;
    if (!is_q && !is_k) {
#pragma unroll
      for (int m = 0; m < NCH; ++m) {
        const int i = lane + 32 * m;
        if (i < n) dst[i] = from_float<T>(val[m]);
      }
      continue;
    }
    if (w) {
      ss = warp_sum(ss);
      const float f = 1.0f / sqrtf(ss / (float)hd + eps);
#pragma unroll
      for (int m = 0; m < NCH; ++m) {
        const int i = lane + 32 * m;
        if (i < n) val[m] = val[m] * f * w[i];
      }
    }
    if (rot_dim > 0) {
      __syncwarp();
#pragma unroll
      for (int m = 0; m < NCH; ++m) {
        const int i = lane + 32 * m;
        if (i < n) mine[i] = val[m];
      }
      __syncwarp();
#pragma unroll
      for (int m = 0; m < NCH; ++m) {
        const int i = lane + 32 * m;
        if (i < rot_dim) {
          const bool first = pairing ? !(i & 1) : i < half;
          const int j = pairing ? i >> 1 : (first ? i : i - half);
          const int partner = pairing ? i ^ 1 : (first ? i + half : i - half);
          const float other = mine[partner];
          // the pair (u, v) becomes (u cos - v sin, v cos + u sin)
          val[m] = first ? val[m] * c[j] - other * s[j] : val[m] * c[j] + other * s[j];
        }
      }
    }
#pragma unroll
    for (int m = 0; m < NCH; ++m) {
      const int i = lane + 32 * m;
      if (i < n) dst[i] = from_float<T>(val[m]);
    }
  }
}

// The mean of `pool` consecutive cached rows' channel c, from position p0: a 32-bit sum in the order
// of the positions.
template <typename T>
__device__ __forceinline__ float pooled_mean(const T* cache, const int* tab, int p0, int pool, int nkv,
                                             int kvh, int bt, int n, int c) {
  float sum = 0.f;
#pragma unroll 4
  for (int r = 0; r < pool; ++r) {
    const int p = p0 + r, blk = max(tab[p / bt], 0);
    sum += to_float(cache[(((size_t)blk * nkv + kvh) * bt + p % bt) * n + c]);
  }
  return sum / (float)pool;
}

// A sequence's entry e (its block of tokens is complete) -> the entries' cache, by the threads
// tid, tid + threads, ... of a CTA, for the key/value heads kv0 .. kv1 - 1.
template <typename T>
__device__ __forceinline__ void write_entry(const T* kc, const T* vc, const int* tab, T* pk, T* pv,
                                            const int* ptab, int pool, int e, int nkv, int kv0,
                                            int kv1, int hd, int vd, int bt, int tid, int threads,
                                            unsigned int* fault) {
  const int blk = ptab[e / bt];
  if (blk < 0) {
    if (tid == 0) atomicOr(fault, kFaultBlockTable);
    return;
  }
  const int per = hd + vd;
  for (int idx = tid; idx < (kv1 - kv0) * per; idx += threads) {
    const int kvh = kv0 + idx / per, c = idx % per;
    const size_t row = ((size_t)blk * nkv + kvh) * bt + e % bt;
    if (c < hd)
      pk[row * hd + c] = from_float<T>(pooled_mean(kc, tab, e * pool, pool, nkv, kvh, bt, hd, c));
    else
      pv[row * vd + c - hd] =
          from_float<T>(pooled_mean(vc, tab, e * pool, pool, nkv, kvh, bt, vd, c - hd));
  }
}

// Eight channels a thread (bfloat16, head sizes multiples of eight): grid (entries, 1, B), the threads
// of a CTA take a token block's heads and channels in turn.
__global__ void __launch_bounds__(256)
pool_kv8_kernel(const __nv_bfloat16* kc, const __nv_bfloat16* vc, const int* __restrict__ table,
                int table_stride, __nv_bfloat16* pk, __nv_bfloat16* pv,
                const int* __restrict__ pool_table, int pool_stride, int pool,
                const int* __restrict__ cu_seqlens, const int* __restrict__ seq_start,
                const int* __restrict__ seq_slot, int nkv, int hd, int vd, int bt,
                unsigned int* __restrict__ fault) {
  const int b = blockIdx.z;
  const int start = seq_start[b], end = start + cu_seqlens[b + 1] - cu_seqlens[b];
  const int e = start / pool + blockIdx.x;
  if (e >= end / pool) return;
  const int slot = seq_slot[b];
  const int* tab = table + (size_t)slot * table_stride;
  const int blk = pool_table[(size_t)slot * pool_stride + e / bt];
  if (blk < 0) {
    if (threadIdx.x == 0) atomicOr(fault, kFaultBlockTable);
    return;
  }
  const int per = (hd + vd) >> 3;
  for (int idx = threadIdx.x; idx < nkv * per; idx += 256) {
    const int kvh = idx / per;
    int c = (idx - kvh * per) << 3;
    const bool is_k = c < hd;
    if (!is_k) c -= hd;
    const __nv_bfloat16* cache = is_k ? kc : vc;
    const int n = is_k ? hd : vd;
    float sum[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) sum[u] = 0.f;
#pragma unroll 8
    for (int r = 0; r < pool; ++r) {
      const int p = e * pool + r, from = max(tab[p / bt], 0);
      float x[8];
      load8(cache + (((size_t)from * nkv + kvh) * bt + p % bt) * n + c, x);
#pragma unroll
      for (int u = 0; u < 8; ++u) sum[u] += x[u];
    }
#pragma unroll
    for (int u = 0; u < 8; ++u) sum[u] /= (float)pool;
    store8((is_k ? pk : pv) + (((size_t)blk * nkv + kvh) * bt + e % bt) * n + c, sum);
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
pool_kv_kernel(const T* kc, const T* vc, const int* __restrict__ table, int table_stride, T* pk, T* pv,
               const int* __restrict__ pool_table, int pool_stride, int pool,
               const int* __restrict__ cu_seqlens, const int* __restrict__ seq_start,
               const int* __restrict__ seq_slot, int nkv, int hd, int vd, int bt,
               unsigned int* __restrict__ fault) {
  const int b = blockIdx.z, kvh = blockIdx.y;
  const int start = seq_start[b], end = start + cu_seqlens[b + 1] - cu_seqlens[b];
  const int e = start / pool + blockIdx.x;
  if (e >= end / pool) return;
  const int slot = seq_slot[b];
  write_entry(kc, vc, table + (size_t)slot * table_stride, pk, pv,
              pool_table + (size_t)slot * pool_stride, pool, e, nkv, kvh, kvh + 1, hd, vd, bt,
              (int)threadIdx.x, (int)blockDim.x, fault);
}

// VEC: four channels a thread (head size, rotated part and addresses allow it).  NT threads a token:
// a step of few tokens takes 1024, so that a row is one turn of loads, prompts take 256.
__device__ __forceinline__ float4 hn_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void hn_st4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void hn_st4(__nv_bfloat16* p, const float4& v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&lo);
  u.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}

// The convolution in front of the norms.  w [taps, C]: a tap's weights lie side by side.
struct ProjConv {
  const float* w;
  float* state;
  size_t stride;
  const int* seq_start;
  int taps, C, save;
};

// TAPS: 0 no convolution; 2, 3, 4: that many taps, four channels at a time; -1: any number, a channel
// at a time.
template <typename T, bool VEC, int NT, int TAPS>
__global__ void __launch_bounds__(NT)
projnorm_rope_kv_append_kernel(const float* __restrict__ proj, int ldp,
                               const float* __restrict__ bias, const float* __restrict__ wq,
                               const float* __restrict__ wk, float eps,
                               const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                               int pairing, int rot_dim, const int* __restrict__ tok_pos,
                               const int* __restrict__ tok_seq, const int* __restrict__ seq_slot,
                               int nh, int nkv, int hd, int vd, float v_scale,
                               T* __restrict__ q_out, int ldq, const int* __restrict__ table,
                               int table_stride, T* kc, T* vc, int bt, int write_cache, T* pk, T* pv,
                               const int* __restrict__ pool_table, int pool_stride, int pool,
                               const ProjConv conv, unsigned int* __restrict__ fault) {
  extern __shared__ __align__(16) float row_s[];       // q | k with the bias
  __shared__ float sums[NT / 32][2];
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = tok_pos[t];
  const float* row = proj + (size_t)t * ldp;
  const int nq = nh * hd, nk = nkv * hd, nqk = nq + nk;
  float ssq = 0.f, ssk = 0.f;
  int slot = 0, blk = -1;
  if (write_cache) {                  // (a chain of loads: asked for before the row)
    slot = seq_slot[tok_seq[t]];
    blk = table[(size_t)slot * table_stride + pos / bt];
    if (blk < 0 && tid == 0) atomicOr(fault, kFaultBlockTable);
  }
  const int half = rot_dim >> 1;
  const float* c = cos_t + (size_t)pos * half;
  const float* s = sin_t + (size_t)pos * half;
  int lt = 0, keep = 0;               // tokens of the sequence before t in the step; saved inputs
  float* st = nullptr;
  if (TAPS != 0) {
    const int b = tok_seq[t];
    lt = pos - conv.seq_start[b];
    keep = conv.taps - 1;
    if (keep) st = conv.state + (size_t)seq_slot[b] * conv.stride;
  }
  auto conv1 = [&](int ch) {
    float acc = 0.f;
    for (int j = 0; j <= keep; ++j) {
      const int back = keep - j;
      const float u = back <= lt ? row[ch - (ptrdiff_t)back * ldp]
                                 : st[(size_t)ch * keep + keep - (back - lt)];
      acc = fmaf(conv.w[(size_t)j * conv.C + ch], u, acc);
    }
    if (conv.save && keep) {
      float* mine = st + (size_t)ch * keep;
      for (int j = 0; j + 1 < keep; ++j) mine[j] = mine[j + 1];
      mine[keep - 1] = row[ch];
    }
    return acc;
  };
  auto conv4 = [&](int ch) {
    constexpr int K = TAPS > 1 ? TAPS - 1 : 1;
    float4 u[K + 1];
    float4 w[K + 1];
    u[K] = hn_ld4(row + ch);
#pragma unroll
    for (int j = 0; j <= K; ++j) w[j] = hn_ld4(conv.w + (size_t)j * conv.C + ch);
    float4 saved[K];                   // four channels' saved inputs: channel u's are 4 / K apart
    float* f = reinterpret_cast<float*>(saved);
    float* mine = st + (size_t)ch * K;
    if (lt < K) {
#pragma unroll
      for (int j = 0; j < K; ++j) saved[j] = hn_ld4(mine + 4 * j);
    }
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int back = K - j;
      if (back <= lt) {
        u[j] = hn_ld4(row + ch - (ptrdiff_t)back * ldp);
      } else {                         // entry K - (back - lt) = j + lt of every channel
        u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < K; ++i)
          if (i == j + lt) u[j] = make_float4(f[i], f[K + i], f[2 * K + i], f[3 * K + i]);
      }
    }
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j <= K; ++j) {
      acc.x = fmaf(w[j].x, u[j].x, acc.x);
      acc.y = fmaf(w[j].y, u[j].y, acc.y);
      acc.z = fmaf(w[j].z, u[j].z, acc.z);
      acc.w = fmaf(w[j].w, u[j].w, acc.w);
    }
    if (conv.save) {                   // (lt is zero)
      float g[4 * K];
#pragma unroll
      for (int i = 0; i < K; ++i) {
        const float4& v = u[i + 1];
        g[i] = v.x; g[K + i] = v.y; g[2 * K + i] = v.z; g[3 * K + i] = v.w;
      }
#pragma unroll
      for (int j = 0; j < K; ++j)
        hn_st4(mine + 4 * j, make_float4(g[4 * j], g[4 * j + 1], g[4 * j + 2], g[4 * j + 3]));
    }
    return acc;
  };
  if (VEC) {
    // (few tokens: what the thread's first turn reads after the row's sums are known)
    if (NT > 256 && 4 * tid < nkv * vd) {
      asm volatile("prefetch.global.L1 [%0];" ::"l"(row + nqk + 4 * tid));
      if (bias) asm volatile("prefetch.global.L1 [%0];" ::"l"(bias + nqk + 4 * tid));
    }
    if (NT > 256 && 4 * tid < nqk) {
      const int i = 4 * tid % hd;
      asm volatile("prefetch.global.L1 [%0];" ::"l"(4 * tid < nq ? wq + 4 * tid : wk + 4 * tid - nq));
      if (i < half) {
        asm volatile("prefetch.global.L1 [%0];" ::"l"(c + i));
        asm volatile("prefetch.global.L1 [%0];" ::"l"(s + i));
      }
    }
    for (int i = 4 * tid; i < nqk; i += 4 * NT) {
      float4 v = TAPS != 0 ? conv4(i) : hn_ld4(row + i);
      if (TAPS == 0 && bias) {
        const float4 b4 = *reinterpret_cast<const float4*>(bias + i);
        v.x += b4.x; v.y += b4.y; v.z += b4.z; v.w += b4.w;
      }
      *reinterpret_cast<float4*>(row_s + i) = v;
      const float s4 = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      if (i < nq) ssq += s4; else ssk += s4;
    }
  } else {
    for (int i = tid; i < nqk; i += NT) {
      const float v = TAPS != 0 ? conv1(i) : row[i] + (bias ? bias[i] : 0.f);
      row_s[i] = v;
      if (i < nq) ssq += v * v; else ssk += v * v;
    }
  }
  ssq = warp_sum(ssq);
  ssk = warp_sum(ssk);
  if (lane == 0) { sums[warp][0] = ssq; sums[warp][1] = ssk; }
  __syncthreads();
  ssq = warp_sum(lane < NT / 32 ? sums[lane][0] : 0.f);
  ssk = warp_sum(lane < NT / 32 ? sums[lane][1] : 0.f);
  const float fq = 1.0f / sqrtf(ssq / (float)nq + eps);
  const float fk = nk ? 1.0f / sqrtf(ssk / (float)nk + eps) : 0.f;
  const int n_write = write_cache && blk >= 0 ? nqk : nq;
  auto normed = [&](int idx) {
    return idx < nq ? row_s[idx] * fq * wq[idx] : row_s[idx] * fk * wk[idx - nq];
  };
  auto target = [&](int idx, int i) {              // where channel i of the head of column idx goes
    if (idx < nq) return q_out + (size_t)t * ldq + idx;
    const int kvh = (idx - nq) / hd;
    return kc + (((size_t)blk * nkv + kvh) * bt + pos % bt) * hd + i;
  };
  if (VEC) {
    auto normed4 = [&](int idx) {
      float4 x = hn_ld4(row_s + idx);
      const bool is_q = idx < nq;
      const float4 w = hn_ld4(is_q ? wq + idx : wk + idx - nq);
      const float f = is_q ? fq : fk;
      x.x *= f * w.x; x.y *= f * w.y; x.z *= f * w.z; x.w *= f * w.w;
      return x;
    };
    for (int idx = 4 * tid; idx < n_write; idx += 4 * NT) {
      const int i = idx % hd;
      float4 v = normed4(idx);
      if (i < rot_dim) {
        if (pairing) {
          const int j = i >> 1;
          const float2 c2 = *reinterpret_cast<const float2*>(c + j);
          const float2 s2 = *reinterpret_cast<const float2*>(s + j);
          v = make_float4(v.x * c2.x - v.y * s2.x, v.y * c2.x + v.x * s2.x,
                          v.z * c2.y - v.w * s2.y, v.w * c2.y + v.z * s2.y);
        } else {
          const bool first = i < half;
          const int j = first ? i : i - half;
          const float4 c4 = hn_ld4(c + j), o = normed4(idx + (first ? half : -half));
          float4 s4 = hn_ld4(s + j);
          if (first) s4 = make_float4(-s4.x, -s4.y, -s4.z, -s4.w);
          v = make_float4(v.x * c4.x + o.x * s4.x, v.y * c4.y + o.y * s4.y, v.z * c4.z + o.z * s4.z,
                          v.w * c4.w + o.w * s4.w);
        }
      }
      hn_st4(target(idx, i), v);
    }
  } else {
    for (int idx = tid; idx < n_write; idx += NT) {
      const int i = idx % hd;
      float v = normed(idx);
      if (i < rot_dim) {
        const bool first = pairing ? !(i & 1) : i < half;
        const int j = pairing ? i >> 1 : (first ? i : i - half);
        const int partner = pairing ? i ^ 1 : (first ? i + half : i - half);
        const float other = normed(idx - i + partner);
        v = first ? v * c[j] - other * s[j] : v * c[j] + other * s[j];
      }
      *target(idx, i) = from_float<T>(v);
    }
  }
  if (!write_cache || blk < 0) return;
  const bool vec_v = VEC && (vd & 3) == 0 && (reinterpret_cast<uintptr_t>(vc) & 15) == 0;
  for (int idx = 4 * tid; vec_v && idx < nkv * vd; idx += 4 * NT) {
    const int kvh = idx / vd, i = idx - kvh * vd;
    float4 v = TAPS != 0 ? conv4(nqk + idx) : hn_ld4(row + nqk + idx);
    if (TAPS == 0 && bias) {
      const float4 b4 = hn_ld4(bias + nqk + idx);
      v.x += b4.x; v.y += b4.y; v.z += b4.z; v.w += b4.w;
    }
    v.x *= v_scale; v.y *= v_scale; v.z *= v_scale; v.w *= v_scale;
    hn_st4(vc + (((size_t)blk * nkv + kvh) * bt + pos % bt) * vd + i, v);
  }
  for (int idx = tid; !vec_v && idx < nkv * vd; idx += NT) {
    const int kvh = idx / vd, i = idx - kvh * vd;
    const float v = TAPS != 0 ? conv1(nqk + idx) : row[nqk + idx] + (bias ? bias[nqk + idx] : 0.f);
    vc[(((size_t)blk * nkv + kvh) * bt + pos % bt) * vd + i] = from_float<T>(v * v_scale);
  }
  if (pool_table && (pos + 1) % pool == 0) {       // (one token a sequence: this one ends a block)
    __syncthreads();
    write_entry<T>(kc, vc, table + (size_t)slot * table_stride, pk, pv,
                   pool_table + (size_t)slot * pool_stride, pool, pos / pool, nkv, 0, nkv, hd, vd, bt,
                   tid, NT, fault);
  }
}

// o[t, h, :] *= sigmoid(g[t, h]): a gate per head from a float32 column of the projections.
template <typename T>
__global__ void gate_heads_kernel(T* __restrict__ o, int ldo, const float* __restrict__ g, int ldg,
                                  int nh, int vd, long long total) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const int w = nh * vd;
  const long long t = idx / w;
  const int col = (int)(idx - t * w);
  const float z = g[(size_t)t * ldg + col / vd];
  const float gate = 1.0f / (1.0f + expf(-z));
  T* p = o + (size_t)t * ldo + col;
  *p = from_float<T>(to_float(*p) * gate);
}

// The same for bfloat16 rows whose heads are whole groups of eight channels: a thread takes 16
// bytes of a head.
__global__ void gate_heads8_kernel(__nv_bfloat16* __restrict__ o, int ldo,
                                   const float* __restrict__ g, int ldg, int nh, int vd,
                                   long long groups) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= groups) return;
  const int per_row = nh * vd / 8;
  const long long t = idx / per_row;
  const int col = (int)(idx - t * per_row) * 8;
  const float z = g[(size_t)t * ldg + col / vd];
  const float gate = 1.0f / (1.0f + expf(-z));
  uint4* p = reinterpret_cast<uint4*>(o + (size_t)t * ldo + col);
  uint4 raw = *p;
  __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = __bfloat1622float2(h2[e]);
    h2[e] = __floats2bfloat162_rn(f.x * gate, f.y * gate);
  }
  *p = raw;
}

// A gate per channel (value size 1: every column is a head of its own), bfloat16 rows: a thread
// takes eight channels and their eight gates.
__global__ void gate_channels8_kernel(__nv_bfloat16* __restrict__ o, int ldo,
                                      const float* __restrict__ g, int ldg, int width,
                                      long long groups) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= groups) return;
  const int per_row = width / 8;
  const long long t = idx / per_row;
  const int col = (int)(idx - t * per_row) * 8;
  const float* gp = g + (size_t)t * ldg + col;
  uint4* p = reinterpret_cast<uint4*>(o + (size_t)t * ldo + col);
  uint4 raw = *p;
  __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = __bfloat1622float2(h2[e]);
    h2[e] = __floats2bfloat162_rn(f.x / (1.0f + expf(-gp[2 * e])),
                                  f.y / (1.0f + expf(-gp[2 * e + 1])));
  }
  *p = raw;
}

template <typename TI, typename TO>
__global__ void activation_kernel(const TI* __restrict__ in, int ldi, TO* __restrict__ out, int ldo,
                                  int width, long long total, int kind, const TO* __restrict__ mul,
                                  int mul_ld, int mul_rows, const int* __restrict__ mul_ids) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const long long t = idx / width;
  const int col = (int)(idx - t * width);
  float v = unary_activation(to_float(in[(size_t)t * ldi + col]), kind);
  if (mul) {                          // times the token's row of a table
    const int id = mul_ids[t];
    v *= id >= 0 && id < mul_rows ? to_float(mul[(size_t)id * mul_ld + col]) : 0.f;
  }
  out[(size_t)t * ldo + col] = from_float<TO>(v);
}

// z <- cap * tanh(z / cap), in place, 32-bit.
__global__ void softcap_kernel(float* __restrict__ z, long long total, float cap) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx < total) z[idx] = cap * tanhf(z[idx] / cap);
}

__global__ void scale_kernel(float* __restrict__ z, long long total, float factor) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx < total) z[idx] *= factor;
}

// h += alpha * y, 32-bit (y float32 or bfloat16).
template <typename TY>
__global__ void axpy_rows_kernel(float* __restrict__ h, const TY* __restrict__ y, float alpha,
                                 long long total) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx < total) h[idx] = fmaf(alpha, to_float(y[idx]), h[idx]);
}
}  // namespace
}  // namespace cretif

using namespace cretif;

extern "C" int cretif_headnorm_rope_kv_append(
    const void* proj, int ldp, int proj_dt, const float* bias, const float* wq, const float* wk,
    float eps, const float* cos_t, const float* sin_t, int pairing, int rot_dim,
    const int* tok_pos, const int* tok_seq, const int* seq_slot, int nh, int nkv, int hd, int vd,
    void* q_out, int ldq, int dt, const int* table, int table_stride, void* kc, void* vc, int bt,
    int write_cache, int T, unsigned int* fault, void* stream) {
  if (T <= 0) return kOk;
  if (nh <= 0 || nkv < 0 || hd <= 0 || hd > kHnMaxD || vd <= 0 || vd > kHnMaxD || ldq < nh * hd ||
      rot_dim < 0 || rot_dim > hd || (rot_dim & 1) || (!wq) != (!wk))
    return kBadArgument;
  if (rot_dim > 0 && (!cos_t || !sin_t)) return kBadArgument;
  if (write_cache && (bt <= 0 || !kc || !vc || !table || !tok_seq || !seq_slot)) return kBadArgument;
  if (ldp < (nh + nkv) * hd + nkv * vd) return kBadArgument;
  if (!write_cache) nkv = 0;                     // nothing to store: only the queries are made
  const int units = nh + 2 * nkv;
  dim3 grid(T, T >= 256 ? 1 : (units + kHnWarps - 1) / kHnWarps);
  if (grid.y > 65535) return kBadArgument;
  cudaStream_t st = (cudaStream_t)stream;
  const int widest = vd > hd ? vd : hd;
#define CRETIF_HN(TI, TT, NCH)                                                                   \
  headnorm_rope_kv_append_kernel<TI, TT, NCH><<<grid, kHnWarps * 32, 0, st>>>(                    \
      (const TI*)proj, ldp, bias, wq, wk, eps, cos_t, sin_t, pairing, rot_dim, tok_pos, tok_seq,  \
      seq_slot, nh, nkv, hd, vd, (TT*)q_out, ldq, table, table_stride, (TT*)kc, (TT*)vc, bt,      \
      write_cache, fault)
#define CRETIF_HN_T(TI, TT)                                                                      \
  do {                                                                                           \
    if (widest <= 64) CRETIF_HN(TI, TT, 2);                                                       \
    else if (widest <= 128) CRETIF_HN(TI, TT, 4);                                                 \
    else if (widest <= 256) CRETIF_HN(TI, TT, 8);                                                 \
    else CRETIF_HN(TI, TT, 16);                                                                   \
  } while (0)
  if (proj_dt == kF32 && dt == kF32)
    CRETIF_HN_T(float, float);
  else if (proj_dt == kF32 && dt == kBF16)
    CRETIF_HN_T(float, __nv_bfloat16);
  else if (proj_dt == kBF16 && dt == kBF16)
    CRETIF_HN_T(__nv_bfloat16, __nv_bfloat16);
  else
    return kBadDType;
#undef CRETIF_HN_T
#undef CRETIF_HN
  return launch_status();
}

// proj float32; pool_table non-null: the step brings one token a sequence and the entry of a block
// that a token completes is written here.
extern "C" int cretif_projnorm_rope_kv_append(
    const float* proj, int ldp, const float* bias, const float* wq, const float* wk, float eps,
    const float* cos_t, const float* sin_t, int pairing, int rot_dim, const int* tok_pos,
    const int* tok_seq, const int* seq_slot, int nh, int nkv, int hd, int vd, float v_scale,
    void* q_out, int ldq, int dt, const int* table, int table_stride, void* kc, void* vc, int bt,
    int write_cache, void* pool_k, void* pool_v, const int* pool_table, int pool_stride, int pool,
    const float* conv_w, int taps, float* conv_state, long long conv_stride, const int* seq_start,
    int save_inputs, int T, unsigned int* fault, void* stream) {
  if (T <= 0) return kOk;
  if (conv_w && (taps < 1 || bias || !write_cache || !seq_start ||
                 (taps > 1 && (!conv_state ||
                               conv_stride < (long long)((nh + nkv) * hd + nkv * vd) * (taps - 1)))))
    return kBadArgument;
  const ProjConv conv{conv_w, conv_state, (size_t)conv_stride, seq_start, taps,
                      (nh + nkv) * hd + nkv * vd, save_inputs};
  if (nh <= 0 || nkv < 0 || hd <= 0 || vd <= 0 || ldq < nh * hd || rot_dim < 0 || rot_dim > hd ||
      (rot_dim & 1) || !wq || (nkv && !wk) || ldp < (nh + nkv) * hd + nkv * vd)
    return kBadArgument;
  if (rot_dim > 0 && (!cos_t || !sin_t)) return kBadArgument;
  if (write_cache && (bt <= 0 || nkv <= 0 || !kc || !vc || !table || !tok_seq || !seq_slot))
    return kBadArgument;
  if (pool_table && (!write_cache || pool <= 0 || !pool_k || !pool_v)) return kBadArgument;
  const size_t smem = sizeof(float) * (size_t)(nh + nkv) * hd;
  if (smem > 200 * 1024) return kBadArgument;
  const bool vec = hd % 4 == 0 && ldp % 4 == 0 && ldq % 4 == 0 &&
                   (pairing ? rot_dim % 4 == 0 : rot_dim % 8 == 0) &&
                   (((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)q_out | (uintptr_t)kc | (uintptr_t)wq |
                     (uintptr_t)wk | (uintptr_t)cos_t | (uintptr_t)sin_t) & 15) == 0 &&
                   (!conv_w || (taps >= 2 && taps <= 4 && conv.C % 4 == 0 && vd % 4 == 0 &&
                                conv_stride % 4 == 0 &&
                                (((uintptr_t)conv_w | (uintptr_t)conv_state | (uintptr_t)vc) & 15) == 0));
  cudaStream_t st = (cudaStream_t)stream;
#define CRETIF_PN(TT, VEC, TAPS)                                                                  \
  do {                                                                                            \
    if (T < 64) CRETIF_PN_N(TT, VEC, 1024, TAPS);                                                 \
    else CRETIF_PN_N(TT, VEC, 256, TAPS);                                                         \
  } while (0)
#define CRETIF_PN_T(TT)                                                                           \
  do {                                                                                            \
    if (vec && !conv_w) CRETIF_PN(TT, true, 0);                                                   \
    else if (vec && taps == 2) CRETIF_PN(TT, true, 2);                                            \
    else if (vec && taps == 3) CRETIF_PN(TT, true, 3);                                            \
    else if (vec) CRETIF_PN(TT, true, 4);                                                         \
    else if (!conv_w) CRETIF_PN(TT, false, 0);                                                    \
    else CRETIF_PN(TT, false, -1);                                                                \
  } while (0)
#define CRETIF_PN_N(TT, VEC, NT, TAPS)                                                            \
  do {                                                                                            \
    if (smem > 40 * 1024) {                                                                       \
      cudaError_t err = cudaFuncSetAttribute(projnorm_rope_kv_append_kernel<TT, VEC, NT, TAPS>,   \
                                             cudaFuncAttributeMaxDynamicSharedMemorySize,         \
                                             (int)smem);                                          \
      if (err != cudaSuccess) return (int)err;                                                    \
    }                                                                                             \
    projnorm_rope_kv_append_kernel<TT, VEC, NT, TAPS><<<T, NT, smem, st>>>(                       \
        proj, ldp, bias, wq, wk, eps, cos_t, sin_t, pairing, rot_dim, tok_pos, tok_seq, seq_slot, \
        nh, nkv, hd, vd, v_scale, (TT*)q_out, ldq, table, table_stride, (TT*)kc, (TT*)vc, bt,     \
        write_cache, (TT*)pool_k, (TT*)pool_v, pool_table, pool_stride, pool, conv, fault);       \
  } while (0)
  if (dt == kF32) {
    CRETIF_PN_T(float);
  } else if (dt == kBF16) {
    CRETIF_PN_T(__nv_bfloat16);
  } else {
    return kBadDType;
  }
#undef CRETIF_PN_N
#undef CRETIF_PN_T
#undef CRETIF_PN
  return launch_status();
}

extern "C" int cretif_pool_kv(const void* kc, const void* vc, int dt, const int* table,
                              int table_stride, void* pool_k, void* pool_v, const int* pool_table,
                              int pool_stride, int pool, const int* cu_seqlens, const int* seq_start,
                              const int* seq_slot, int nkv, int hd, int vd, int bt, int B,
                              int max_new, unsigned int* fault, void* stream) {
  if (B <= 0 || max_new <= 0) return kOk;
  if (pool <= 0 || nkv <= 0 || nkv > 65535 || B > 65535 || hd <= 0 || vd <= 0 || bt <= 0 || !table ||
      !pool_table || !pool_k || !pool_v)
    return kBadArgument;
  // (n new tokens complete at most ceil(n / pool) blocks)
  const dim3 grid((max_new + pool - 1) / pool, nkv, B);
  cudaStream_t st = (cudaStream_t)stream;
  if (dt == kF32)
    pool_kv_kernel<float><<<grid, 128, 0, st>>>(
        (const float*)kc, (const float*)vc, table, table_stride, (float*)pool_k, (float*)pool_v,
        pool_table, pool_stride, pool, cu_seqlens, seq_start, seq_slot, nkv, hd, vd, bt, fault);
  else if (dt == kBF16 && hd % 8 == 0 && vd % 8 == 0 &&
           (((uintptr_t)kc | (uintptr_t)vc | (uintptr_t)pool_k | (uintptr_t)pool_v) & 15) == 0)
    pool_kv8_kernel<<<dim3(grid.x, 1, B), 256, 0, st>>>(
        (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, table, table_stride,
        (__nv_bfloat16*)pool_k, (__nv_bfloat16*)pool_v, pool_table, pool_stride, pool, cu_seqlens,
        seq_start, seq_slot, nkv, hd, vd, bt, fault);
  else if (dt == kBF16)
    pool_kv_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(
        (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, table, table_stride,
        (__nv_bfloat16*)pool_k, (__nv_bfloat16*)pool_v, pool_table, pool_stride, pool, cu_seqlens,
        seq_start, seq_slot, nkv, hd, vd, bt, fault);
  else
    return kBadDType;
  return launch_status();
}

extern "C" int cretif_scale(float* z, long long total, float factor, void* stream) {
  if (total <= 0) return kOk;
  scale_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(z, total, factor);
  return launch_status();
}

extern "C" int cretif_gate_heads(void* o, int ldo, int dt, const float* g, int ldg, int nh, int vd,
                                 int T, void* stream) {
  if (T <= 0) return kOk;
  if (nh <= 0 || vd <= 0 || ldo < nh * vd || ldg < nh) return kBadArgument;
  const long long total = (long long)T * nh * vd;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (dt == kF32)
    gate_heads_kernel<float><<<blocks, 256, 0, st>>>((float*)o, ldo, g, ldg, nh, vd, total);
  else if (dt == kBF16 && vd == 1 && nh % 8 == 0 && ldo % 8 == 0 && ((uintptr_t)o & 15) == 0)
    gate_channels8_kernel<<<(unsigned)((total / 8 + 255) / 256), 256, 0, st>>>(
        (__nv_bfloat16*)o, ldo, g, ldg, nh, total / 8);
  else if (dt == kBF16 && vd % 8 == 0 && ldo % 8 == 0 && ((uintptr_t)o & 15) == 0)
    gate_heads8_kernel<<<(unsigned)((total / 8 + 255) / 256), 256, 0, st>>>(
        (__nv_bfloat16*)o, ldo, g, ldg, nh, vd, total / 8);
  else if (dt == kBF16)
    gate_heads_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>((__nv_bfloat16*)o, ldo, g, ldg, nh,
                                                            vd, total);
  else
    return kBadDType;
  return launch_status();
}

extern "C" int cretif_activation(const void* in, int ldi, int in_dt, void* out, int ldo, int out_dt,
                                 int T, int width, int kind, const void* mul, int mul_ld,
                                 int mul_rows, const int* mul_ids, void* stream) {
  if (T <= 0 || width <= 0) return kOk;
  if (ldi < width || ldo < width || kind < 0 || kind >= kUnaryKinds) return kBadArgument;
  if (mul && (!mul_ids || mul_ld < width)) return kBadArgument;
  const long long total = (long long)T * width;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (in_dt == kF32 && out_dt == kF32)
    activation_kernel<float, float><<<blocks, 256, 0, st>>>((const float*)in, ldi, (float*)out,
                                                            ldo, width, total, kind,
                                                            (const float*)mul, mul_ld, mul_rows, mul_ids);
  else if (in_dt == kF32 && out_dt == kBF16)
    activation_kernel<float, __nv_bfloat16><<<blocks, 256, 0, st>>>(
        (const float*)in, ldi, (__nv_bfloat16*)out, ldo, width, total, kind,
        (const __nv_bfloat16*)mul, mul_ld, mul_rows, mul_ids);
  else if (in_dt == kBF16 && out_dt == kBF16)
    activation_kernel<__nv_bfloat16, __nv_bfloat16><<<blocks, 256, 0, st>>>(
        (const __nv_bfloat16*)in, ldi, (__nv_bfloat16*)out, ldo, width, total, kind,
        (const __nv_bfloat16*)mul, mul_ld, mul_rows, mul_ids);
  else
    return kBadDType;
  return launch_status();
}

extern "C" int cretif_softcap(float* z, long long total, float cap, void* stream) {
  if (total <= 0) return kOk;
  if (!(cap > 0.f)) return kBadArgument;
  softcap_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(z, total, cap);
  return launch_status();
}

extern "C" int cretif_axpy_rows(float* h, const void* y, int y_dt, float alpha, long long total,
                                void* stream) {
  if (total <= 0) return kOk;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (y_dt == kF32)
    axpy_rows_kernel<float><<<blocks, 256, 0, st>>>(h, (const float*)y, alpha, total);
  else if (y_dt == kBF16)
    axpy_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(h, (const __nv_bfloat16*)y, alpha,
                                                           total);
  else
    return kBadDType;
  return launch_status();
}
