// Causal grouped-query attention over the block cache, one CTA per (token, query head).
//
// The plain attention kernel: it serves prefill and decode alike, in 32-bit and in
// bfloat16 storage, for any number of heads and groups, any head size up to 512 (16-byte
// loads where it is a multiple of 8), a value size of its own, an optional sliding window, an
// optional per-head sink in the softmax's denominator and an optional learned bias by distance
// (below), and it is the kernel the faster ones are checked against.  Maths as in the reference: s = (q·k)·scale with the scale applied after the
// dot (src/attention.cu:690-692), keys after the query's position are masked (:60-77),
// softmax with running maximum and sum in 32-bit as in the reference's decode kernel
// (:451-493), query head h reads key/value head h / (heads / kv_heads) (:421-422).
// The CTA's eight warps take the keys in blocks of 32 in turn (warp w: blocks w, w + 8, ...),
// each with its own running maximum, sum and output, and warp 0 folds the eight results
// together in the order of the warps: a decode step, whose one query per head would otherwise
// be one warp walking thousands of keys with every load's latency exposed, is eight chains
// of an eighth the length.  A (token, head) is always reduced in the same order, so its
// output does not depend on what else is in the batch or on how the tokens were cut into
// steps.
//
// Bias by distance: a table bias[rows, heads] and ascending edges[rows] (edges[0] = 0); a key
// n = pos - key positions back adds bias[r, h] to its scaled score, where r is the last row
// with edges[r] <= n.  The host lays the edges out (a row per distance, then rows spaced by the
// logarithm, or anything else that is monotone); the kernel only searches them.
//
// Slope by distance: slope[heads]; a key n positions back has slope[h] * n taken off its scaled
// score.  The mask is first_visible_key(pos, window): every key, a sliding window, or the
// query's own chunk of positions.
//
// Pooled entries (PooledKeys, common.cuh): the entries that a query sees are walked like keys, after
// the tokens and in the same softmax; bias and slope are the tokens' only.
#include <type_traits>

#include "api.h"
#include "common.cuh"

namespace cretif {

constexpr int kWarps = 8;
constexpr int kMaxHd = 512;
constexpr int kMaxBiasRows = 1024;

template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
attn_simt_kernel(const T* __restrict__ q, int ldq, T* __restrict__ out, int ldo,
                 const T* __restrict__ kc, const T* __restrict__ vc,
                 const int* __restrict__ table, int table_stride,
                 const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                 const int* __restrict__ seq_slot, int nh, int nkv, int hd, float scale,
                 int window, int bt, int T_tokens, const float* __restrict__ sink, int vd,
                 const float* __restrict__ bias, const int* __restrict__ bias_edges,
                 int bias_rows, const float* __restrict__ slope, const PooledKeys pooled) {
  __shared__ float qs[kMaxHd];
  __shared__ float bias_s[kMaxBiasRows];
  __shared__ int edge_s[kMaxBiasRows];
  __shared__ float part_acc[kWarps][kMaxHd];
  __shared__ float part_m[kWarps], part_l[kWarps];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = blockIdx.x;
  const int t = (int)(item / nh), h = (int)(item - (long long)t * nh);
  const int kvh = h / (nh / nkv);
  const int pos = tok_pos[t];
  const int slot = seq_slot[tok_seq[t]];
  const int* tab = table + (size_t)slot * table_stride;
  const int first = first_visible_key(pos, window);
  const float tilt = slope ? slope[h] : 0.f;

  const T* qrow = q + (size_t)t * ldq + (size_t)h * hd;
  for (int d = threadIdx.x; d < hd; d += kWarps * 32) qs[d] = to_float(qrow[d]);
  if (bias)
    for (int r = threadIdx.x; r < bias_rows; r += kWarps * 32) {
      bias_s[r] = bias[(size_t)r * nh + h];
      edge_s[r] = bias_edges[r];
    }
  __syncthreads();

  float m = -INFINITY, l = 0.f;
  float acc[kMaxHd / 32];
#pragma unroll
  for (int i = 0; i < kMaxHd / 32; ++i) acc[i] = 0.f;

  // Keys lo .. hi of one block cache join the softmax.  TOKENS: the sequence's own keys (a bias or
  // slope by distance applies), else its pooled entries.
  auto walk = [&](auto tokens, int lo, int hi, const T* kbase, const T* vbase, const int* tbl) {
    constexpr bool TOKENS = decltype(tokens)::value;
    for (int base = lo + 32 * warp; base <= hi; base += 32 * kWarps) {
      const int key = base + lane;
      bool valid = key <= hi;
      float s = -INFINITY;
      unsigned long long row = 0;
      const int blk = valid ? tbl[key / bt] : -1;
      valid = blk >= 0;                 // a position without a block counts as masked
      if (valid) {
        row = ((unsigned long long)blk * nkv + kvh) * bt + (key % bt);
        const T* kp = kbase + row * hd;
        float dot = 0.f;
        if ((hd & 7) == 0) {
#pragma unroll 4
          for (int d = 0; d < hd; d += 8) {
            float kv[8];
            load8(kp + d, kv);
#pragma unroll
            for (int e = 0; e < 8; ++e) dot = fmaf(qs[d + e], kv[e], dot);
          }
        } else {                        // a head size that is no multiple of 8: element by element
          for (int d = 0; d < hd; ++d) dot = fmaf(qs[d], to_float(kp[d]), dot);
        }
        s = dot * scale;
        if (TOKENS && slope) s -= tilt * (float)(pos - key);
        if (TOKENS && bias) {
          // the last row whose edge is at or below the distance
          const int n = pos - key;
          int lo = 0, hi = bias_rows - 1;
          while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (edge_s[mid] <= n) lo = mid; else hi = mid - 1;
          }
          s += bias_s[lo];
        }
      }
      const float m_new = fmaxf(m, warp_max(s));
      const float p = valid ? expf(s - m_new) : 0.f;
      const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);   // nothing summed yet
      l = l * corr + warp_sum(p);
#pragma unroll
      for (int i = 0; i < kMaxHd / 32; ++i) acc[i] *= corr;
      m = m_new;
      // Values: keys in ascending order, eight at a time so that their loads travel together
      // (a decode step has one warp per head and nothing else to hide a load behind).  A key
      // with p = 0 (masked, or underflowed) adds nothing and is not read.
      const int n_valid = min(32, hi + 1 - base);
      constexpr int kAhead = 8;
      for (int j0 = 0; j0 < n_valid; j0 += kAhead) {
        float pj[kAhead];
        const T* vp[kAhead];
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
          const int j = min(j0 + u, 31);
          const float pu = __shfl_sync(0xffffffffu, p, j);
          const unsigned long long ru = __shfl_sync(0xffffffffu, row, j);
          pj[u] = j0 + u < n_valid ? pu : 0.f;
          vp[u] = vbase + ru * vd;
        }
#pragma unroll
        for (int i = 0; i < kMaxHd / 32; ++i) {
          const int d = lane + 32 * i;
          if (d < vd) {
            float v[kAhead];
#pragma unroll
            for (int u = 0; u < kAhead; ++u) v[u] = pj[u] != 0.f ? to_float(vp[u][d]) : 0.f;
#pragma unroll
            for (int u = 0; u < kAhead; ++u)
              if (pj[u] != 0.f) acc[i] = fmaf(pj[u], v[u], acc[i]);
          }
        }
      }
    }
  };
  walk(std::true_type{}, first, pos, kc, vc, tab);
  if (pooled.table)
    walk(std::false_type{}, 0, visible_pooled(pos, window, pooled.pool) - 1, (const T*)pooled.k,
         (const T*)pooled.v, pooled.table + (size_t)slot * pooled.table_stride);
  // the warps' results meet in shared memory; warp 0 folds them in the warps' order
  if (lane == 0) {
    part_m[warp] = m;
    part_l[warp] = l;
  }
#pragma unroll
  for (int i = 0; i < kMaxHd / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < vd) part_acc[warp][d] = acc[i];
  }
  __syncthreads();
  if (warp != 0) return;
  float m_all = -INFINITY;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) m_all = fmaxf(m_all, part_m[w]);
  float l_all = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxHd / 32; ++i) acc[i] = 0.f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    const float mw = part_m[w];
    if (mw == -INFINITY) continue;              // a warp without a visible key adds nothing
    const float a = expf(mw - m_all);
    l_all += part_l[w] * a;
#pragma unroll
    for (int i = 0; i < kMaxHd / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < vd) acc[i] = fmaf(part_acc[w][d], a, acc[i]);
    }
  }
  if (sink) {
    // a sink: one more term exp(sink_h) in the denominator, with no key and no value
    const float sk = sink[h];
    const float m2 = fmaxf(m_all, sk);
    const float a = m_all == -INFINITY ? 0.f : expf(m_all - m2);
    l_all = l_all * a + expf(sk - m2);
#pragma unroll
    for (int i = 0; i < kMaxHd / 32; ++i) acc[i] *= a;
  }
  const float inv = 1.0f / l_all;
  T* orow = out + (size_t)t * ldo + (size_t)h * vd;
#pragma unroll
  for (int i = 0; i < kMaxHd / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < vd) orow[d] = from_float<T>(acc[i] * inv);
  }
}

}  // namespace cretif

using namespace cretif;

extern "C" int cretif_attn_simt(const void* q, int ldq, void* out, int ldo, int dt, const void* kc,
                                const void* vc, const int* table, int table_stride,
                                const int* tok_pos, const int* tok_seq, const int* seq_slot,
                                int nh, int nkv, int hd, float scale, int window, int bt, int T,
                                const float* sink, int vd, const float* bias,
                                const int* bias_edges, int bias_rows, const float* slope,
                                void* stream) {
  return cretif_attn_simt_pooled(q, ldq, out, ldo, dt, kc, vc, table, table_stride, tok_pos, tok_seq,
                                 seq_slot, nh, nkv, hd, scale, window, bt, T, sink, vd, bias,
                                 bias_edges, bias_rows, slope, nullptr, nullptr, nullptr, 0, 0, stream);
}

// pool_k, pool_v [blocks, nkv, bt, hd or vd], pool_table [slots, pool_stride]: the entries per
// complete block of `pool` tokens (pool_table null: none; they need a sliding window).
extern "C" int cretif_attn_simt_pooled(
    const void* q, int ldq, void* out, int ldo, int dt, const void* kc, const void* vc,
    const int* table, int table_stride, const int* tok_pos, const int* tok_seq, const int* seq_slot,
    int nh, int nkv, int hd, float scale, int window, int bt, int T, const float* sink, int vd,
    const float* bias, const int* bias_edges, int bias_rows, const float* slope, const void* pool_k,
    const void* pool_v, const int* pool_table, int pool_stride, int pool, void* stream) {
  if (T <= 0) return kOk;
  if (pool_table && (!pool_k || !pool_v || pool <= 0 || window <= 0)) return kBadArgument;
  const PooledKeys pooled{pool_k, pool_v, pool_table, pool_stride, pool, 0};
  if (nh <= 0 || nkv <= 0 || nh % nkv || hd <= 0 || hd > kMaxHd || bt <= 0 ||
      vd <= 0 || vd > kMaxHd)
    return kBadArgument;
  if (bias && (!bias_edges || bias_rows <= 0 || bias_rows > kMaxBiasRows)) return kBadArgument;
  cudaStream_t st = (cudaStream_t)stream;
  const long long items = (long long)T * nh;
  if (items > 0x7fffffffLL) return kBadArgument;
  const unsigned blocks = (unsigned)items;
  if (dt == kF32)
    attn_simt_kernel<float><<<blocks, kWarps * 32, 0, st>>>(
        (const float*)q, ldq, (float*)out, ldo, (const float*)kc, (const float*)vc, table,
        table_stride, tok_pos, tok_seq, seq_slot, nh, nkv, hd, scale, window, bt, T, sink, vd, bias,
        bias_edges, bias_rows, slope, pooled);
  else if (dt == kBF16)
    attn_simt_kernel<__nv_bfloat16><<<blocks, kWarps * 32, 0, st>>>(
        (const __nv_bfloat16*)q, ldq, (__nv_bfloat16*)out, ldo, (const __nv_bfloat16*)kc,
        (const __nv_bfloat16*)vc, table, table_stride, tok_pos, tok_seq, seq_slot, nh, nkv, hd,
        scale, window, bt, T, sink, vd, bias, bias_edges, bias_rows, slope, pooled);
  else
    return kBadDType;
  return launch_status();
}
