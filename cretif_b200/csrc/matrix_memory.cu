// Matrix memory with exponential gates (the mLSTM recurrence of xLSTM): linear attention whose decay
// and input weight are learned per token and head, kept in range by a running maximum.
//
// Per token and head, with state S [d, e], n [d] and m (32-bit, all zero at a sequence's start), the
// logarithms of the input and the forget gate
//     i = cap tanh((z_i + b_i) / cap),   f = log sigmoid(cap tanh((z_f + b_f) / cap))
// and q scaled by q_scale:
//     m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k v^T;   n likewise with k alone
//     o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)
// Everything is 32-bit; sums of f are carried in 64-bit, because what enters the exponentials are
// differences of them.
//
// * memory_token_kernel (a CTA per (sequence, head, slice of columns)): token by token, the thread
//   layout of the retention's recurrence (retention.cu).  The first slice's first warp also carries n.
// * memory_intra_kernel + memory_carry_kernel: 64 tokens at a time, below.
// * memory_out_kernel (a warp per (token, head)): the division, the norm per head, the output gate,
//   and the sequence's new m (it is written here, after every CTA of the kernels above has read it).
//
// proj rows (float32): [q (H d) | k (H d) | v (H e) | gate (H e) | z_i (H) | z_f (H) | ...].
// A slot's state: [S (H d e) | n (H d) | m (H)].  Between the kernels: o_raw [T, H e] the numerators,
// den [T, H] n . q, ref [T, H] m'.
#include "api.h"
#include "common.cuh"

namespace cretif {

namespace {

constexpr float kMemEps = 1e-6f;

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float c = cap * tanhf(z / cap);
  return fminf(c, 0.f) - log1pf(expf(-fabsf(c)));
}

// What every kernel reads of a layer.
struct MemArgs {
  const float* proj;
  int ldp;
  const float* bias_i;
  const float* bias_f;
  float cap, q_scale;
  float* state;
  size_t state_stride;
  const int* cu;
  const int* slot;
  int B, H, d, e, T;
  float* o_raw;
  float* den;
  float* ref;
  int write_state;
  __device__ const float* q(int t, int h) const { return proj + (size_t)t * ldp + (size_t)h * d; }
  __device__ const float* k(int t, int h) const { return q(t, h) + (size_t)H * d; }
  __device__ const float* v(int t, int h) const {
    return proj + (size_t)t * ldp + (size_t)2 * H * d + (size_t)h * e;
  }
  __device__ float log_i(int t, int h) const {
    return log_input_gate(proj[(size_t)t * ldp + 2 * (size_t)H * (d + e) + h] + bias_i[h], cap);
  }
  __device__ float log_f(int t, int h) const {
    return log_forget_gate(proj[(size_t)t * ldp + 2 * (size_t)H * (d + e) + H + h] + bias_f[h], cap);
  }
  __device__ float* S(int b, int h) const {
    return state + (size_t)slot[b] * state_stride + (size_t)h * d * e;
  }
  __device__ float* n(int b, int h) const {
    return state + (size_t)slot[b] * state_stride + (size_t)H * d * e + (size_t)h * d;
  }
  __device__ float* m(int b, int h) const {
    return state + (size_t)slot[b] * state_stride + (size_t)H * d * (e + 1) + h;
  }
};

constexpr int kMemChunk = 16;

// blockDim.x = ecols * P threads (at most 256), rounded up to whole warps: thread = column * P + part,
// a lane owns R contiguous rows of its column.
template <int R>
__global__ void __launch_bounds__(256)
memory_token_kernel(const MemArgs a, int P, int ecols) {
  extern __shared__ __align__(16) float smem[];
  const int b = blockIdx.x, h = blockIdx.y, H = a.H, d = a.d, e = a.e;
  const int col0 = blockIdx.z * ecols;
  const int t0 = a.cu[b], t1 = a.cu[b + 1];
  const int part = threadIdx.x % P, jc = threadIdx.x / P;
  const int col = col0 + jc;
  const bool active = jc < ecols && col < e;
  const bool keeps_n = blockIdx.z == 0 && threadIdx.x < 32;      // (a whole warp)
  const int slice = R + 4;                       // a lane's rows of q or k, padded
  float* sq = smem;                              // [chunk][P * slice]
  float* sk = sq + kMemChunk * P * slice;        // [chunk][P * slice]
  float* sv = sk + kMemChunk * P * slice;        // [chunk][ecols]
  float* so = sv + kMemChunk * ecols;            // [chunk][ecols]
  float* gi = so + kMemChunk * ecols;            // [chunk] log gates, then the factors
  float* gf = gi + kMemChunk;
  float* gm = gf + kMemChunk;                    // [chunk + 1] m before each token, and after the last
  float* M = a.S(b, h);
  float S[R], N[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = part * R + r;
    S[r] = (active && i < d) ? M[(size_t)i * e + col] : 0.f;
    N[r] = (keeps_n && i < d) ? a.n(b, h)[i] : 0.f;
  }
  if (threadIdx.x == 0) gm[0] = *a.m(b, h);
  const int rows_padded = P * R;
  for (int c0 = t0; c0 < t1; c0 += kMemChunk) {
    const int nt = min(kMemChunk, t1 - c0);
    __syncthreads();                             // the chunk before has been read and written out
    for (int idx = threadIdx.x; idx < nt * rows_padded; idx += blockDim.x) {
      const int tt = idx / rows_padded, i = idx - tt * rows_padded;
      const int p = i / R, r = i - p * R;
      sq[(tt * P + p) * slice + r] = i < d ? a.q(c0 + tt, h)[i] * a.q_scale : 0.f;
      sk[(tt * P + p) * slice + r] = i < d ? a.k(c0 + tt, h)[i] : 0.f;
    }
    for (int idx = threadIdx.x; idx < nt * ecols; idx += blockDim.x) {
      const int tt = idx / ecols, j = idx - tt * ecols;
      sv[idx] = col0 + j < e ? a.v(c0 + tt, h)[col0 + j] : 0.f;
    }
    if (threadIdx.x < nt) {
      gi[threadIdx.x] = a.log_i(c0 + threadIdx.x, h);
      gf[threadIdx.x] = a.log_f(c0 + threadIdx.x, h);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
      if (c0 > t0) gm[0] = gm[kMemChunk];        // (every chunk but the last is full)
      for (int tt = 0; tt < nt; ++tt) gm[tt + 1] = fmaxf(gf[tt] + gm[tt], gi[tt]);
    }
    __syncthreads();
    if (threadIdx.x < nt) {
      const int tt = threadIdx.x;
      const float m1 = gm[tt + 1];
      gf[tt] = expf(gf[tt] + gm[tt] - m1);
      gi[tt] = expf(gi[tt] - m1);
      if (blockIdx.z == 0) a.ref[(size_t)(c0 + tt) * H + h] = m1;
    }
    __syncthreads();
    {
      // every lane goes through the loop (the shuffles want whole warps); lanes beyond the
      // slice work on zeros and store nothing
      const int jv = jc < ecols ? jc : 0;
      for (int tt = 0; tt < nt; ++tt) {
        const float* q = sq + (tt * P + part) * slice;
        const float* k = sk + (tt * P + part) * slice;
        const float keep = gf[tt], add = gi[tt];
        const float vt = add * sv[tt * ecols + jv];
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int r = 0; r < R; r += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(k + r);
          const float4 q4 = *reinterpret_cast<const float4*>(q + r);
          S[r] = fmaf(k4.x, vt, keep * S[r]);
          S[r + 1] = fmaf(k4.y, vt, keep * S[r + 1]);
          S[r + 2] = fmaf(k4.z, vt, keep * S[r + 2]);
          S[r + 3] = fmaf(k4.w, vt, keep * S[r + 3]);
          acc[0] = fmaf(S[r], q4.x, acc[0]);
          acc[1] = fmaf(S[r + 1], q4.y, acc[1]);
          acc[2] = fmaf(S[r + 2], q4.z, acc[2]);
          acc[3] = fmaf(S[r + 3], q4.w, acc[3]);
        }
        float o = (acc[0] + acc[1]) + (acc[2] + acc[3]);
        for (int off = P >> 1; off > 0; off >>= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
        if (part == 0 && jc < ecols) so[tt * ecols + jc] = o;
        if (keeps_n) {
          float nq = 0.f;
#pragma unroll
          for (int r = 0; r < R; ++r) {
            N[r] = fmaf(k[r], add, keep * N[r]);
            nq = fmaf(N[r], q[r], nq);
          }
          for (int off = P >> 1; off > 0; off >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, off);
          if (threadIdx.x == 0) a.den[(size_t)(c0 + tt) * H + h] = nq;
        }
      }
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nt * ecols; idx += blockDim.x) {
      const int tt = idx / ecols, j = idx - tt * ecols;
      if (col0 + j < e) a.o_raw[(size_t)(c0 + tt) * H * e + (size_t)h * e + col0 + j] = so[idx];
    }
  }
  if (a.write_state) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = part * R + r;
      if (active && i < d) M[(size_t)i * e + col] = S[r];
      if (keeps_n && jc == 0 && i < d) a.n(b, h)[i] = N[r];
    }
  }
}

template <int R>
int launch_memory_token(const MemArgs& a, int P, int ecols, cudaStream_t st) {
  const int threads = ((ecols * P + 31) / 32) * 32;
  const size_t smem = sizeof(float) * (kMemChunk * (2 * (size_t)P * (R + 4) + 2 * (size_t)ecols) +
                                       3 * kMemChunk + 4);
  auto kern = memory_token_kernel<R>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return kBadArgument;
    cudaError_t err =
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  const int slices = (a.e + ecols - 1) / ecols;
  if (a.H > 65535 || slices > 65535) return kBadArgument;
  kern<<<dim3(a.B, a.H, slices), threads, smem, st>>>(a, P, ecols);
  return launch_status();
}

// ---------------------------------------------------------------------------------------------
// 64 tokens at a time.  Within a chunk let F_t be the sum of f up to and with token t, u_s = i_s - F_s
// and U_t = max of u_s for s <= t; m0, S0, n0 are the state before the chunk.  Then
//     m_t = F_t + X_t,   X_t = max(m0, U_t)
//     S_t^T q_t = exp(m0 - X_t) S0^T q_t + exp(U_t - X_t) sum_{s<=t} exp(u_s - U_t) (q_t . k_s) v_s
//     S_n = exp(m0 - X_n) S0 + sum_s exp(u_s - X_n) k_s v_s^T
// (n and n . q the same way without v), and no exponent is ever above zero.
//
// * memory_intra_kernel (a CTA per (chunk, head); the chunks of all sequences at once): the inner sum,
//   relative to U_t, to o_raw, its share of n . q to den, and u, U and F to gates [3][H][T] (64-bit).
//   Nothing here depends on the state, so a long prompt fills the chip.
// * memory_carry_kernel (a CTA per (sequence, head, EC columns of S), and one more per (sequence,
//   head) that carries n) walks the sequence's chunks with its part of the state in shared memory.
// The matrix products are the retention's (32-bit FMA, 16-byte shared-memory loads, rows padded to
// 4 mod 8 floats).
constexpr int kMcTokens = 64;
constexpr int kMcThreads = 256;
constexpr int kMcScoreLd = kMcTokens + 4;
constexpr int kMcSlab = 64;             // columns of v the intra kernel takes at a time

__device__ __forceinline__ void fma4(float4& a, float s, const float4& v) {
  a.x = fmaf(s, v.x, a.x);
  a.y = fmaf(s, v.y, a.y);
  a.z = fmaf(s, v.z, a.z);
  a.w = fmaf(s, v.w, a.w);
}
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
  acc = fmaf(a.x, b.x, acc);
  acc = fmaf(a.y, b.y, acc);
  acc = fmaf(a.z, b.z, acc);
  return fmaf(a.w, b.w, acc);
}
__device__ __forceinline__ void scale4(float4& a, float s) {
  a.x *= s; a.y *= s; a.z *= s; a.w *= s;
}

__device__ __forceinline__ void mem_cp16(float* dst, const float* src) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ void mem_cp8(double* dst, const double* src) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ void mem_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void mem_cp_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

__host__ __device__ inline int memory_chunk_ld(int d) {
  int ld = d;
  while ((ld & 7) != 4) ++ld;
  return ld;
}
// (the 64-bit gates come first, so that they are 8-byte aligned)
inline size_t memory_intra_smem(int d) {
  return sizeof(double) * 2 * kMcTokens +
         sizeof(float) * (2 * (size_t)kMcTokens * memory_chunk_ld(d) + (size_t)kMcTokens * kMcSlab +
                          (size_t)kMcTokens * kMcScoreLd);
}
inline size_t memory_carry_smem(int d, int ec, int nbuf) {
  return sizeof(double) * 3 * kMcTokens * nbuf +
         sizeof(float) * (nbuf * (2 * (size_t)kMcTokens * memory_chunk_ld(d) + (size_t)kMcTokens * ec) +
                          (size_t)d * ec + kMcTokens);
}

__global__ void __launch_bounds__(kMcThreads)
memory_intra_kernel(const MemArgs a, double* __restrict__ gates) {
  extern __shared__ __align__(16) float smem[];
  constexpr int C = kMcTokens;
  constexpr int LP = kMcScoreLd;
  const int tid = threadIdx.x, H = a.H, d = a.d, e = a.e;
  const int h = blockIdx.y;
  // which sequence's which chunk: the grid has a CTA for every chunk there can be
  int left = blockIdx.x, c0 = -1, t1 = 0;
  for (int b = 0; b < a.B; ++b) {
    const int s0 = a.cu[b], s1 = a.cu[b + 1];
    const int chunks = (s1 - s0 + C - 1) / C;
    if (left < chunks) {
      c0 = s0 + left * C;
      t1 = s1;
      break;
    }
    left -= chunks;
  }
  if (c0 < 0) return;
  const int nt = min(C, t1 - c0);
  const int ldq = memory_chunk_ld(d);
  const int d4 = d >> 2;
  double* su = reinterpret_cast<double*>(smem);      // [C] u
  double* sU = su + C;                               // [C] U
  float* sQ = reinterpret_cast<float*>(sU + C);      // [C][ldq]
  float* sK = sQ + C * ldq;                          // [C][ldq]
  float* sV = sK + C * ldq;                          // [C][kMcSlab]
  float* sP = sV + C * kMcSlab;                      // [C][LP]
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  // q and k of the chunk's tokens, copied asynchronously.  Rows beyond the chunk's last token stay as
  // they are: they reach only scores of rows that are not stored, or of keys after the row, which
  // are set to zero.
  for (int idx = tid; idx < nt * d4; idx += kMcThreads) {
    const int tt = idx / d4, i4 = idx - tt * d4;
    mem_cp16(sQ + tt * ldq + 4 * i4, a.q(c0 + tt, h) + 4 * i4);
    mem_cp16(sK + tt * ldq + 4 * i4, a.k(c0 + tt, h) + 4 * i4);
  }
  mem_cp_commit();
  // a slab of v: rows beyond the last token and columns beyond the slab are zero (a zero score
  // times whatever lay there must stay zero)
  auto stage_v = [&](int j0, int width) {
    for (int idx = tid; idx < C * (kMcSlab / 4); idx += kMcThreads) {
      const int tt = idx >> 4, jg = idx & 15;
      float* dst = sV + tt * kMcSlab + 4 * jg;
      if (tt < nt && 4 * jg < width)
        mem_cp16(dst, a.v(c0 + tt, h) + j0 + 4 * jg);
      else
        *reinterpret_cast<float4*>(dst) = zero4;
    }
    mem_cp_commit();
  };
  stage_v(0, min(kMcSlab, e));
  if (tid < 32) {
    // the gates' scans: lane l has tokens 2 l and 2 l + 1 (beyond the last: f = 0, i = -inf)
    double f[2], u[2];
    float li[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int tt = 2 * tid + x;
      f[x] = tt < nt ? (double)a.log_f(c0 + tt, h) : 0.0;
      li[x] = tt < nt ? a.log_i(c0 + tt, h) : -INFINITY;
    }
    f[1] += f[0];
    double run = f[1];
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, run, off);
      if (tid >= off) run += other;
    }
    const double before = run - f[1];            // (the sum of the lanes below, exactly enough)
    f[0] += before;
    f[1] += before;
    u[0] = (double)li[0] - f[0];
    u[1] = (double)li[1] - f[1];
    double top = fmax(u[0], u[1]);
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, top, off);
      if (tid >= off) top = fmax(top, other);
    }
    double below = __shfl_up_sync(0xffffffffu, top, 1);
    if (tid == 0) below = u[0];
    const double U0 = fmax(below, u[0]), U1 = fmax(U0, u[1]);
    su[2 * tid] = u[0]; su[2 * tid + 1] = u[1];
    sU[2 * tid] = U0; sU[2 * tid + 1] = U1;
    double* g = gates + (size_t)h * a.T + c0;
    const size_t plane = (size_t)H * a.T;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int tt = 2 * tid + x;
      if (tt < nt) {
        g[tt] = u[x];
        g[plane + tt] = x ? U1 : U0;
        g[2 * plane + tt] = f[x];
      }
    }
  }
  mem_cp_wait<1>();                        // q and k have arrived
  __syncthreads();
  const int ti = tid >> 4, si = tid & 15;
  {
    // scores: thread (ti, si) owns rows ti + 16 r and keys si + 16 c; key blocks ahead of the
    // row block are never computed
    float acc[4][4];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[r][c] = 0.f;
    for (int kk = 0; kk < d; kk += 4) {
      float4 q4[4], k4[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        q4[r] = *reinterpret_cast<const float4*>(sQ + (ti + 16 * r) * ldq + kk);
        k4[r] = *reinterpret_cast<const float4*>(sK + (si + 16 * r) * ldq + kk);
      }
#pragma unroll
      for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c <= r; ++c) acc[r][c] = dot4(q4[r], k4[c], acc[r][c]);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int t = ti + 16 * r;
      const double Ut = sU[t];
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int s = si + 16 * c;
        float p = 0.f;
        if (c < r || (c == r && si <= ti))
          p = acc[r][c] * a.q_scale * expf((float)(su[s] - Ut));
        sP[t * LP + s] = p;
        sum += p;
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      if (si == 0 && t < nt) a.den[(size_t)(c0 + t) * H + h] = sum;
    }
  }
  // scores times v, 64 columns at a time: rows ti + 16 r, columns 4 si .. 4 si + 3 of the slab
  for (int j0 = 0; j0 < e; j0 += kMcSlab) {
    const int width = min(kMcSlab, e - j0);            // a multiple of 4
    if (j0 > 0) {
      __syncthreads();                                 // the slab before has been read
      stage_v(j0, width);
    }
    mem_cp_wait<0>();
    __syncthreads();                                   // the slab and the scores are in place
    if (4 * si >= width) continue;
    float4 acc[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) acc[r] = zero4;
    const int smax = min(nt, ti + 49);
    for (int s = 0; s < smax; s += 4) {
      const float4 v0 = *reinterpret_cast<const float4*>(sV + (s + 0) * kMcSlab + 4 * si);
      const float4 v1 = *reinterpret_cast<const float4*>(sV + (s + 1) * kMcSlab + 4 * si);
      const float4 v2 = *reinterpret_cast<const float4*>(sV + (s + 2) * kMcSlab + 4 * si);
      const float4 v3 = *reinterpret_cast<const float4*>(sV + (s + 3) * kMcSlab + 4 * si);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        if (s > ti + 16 * r) continue;                 // keys after the row: the scores are zero
        const float4 p = *reinterpret_cast<const float4*>(sP + (ti + 16 * r) * LP + s);
        fma4(acc[r], p.x, v0);
        fma4(acc[r], p.y, v1);
        fma4(acc[r], p.z, v2);
        fma4(acc[r], p.w, v3);
      }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int t = ti + 16 * r;
      if (t < nt)
        *reinterpret_cast<float4*>(a.o_raw + (size_t)(c0 + t) * H * e + (size_t)h * e + j0 + 4 * si) =
            acc[r];
    }
  }
}

// Two buffers for q, k, v and the gates where they fit (nbuf = 2): a chunk's copies are under way
// while the chunk before is computed.
template <int EC>
__global__ void __launch_bounds__(kMcThreads)
memory_carry_kernel(const MemArgs a, const double* __restrict__ gates, int nbuf) {
  extern __shared__ __align__(16) float smem[];
  constexpr int C = kMcTokens;
  constexpr int CG = EC / 4;               // groups of four columns
  constexpr int NR = kMcThreads / CG;      // threads along the rows
  constexpr int RT = C / NR;               // read-out rows a thread
  const int tid = threadIdx.x, H = a.H, d = a.d, e = a.e;
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * EC;
  const bool carries_n = col0 >= e;        // the one CTA beyond the columns' slices
  const int t0 = a.cu[b], t1 = a.cu[b + 1];
  if (t1 <= t0) return;
  const int ldq = memory_chunk_ld(d);
  const int d4 = d >> 2;
  double* sG = reinterpret_cast<double*>(smem);          // [nbuf][u, U, F][C]
  float* bufs = reinterpret_cast<float*>(sG + nbuf * 3 * C);
  const int buf_floats = 2 * C * ldq + C * EC;           // q [C][ldq] | k [C][ldq] | v [C][EC]
  float* sS = bufs + nbuf * buf_floats;                  // [d][EC]
  float* sW = sS + d * EC;                               // [C] a token's weight in the state's update
  float* M = a.S(b, h) + (carries_n ? 0 : col0);
  if (carries_n) {
    for (int i = tid; i < d; i += kMcThreads) sS[i] = a.n(b, h)[i];
  } else {
    for (int idx = tid; idx < d * CG; idx += kMcThreads) {
      const int i = idx / CG, jg = idx - i * CG;
      *reinterpret_cast<float4*>(sS + i * EC + 4 * jg) =
          *reinterpret_cast<const float4*>(M + (size_t)i * e + 4 * jg);
    }
  }
  double m0 = (double)*a.m(b, h);
  const int tj = tid % CG, tr = tid / CG;
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  // Rows beyond a chunk's last token are not copied: of q they reach only read-outs that are
  // not stored, of k and v nothing (the update stops at the last token).
  auto stage = [&](int c0, int which) {
    const int nt = min(C, t1 - c0);
    float* buf = bufs + which * buf_floats;
    for (int idx = tid; idx < nt * d4; idx += kMcThreads) {
      const int tt = idx / d4, i4 = idx - tt * d4;
      mem_cp16(buf + tt * ldq + 4 * i4, a.q(c0 + tt, h) + 4 * i4);
      mem_cp16(buf + C * ldq + tt * ldq + 4 * i4, a.k(c0 + tt, h) + 4 * i4);
    }
    if (!carries_n)
      for (int idx = tid; idx < nt * CG; idx += kMcThreads) {
        const int tt = idx / CG, jg = idx - tt * CG;
        mem_cp16(buf + 2 * C * ldq + tt * EC + 4 * jg, a.v(c0 + tt, h) + col0 + 4 * jg);
      }
    for (int idx = tid; idx < 3 * C; idx += kMcThreads) {
      const int plane = idx / C, tt = idx - plane * C;
      if (tt < nt)
        mem_cp8(sG + (which * 3 + plane) * C + tt,
                gates + ((size_t)plane * H + h) * a.T + c0 + tt);
    }
    mem_cp_commit();
  };
  stage(t0, 0);
  int turn = 0;
  for (int c0 = t0; c0 < t1; c0 += C, ++turn) {
    const int nt = min(C, t1 - c0);
    const bool last = c0 + C >= t1;
    const int which = nbuf == 2 ? (turn & 1) : 0;
    const double* su = sG + which * 3 * C;
    const double* sU = su + C;
    const double* sF = sU + C;
    float* sQ = bufs + which * buf_floats;
    float* sK = sQ + C * ldq;
    float* sV = sK + C * ldq;
    mem_cp_wait<0>();
    __syncthreads();                       // the chunk is in place; the chunk before is done
    if (nbuf == 2 && !last) stage(c0 + C, (turn + 1) & 1);
    const double Xn = fmax(m0, sU[nt - 1]);
    const float keep = expf((float)(m0 - Xn));
    if (tid < nt) sW[tid] = expf((float)(su[tid] - Xn));
    if (carries_n) {
      // n . q of every row: four lanes a row
      const int t = tid >> 2, part = tid & 3;
      float acc = 0.f;
      for (int i4 = part; i4 < d4; i4 += 4)
        acc = dot4(*reinterpret_cast<const float4*>(sQ + t * ldq + 4 * i4),
                   *reinterpret_cast<const float4*>(sS + 4 * i4), acc);
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      if (part == 0 && t < nt) {
        const double X = fmax(m0, sU[t]);
        const size_t at = (size_t)(c0 + t) * H + h;
        a.den[at] = expf((float)(m0 - X)) * a.q_scale * acc + expf((float)(sU[t] - X)) * a.den[at];
        a.ref[at] = (float)(sF[t] + X);
      }
      __syncthreads();                     // everybody has read n; the weights are in place
      for (int i = tid; i < d; i += kMcThreads) {
        float v = keep * sS[i];
#pragma unroll 8
        for (int s = 0; s < nt; ++s) v = fmaf(sW[s], sK[s * ldq + i], v);
        sS[i] = v;
      }
    } else {
      {
        // what the state before the chunk gives every row: rows tr + NR r, columns 4 tj .. + 3
        float4 acc[RT], old[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          acc[r] = zero4;
          const int t = tr + NR * r;
          old[r] = t < nt ? __ldcg(reinterpret_cast<const float4*>(
                                a.o_raw + (size_t)(c0 + t) * H * e + (size_t)h * e + col0 + 4 * tj))
                          : zero4;
        }
#pragma unroll 2
        for (int i = 0; i < d; i += 4) {
          const float4 s0 = *reinterpret_cast<const float4*>(sS + (i + 0) * EC + 4 * tj);
          const float4 s1 = *reinterpret_cast<const float4*>(sS + (i + 1) * EC + 4 * tj);
          const float4 s2 = *reinterpret_cast<const float4*>(sS + (i + 2) * EC + 4 * tj);
          const float4 s3 = *reinterpret_cast<const float4*>(sS + (i + 3) * EC + 4 * tj);
#pragma unroll
          for (int r = 0; r < RT; ++r) {
            const float4 q = *reinterpret_cast<const float4*>(sQ + (tr + NR * r) * ldq + i);
            fma4(acc[r], q.x, s0);
            fma4(acc[r], q.y, s1);
            fma4(acc[r], q.z, s2);
            fma4(acc[r], q.w, s3);
          }
        }
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          const int t = tr + NR * r;
          if (t < nt) {
            const double X = fmax(m0, sU[t]);
            const float w0 = expf((float)(m0 - X)) * a.q_scale, w1 = expf((float)(sU[t] - X));
            float4 o = old[r];
            scale4(o, w1);
            fma4(o, w0, acc[r]);
            *reinterpret_cast<float4*>(a.o_raw + (size_t)(c0 + t) * H * e + (size_t)h * e + col0 +
                                       4 * tj) = o;
          }
        }
      }
      if (last && !a.write_state) break;   // nobody reads the state after the last chunk
      __syncthreads();                     // everybody has read the old state; the weights are in place
      // v takes the weight it has in the state's update (the read-out does not use v)
      for (int idx = tid; idx < nt * CG; idx += kMcThreads) {
        const int tt = idx / CG, jg = idx - tt * CG;
        float4 v4 = *reinterpret_cast<float4*>(sV + tt * EC + 4 * jg);
        scale4(v4, sW[tt]);
        *reinterpret_cast<float4*>(sV + tt * EC + 4 * jg) = v4;
      }
      __syncthreads();
      for (int ig = tr; ig < d4; ig += NR) {
        float* srow = sS + (4 * ig) * EC + 4 * tj;
        float4 a0 = *reinterpret_cast<float4*>(srow);
        float4 a1 = *reinterpret_cast<float4*>(srow + EC);
        float4 a2 = *reinterpret_cast<float4*>(srow + 2 * EC);
        float4 a3 = *reinterpret_cast<float4*>(srow + 3 * EC);
        scale4(a0, keep);
        scale4(a1, keep);
        scale4(a2, keep);
        scale4(a3, keep);
#pragma unroll 4
        for (int s = 0; s < nt; ++s) {
          const float4 k4 = *reinterpret_cast<const float4*>(sK + s * ldq + 4 * ig);
          const float4 v4 = *reinterpret_cast<const float4*>(sV + s * EC + 4 * tj);
          fma4(a0, k4.x, v4);
          fma4(a1, k4.y, v4);
          fma4(a2, k4.z, v4);
          fma4(a3, k4.w, v4);
        }
        *reinterpret_cast<float4*>(srow) = a0;
        *reinterpret_cast<float4*>(srow + EC) = a1;
        *reinterpret_cast<float4*>(srow + 2 * EC) = a2;
        *reinterpret_cast<float4*>(srow + 3 * EC) = a3;
      }
    }
    m0 = sF[nt - 1] + Xn;
    if (nbuf != 2 && !last) {
      __syncthreads();                     // the one buffer has been read
      stage(c0 + C, 0);
    }
  }
  if (a.write_state) {
    __syncthreads();
    if (carries_n) {
      for (int i = tid; i < d; i += kMcThreads) a.n(b, h)[i] = sS[i];
    } else {
      for (int idx = tid; idx < d * CG; idx += kMcThreads) {
        const int i = idx / CG, jg = idx - i * CG;
        *reinterpret_cast<float4*>(M + (size_t)i * e + 4 * jg) =
            *reinterpret_cast<const float4*>(sS + i * EC + 4 * jg);
      }
    }
  }
}

template <int EC>
int launch_memory_carry(const MemArgs& a, const double* gates, cudaStream_t st) {
  const int nbuf = memory_carry_smem(a.d, EC, 2) <= 220 * 1024 ? 2 : 1;
  const size_t smem = memory_carry_smem(a.d, EC, nbuf);
  auto kern = memory_carry_kernel<EC>;
  if (smem > 48 * 1024) {
    cudaError_t err =
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  kern<<<dim3(a.B, a.H, a.e / EC + 1), kMcThreads, smem, st>>>(a, gates, nbuf);
  return launch_status();
}

int launch_memory_intra(const MemArgs& a, double* gates, cudaStream_t st) {
  const size_t smem = memory_intra_smem(a.d);
  if (smem > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(
        memory_intra_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  // every sequence has at most one chunk that is not full
  const long long chunks = (long long)a.T / kMcTokens + a.B;
  if (chunks > 0x7fffffffLL) return kBadArgument;
  memory_intra_kernel<<<dim3((unsigned)chunks, a.H), kMcThreads, smem, st>>>(a, gates);
  return launch_status();
}

// out[t, h] = x / sqrt(mean(x^2) + eps) * norm_w * sigmoid(gate), x = o_raw / (max(|den|, exp(-ref)) +
// 1e-6); the warp of a sequence's last token leaves ref as the sequence's m.
template <typename TO>
__global__ void __launch_bounds__(256)
memory_out_kernel(const MemArgs a, const int* __restrict__ tok_seq, const float* __restrict__ norm_w,
                  float eps, TO* __restrict__ out, int ldo, long long items) {
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= items) return;
  const int H = a.H, e = a.e;
  const int t = (int)(item / H), h = (int)(item - (long long)t * H);
  const float ref = a.ref[item];
  const float inv = 1.0f / (fmaxf(fabsf(a.den[item]), expf(-ref)) + kMemEps);
  const float* o = a.o_raw + (size_t)t * H * e + (size_t)h * e;
  const float* gate = a.proj + (size_t)t * a.ldp + (size_t)2 * H * a.d + (size_t)H * e + (size_t)h * e;
  TO* dst = out + (size_t)t * ldo + (size_t)h * e;
  constexpr int kKeep = 8;
  float x[kKeep], g[kKeep];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = lane + 32 * u;
    x[u] = i < e ? o[i] * inv : 0.f;
    g[u] = i < e ? gate[i] : 0.f;
    ss += x[u] * x[u];
  }
  for (int i = lane + 32 * kKeep; i < e; i += 32) {
    const float v = o[i] * inv;
    ss += v * v;
  }
  ss = warp_sum(ss);
  const float f = 1.0f / sqrtf(ss / (float)e + eps);
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = lane + 32 * u;
    if (i < e) dst[i] = from_float<TO>(x[u] * f * norm_w[h * e + i] / (1.0f + expf(-g[u])));
  }
  for (int i = lane + 32 * kKeep; i < e; i += 32)
    dst[i] = from_float<TO>(o[i] * inv * f * norm_w[h * e + i] / (1.0f + expf(-gate[i])));
  if (a.write_state && lane == 0) {
    const int b = tok_seq[t];
    if (t + 1 == a.cu[b + 1]) *a.m(b, h) = ref;
  }
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
}  // namespace
}  // namespace cretif

using namespace cretif;

// gates: float64 [3, H, T] scratch; form 0 chooses, 1 token by token, 2 chunks (refused where the
// sizes or addresses rule out 16-byte accesses).
extern "C" int cretif_matrix_memory(const float* proj, int ldp, const float* bias_i,
                                    const float* bias_f, float cap, float q_scale, float* state,
                                    long long state_stride, const int* cu_seqlens,
                                    const int* seq_slot, const int* tok_seq, int B, int H, int d,
                                    int e, const float* norm_w, float eps, float* o_raw, float* den,
                                    float* ref, double* gates, void* out, int out_dt, int ldo,
                                    int write_state, int T, int form, void* stream) {
  if (B <= 0 || T <= 0) return kOk;
  if (H <= 0 || d <= 0 || e <= 0 || !proj || !bias_i || !bias_f || !state || !norm_w || !o_raw ||
      !den || !ref || !(cap > 0.f) || ldp < 2 * H * (d + e) + 2 * H || ldo < H * e ||
      state_stride < (long long)H * d * (e + 1) + H || form < 0 || form > 2)
    return kBadArgument;
  static int sm_count = 0;
  if (!sm_count) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sm_count, cudaDevAttrMultiProcessorCount, dev);
    if (sm_count <= 0) sm_count = 148;
  }
  cudaStream_t st = (cudaStream_t)stream;
  const MemArgs a{proj, ldp, bias_i, bias_f, cap, q_scale, state, (size_t)state_stride, cu_seqlens,
                  seq_slot, B, H, d, e, T, o_raw, den, ref, write_state};
  int rc = kBadArgument;
  bool done = false;
  // 64 tokens at a time where the step brings a sequence 16 tokens or more on average and the
  // sizes allow 16-byte accesses throughout; token by token otherwise.
  if (form == 2 || (form == 0 && (long long)T >= 16LL * B)) {
    const bool fits = d % 4 == 0 && e % 16 == 0 && ldp % 4 == 0 && state_stride % 4 == 0 && gates &&
                      aligned16(proj) && aligned16(state) && aligned16(o_raw) && H <= 65535 &&
                      memory_carry_smem(d, 16, 1) <= 220 * 1024 &&
                      memory_intra_smem(d) <= 220 * 1024;
    if (fits) {
      rc = launch_memory_intra(a, gates, st);
      if (rc != kOk) return rc;
      // columns a CTA: as many as divide e and fit, fewer while the chip is not filled
      int ec = e % 64 == 0 ? 64 : e % 32 == 0 ? 32 : 16;
      while (ec > 16 && (memory_carry_smem(d, ec, 1) > 220 * 1024 ||
                         (long long)B * H * (e / ec) < (long long)sm_count))
        ec /= 2;
      rc = ec == 64   ? launch_memory_carry<64>(a, gates, st)
           : ec == 32 ? launch_memory_carry<32>(a, gates, st)
                      : launch_memory_carry<16>(a, gates, st);
      if (rc != kOk) return rc;
      done = true;
    } else if (form == 2) {
      return kBadArgument;
    }
  }
  if (!done) {
    // R rows a lane (a power of two from 4 to 32, about a quarter of d), P lanes a column
    int R = 4;
    while (R < 32 && R * 4 < d) R *= 2;
    int P = 1;
    while (P < 32 && P * R < d) P *= 2;
    if (P * R < d) return kBadArgument;            // d > 1024
    // columns a CTA: a head's columns are cut into slices while the (sequence, head) pairs alone
    // do not fill the chip twice over, down to two warps a CTA, and as far as 256 threads demand
    int ecols = e;
    while (ecols * P > 256) ecols = (ecols + 1) / 2;
    while ((long long)B * H * ((e + ecols - 1) / ecols) < 2LL * sm_count && ecols * P >= 128 &&
           ecols % 2 == 0)
      ecols /= 2;
    rc = R == 4    ? launch_memory_token<4>(a, P, ecols, st)
         : R == 8  ? launch_memory_token<8>(a, P, ecols, st)
         : R == 16 ? launch_memory_token<16>(a, P, ecols, st)
                   : launch_memory_token<32>(a, P, ecols, st);
    if (rc != kOk) return rc;
  }
  const long long items = (long long)T * H;
  const unsigned blocks = (unsigned)((items + 7) / 8);
  if (out_dt == kF32)
    memory_out_kernel<float><<<blocks, 256, 0, st>>>(a, tok_seq, norm_w, eps, (float*)out, ldo, items);
  else if (out_dt == kBF16)
    memory_out_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(a, tok_seq, norm_w, eps,
                                                             (__nv_bfloat16*)out, ldo, items);
  else
    return kBadDType;
  return launch_status();
}
