// The Mamba-2 recurrence (state-space duality): linear attention whose decay is learned per token and
// head, whose read and write vectors are shared by the heads of a group, behind a short causal
// convolution.
//
// Per token, with the projected channels u = [x (H e) | B (G N) | C (G N)] and dt_raw (H):
//     [x | B | C] = silu(conv(u) + conv_b),   dt = softplus(dt_raw + dt_bias),   a = -exp(A_log)
// and per head, with state S [N, e] (32-bit, zero at a sequence's start), B and C of the head's group:
//     S <- exp(a dt) S + dt B x^T;   y = S^T C + D x
// then y silu(z) is divided by its root mean square in `parts` equal parts and multiplied by a weight
// per channel.  Everything is 32-bit; sums of a dt are carried in 64-bit, because what enters the
// exponentials are differences of them.
//
// * ssm_prepare_kernel: the convolved channels and the step sizes.  A thread has a channel and eight
//   tokens in turn, so that a projected row is read once, or (few tokens) a channel and one token.  In a
//   step of one token a sequence it also brings the convolution's saved inputs up to date: each is read
//   and replaced by one thread.  After any other step delta_conv_state (delta_rule.cu) does.
// * ssm_token_kernel (a CTA per (sequence, head, slice of columns)): token by token, the thread layout
//   of the retention's recurrence (retention.cu).
// * ssm_intra_kernel + ssm_carry_kernel: 64 tokens at a time, below.
// * ssm_out_kernel: the gate, the norms and the weight.
//
// A slot's state: [S (H N e) | the last taps - 1 inputs of every convolved channel (C' (taps - 1))].
#include "api.h"
#include "common.cuh"

namespace cretif {

namespace {

// (the quotient by an approximate reciprocal: two units in the last place of 32 bits)
__device__ __forceinline__ float ssm_silu(float z) { return __fdividef(z, 1.0f + expf(-z)); }
__device__ __forceinline__ float ssm_softplus(float z) {
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

// What every kernel reads of a layer.
struct SsmArgs {
  const float* proj;        // rows [z (H e) | u (C') | dt (H) | ...]
  int ldp;
  const float* conv_w;      // [taps, C']
  const float* conv_b;      // [C']
  int taps;
  const float* a_log;
  const float* dt_bias;
  const float* d_skip;
  float* state;
  size_t stride;            // floats a slot
  size_t inputs;            // where a slot's saved inputs begin
  const int* cu;
  const int* slot;
  const int* tok_seq;
  int B, H, G, N, e, T;
  float* y;                 // [T, H e]
  float* xbc;               // [T, ldx] the convolved channels
  int ldx;
  float* dts;               // [H, T] step sizes
  double* sums;             // chunks: [H, T] sums of a dt from the chunk's start
  int write_state;
  __device__ int inner() const { return H * e; }
  __device__ int channels() const { return H * e + 2 * G * N; }
  __device__ const float* u(int t) const { return proj + (size_t)t * ldp + inner(); }
  __device__ float step(int t, int h) const {
    return ssm_softplus(proj[(size_t)t * ldp + inner() + channels() + h] + dt_bias[h]);
  }
  __device__ float rate(int h) const { return -expf(a_log[h]); }
  __device__ float* S(int b, int h) const {
    return state + (size_t)slot[b] * stride + (size_t)h * N * e;
  }
  // a sequence's last taps - 1 inputs of channel c, the oldest first
  __device__ float* saved(int b, int c) const {
    return state + (size_t)slot[b] * stride + inputs + (size_t)c * (taps - 1);
  }
};

constexpr int kSpTokens = 8;

// TAPS: the number of taps when it is 2, 3 or 4, 0 for any number.  NT: tokens a thread (one where
// the inputs are saved).
template <int TAPS, int NT>
__global__ void __launch_bounds__(256)
ssm_prepare_kernel(const SsmArgs a, int save) {
  const int C = a.channels();
  const int c = blockIdx.y * 256 + threadIdx.x;
  const int first = blockIdx.x * NT, last = min(first + NT, a.T);
  if (c >= C) {                         // behind the channels: the heads' step sizes
    const int h = c - C;
    if (h < a.H)
      for (int t = first; t < last; ++t) a.dts[(size_t)h * a.T + t] = a.step(t, h);
    return;
  }
  if (TAPS == 0) {
    const int keep = a.taps - 1;
    for (int t = first; t < last; ++t) {
      const int b = a.tok_seq[t], lt = t - a.cu[b];
      float* st = a.saved(b, c);
      float acc = a.conv_b[c];
      for (int j = 0; j <= keep; ++j) {
        const int back = keep - j;
        const float v = back <= lt ? a.u(t - back)[c] : st[keep - (back - lt)];
        acc = fmaf(a.conv_w[(size_t)j * C + c], v, acc);
      }
      a.xbc[(size_t)t * a.ldx + c] = ssm_silu(acc);
      if (save && keep) {
        for (int j = 0; j + 1 < keep; ++j) st[j] = st[j + 1];
        st[keep - 1] = a.u(t)[c];
      }
    }
    return;
  }
  constexpr int K = TAPS > 1 ? TAPS - 1 : 1;
  float w[TAPS > 0 ? TAPS : 1], back[K];          // back[k]: the input k + 1 tokens before
  float in[NT];
#pragma unroll
  for (int i = 0; i < NT; ++i) in[i] = first + i < last ? a.u(first + i)[c] : 0.f;
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = a.conv_w[(size_t)j * C + c];
  const float bias = a.conv_b[c];
  const bool one = a.tok_seq[first] == a.tok_seq[last - 1];       // all of one sequence
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int t = first + i;
    if (t >= last) break;
    if (i == 0 || !one) {
      const int b = a.tok_seq[t], lt = t - a.cu[b];
      if (i == 0 || lt == 0) {
        const float* st = a.saved(b, c);
#pragma unroll
        for (int k = 0; k < K; ++k) back[k] = k + 1 <= lt ? a.u(t - k - 1)[c] : st[K - (k + 1 - lt)];
      }
    }
    float acc = bias;
#pragma unroll
    for (int k = K; k >= 1; --k) acc = fmaf(w[TAPS > 0 ? TAPS - 1 - k : 0], back[k - 1], acc);
    acc = fmaf(w[TAPS > 0 ? TAPS - 1 : 0], in[i], acc);
    a.xbc[(size_t)t * a.ldx + c] = ssm_silu(acc);
#pragma unroll
    for (int k = K - 1; k > 0; --k) back[k] = back[k - 1];
    back[0] = in[i];
    if (NT == 1 && save) {
      float* st = a.saved(a.tok_seq[t], c);
#pragma unroll
      for (int k = 0; k < K; ++k) st[K - 1 - k] = back[k];
    }
  }
}

int launch_ssm_prepare(const SsmArgs& a, int save, cudaStream_t st) {
  const bool few = a.T <= 256 || save;
  const int tokens = few ? 1 : kSpTokens;
  const dim3 grid((a.T + tokens - 1) / tokens, (a.H * a.e + 2 * a.G * a.N + a.H + 255) / 256);
  if (grid.y > 65535) return kBadArgument;
#define CRETIF_SSM_PREP(TAPS)                                                        \
  do {                                                                               \
    if (few) ssm_prepare_kernel<TAPS, 1><<<grid, 256, 0, st>>>(a, save);             \
    else ssm_prepare_kernel<TAPS, kSpTokens><<<grid, 256, 0, st>>>(a, save);         \
  } while (0)
  if (a.taps == 4) CRETIF_SSM_PREP(4);
  else if (a.taps == 3) CRETIF_SSM_PREP(3);
  else if (a.taps == 2) CRETIF_SSM_PREP(2);
  else CRETIF_SSM_PREP(0);
#undef CRETIF_SSM_PREP
  return launch_status();
}

constexpr int kSsmChunk = 16;

// blockDim.x = ecols * P threads (at most 256), rounded up to whole warps: thread = column * P + part,
// a lane owns R contiguous rows of its column.
template <int R>
__global__ void __launch_bounds__(256)
ssm_token_kernel(const SsmArgs a, int P, int ecols) {
  extern __shared__ __align__(16) float smem[];
  const int b = blockIdx.x, h = blockIdx.y, N = a.N, e = a.e;
  const int col0 = blockIdx.z * ecols;
  const int t0 = a.cu[b], t1 = a.cu[b + 1];
  const int part = threadIdx.x % P, jc = threadIdx.x / P;
  const int col = col0 + jc;
  const bool active = jc < ecols && col < e;
  const int slice = R + 4;                       // a lane's rows of C or B, padded
  float* sc = smem;                              // [chunk][P * slice]
  float* sb = sc + kSsmChunk * P * slice;        // [chunk][P * slice]
  float* sx = sb + kSsmChunk * P * slice;        // [chunk][ecols]
  float* so = sx + kSsmChunk * ecols;            // [chunk][ecols]
  float* sk = so + kSsmChunk * ecols;            // [chunk] decay
  float* sd = sk + kSsmChunk;                    // [chunk] step size
  float* M = a.S(b, h);
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = part * R + r;
    S[r] = (active && i < N) ? M[(size_t)i * e + col] : 0.f;
  }
  const int rows_padded = P * R;
  const int grp = h / (a.H / a.G);
  const int cb = a.inner() + grp * N, cc = cb + a.G * N, cx = h * e;
  const float rate = a.rate(h), skip = a.d_skip[h];
  auto value = [&](int t, int c) { return a.xbc[(size_t)t * a.ldx + c]; };
  for (int c0 = t0; c0 < t1; c0 += kSsmChunk) {
    const int nt = min(kSsmChunk, t1 - c0);
    const float dt = threadIdx.x < nt ? a.dts[(size_t)h * a.T + c0 + threadIdx.x] : 0.f;
    __syncthreads();                             // the chunk before has been read and written out
    for (int idx = threadIdx.x; idx < nt * rows_padded; idx += blockDim.x) {
      const int tt = idx / rows_padded, i = idx - tt * rows_padded;
      const int p = i / R, r = i - p * R, t = c0 + tt;
      sc[(tt * P + p) * slice + r] = i < N ? value(t, cc + i) : 0.f;
      sb[(tt * P + p) * slice + r] = i < N ? value(t, cb + i) : 0.f;
    }
    for (int idx = threadIdx.x; idx < nt * ecols; idx += blockDim.x) {
      const int tt = idx / ecols, j = idx - tt * ecols, t = c0 + tt;
      sx[idx] = col0 + j < e ? value(t, cx + col0 + j) : 0.f;
    }
    if (threadIdx.x < nt) {
      sd[threadIdx.x] = dt;
      sk[threadIdx.x] = expf(rate * dt);
    }
    __syncthreads();
    {
      // every lane goes through the loop (the shuffles want whole warps); lanes beyond the
      // slice work on zeros and store nothing
      const int jv = jc < ecols ? jc : 0;
      for (int tt = 0; tt < nt; ++tt) {
        const float* q = sc + (tt * P + part) * slice;
        const float* k = sb + (tt * P + part) * slice;
        const float keep = sk[tt], x = sx[tt * ecols + jv];
        const float vt = sd[tt] * x;
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
        if (part == 0 && jc < ecols) so[tt * ecols + jc] = fmaf(skip, x, o);
      }
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nt * ecols; idx += blockDim.x) {
      const int tt = idx / ecols, j = idx - tt * ecols;
      if (col0 + j < e) a.y[(size_t)(c0 + tt) * a.inner() + (size_t)h * e + col0 + j] = so[idx];
    }
  }
  if (a.write_state) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = part * R + r;
      if (active && i < N) M[(size_t)i * e + col] = S[r];
    }
  }
}

template <int R>
int launch_ssm_token(const SsmArgs& a, int P, int ecols, cudaStream_t st) {
  const int threads = ((ecols * P + 31) / 32) * 32;
  const size_t smem = sizeof(float) * (kSsmChunk * (2 * (size_t)P * (R + 4) + 2 * (size_t)ecols) +
                                       2 * kSsmChunk);
  auto kern = ssm_token_kernel<R>;
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
// 64 tokens at a time.  Within a chunk let F_t be the sum of a dt up to and with token t, S0 the state
// before the chunk.  Then
//     y_t = exp(F_t) S0^T C_t + sum_{s<=t} exp(F_t - F_s) dt_s (C_t . B_s) x_s + D x_t
//     S_n = exp(F_n) S0 + sum_s exp(F_n - F_s) dt_s B_s x_s^T
// and no exponent is ever above zero.
//
// * ssm_intra_kernel (a CTA per (chunk, few heads of one group); the chunks of all sequences at once):
//   the second and third term to y, the sums F to memory.  The scores C . B are computed once for the
//   CTA's heads.  Nothing here depends on the state, so a long prompt fills the chip.
// * ssm_carry_kernel (a CTA per (sequence, head, EC columns of S)) walks the sequence's chunks with its
//   part of the state in shared memory.
// The matrix products are the retention's (32-bit FMA, 16-byte shared-memory loads, rows padded to
// 4 mod 8 floats).
constexpr int kScTokens = 64;
constexpr int kScThreads = 256;
constexpr int kScScoreLd = kScTokens + 4;
constexpr int kScSlab = 64;             // columns of x the intra kernel takes at a time
constexpr int kScHeads = 8;             // heads an intra CTA takes at most (a warp each scans the sums)

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
__device__ __forceinline__ void ssm_cp16(float* dst, const float* src) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}
template <typename T>
__device__ __forceinline__ void ssm_cp_one(T* dst, const T* src) {      // 4 or 8 bytes
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(a), "l"(src), "n"(sizeof(T))
               : "memory");
}
__device__ __forceinline__ void ssm_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ssm_cp_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

__host__ __device__ inline int ssm_chunk_ld(int n) {
  int ld = n;
  while ((ld & 7) != 4) ++ld;
  return ld;
}
// C and B, whose place the scores and x take once the raw scores are in registers
__host__ __device__ inline size_t ssm_intra_floats(int n) {
  const size_t in = 2 * (size_t)kScTokens * ssm_chunk_ld(n);
  const size_t out = (size_t)kScTokens * (kScScoreLd + kScSlab);
  return in > out ? in : out;
}
inline size_t ssm_intra_smem(int n) {
  return sizeof(double) * kScHeads * kScTokens + sizeof(float) * (kScHeads * kScTokens +
                                                                  ssm_intra_floats(n));
}
// (the 64-bit sums come first, so that they are 8-byte aligned)
inline size_t ssm_carry_smem(int n, int ec, int nbuf) {
  return nbuf * kScTokens * (sizeof(double) + sizeof(float)) +
         sizeof(float) * (nbuf * (2 * (size_t)kScTokens * ssm_chunk_ld(n) + (size_t)kScTokens * ec) +
                          (size_t)n * ec);
}
// The pieces tid, tid + kScThreads, ... of a [rows][n4] block without a division a piece.
struct SsmWalk {
  int row, col, n4, dr, dc;
  __device__ SsmWalk(int tid, int n4_)
      : row(tid / n4_), col(tid % n4_), n4(n4_), dr(kScThreads / n4_), dc(kScThreads % n4_) {}
  __device__ void next() {
    row += dr;
    col += dc;
    if (col >= n4) { col -= n4; ++row; }
  }
};

__global__ void __launch_bounds__(kScThreads)
ssm_intra_kernel(const SsmArgs a, int heads) {
  extern __shared__ __align__(16) float smem[];
  constexpr int C = kScTokens;
  constexpr int LP = kScScoreLd;
  const int tid = threadIdx.x, H = a.H, N = a.N, e = a.e;
  const int h0 = blockIdx.y * heads;
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
  const int ldq = ssm_chunk_ld(N);
  const int n4 = N >> 2;
  double* sF = reinterpret_cast<double*>(smem);          // [heads][C]
  float* sT = reinterpret_cast<float*>(sF + kScHeads * C);   // [heads][C] step sizes
  float* sC = sT + kScHeads * C;                         // [C][ldq]
  float* sB = sC + C * ldq;                              // [C][ldq]
  float* sP = sC;                                        // [C][LP]
  float* sX = sC + C * LP;                               // [C][kScSlab]
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  const int grp = h0 / (H / a.G);
  const int cb = a.inner() + grp * N, cc = cb + a.G * N;
  // Rows beyond the chunk's last token stay as they are: they reach only scores of rows that are
  // not stored, or of keys after the row, which are set to zero.
  for (SsmWalk w(tid, n4); w.row < nt; w.next()) {
    const float* row = a.xbc + (size_t)(c0 + w.row) * a.ldx + 4 * w.col;
    ssm_cp16(sC + w.row * ldq + 4 * w.col, row + cc);
    ssm_cp16(sB + w.row * ldq + 4 * w.col, row + cb);
  }
  ssm_cp_commit();
  for (int hh = tid >> 5; hh < heads; hh += kScThreads / 32) {
    // a head's sums: lane l has tokens 2 l and 2 l + 1
    const int lane = tid & 31, h = h0 + hh;
    const double rate = (double)a.rate(h);
    double f[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int tt = 2 * lane + x;
      const float dt = tt < nt ? a.dts[(size_t)h * a.T + c0 + tt] : 0.f;
      sT[hh * C + tt] = dt;
      f[x] = rate * (double)dt;
    }
    f[1] += f[0];
    double run = f[1];
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, run, off);
      if (lane >= off) run += other;
    }
    double before = __shfl_up_sync(0xffffffffu, run, 1);
    if (lane == 0) before = 0.0;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int tt = 2 * lane + x;
      const double v = before + f[x];
      sF[hh * C + tt] = v;
      if (tt < nt) a.sums[(size_t)h * a.T + c0 + tt] = v;
    }
  }
  ssm_cp_wait<0>();
  __syncthreads();
  const int ti = tid >> 4, si = tid & 15;
  // raw scores: thread (ti, si) owns rows ti + 16 r and keys si + 16 c; key blocks ahead of the
  // row block are never computed
  float raw[4][4];
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) raw[r][c] = 0.f;
  for (int kk = 0; kk < N; kk += 4) {
    float4 q4[4], k4[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      q4[r] = *reinterpret_cast<const float4*>(sC + (ti + 16 * r) * ldq + kk);
      k4[r] = *reinterpret_cast<const float4*>(sB + (si + 16 * r) * ldq + kk);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int c = 0; c <= r; ++c) raw[r][c] = dot4(q4[r], k4[c], raw[r][c]);
  }
  __syncthreads();                       // C and B have been read: their place is free
  for (int hh = 0; hh < heads; ++hh) {
    const int h = h0 + hh;
    const float skip = a.d_skip[h];
    // x, 64 columns at a time: rows beyond the last token and columns beyond the slab are zero (a
    // zero score times whatever lay there must stay zero)
    for (int j0 = 0; j0 < e; j0 += kScSlab) {
      const int width = min(kScSlab, e - j0);            // a multiple of 4
      for (int idx = tid; idx < C * (kScSlab / 4); idx += kScThreads) {
        const int tt = idx >> 4, jg = idx & 15;
        float* dst = sX + tt * kScSlab + 4 * jg;
        if (tt < nt && 4 * jg < width)
          ssm_cp16(dst, a.xbc + (size_t)(c0 + tt) * a.ldx + (size_t)h * e + j0 + 4 * jg);
        else
          *reinterpret_cast<float4*>(dst) = zero4;
      }
      ssm_cp_commit();
      if (j0 == 0) {
        const double* F = sF + hh * C;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const int t = ti + 16 * r;
          const double Ft = F[t];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int s = si + 16 * c;
            sP[t * LP + s] = (c < r || (c == r && si <= ti))
                                 ? raw[r][c] * expf((float)(Ft - F[s])) * sT[hh * C + s] : 0.f;
          }
        }
      }
      ssm_cp_wait<0>();
      __syncthreads();                                   // the slab and the scores are in place
      if (4 * si < width) {
        float4 acc[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) acc[r] = zero4;
        const int smax = min(nt, ti + 49);
        for (int s = 0; s < smax; s += 4) {
          const float4 v0 = *reinterpret_cast<const float4*>(sX + (s + 0) * kScSlab + 4 * si);
          const float4 v1 = *reinterpret_cast<const float4*>(sX + (s + 1) * kScSlab + 4 * si);
          const float4 v2 = *reinterpret_cast<const float4*>(sX + (s + 2) * kScSlab + 4 * si);
          const float4 v3 = *reinterpret_cast<const float4*>(sX + (s + 3) * kScSlab + 4 * si);
#pragma unroll
          for (int r = 0; r < 4; ++r) {
            if (s > ti + 16 * r) continue;               // keys after the row: the scores are zero
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
          if (t < nt) {
            fma4(acc[r], skip, *reinterpret_cast<const float4*>(sX + t * kScSlab + 4 * si));
            *reinterpret_cast<float4*>(a.y + (size_t)(c0 + t) * a.inner() + (size_t)h * e + j0 +
                                       4 * si) = acc[r];
          }
        }
      }
      __syncthreads();                                   // the slab and the scores have been read
    }
  }
}

// Two buffers for C, B and x where they fit (nbuf = 2): a chunk's copies are under way while the chunk
// before is computed.
template <int EC>
__global__ void __launch_bounds__(kScThreads)
ssm_carry_kernel(const SsmArgs a, int nbuf) {
  extern __shared__ __align__(16) float smem[];
  constexpr int C = kScTokens;
  constexpr int CG = EC / 4;               // groups of four columns
  constexpr int NR = kScThreads / CG;      // threads along the rows
  constexpr int RT = C / NR;               // read-out rows a thread
  const int tid = threadIdx.x, H = a.H, N = a.N, e = a.e;
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * EC;
  const int t0 = a.cu[b], t1 = a.cu[b + 1];
  if (t1 <= t0) return;
  const int ldq = ssm_chunk_ld(N);
  const int n4 = N >> 2;
  const int buf_floats = 2 * C * ldq + C * EC;   // C [C][ldq] | B [C][ldq] | x [C][EC]
  double* sums = reinterpret_cast<double*>(smem);           // [nbuf][C] F
  float* steps = reinterpret_cast<float*>(sums + nbuf * C); // [nbuf][C] dt
  float* bufs = steps + nbuf * C;
  float* sS = bufs + nbuf * buf_floats;          // [N][EC]
  const int grp = h / (H / a.G);
  const int cb = a.inner() + grp * N, cc = cb + a.G * N, cx = h * e + col0;
  float* M = a.S(b, h) + col0;
  for (int idx = tid; idx < N * CG; idx += kScThreads) {
    const int i = idx / CG, jg = idx - i * CG;
    *reinterpret_cast<float4*>(sS + i * EC + 4 * jg) =
        *reinterpret_cast<const float4*>(M + (size_t)i * e + 4 * jg);
  }
  const double* F = a.sums + (size_t)h * a.T;
  const float* dts = a.dts + (size_t)h * a.T;
  const int tj = tid % CG, tr = tid / CG;
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  // Rows beyond a chunk's last token are not copied: of C they reach only read-outs that are not
  // stored, of B and x nothing (the update stops at the last token).
  auto stage = [&](int c0, int which) {
    const int nt = min(C, t1 - c0);
    float* buf = bufs + which * buf_floats;
    for (SsmWalk w(tid, n4); w.row < nt; w.next()) {
      const float* row = a.xbc + (size_t)(c0 + w.row) * a.ldx + 4 * w.col;
      float* to = buf + w.row * ldq + 4 * w.col;
      ssm_cp16(to, row + cc);
      ssm_cp16(to + C * ldq, row + cb);
    }
    if (tid < nt) {
      ssm_cp_one(sums + which * C + tid, F + c0 + tid);
      ssm_cp_one(steps + which * C + tid, dts + c0 + tid);
    }
    for (int idx = tid; idx < nt * CG; idx += kScThreads) {
      const int tt = idx / CG, jg = idx - tt * CG;
      ssm_cp16(buf + 2 * C * ldq + tt * EC + 4 * jg,
               a.xbc + (size_t)(c0 + tt) * a.ldx + cx + 4 * jg);
    }
    ssm_cp_commit();
  };
  stage(t0, 0);
  int turn = 0;
  for (int c0 = t0; c0 < t1; c0 += C, ++turn) {
    const int nt = min(C, t1 - c0);
    const bool last = c0 + C >= t1;
    const int which = nbuf == 2 ? (turn & 1) : 0;
    float* sC = bufs + which * buf_floats;
    float* sB = sC + C * ldq;
    float* sX = sB + C * ldq;
    const double* sF = sums + which * C;
    const float* sD = steps + which * C;
    ssm_cp_wait<0>();
    __syncthreads();                       // the chunk is in place; the chunk before is done
    if (nbuf == 2 && !last) stage(c0 + C, which ^ 1);
    const double Fn = sF[nt - 1];
    const float keep = expf((float)Fn);
    {
      // what the state before the chunk gives every row: rows tr + NR r, columns 4 tj .. + 3
      float4 acc[RT], old[RT];
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        acc[r] = zero4;
        const int t = tr + NR * r;
        old[r] = t < nt ? __ldcg(reinterpret_cast<const float4*>(
                              a.y + (size_t)(c0 + t) * a.inner() + cx + 4 * tj))
                        : zero4;
      }
#pragma unroll (RT == 1 ? 4 : 2)
      for (int i = 0; i < N; i += 4) {
        const float4 s0 = *reinterpret_cast<const float4*>(sS + (i + 0) * EC + 4 * tj);
        const float4 s1 = *reinterpret_cast<const float4*>(sS + (i + 1) * EC + 4 * tj);
        const float4 s2 = *reinterpret_cast<const float4*>(sS + (i + 2) * EC + 4 * tj);
        const float4 s3 = *reinterpret_cast<const float4*>(sS + (i + 3) * EC + 4 * tj);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          const float4 q = *reinterpret_cast<const float4*>(sC + (tr + NR * r) * ldq + i);
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
          float4 o = old[r];
          fma4(o, expf((float)sF[t]), acc[r]);
          *reinterpret_cast<float4*>(a.y + (size_t)(c0 + t) * a.inner() + cx + 4 * tj) = o;
        }
      }
    }
    if (last && !a.write_state) break;     // nobody reads the state after the last chunk
    // x takes the weight it has in the state's update (the read-out does not use x)
    for (int idx = tid; idx < nt * CG; idx += kScThreads) {
      const int tt = idx / CG, jg = idx - tt * CG;
      float4 v4 = *reinterpret_cast<float4*>(sX + tt * EC + 4 * jg);
      scale4(v4, expf((float)(Fn - sF[tt])) * sD[tt]);
      *reinterpret_cast<float4*>(sX + tt * EC + 4 * jg) = v4;
    }
    __syncthreads();                       // everybody has read the old state; x is weighted
    // (few rows for many threads: two rows a thread, so that all have some)
    if (n4 < NR) {
      for (int ig = tr; ig < 2 * n4; ig += NR) {
        float* srow = sS + (2 * ig) * EC + 4 * tj;
        float4 a0 = *reinterpret_cast<float4*>(srow);
        float4 a1 = *reinterpret_cast<float4*>(srow + EC);
        scale4(a0, keep);
        scale4(a1, keep);
#pragma unroll 8
        for (int s = 0; s < nt; ++s) {
          const float2 k2 = *reinterpret_cast<const float2*>(sB + s * ldq + 2 * ig);
          const float4 v4 = *reinterpret_cast<const float4*>(sX + s * EC + 4 * tj);
          fma4(a0, k2.x, v4);
          fma4(a1, k2.y, v4);
        }
        *reinterpret_cast<float4*>(srow) = a0;
        *reinterpret_cast<float4*>(srow + EC) = a1;
      }
    } else for (int ig = tr; ig < n4; ig += NR) {
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
        const float4 k4 = *reinterpret_cast<const float4*>(sB + s * ldq + 4 * ig);
        const float4 v4 = *reinterpret_cast<const float4*>(sX + s * EC + 4 * tj);
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
    if (nbuf != 2 && !last) {
      __syncthreads();                     // the one buffer has been read
      stage(c0 + C, 0);
    }
  }
  if (a.write_state) {
    __syncthreads();
    for (int idx = tid; idx < N * CG; idx += kScThreads) {
      const int i = idx / CG, jg = idx - i * CG;
      *reinterpret_cast<float4*>(M + (size_t)i * e + 4 * jg) =
          *reinterpret_cast<const float4*>(sS + i * EC + 4 * jg);
    }
  }
}

template <int EC>
int launch_ssm_carry(const SsmArgs& a, cudaStream_t st) {
  const int nbuf = ssm_carry_smem(a.N, EC, 2) <= 220 * 1024 ? 2 : 1;
  const size_t smem = ssm_carry_smem(a.N, EC, nbuf);
  auto kern = ssm_carry_kernel<EC>;
  if (smem > 48 * 1024) {
    cudaError_t err =
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  kern<<<dim3(a.B, a.H, a.e / EC), kScThreads, smem, st>>>(a, nbuf);
  return launch_status();
}

int launch_ssm_intra(const SsmArgs& a, int sm_count, cudaStream_t st) {
  const size_t smem = ssm_intra_smem(a.N);
  if (smem > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(
        ssm_intra_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  // every sequence has at most one chunk that is not full
  const long long chunks = (long long)a.T / kScTokens + a.B;
  if (chunks > 0x7fffffffLL) return kBadArgument;
  // heads a CTA: those of one group, as many as leave the chip filled twice over
  const int per = a.H / a.G;
  int heads = 1;
  for (int n = 2; n <= kScHeads && n <= per; ++n)
    if (per % n == 0 && chunks * (a.H / n) >= 2LL * sm_count) heads = n;
  ssm_intra_kernel<<<dim3((unsigned)chunks, a.H / heads), kScThreads, smem, st>>>(a, heads);
  return launch_status();
}

// out[t, part] = v / sqrt(mean(v^2) + eps) * w,  v = y silu(z) over the part's channels.  NT threads a
// (token, part): 32 or 256; VEC: four channels at a time, 16 NT of them kept in registers between the
// sum and the store, what lies beyond is computed again.
template <int NT, bool VEC, typename TO>
__global__ void __launch_bounds__(256)
ssm_out_kernel(const SsmArgs a, int parts, const float* __restrict__ norm_w, float eps,
               TO* __restrict__ out, int ldo, long long items) {
  __shared__ float scratch[33];
  const long long item = (long long)blockIdx.x * (256 / NT) + threadIdx.x / NT;
  const int tid = threadIdx.x % NT;
  if (item >= items) return;             // (whole warps; with a CTA an item there is none beyond)
  const int n = a.inner() / parts;
  const int t = (int)(item / parts), c0 = (int)(item - (long long)t * parts) * n;
  const float* y = a.y + (size_t)t * a.inner() + c0;
  const float* z = a.proj + (size_t)t * a.ldp + c0;
  const float* w = norm_w + c0;
  TO* o = out + (size_t)t * ldo + c0;
  auto total = [&](float v) { return NT == 32 ? warp_sum(v) : block_sum(v, scratch); };
  float ss = 0.f;
  if (VEC) {
    constexpr int kKeep = 4;
    const int n4 = n >> 2;
    auto value = [&](int i) {
      float4 v = *reinterpret_cast<const float4*>(y + 4 * i);
      const float4 g = *reinterpret_cast<const float4*>(z + 4 * i);
      v.x *= ssm_silu(g.x); v.y *= ssm_silu(g.y); v.z *= ssm_silu(g.z); v.w *= ssm_silu(g.w);
      return v;
    };
    float4 keep[kKeep];
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int i = u * NT + tid;
      keep[u] = i < n4 ? value(i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss = dot4(keep[u], keep[u], ss);
    }
    for (int i = kKeep * NT + tid; i < n4; i += NT) {
      const float4 v = value(i);
      ss = dot4(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(total(ss) / (float)n + eps);
    auto put = [&](int i, float4 v) {
      const float4 g = *reinterpret_cast<const float4*>(w + 4 * i);
      v.x *= inv * g.x; v.y *= inv * g.y; v.z *= inv * g.z; v.w *= inv * g.w;
      if constexpr (sizeof(TO) == 4) {
        *reinterpret_cast<float4*>(o + 4 * i) = v;
      } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        uint2 p;
        p.x = *reinterpret_cast<uint32_t*>(&lo);
        p.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(o + 4 * i) = p;
      }
    };
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int i = u * NT + tid;
      if (i < n4) put(i, keep[u]);
    }
    for (int i = kKeep * NT + tid; i < n4; i += NT) put(i, value(i));
  } else {
    for (int i = tid; i < n; i += NT) {
      const float v = y[i] * ssm_silu(z[i]);
      ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(total(ss) / (float)n + eps);
    for (int i = tid; i < n; i += NT) o[i] = from_float<TO>(y[i] * ssm_silu(z[i]) * inv * w[i]);
  }
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename TO>
int launch_ssm_out(const SsmArgs& a, int parts, const float* norm_w, float eps, TO* out, int ldo,
                   cudaStream_t st) {
  const int inner = a.H * a.e, n = inner / parts;
  const bool vec = n % 4 == 0 && a.ldp % 4 == 0 && ldo % 4 == 0 && inner % 4 == 0 && aligned16(a.y) &&
                   aligned16(a.proj) && aligned16(norm_w) && aligned16(out);
  const long long items = (long long)a.T * parts;
  const bool warps = n <= 1024 && items >= 1024;
  const long long blocks = warps ? (items + 7) / 8 : items;
  if (blocks > 0x7fffffffLL) return kBadArgument;
  const unsigned grid = (unsigned)blocks;
  if (warps) {
    if (vec) ssm_out_kernel<32, true, TO><<<grid, 256, 0, st>>>(a, parts, norm_w, eps, out, ldo, items);
    else ssm_out_kernel<32, false, TO><<<grid, 256, 0, st>>>(a, parts, norm_w, eps, out, ldo, items);
  } else {
    if (vec) ssm_out_kernel<256, true, TO><<<grid, 256, 0, st>>>(a, parts, norm_w, eps, out, ldo, items);
    else ssm_out_kernel<256, false, TO><<<grid, 256, 0, st>>>(a, parts, norm_w, eps, out, ldo, items);
  }
  return launch_status();
}
}  // namespace
}  // namespace cretif

using namespace cretif;

// form 0 chooses, 1 token by token, 2 chunks (refused where the sizes or addresses rule out 16-byte
// accesses).  Scratch: y [T, H e], xbc [T, ldx] and dts [H, T]; sums (float64) [H, T] for the chunks.  save_inputs: the step brings one token a sequence and the saved inputs are brought up to
// date here.
extern "C" int cretif_state_space(const float* proj, int ldp, const float* conv_w, const float* conv_b,
                                  int taps, const float* a_log, const float* dt_bias,
                                  const float* d_skip, float* state, long long state_stride,
                                  long long inputs_at, const int* cu_seqlens, const int* seq_slot,
                                  const int* tok_seq, int B, int H, int G, int N, int e, float* y,
                                  float* xbc, int ldx, float* dts, double* sums, int parts,
                                  const float* norm_w, float eps, void* out, int out_dt, int ldo,
                                  int write_state, int save_inputs, int T, int form, void* stream) {
  if (B <= 0 || T <= 0) return kOk;
  if (H <= 0 || G <= 0 || H % G || N <= 0 || e <= 0 || taps < 1 || parts <= 0 || (H * e) % parts ||
      !proj || !conv_w || !conv_b || !a_log || !dt_bias || !d_skip || !state || !norm_w || !y || !xbc || !dts ||
      form < 0 || form > 2)
    return kBadArgument;
  const int inner = H * e, C = inner + 2 * G * N;
  if (ldp < inner + C + H || ldo < inner || inputs_at < (long long)H * N * e ||
      state_stride < inputs_at + (long long)C * (taps - 1) || ldx < C ||
      (save_inputs && T != B))
    return kBadArgument;
  static int sm_count = 0;
  if (!sm_count) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sm_count, cudaDevAttrMultiProcessorCount, dev);
    if (sm_count <= 0) sm_count = 148;
  }
  cudaStream_t st = (cudaStream_t)stream;
  const SsmArgs a{proj, ldp, conv_w, conv_b, taps, a_log, dt_bias, d_skip, state, (size_t)state_stride,
                  (size_t)inputs_at, cu_seqlens, seq_slot, tok_seq, B, H, G, N, e, T, y, xbc, ldx, dts,
                  sums, write_state};
  int rc = launch_ssm_prepare(a, save_inputs && taps > 1, st);
  if (rc != kOk) return rc;
  bool done = false;
  // 64 tokens at a time where the step brings a sequence 16 tokens or more on average and the
  // sizes allow 16-byte accesses throughout; token by token otherwise.
  if (form == 2 || (form == 0 && (long long)T >= 16LL * B)) {
    const bool fits = N % 4 == 0 && e % 16 == 0 && state_stride % 4 == 0 && sums && ldx % 4 == 0 && aligned16(xbc) && aligned16(state) && aligned16(y) &&
                      H <= 65535 && ssm_carry_smem(N, 16, 1) <= 220 * 1024 &&
                      ssm_intra_smem(N) <= 220 * 1024;
    if (fits) {
      rc = launch_ssm_intra(a, sm_count, st);
      if (rc != kOk) return rc;
      // columns a CTA: a chunk takes about 40 + columns units of time, a wave of CTAs (one an SM) a
      // chunk after the other (measured with N = 128: 205, 250 and 390 us for 2,048 tokens at 16, 32
      // and 64 columns)
      int ec = 16;
      double best = 0.0;
      for (int n = 16; n <= 64 && e % n == 0 && ssm_carry_smem(N, n, 1) <= 220 * 1024; n *= 2) {
        const double waves = (double)B * H * (e / n) / sm_count;
        const double cost = (waves > 1.0 ? waves : 1.0) * (40 + n);
        if (n == 16 || cost < best) { best = cost; ec = n; }
      }
      rc = ec == 64   ? launch_ssm_carry<64>(a, st)
           : ec == 32 ? launch_ssm_carry<32>(a, st)
                      : launch_ssm_carry<16>(a, st);
      if (rc != kOk) return rc;
      done = true;
    } else if (form == 2) {
      return kBadArgument;
    }
  }
  if (!done) {
    // R rows a lane (a power of two from 4 to 32, about a quarter of N), P lanes a column
    int R = 4;
    while (R < 32 && R * 4 < N) R *= 2;
    int P = 1;
    while (P < 32 && P * R < N) P *= 2;
    if (P * R < N) return kBadArgument;            // N > 1024
    // columns a CTA: a head's columns are cut into slices while the (sequence, head) pairs alone
    // do not fill the chip twice over, down to two warps a CTA, and as far as 256 threads demand
    int ecols = e;
    while (ecols * P > 256) ecols = (ecols + 1) / 2;
    while ((long long)B * H * ((e + ecols - 1) / ecols) < 2LL * sm_count && ecols * P >= 128 &&
           ecols % 2 == 0)
      ecols /= 2;
    rc = R == 4    ? launch_ssm_token<4>(a, P, ecols, st)
         : R == 8  ? launch_ssm_token<8>(a, P, ecols, st)
         : R == 16 ? launch_ssm_token<16>(a, P, ecols, st)
                   : launch_ssm_token<32>(a, P, ecols, st);
    if (rc != kOk) return rc;
  }
  if (out_dt == kF32)
    return launch_ssm_out(a, parts, norm_w, eps, (float*)out, ldo, st);
  if (out_dt == kBF16)
    return launch_ssm_out(a, parts, norm_w, eps, (__nv_bfloat16*)out, ldo, st);
  return kBadDType;
}
