// Norms that sit elsewhere than in front of a sublayer.
//
// * rmsnorm_add: a norm on a sublayer's OUTPUT, fused with the residual addition:
//   h[t] += y[t] * w * rsqrt(mean(y[t]^2) + eps).  Sum, scaling and addition are 32-bit.  The
//   kernel can also leave the new rows in bfloat16 for the sublayer that reads them next.
// * add_layernorm: the norm with the mean taken off and a bias, in front of a sublayer, fused with the
//   residual addition that precedes it (the RMS norm's counterpart is in elementwise.cu).
// * convert_rows: the residual stream handed to a sublayer that reads it without a norm
//   (float32 -> the compute type).
// * proj_norm_kv_append: RMS norms over whole query / key projections (all heads of a token
//   at once, one weight per channel), fused with the write into the block cache.  The key
//   part of a row is normed and stored as the key; when a value cache is given, the SAME
//   columns as projected (before the norm) are stored as the value: a layer whose values are
//   its keys needs no value projection.  Without query weights the query part is left alone,
//   without a value cache only keys are stored (a latent that serves as key and value).
#include "api.h"
#include "common.cuh"

namespace cretif {

namespace {
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u),
                     __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void st4_bf16(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&lo);
  u.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}
}  // namespace

// A warp per row, no block-wide barrier.  VEC: rows are read and written four columns at a time
// (H and the row strides multiples of 4, 16-byte aligned bases) and a row of up to 2048 columns
// stays in registers between the sum of squares and the addition; every loop is unrolled so
// that a lane's loads are in flight together (a step of one token is one warp, and a loop that
// waited for each load in turn took longer than the product before it).
template <typename TY, bool VEC>
__global__ void __launch_bounds__(256)
rmsnorm_add_kernel(float* __restrict__ h, const TY* __restrict__ y, int ldy,
                   const float* __restrict__ weight, int R, int H, float eps,
                   __nv_bfloat16* __restrict__ x_out) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.x * 8 + warp;
  if (r >= R) return;
  const TY* yrow = y + (size_t)r * ldy;
  float* hrow = h + (size_t)r * H;
  __nv_bfloat16* xrow = x_out ? x_out + (size_t)r * H : nullptr;
  if (VEC) {
    constexpr int kKeep = 16;
    const int n4 = H >> 2;
    float4 keep[kKeep];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int i = u * 32 + lane;
      keep[u] = i < n4 ? ld4(yrow + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[u].x * keep[u].x + keep[u].y * keep[u].y + keep[u].z * keep[u].z +
            keep[u].w * keep[u].w;
    }
#pragma unroll 4
    for (int i = kKeep * 32 + lane; i < n4; i += 32) {
      const float4 v = ld4(yrow + 4 * i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int i = u * 32 + lane;
      if (i < n4) {
        const float4 w = ld4(weight + 4 * i);
        float4 v = ld4(hrow + 4 * i);
        v.x += keep[u].x * inv * w.x; v.y += keep[u].y * inv * w.y;
        v.z += keep[u].z * inv * w.z; v.w += keep[u].w * inv * w.w;
        *reinterpret_cast<float4*>(hrow + 4 * i) = v;
        if (xrow) st4_bf16(xrow + 4 * i, v);
      }
    }
#pragma unroll 4
    for (int i = kKeep * 32 + lane; i < n4; i += 32) {
      const float4 w = ld4(weight + 4 * i), a = ld4(yrow + 4 * i);
      float4 v = ld4(hrow + 4 * i);
      v.x += a.x * inv * w.x; v.y += a.y * inv * w.y; v.z += a.z * inv * w.z; v.w += a.w * inv * w.w;
      *reinterpret_cast<float4*>(hrow + 4 * i) = v;
      if (xrow) st4_bf16(xrow + 4 * i, v);
    }
    return;
  }
  float ss = 0.f;
#pragma unroll 8
  for (int i = lane; i < H; i += 32) {
    const float v = to_float(yrow[i]);
    ss += v * v;
  }
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
#pragma unroll 8
  for (int i = lane; i < H; i += 32) {
    const float v = hrow[i] + to_float(yrow[i]) * inv * weight[i];
    hrow[i] = v;
    if (xrow) xrow[i] = __float2bfloat16_rn(v);
  }
}

// The same for few rows (a decode step): a CTA per row, four columns a thread and turn, everything a
// thread reads asked for before the row's sum is known.  Up to 2 x 1024 columns stay in registers.
template <typename TY>
__global__ void __launch_bounds__(256)
rmsnorm_add_row_block_kernel(float* __restrict__ h, const TY* __restrict__ y, int ldy,
                             const float* __restrict__ weight, int H, float eps,
                             __nv_bfloat16* __restrict__ x_out) {
  __shared__ float sums[8];
  const int r = blockIdx.x, tid = threadIdx.x, n4 = H >> 2;
  const TY* yrow = y + (size_t)r * ldy;
  float* hrow = h + (size_t)r * H;
  __nv_bfloat16* xrow = x_out ? x_out + (size_t)r * H : nullptr;
  constexpr int kKeep = 2;
  float4 a[kKeep], w[kKeep], v[kKeep];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * 256 + tid;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    a[u] = i < n4 ? ld4(yrow + 4 * i) : zero;
    w[u] = i < n4 ? ld4(weight + 4 * i) : zero;
    v[u] = i < n4 ? ld4(hrow + 4 * i) : zero;
    ss += a[u].x * a[u].x + a[u].y * a[u].y + a[u].z * a[u].z + a[u].w * a[u].w;
  }
  for (int i = kKeep * 256 + tid; i < n4; i += 256) {
    const float4 b = ld4(yrow + 4 * i);
    ss += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) sums[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int u = 0; u < 8; ++u) ss += sums[u];
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  auto put = [&](int i, float4 b, float4 g, float4 t) {
    t.x += b.x * inv * g.x; t.y += b.y * inv * g.y;
    t.z += b.z * inv * g.z; t.w += b.w * inv * g.w;
    *reinterpret_cast<float4*>(hrow + 4 * i) = t;
    if (xrow) st4_bf16(xrow + 4 * i, t);
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * 256 + tid;
    if (i < n4) put(i, a[u], w[u], v[u]);
  }
  for (int i = kKeep * 256 + tid; i < n4; i += 256)
    put(i, ld4(yrow + 4 * i), ld4(weight + 4 * i), ld4(hrow + 4 * i));
}

// Layer norm: v = h[src] (+ delta[src]); h[src] = v when write_h;
// out[r] = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w + b.  NT threads a row: 32 (many rows) or
// 256 (fewer, a CTA each).  A row of up to 2048 columns stays in the threads' registers between
// the sums (VEC); beyond that, and without VEC, it is read again.
template <int NT, bool VEC, typename TD, typename TO>
__global__ void __launch_bounds__(256)
add_layernorm_kernel(float* h, const TD* __restrict__ delta, const float* __restrict__ weight,
                     const float* __restrict__ bias, TO* __restrict__ out,
                     const int* __restrict__ rows, int R, int H, float eps, int write_h) {
  __shared__ float scratch[33];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int r = blockIdx.x * (256 / NT) + threadIdx.x / NT, tid = threadIdx.x % NT;
  constexpr int kKeep = 512 / NT;
  const int n4 = VEC ? H >> 2 : 0;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w[NT == 256 ? kKeep : 1], b[NT == 256 ? kKeep : 1];
  if (VEC && NT == 256) {             // (they do not wait for the kernel before)
#pragma unroll
    for (int u = 0; u < kKeep; ++u) {
      const int i = u * NT + tid;
      w[NT == 256 ? u : 0] = i < n4 ? ld4(weight + 4 * i) : zero;
      b[NT == 256 ? u : 0] = i < n4 ? ld4(bias + 4 * i) : zero;
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  if (r >= R) return;                 // (whole warps; with a CTA a row there is none beyond R)
  auto total = [&](float v) { return NT == 32 ? warp_sum(v) : block_sum(v, scratch); };
  const int src = rows ? rows[r] : r;
  float* hrow = h + (size_t)src * H;
  const TD* drow = delta ? delta + (size_t)src * H : nullptr;
  TO* orow = out + (size_t)r * H;
  if (!VEC) {
    auto value = [&](int i) { return hrow[i] + (drow ? to_float(drow[i]) : 0.f); };
    float s = 0.f, ss = 0.f;
    for (int i = tid; i < H; i += NT) s += value(i);
    const float mean = total(s) / (float)H;
    for (int i = tid; i < H; i += NT) { const float d = value(i) - mean; ss += d * d; }
    const float inv = rsqrtf(total(ss) / (float)H + eps);
    for (int i = tid; i < H; i += NT) {
      const float v = value(i);       // (read before the same thread replaces it)
      if (write_h) hrow[i] = v;
      orow[i] = from_float<TO>((v - mean) * inv * weight[i] + bias[i]);
    }
    return;
  }
  auto value = [&](int i) {
    float4 v = ld4(hrow + 4 * i);
    if (drow) {
      const float4 d = ld4(drow + 4 * i);
      v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
    }
    return v;
  };
  auto squares = [](const float4& v, float m) {
    const float a = v.x - m, c = v.y - m, d = v.z - m, e = v.w - m;
    return a * a + c * c + d * d + e * e;
  };
  float4 keep[kKeep];
  float s = 0.f, ss = 0.f;
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * NT + tid;
    keep[u] = i < n4 ? value(i) : zero;
    s += (keep[u].x + keep[u].y) + (keep[u].z + keep[u].w);
  }
  for (int i = kKeep * NT + tid; i < n4; i += NT) {
    const float4 v = value(i);
    s += (v.x + v.y) + (v.z + v.w);
  }
  const float mean = total(s) / (float)H;
#pragma unroll
  for (int u = 0; u < kKeep; ++u)
    if (u * NT + tid < n4) ss += squares(keep[u], mean);
  for (int i = kKeep * NT + tid; i < n4; i += NT) ss += squares(value(i), mean);
  const float inv = rsqrtf(total(ss) / (float)H + eps);
  auto put = [&](int i, const float4& v, const float4& g, const float4& c) {
    if (write_h) *reinterpret_cast<float4*>(hrow + 4 * i) = v;
    const float4 y = make_float4((v.x - mean) * inv * g.x + c.x, (v.y - mean) * inv * g.y + c.y,
                                 (v.z - mean) * inv * g.z + c.z, (v.w - mean) * inv * g.w + c.w);
    if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(orow + 4 * i) = y;
    else st4_bf16(orow + 4 * i, y);
  };
#pragma unroll
  for (int u = 0; u < kKeep; ++u) {
    const int i = u * NT + tid;
    if (i < n4)
      put(i, keep[u], NT == 256 ? w[NT == 256 ? u : 0] : ld4(weight + 4 * i),
          NT == 256 ? b[NT == 256 ? u : 0] : ld4(bias + 4 * i));
  }
  for (int i = kKeep * NT + tid; i < n4; i += NT)
    put(i, value(i), ld4(weight + 4 * i), ld4(bias + 4 * i));
}

template <typename TD, typename TO>
static int launch_layernorm(float* h, const TD* delta, const float* w, const float* b, TO* out,
                            const int* rows, int R, int H, float eps, int write_h, cudaStream_t st) {
  const bool vec = H % 4 == 0 && (((uintptr_t)h | (uintptr_t)delta | (uintptr_t)w | (uintptr_t)b |
                                   (uintptr_t)out) & 15) == 0;
  cudaLaunchConfig_t cfg = {};
  // a CTA a row while the rows are few for the chip, a warp a row beyond (measured at width 2,048:
  // 24.6 against 27.6 us for 2,048 rows, 74.8 against 58.3 us for 16,384)
  const bool cta = R < 256 || (H >= 1024 && R < 8192);
  cfg.gridDim = dim3(cta ? R : (R + 7) / 8);
  cfg.blockDim = dim3(256);
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = dependent_launch_enabled();
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  cudaError_t e;
  if (cta)
    e = vec ? cudaLaunchKernelEx(&cfg, add_layernorm_kernel<256, true, TD, TO>, h, delta, w, b, out,
                                 rows, R, H, eps, write_h)
            : cudaLaunchKernelEx(&cfg, add_layernorm_kernel<256, false, TD, TO>, h, delta, w, b, out,
                                 rows, R, H, eps, write_h);
  else
    e = vec ? cudaLaunchKernelEx(&cfg, add_layernorm_kernel<32, true, TD, TO>, h, delta, w, b, out,
                                 rows, R, H, eps, write_h)
            : cudaLaunchKernelEx(&cfg, add_layernorm_kernel<32, false, TD, TO>, h, delta, w, b, out,
                                 rows, R, H, eps, write_h);
  return e == cudaSuccess ? launch_status() : (int)e;
}

template <typename TO>
__global__ void convert_rows_kernel(const float* __restrict__ h, TO* __restrict__ out,
                                    size_t total) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < total) out[i] = from_float<TO>(h[i]);
}

// The same into some columns of a wider matrix, V columns a thread.
template <typename TO, int V>
__global__ void __launch_bounds__(256)
convert_into_kernel(const float* __restrict__ h, TO* __restrict__ out, int ldo, int H, long long total) {
  const long long idx = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (idx >= total) return;
  const long long r = idx / H;
  TO* to = out + (size_t)r * ldo + (size_t)(idx - r * H);
  if constexpr (V == 4) {
    const float4 v = ld4(h + idx);
    if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(to) = v;
    else st4_bf16(to, v);
  } else {
    *to = from_float<TO>(h[idx]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
proj_norm_kv_append_kernel(T* __restrict__ row0, int ld, int q_dim, const float* __restrict__ wq,
                           int nkv, int hd, const float* __restrict__ wk, float eps,
                           const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                           const int* __restrict__ seq_slot, const int* __restrict__ table,
                           int table_stride, T* __restrict__ kc, T* __restrict__ vc, int bt,
                           int write_cache, unsigned int* __restrict__ fault) {
  __shared__ float scratch[33];
  const int t = blockIdx.x;
  T* row = row0 + (size_t)t * ld;
  const int kv_dim = nkv * hd;
  if (wq) {
    float ss = 0.f;
#pragma unroll 4
    for (int i = threadIdx.x; i < q_dim; i += blockDim.x) {
      const float v = to_float(row[i]);
      ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)q_dim + eps);
#pragma unroll 4
    for (int i = threadIdx.x; i < q_dim; i += blockDim.x)
      row[i] = from_float<T>(to_float(row[i]) * inv * wq[i]);
  }
  T* krow = row + q_dim;
  float ss = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x; i < kv_dim; i += blockDim.x) {
    const float v = to_float(krow[i]);
    ss += v * v;
  }
  ss = block_sum(ss, scratch);
  if (!write_cache) return;
  const float inv = 1.0f / sqrtf(ss / (float)kv_dim + eps);
  const int pos = tok_pos[t];
  const int slot = seq_slot[tok_seq[t]];
  const int blk = table[(size_t)slot * table_stride + pos / bt];
  if (blk < 0) {
    if (threadIdx.x == 0) atomicOr(fault, kFaultBlockTable);
    return;
  }
  const size_t cache_row = (size_t)blk * nkv * bt + (pos % bt);
#pragma unroll 4
  for (int i = threadIdx.x; i < kv_dim; i += blockDim.x) {
    const int kvh = i / hd, d = i - kvh * hd;
    const size_t at = (cache_row + (size_t)kvh * bt) * hd + d;
    const T raw = krow[i];
    kc[at] = from_float<T>(to_float(raw) * inv * wk[i]);
    if (vc) vc[at] = raw;
  }
}

}  // namespace cretif

using namespace cretif;

extern "C" int cretif_rmsnorm_add(float* h, const void* y, int y_dt, int ldy, const float* weight,
                                  int R, int H, float eps, void* x_out, void* stream) {
  if (R <= 0) return kOk;
  if (H <= 0 || ldy < H) return kBadArgument;
  cudaStream_t st = (cudaStream_t)stream;
  const unsigned blocks = (unsigned)((R + 7) / 8);
  const bool vec = H % 4 == 0 && ldy % 4 == 0 &&
                   (((uintptr_t)h | (uintptr_t)y | (uintptr_t)weight | (uintptr_t)x_out) & 15) == 0;
  __nv_bfloat16* xo = (__nv_bfloat16*)x_out;
  if (vec && R < 256 && H >= 512) {
    if (y_dt == kF32)
      rmsnorm_add_row_block_kernel<float><<<R, 256, 0, st>>>(h, (const float*)y, ldy, weight, H, eps, xo);
    else if (y_dt == kBF16)
      rmsnorm_add_row_block_kernel<__nv_bfloat16><<<R, 256, 0, st>>>(h, (const __nv_bfloat16*)y, ldy,
                                                                     weight, H, eps, xo);
    else
      return kBadDType;
    return launch_status();
  }
  if (y_dt == kF32) {
    if (vec) rmsnorm_add_kernel<float, true><<<blocks, 256, 0, st>>>(h, (const float*)y, ldy, weight, R, H, eps, xo);
    else rmsnorm_add_kernel<float, false><<<blocks, 256, 0, st>>>(h, (const float*)y, ldy, weight, R, H, eps, xo);
  } else if (y_dt == kBF16) {
    typedef __nv_bfloat16 bf16;
    if (vec) rmsnorm_add_kernel<bf16, true><<<blocks, 256, 0, st>>>(h, (const bf16*)y, ldy, weight, R, H, eps, xo);
    else rmsnorm_add_kernel<bf16, false><<<blocks, 256, 0, st>>>(h, (const bf16*)y, ldy, weight, R, H, eps, xo);
  } else {
    return kBadDType;
  }
  return launch_status();
}

extern "C" int cretif_add_layernorm(float* h, const void* delta, int delta_dt, const float* weight,
                                    const float* bias, void* out, int out_dt, const int* rows, int R,
                                    int H, float eps, int write_h, void* stream) {
  if (R <= 0) return kOk;
  if (H <= 0 || !weight || !bias || (rows && write_h)) return kBadArgument;
  if ((delta && delta_dt != kF32 && delta_dt != kBF16) || (out_dt != kF32 && out_dt != kBF16))
    return kBadDType;
  cudaStream_t st = (cudaStream_t)stream;
  typedef __nv_bfloat16 bf16;
  const bool dbf = delta && delta_dt == kBF16;
  if (out_dt == kF32)
    return dbf ? launch_layernorm(h, (const bf16*)delta, weight, bias, (float*)out, rows, R, H, eps,
                                  write_h, st)
               : launch_layernorm(h, (const float*)delta, weight, bias, (float*)out, rows, R, H, eps,
                                  write_h, st);
  return dbf ? launch_layernorm(h, (const bf16*)delta, weight, bias, (bf16*)out, rows, R, H, eps,
                                write_h, st)
             : launch_layernorm(h, (const float*)delta, weight, bias, (bf16*)out, rows, R, H, eps,
                                write_h, st);
}

extern "C" int cretif_convert_rows(const float* h, void* out, int out_dt, long long total,
                                   void* stream) {
  if (total <= 0) return kOk;
  cudaStream_t st = (cudaStream_t)stream;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  if (out_dt == kF32)
    convert_rows_kernel<float><<<blocks, 256, 0, st>>>(h, (float*)out, (size_t)total);
  else if (out_dt == kBF16)
    convert_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(h, (__nv_bfloat16*)out,
                                                              (size_t)total);
  else
    return kBadDType;
  return launch_status();
}

extern "C" int cretif_convert_into(const float* h, void* out, int out_dt, int ldo, int R, int H,
                                   void* stream) {
  if (R <= 0) return kOk;
  if (H <= 0 || ldo < H) return kBadArgument;
  if (out_dt != kF32 && out_dt != kBF16) return kBadDType;
  cudaStream_t st = (cudaStream_t)stream;
  const long long total = (long long)R * H;
  const bool vec = H % 4 == 0 && ldo % 4 == 0 && (((uintptr_t)h | (uintptr_t)out) & 15) == 0;
  const unsigned blocks = (unsigned)(((vec ? total / 4 : total) + 255) / 256);
  if (out_dt == kF32) {
    if (vec) convert_into_kernel<float, 4><<<blocks, 256, 0, st>>>(h, (float*)out, ldo, H, total);
    else convert_into_kernel<float, 1><<<blocks, 256, 0, st>>>(h, (float*)out, ldo, H, total);
  } else {
    typedef __nv_bfloat16 bf16;
    if (vec) convert_into_kernel<bf16, 4><<<blocks, 256, 0, st>>>(h, (bf16*)out, ldo, H, total);
    else convert_into_kernel<bf16, 1><<<blocks, 256, 0, st>>>(h, (bf16*)out, ldo, H, total);
  }
  return launch_status();
}

extern "C" int cretif_proj_norm_kv_append(void* rows, int ld, int dt, int q_dim, const float* wq,
                                          int nkv, int hd, const float* wk, float eps,
                                          const int* tok_pos, const int* tok_seq,
                                          const int* seq_slot, const int* table, int table_stride,
                                          void* kc, void* vc, int bt, int write_cache, int T,
                                          unsigned int* fault, void* stream) {
  if (T <= 0) return kOk;
  if (q_dim < 0 || nkv <= 0 || hd <= 0 || bt <= 0 || ld < q_dim + nkv * hd || !wk)
    return kBadArgument;
  cudaStream_t st = (cudaStream_t)stream;
  if (dt == kF32)
    proj_norm_kv_append_kernel<float><<<T, 256, 0, st>>>(
        (float*)rows, ld, q_dim, wq, nkv, hd, wk, eps, tok_pos, tok_seq, seq_slot, table,
        table_stride, (float*)kc, (float*)vc, bt, write_cache, fault);
  else if (dt == kBF16)
    proj_norm_kv_append_kernel<__nv_bfloat16><<<T, 256, 0, st>>>(
        (__nv_bfloat16*)rows, ld, q_dim, wq, nkv, hd, wk, eps, tok_pos, tok_seq, seq_slot, table,
        table_stride, (__nv_bfloat16*)kc, (__nv_bfloat16*)vc, bt, write_cache, fault);
  else
    return kBadDType;
  return launch_status();
}
