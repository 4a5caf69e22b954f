// Residual streams: the layers work on `S` rows per token instead of one.  x float32 [S, n, D], plane s holding stream s.
//
//   stream_norm:  u = sum_s a[s] x_s,  y = rms(u) * w                        what a sublayer reads (a null: ones)
//   stream_step:  x_t <- sum_s mix[s, t] x_s + out[t] * y  for all t at once from the old x, then, with a second set of
//                 weights, the same u and norm of the NEW streams for the sublayer that reads them next: the streams are
//                 read once and written once per sublayer, and the next sublayer's input costs no pass of its own.
//
// Everything is float32; only the normalised rows leave in the run dtype.  One block per row; sums over the streams run in
// the order of the streams, the sum of squares in an order that the thread layout alone fixes, so a row's result does not
// depend on the batch.
#include "common.cuh"
#include <stdint.h>

#define ST_MAX 16      // most streams
#define ST_KEEP 4      // float4s of u a thread keeps between the sum of squares and the scaling

template <typename TO>
__device__ __forceinline__ void put4(TO* y, int d4, float4 v) {
  if constexpr (sizeof(TO) == 4) {
    reinterpret_cast<float4*>(y)[d4] = v;
  } else {
    __nv_bfloat162 p[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    reinterpret_cast<uint2*>(y)[d4] = *reinterpret_cast<const uint2*>(p);
  }
}

__device__ __forceinline__ void axpy4(float a, const float4& v, float4& acc) {
  acc.x = fmaf(a, v.x, acc.x);
  acc.y = fmaf(a, v.y, acc.y);
  acc.z = fmaf(a, v.z, acc.z);
  acc.w = fmaf(a, v.w, acc.w);
}

// The shared tail: u of this thread's float4s -> y = rms(u) * w.
template <typename TO>
__device__ __forceinline__ void norm_tail(const float4 (&u)[ST_KEEP], int n4, int dim, const float* __restrict__ w, TO* __restrict__ yr,
                                          float eps, float* scratch) {
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ST_KEEP; ++i) {
    ss = fmaf(u[i].x, u[i].x, ss);
    ss = fmaf(u[i].y, u[i].y, ss);
    ss = fmaf(u[i].z, u[i].z, ss);
    ss = fmaf(u[i].w, u[i].w, ss);
  }
  ss = block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)dim + eps);
#pragma unroll
  for (int i = 0; i < ST_KEEP; ++i) {
    const int d = threadIdx.x + i * blockDim.x;
    if (d >= n4) continue;
    const float4 wv = reinterpret_cast<const float4*>(w)[d];
    put4(yr, d, make_float4((u[i].x * scale) * wv.x, (u[i].y * scale) * wv.y, (u[i].z * scale) * wv.z, (u[i].w * scale) * wv.w));
  }
}

// 16-byte form: dim a multiple of 4, at most ST_KEEP float4s a thread.  rows: the token rows wanted (null: all).
template <typename TO>
__global__ void stream_norm_vec4_kernel(const float* __restrict__ x, size_t plane, const float* __restrict__ a, int S,
                                        const int* __restrict__ rows, const float* __restrict__ w, TO* __restrict__ y, int dim,
                                        float eps) {
  __shared__ float scratch[32];
  zk_let_next_start();
  zk_wait_prior();
  const int r = blockIdx.x, n4 = dim >> 2;
  const float* xr = x + (size_t)(rows ? rows[r] : r) * dim;
  float4 u[ST_KEEP];
#pragma unroll
  for (int i = 0; i < ST_KEEP; ++i) u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s = 0; s < S; ++s) {
    const float as = a ? a[s] : 1.0f;
    const float4* p = reinterpret_cast<const float4*>(xr + s * plane);
#pragma unroll
    for (int i = 0; i < ST_KEEP; ++i) {
      const int d = threadIdx.x + i * blockDim.x;
      if (d < n4) axpy4(as, p[d], u[i]);
    }
  }
  norm_tail(u, n4, dim, w, y + (size_t)r * dim, eps, scratch);
}

template <typename TO, int S>
__global__ void stream_step_vec4_kernel(float* __restrict__ x, size_t plane, const float* __restrict__ y, const float* __restrict__ mix,
                                        const float* __restrict__ out, const float* __restrict__ a, const float* __restrict__ w,
                                        TO* __restrict__ h, int dim, float eps, int want_norm) {
  __shared__ float scratch[32];
  // what no kernel writes: the weights of the mix
  float m[S][S], o[S], an[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    o[s] = out[s];
    an[s] = a ? a[s] : 1.0f;
#pragma unroll
    for (int t = 0; t < S; ++t) m[s][t] = mix[s * S + t];
  }
  zk_let_next_start();
  zk_wait_prior();
  const int r = blockIdx.x, n4 = dim >> 2;
  float* xr = x + (size_t)r * dim;
  const float4* yr = reinterpret_cast<const float4*>(y + (size_t)r * dim);
  float4 u[ST_KEEP];
#pragma unroll
  for (int i = 0; i < ST_KEEP; ++i) {
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    const int d = threadIdx.x + i * blockDim.x;
    if (d >= n4) continue;
    float4 old[S];
#pragma unroll
    for (int s = 0; s < S; ++s) old[s] = reinterpret_cast<const float4*>(xr + s * plane)[d];
    const float4 yv = yr[d];
#pragma unroll
    for (int t = 0; t < S; ++t) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < S; ++s) axpy4(m[s][t], old[s], v);
      axpy4(o[t], yv, v);
      reinterpret_cast<float4*>(xr + t * plane)[d] = v;
      axpy4(an[t], v, u[i]);
    }
  }
  if (want_norm) norm_tail(u, n4, dim, w, h + (size_t)r * dim, eps, scratch);
}

// Any width, any number of streams up to ST_MAX; u is formed twice.
template <typename TO>
__global__ void stream_norm_kernel(const float* __restrict__ x, size_t plane, const float* __restrict__ a, int S,
                                   const int* __restrict__ rows, const float* __restrict__ w, TO* __restrict__ y, int dim, float eps) {
  __shared__ float scratch[32];
  zk_let_next_start();
  zk_wait_prior();
  const int r = blockIdx.x;
  const float* xr = x + (size_t)(rows ? rows[r] : r) * dim;
  auto read = [&](int d) {
    float u = 0.f;
    for (int s = 0; s < S; ++s) u = fmaf(a ? a[s] : 1.0f, xr[s * plane + d], u);
    return u;
  };
  float ss = 0.f;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) {
    const float u = read(d);
    ss = fmaf(u, u, ss);
  }
  ss = block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)dim + eps);
  for (int d = threadIdx.x; d < dim; d += blockDim.x) y[(size_t)r * dim + d] = from_f32<TO>((read(d) * scale) * w[d]);
}

template <typename TO>
__global__ void stream_step_kernel(float* __restrict__ x, size_t plane, const float* __restrict__ y, const float* __restrict__ mix,
                                   const float* __restrict__ out, int S, const float* __restrict__ a, const float* __restrict__ w,
                                   TO* __restrict__ h, int dim, float eps, int want_norm) {
  __shared__ float scratch[32];
  zk_let_next_start();
  zk_wait_prior();
  const int r = blockIdx.x;
  float* xr = x + (size_t)r * dim;
  float ss = 0.f;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) {
    float old[ST_MAX], u = 0.f;
    const float yv = y[(size_t)r * dim + d];
    for (int s = 0; s < S; ++s) old[s] = xr[s * plane + d];
    for (int t = 0; t < S; ++t) {
      float v = 0.f;
      for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + t], old[s], v);
      v = fmaf(out[t], yv, v);
      xr[t * plane + d] = v;
      u = fmaf(a ? a[t] : 1.0f, v, u);
    }
    ss = fmaf(u, u, ss);
  }
  if (!want_norm) return;
  ss = block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)dim + eps);
  for (int d = threadIdx.x; d < dim; d += blockDim.x) {
    float u = 0.f;
    for (int t = 0; t < S; ++t) u = fmaf(a ? a[t] : 1.0f, xr[t * plane + d], u);    // this thread's own stores
    h[(size_t)r * dim + d] = from_f32<TO>((u * scale) * w[d]);
  }
}

namespace {

bool plan(int dim, bool aligned, int* threads) {
  int t = 32;
  while (t < 512 && t * 4 < dim) t <<= 1;
  const bool vec = dim % 4 == 0 && aligned && dim <= 4 * ST_KEEP * t;
  if (vec)
    while (t > 32 && t * 8 >= 2 * dim) t >>= 1;      // two float4s a thread where the row is short enough
  *threads = t;
  return vec;
}

bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

template <typename TO>
int norm_any(const float* x, long long plane, const float* a, int S, const int* rows, const float* w, TO* y, int n_out, int dim,
             float eps, cudaStream_t stream) {
  int threads;
  if (plan(dim, aligned16(x) && aligned16(w) && aligned16(y) && plane % 4 == 0, &threads))
    return zk_launch_dependent(stream_norm_vec4_kernel<TO>, dim3(n_out), dim3(threads), 0, stream, x, (size_t)plane, a, S, rows, w, y,
                               dim, eps);
  return zk_launch_dependent(stream_norm_kernel<TO>, dim3(n_out), dim3(threads), 0, stream, x, (size_t)plane, a, S, rows, w, y, dim, eps);
}

template <typename TO>
int step_any(float* x, long long plane, const float* y, const float* mix, const float* out, int S, const float* a, const float* w,
             TO* h, int n, int dim, float eps, int want_norm, cudaStream_t stream) {
  int threads;
  const bool ok = aligned16(x) && aligned16(y) && (!want_norm || (aligned16(w) && aligned16(h))) && plane % 4 == 0;
#define ZK_ST(NS)                                                                                                         \
  return zk_launch_dependent(stream_step_vec4_kernel<TO, NS>, dim3(n), dim3(threads), 0, stream, x, (size_t)plane, y, mix, out, a, w, h, \
                             dim, eps, want_norm)
  if (plan(dim, ok, &threads)) {
    if (S == 1) ZK_ST(1);
    if (S == 2) ZK_ST(2);
    if (S == 3) ZK_ST(3);
    if (S == 4) ZK_ST(4);
  }
#undef ZK_ST
  return zk_launch_dependent(stream_step_kernel<TO>, dim3(n), dim3(threads), 0, stream, x, (size_t)plane, y, mix, out, S, a, w, h, dim,
                             eps, want_norm);
}

}  // namespace

extern "C" {

int zk_stream_max() { return ST_MAX; }

// x [S, n, dim] (planes `plane` floats apart), a [S] or null (ones), w [dim], rows null or n_out row numbers, y [n_out, dim].
int zk_stream_norm(const float* x, long long plane, const float* a, int S, const int* rows, const float* w, void* y, int n_out,
                   int dim, float eps, int out_dtype, cudaStream_t stream) {
  if (n_out <= 0) return 0;
  if (S < 1 || S > ST_MAX || dim <= 0 || !w) return ZK_EINVAL;
  if (out_dtype == ZK_F32) return norm_any<float>(x, plane, a, S, rows, w, (float*)y, n_out, dim, eps, stream);
  if (out_dtype == ZK_BF16) return norm_any<bf16>(x, plane, a, S, rows, w, (bf16*)y, n_out, dim, eps, stream);
  return ZK_EINVAL;
}

// x [S, n, dim] in place; y [n, dim]; mix [S, S] (from, to), out [S].  With w the normalised u = sum_s a[s] x_s (a null: ones) of the
// new streams goes to h [n, dim].
int zk_stream_step(float* x, long long plane, const float* y, const float* mix, const float* out, int S, const float* a,
                   const float* w, void* h, int n, int dim, float eps, int out_dtype, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (S < 1 || S > ST_MAX || dim <= 0 || (w && !h)) return ZK_EINVAL;
  const int want = w != nullptr;
  if (out_dtype == ZK_F32) return step_any<float>(x, plane, y, mix, out, S, a, w, (float*)h, n, dim, eps, want, stream);
  if (out_dtype == ZK_BF16) return step_any<bf16>(x, plane, y, mix, out, S, a, w, (bf16*)h, n, dim, eps, want, stream);
  return ZK_EINVAL;
}

}  // extern "C"
