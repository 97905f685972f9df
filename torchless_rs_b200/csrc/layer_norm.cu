// Layer norms of the 32-bit stream,  N(u) = (u - mean(u)) / sqrt(mean((u - mean(u))^2) + eps) * w + b.
//
//   layernorm                 y = N(x) in the activation type, for the rows asked for.
//   layernorm_add_layernorm   x += N_out(y) in the stream, and, if the next norm's weight is given,
//                             xn = N_next(x) in the activation type in the same pass: the stream crosses
//                             memory once per sublayer.
//
// One block per row.  The row stays in registers (16-byte pieces) where its size allows it; the mean is taken
// first and the squared deviations from it after, in 32-bit.  Weights and biases, which no kernel of a step
// writes, are asked for before the wait for the kernels ahead.
#include "common.cuh"

__device__ __forceinline__ void ln_load4(const float* p, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void ln_store4(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void ln_store4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&a);
  u.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// The sum over the block, to every thread, with one barrier: each warp leaves its sum, every warp adds them up.
// Calls in a row take turns between the halves of `scratch` (64 floats).
__device__ __forceinline__ float ln_block_sum(float v, float* scratch, int turn) {
  float* s = scratch + 32 * (turn & 1);
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) s[threadIdx.x >> 5] = v;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  return warp_sum(lane < (int)(blockDim.x >> 5) ? s[lane] : 0.0f);
}

// Mean and 1 / sqrt(variance + eps) of a row that lies in registers, K pieces of four entries per thread.
template <int K>
__device__ __forceinline__ void ln_stats(const float (&v)[K][4], int H, float eps, float* scratch, int turn,
                                         float* mean, float* inv) {
  float s = 0.0f;
#pragma unroll
  for (int j = 0; j < K; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) s += v[j][e];            // entries past the row's end are zero
  const float m = ln_block_sum(s, scratch, turn) / (float)H;
  float q = 0.0f;
#pragma unroll
  for (int j = 0; j < K; ++j)
    if (4 * (int)(threadIdx.x + j * blockDim.x) < H)
#pragma unroll
      for (int e = 0; e < 4; ++e) q = fmaf(v[j][e] - m, v[j][e] - m, q);
  *mean = m;
  *inv = 1.0f / sqrtf(ln_block_sum(q, scratch, turn + 1) / (float)H + eps);
}

// ADD: y is normed with (w, b) and added to x in place; with w2 the new x is normed with (w2, b2) into `out`.
// Otherwise row rows[r] (or r) of x is normed with (w, b) into row r of `out`.  A block takes every gridDim.x-th
// row, so that weights and biases are fetched once for all of them, and asks for its next row while it works on
// one.
template <int K, bool ADD, int THREADS>
__global__ void __launch_bounds__(THREADS)
layernorm_vec_kernel(const float* __restrict__ y, int ldy, float* __restrict__ x, const int* __restrict__ rows,
                     const float* __restrict__ w, const float* __restrict__ b, float eps,
                     const float* __restrict__ w2, const float* __restrict__ b2, float eps2,
                     act_t* __restrict__ out, int n_rows, int H) {
  constexpr int KA = ADD ? K : 1;
  __shared__ float scratch[64];
  float wv[K][4], bv[K][4], wv2[KA][4], bv2[KA][4];
  const bool next = ADD && w2 != nullptr;
#pragma unroll
  for (int j = 0; j < K; ++j) {
    const int i = 4 * (threadIdx.x + j * blockDim.x);
    if (i < H) {
      ln_load4(w + i, wv[j]);
      ln_load4(b + i, bv[j]);
      if (next) { ln_load4(w2 + i, wv2[ADD ? j : 0]); ln_load4(b2 + i, bv2[ADD ? j : 0]); }
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  float v[K][4], xs[KA][4], nv[K][4], nx[KA][4];
  auto fetch = [&](int r) {
    const float* xr = x + (size_t)(!ADD && rows != nullptr ? rows[r] : r) * H;
    const float* src = ADD ? y + (size_t)r * ldy : xr;
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int i = 4 * (threadIdx.x + j * blockDim.x);
      if (i < H) {
        ln_load4(src + i, nv[j]);
        if (ADD) ln_load4(xr + i, nx[ADD ? j : 0]);
      } else {
        nv[j][0] = nv[j][1] = nv[j][2] = nv[j][3] = 0.0f;
      }
    }
  };
  fetch(blockIdx.x);
  for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
#pragma unroll
    for (int j = 0; j < K; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[j][e] = nv[j][e];
        if (ADD) xs[ADD ? j : 0][e] = nx[ADD ? j : 0][e];
      }
    if (r + (int)gridDim.x < n_rows) fetch(r + gridDim.x);
    float mean, inv;
    ln_stats<K>(v, H, eps, scratch, 0, &mean, &inv);
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int i = 4 * (threadIdx.x + j * blockDim.x);
      if (i < H) {
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = fmaf((v[j][e] - mean) * inv, wv[j][e], bv[j][e]);
        if (ADD) {
#pragma unroll
          for (int e = 0; e < 4; ++e) v[j][e] = xs[ADD ? j : 0][e] + o[e];
          ln_store4(x + (size_t)r * H + i, v[j]);
        } else {
          ln_store4(out + (size_t)r * H + i, o);
        }
      }
    }
    if (!next) continue;
    ln_stats<K>(v, H, eps2, scratch, 2, &mean, &inv);
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int i = 4 * (threadIdx.x + j * blockDim.x);
      if (i < H) {
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          o[e] = fmaf((v[j][e] - mean) * inv, wv2[ADD ? j : 0][e], bv2[ADD ? j : 0][e]);
        ln_store4(out + (size_t)r * H + i, o);
      }
    }
  }
}

// The same for rows of any size, read again for every pass.
template <bool ADD>
__global__ void __launch_bounds__(512)
layernorm_any_kernel(const float* __restrict__ y, int ldy, float* x, const int* __restrict__ rows,
                     const float* __restrict__ w, const float* __restrict__ b, float eps,
                     const float* __restrict__ w2, const float* __restrict__ b2, float eps2,
                     act_t* __restrict__ out, int H) {
  __shared__ float scratch[64];
  pdl_wait();
  pdl_launch_dependents();
  const size_t r = blockIdx.x;
  float* xr = x + (size_t)(!ADD && rows != nullptr ? rows[r] : r) * H;
  auto stats = [&](const float* p, float ep, int turn, float* mean, float* inv) {
    float s = 0.0f, q = 0.0f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) s += p[i];
    const float m = ln_block_sum(s, scratch, turn) / (float)H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) q = fmaf(p[i] - m, p[i] - m, q);
    *mean = m;
    *inv = 1.0f / sqrtf(ln_block_sum(q, scratch, turn + 1) / (float)H + ep);
  };
  float mean, inv;
  const float* src = ADD ? y + r * ldy : xr;
  stats(src, eps, 0, &mean, &inv);
  if (!ADD) {
    for (int i = threadIdx.x; i < H; i += blockDim.x)
      out[r * H + i] = from_f32<act_t>(fmaf((xr[i] - mean) * inv, w[i], b[i]));
    return;
  }
  for (int i = threadIdx.x; i < H; i += blockDim.x) xr[i] += fmaf((src[i] - mean) * inv, w[i], b[i]);
  if (w2 == nullptr) return;
  // every thread reads back only what it wrote itself
  stats(xr, eps2, 2, &mean, &inv);
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    out[r * H + i] = from_f32<act_t>(fmaf((xr[i] - mean) * inv, w2[i], b2[i]));
}

template <bool ADD>
static int ln_launch(const float* y, int ldy, float* x, const int* rows, const float* w, const float* b, float eps,
                     const float* w2, const float* b2, float eps2, act_t* out, int n_rows, int H,
                     cudaStream_t stream) {
  const uintptr_t at = (uintptr_t)y | (uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)w2 | (uintptr_t)b2 |
                       (uintptr_t)out;
  if (H % 4 == 0 && ldy % 4 == 0 && H <= 8192 && (at & 15) == 0) {
    // few rows: as many threads a row as it has pieces; many: fewer, so that several rows are in flight on an SM
    const int grid = n_rows < 148 * 4 ? n_rows : 148 * 4;
#define LN_VEC(K_, THREADS_)                                                                                      \
    return tl_launch(layernorm_vec_kernel<K_, ADD, THREADS_>, dim3(grid), dim3(THREADS_), 0, stream, y, ldy, x, rows, w, b, \
                     eps, w2, b2, eps2, out, n_rows, H)
    if (H <= 512) LN_VEC(1, 128);
    if (H <= 1024) LN_VEC(1, 256);
    if (H <= 2048) { if (n_rows < 148) LN_VEC(1, 512); LN_VEC(2, 256); }
    if (H <= 4096) { if (n_rows < 148) LN_VEC(1, 1024); LN_VEC(2, 512); }
    LN_VEC(2, 1024);
#undef LN_VEC
  }
  return tl_launch(layernorm_any_kernel<ADD>, dim3(n_rows), dim3(H >= 2048 ? 512 : 128), 0, stream, y, ldy, x, rows, w,
                   b, eps, w2, b2, eps2, out, H);
}

extern "C" int TL_NAME(tl_layernorm)(const float* x, const int* rows, const float* w, const float* b, float eps,
                                     void* out, int n_rows, int H, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (H <= 0 || w == nullptr || b == nullptr) return TL_ERR_BAD_ARG;
  return ln_launch<false>(nullptr, 0, const_cast<float*>(x), rows, w, b, eps, nullptr, nullptr, 0.0f, (act_t*)out,
                          n_rows, H, stream);
}

extern "C" int TL_NAME(tl_layernorm_add_layernorm)(const float* y, int ldy, const float* w, const float* b, float eps,
                                                   float* x, const float* w2, const float* b2, float eps2, void* out,
                                                   int n_rows, int H, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (H <= 0 || w == nullptr || b == nullptr || (w2 != nullptr && (b2 == nullptr || out == nullptr)))
    return TL_ERR_BAD_ARG;
  return ln_launch<true>(y, ldy, x, nullptr, w, b, eps, w2, b2, eps2, (act_t*)out, n_rows, H, stream);
}
