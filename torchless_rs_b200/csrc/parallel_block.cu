// Closing kernel of a block whose sublayers run side by side and add to the 32-bit stream: one pass over the
// stream takes everything that is still to be added and prepares the next norm.
//   x[t] <- x[t] + sum_k wt[t, k] yk[row_of[t, k]]  +  sigmoid(sg[t]) ys[t]  +  add_rows[t]  +  add_vec
//   xn[t] = x[t] / sqrt(mean(x[t]^2) + eps) * w_next                           (activation type)
// Every term may be absent: the chosen experts' outputs (k in order of the token's choice), a shared expert's
// output with its gate's pre-activation (or none), a row per token, a vector for all tokens, the next norm.
#include "common.cuh"

#define PB_KEEP 4

struct CloseArgs {
  float* x;
  const float* yk;          // [pairs, H]
  const int* row_of;        // [T, top]
  const float* wt;          // [T, top]
  const float* ys;          // [T, H]
  const float* sg;          // [T], stride ld_sg; null: weight one
  const float* add_rows;    // [T, H]
  const float* add_vec;     // [H]
  const float* w_next;      // [H]
  act_t* xn;
  float eps;
  int H, top, ld_sg;
};

template <int V>
__device__ __forceinline__ void pb_load(const float* p, float (&v)[V]) {
  if (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[V > 1 ? 1 : 0] = f.y; v[V > 2 ? 2 : 0] = f.z; v[V > 3 ? 3 : 0] = f.w;
    if (V == 1) v[0] = f.x;
  } else {
    v[0] = *p;
  }
}

template <int V>
__global__ void __launch_bounds__(1024)
close_block_kernel(CloseArgs a) {
  __shared__ float scratch[33];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, H = a.H;
  float* xr = a.x + (size_t)t * H;
  const float gate = a.ys == nullptr ? 0.0f : (a.sg == nullptr ? 1.0f : 1.0f / (1.0f + expf(-a.sg[(size_t)t * a.ld_sg])));
  auto value = [&](int i, float (&v)[V]) {
    float u[V];
    pb_load<V>(xr + i, v);
    if (a.yk != nullptr) {
      float s[V];
#pragma unroll
      for (int e = 0; e < V; ++e) s[e] = 0.0f;
      for (int k = 0; k < a.top; ++k) {
        const float w = a.wt[(size_t)t * a.top + k];
        pb_load<V>(a.yk + (size_t)a.row_of[(size_t)t * a.top + k] * H + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] = fmaf(w, u[e], s[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += s[e];
    }
    if (a.ys != nullptr) {
      pb_load<V>(a.ys + (size_t)t * H + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = fmaf(gate, u[e], v[e]);
    }
    if (a.add_rows != nullptr) {
      pb_load<V>(a.add_rows + (size_t)t * H + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += u[e];
    }
    if (a.add_vec != nullptr) {
      pb_load<V>(a.add_vec + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += u[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) xr[i + e] = v[e];
  };
  const bool fits = H <= (int)blockDim.x * V * PB_KEEP;
  float keep[PB_KEEP][V];
  float ss = 0.0f;
  if (fits) {
#pragma unroll
    for (int j = 0; j < PB_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
#pragma unroll
      for (int e = 0; e < V; ++e) keep[j][e] = 0.0f;
      if (i < H) value(i, keep[j]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(keep[j][e], keep[j][e], ss);
    }
  } else {
    for (int i = V * threadIdx.x; i < H; i += V * blockDim.x) {
      float v[V];
      value(i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    }
  }
  if (a.w_next == nullptr) return;
  ss = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)H + a.eps);
  act_t* o = a.xn + (size_t)t * H;
  if (fits) {
#pragma unroll
    for (int j = 0; j < PB_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
      if (i < H) {
#pragma unroll
        for (int e = 0; e < V; ++e) o[i + e] = from_f32<act_t>(keep[j][e] * inv * a.w_next[i + e]);
      }
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = from_f32<act_t>(xr[i] * inv * a.w_next[i]);
  }
}

extern "C" int TL_NAME(tl_close_block)(float* x, const float* yk, const int* row_of, const float* wt, int top,
                                       const float* ys, const float* sg, int ld_sg, const float* add_rows,
                                       const float* add_vec, const float* w_next, float eps, void* xn, int T, int H,
                                       cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || (yk != nullptr && (row_of == nullptr || wt == nullptr || top < 1)) || (w_next != nullptr && xn == nullptr))
    return TL_ERR_BAD_ARG;
  CloseArgs a = {x, yk, row_of, wt, ys, sg, add_rows, add_vec, w_next, (act_t*)xn, eps, H, top, ld_sg};
  const uintptr_t all = (uintptr_t)x | (uintptr_t)yk | (uintptr_t)ys | (uintptr_t)add_rows | (uintptr_t)add_vec;
  // few rows (decode steps): more threads per row, so that a row's loads are in flight together.  A block that
  // cannot hold its row reads back what its own threads wrote only if a thread's places are the same in both
  // passes, which one value at a time gives.
  const bool vec = H % 4 == 0 && (all & 15) == 0 && H <= 1024 * 4 * PB_KEEP;
  const int per = vec ? 4 : 1;
  int threads = ((H + per - 1) / per + 31) / 32 * 32;
  if (T >= 512) threads = (threads / 2 + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 1024 ? 1024 : threads);
  if (vec) return tl_launch(close_block_kernel<4>, dim3(T), dim3(threads), 0, stream, a);
  return tl_launch(close_block_kernel<1>, dim3(T), dim3(threads), 0, stream, a);
}
