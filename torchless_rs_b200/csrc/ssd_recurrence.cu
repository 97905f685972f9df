// State-space recurrence with one decay per head and token (the state-space duality form of a selective
// scan).  Per head h, which reads the input and read-out vectors of group h / (heads / groups):
//   dt = softplus(zdt + dt_bias),  a = exp(neg_a dt)                                  (per token and head)
//   S <- a S + dt B x^T,   y = S^T C + D x                                            (S: [N, P])
// x, B and C come out of a causal convolution over the last `taps` tokens of each channel (with a bias) and
// a silu; the concatenated heads' y is multiplied by silu(z) and then normed in equal parts.
//
//   ssd_prep         the step's projections -> convolved, activated x, B, C (activation type), dt and the
//                    decay's logarithm per token and head (32-bit); the last taps - 1 inputs go back to
//                    the sequence's slot
//   conv_silu        the convolution alone, on inputs of the activation type
//   ssd_walk         the recurrence token by token from the state in the slot: decode steps, short steps
//                    and the whole of the 32-bit path
//   ssd_chunk_state, ssd_chunk_carry, ssd_chunk_out
//                    long steps in bfloat16: chunks of SSD_Q tokens on the tensor cores.  With L_t the sum of
//                    the decays' logarithms since the chunk's start,
//                      E   = sum over s in the chunk of exp(L_end - L_s) dt_s B_s x_s^T     (all chunks at once)
//                      S_c = exp(L_end) S_(c-1) + E_(c-1)                          (chunk after chunk, per head)
//                      y_t = exp(L_t) S_c^T C_t + sum over s <= t of (C_t . B_s) exp(L_t - L_s) dt_s x_s + D x_t
//                    No quotient of decays is formed (every exponent is <= 0).  x, B and C are bfloat16 as they
//                    come out of the convolution; every factor that is not (the state, the weights with their
//                    decays) enters the tensor cores as the sum of two bfloat16 numbers, which leaves 2^-17 of
//                    it, and all sums are 32-bit.
//   ssd_gate_norm    y silu(z), normed part by part, times a weight
//
// The state and the convolution's kept inputs are 32-bit, live in per-sequence slots and are carried from
// step to step, so a prompt may come in any number of pieces.
#include "common.cuh"

#define SSD_STRIP 16        // tokens of one sequence per block of ssd_prep
#define SSD_MAX_TAPS 16

__device__ __forceinline__ float ssd_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ssd_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// (sequence, first token, token count, index of the piece in its sequence) of piece `id` when every
// sequence's tokens of the step are cut into pieces of `size`
__device__ __forceinline__ bool ssd_find_piece(int id, int size, const int* seq_start, int B, int* b_out, int* t0,
                                               int* n, int* in_seq) {
  for (int b = 0; b < B; ++b) {
    const int cnt = seq_start[b + 1] - seq_start[b];
    const int pieces = (cnt + size - 1) / size;
    if (id < pieces) {
      *b_out = b;
      *in_seq = id;
      *t0 = seq_start[b] + id * size;
      const int left = seq_start[b + 1] - *t0;
      *n = left < size ? left : size;
      return true;
    }
    id -= pieces;
  }
  return false;
}

// z: [T, ld] 32-bit; channels at columns col_x .. col_x + channels - 1, step sizes at col_dt .. col_dt + H - 1.
// xbc: [T, channels]; dtla: [T, H] pairs (dt, neg_a dt).  kept: [slots, taps - 1, channels], oldest first.
// A thread per channel walks a strip of 16 tokens; the thread of a sequence's first strip, the only one that
// looks at the kept inputs, also replaces them.  The blocks past the channels' take the step sizes.
// TAPS: the number of taps, or 0 for any (their inputs are then read where they are needed).
template <int TAPS, typename Z>
__global__ void __launch_bounds__(128)
ssd_prep_kernel(const Z* __restrict__ z, int ld, int col_x, int col_dt, const float* __restrict__ taps_w,
                const float* __restrict__ bias, int taps_rt, float* __restrict__ kept, act_t* __restrict__ xbc,
                float2* __restrict__ dtla, const float* __restrict__ neg_a, const float* __restrict__ dt_bias,
                const int* __restrict__ seq_start, const int* __restrict__ seq_slot, int B, int channels, int H,
                int ch_blocks) {
  pdl_wait();
  pdl_launch_dependents();
  const int taps = TAPS ? TAPS : taps_rt;
  int b, t0, n, strip;
  if (!ssd_find_piece(blockIdx.x, SSD_STRIP, seq_start, B, &b, &t0, &n, &strip)) return;
  if ((int)blockIdx.y >= ch_blocks) {
    for (int i = threadIdx.x + ((int)blockIdx.y - ch_blocks) * blockDim.x; i < n * H;
         i += (gridDim.y - ch_blocks) * blockDim.x) {
      const int t = t0 + i / H, h = i % H;
      const float dt = ssd_softplus(to_f32(z[(size_t)t * ld + col_dt + h]) + dt_bias[h]);
      dtla[(size_t)t * H + h] = make_float2(dt, neg_a[h] * dt);
    }
    return;
  }
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const Z* zc = z + col_x + c;
  float* mine = kept + (size_t)seq_slot[b] * (taps - 1) * channels + c;
  const float bi = bias[c];
  const int first = seq_start[b], count = seq_start[b + 1] - first, j0 = strip * SSD_STRIP;
  // the input at place j of the step (j < 0: kept from before)
  auto input = [&](int j) -> float {
    return j >= 0 ? to_f32(zc[(size_t)(first + j) * ld]) : mine[(size_t)(taps - 1 + j) * channels];
  };
  if (TAPS) {
    float v[SSD_STRIP + (TAPS ? TAPS : 1) - 1], w[TAPS ? TAPS : 1];
#pragma unroll
    for (int i = 0; i < SSD_STRIP + TAPS - 1; ++i) v[i] = i < n + TAPS - 1 ? input(j0 - (TAPS - 1) + i) : 0.0f;
#pragma unroll
    for (int i = 0; i < TAPS; ++i) w[i] = taps_w[(size_t)c * TAPS + i];
#pragma unroll
    for (int j = 0; j < SSD_STRIP; ++j) {
      if (j < n) {
        float acc = bi;
#pragma unroll
        for (int i = 0; i < TAPS; ++i) acc = fmaf(w[i], v[j + i], acc);
        xbc[(size_t)(t0 + j) * channels + c] = from_f32<act_t>(ssd_silu(acc));
      }
    }
  } else {
    for (int j = 0; j < n; ++j) {
      float acc = bi;
      for (int i = 0; i < taps; ++i)
        acc = fmaf(taps_w[(size_t)c * taps + i], input(j0 + j - (taps - 1) + i), acc);
      xbc[(size_t)(t0 + j) * channels + c] = from_f32<act_t>(ssd_silu(acc));
    }
  }
  if (strip == 0 && taps > 1) {
    float k[SSD_MAX_TAPS - 1];
#pragma unroll
    for (int i = 0; i < SSD_MAX_TAPS - 1; ++i) k[i] = i < taps - 1 ? input(count - (taps - 1) + i) : 0.0f;
#pragma unroll
    for (int i = 0; i < SSD_MAX_TAPS - 1; ++i)
      if (i < taps - 1) mine[(size_t)i * channels] = k[i];
  }
}

template <typename Z>
static int ssd_prep_launch(const Z* z, int ld, int col_x, int col_dt, const float* taps_w, const float* bias, int taps,
                           float* kept, void* xbc, float* dtla, const float* neg_a, const float* dt_bias,
                           const int* seq_start, const int* seq_slot, int T, int B, int channels, int H,
                           cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (channels < 1 || H < 0 || taps < 1) return TL_ERR_BAD_ARG;
  if (taps > SSD_MAX_TAPS) return TL_ERR_UNSUPPORTED;
  const int ch_blocks = (channels + 127) / 128;
  const int dt_blocks = (H * (T < SSD_STRIP ? T : SSD_STRIP) + 511) / 512;
  dim3 grid(T / SSD_STRIP + B, ch_blocks + dt_blocks);
  if (grid.y > 65535) return TL_ERR_UNSUPPORTED;
#define PREP(TAPS_)                                                                                            \
  return tl_launch(ssd_prep_kernel<TAPS_, Z>, grid, dim3(128), 0, stream, z, ld, col_x, col_dt, taps_w, bias, taps, \
                   kept, (act_t*)xbc, (float2*)dtla, neg_a, dt_bias, seq_start, seq_slot, B, channels, H, ch_blocks)
  switch (taps) {
    case 1: PREP(1);
    case 2: PREP(2);
    case 3: PREP(3);
    case 4: PREP(4);
    default: PREP(0);
  }
#undef PREP
}

extern "C" int TL_NAME(tl_ssd_prep)(const float* z, int ld, int col_x, int col_dt, const float* taps_w,
                                    const float* bias, int taps, float* kept, void* xbc, float* dtla,
                                    const float* neg_a, const float* dt_bias, const int* seq_start,
                                    const int* seq_slot, int T, int B, int channels, int H, cudaStream_t stream) {
  if (H < 1) return TL_ERR_BAD_ARG;
  return ssd_prep_launch<float>(z, ld, col_x, col_dt, taps_w, bias, taps, kept, xbc, dtla, neg_a, dt_bias, seq_start,
                                seq_slot, T, B, channels, H, stream);
}

// The convolution alone, four channels per thread (16- or 8-byte loads, kept as they came until they are used)
// over a strip of SSD_STRIP tokens.  Everything else as in ssd_prep_kernel.
#if TL_DTYPE == 0
typedef float4 ssd_quad;
__device__ __forceinline__ float ssd_fast_silu(float z) { return ssd_silu(z); }
#else
typedef uint2 ssd_quad;
__device__ __forceinline__ float ssd_fast_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
#endif
__device__ __forceinline__ void ssd_unpack(const float4& f, float (&v)[4]) {
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void ssd_unpack(const uint2& u, float (&v)[4]) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void ssd_store4(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void ssd_store4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&a);
  u.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}
template <int TAPS>
__global__ void __launch_bounds__(128)
conv_silu_vec_kernel(const act_t* __restrict__ z, int ld, const float* __restrict__ taps_w,
                     const float* __restrict__ bias, float* __restrict__ kept, act_t* __restrict__ out,
                     const int* __restrict__ seq_start, const int* __restrict__ seq_slot, int B, int channels) {
  const int c = 4 * (blockIdx.y * blockDim.x + threadIdx.x);
  float w[4 * TAPS], bi[4] = {0.0f, 0.0f, 0.0f, 0.0f};      // w: channel after channel, its taps in a row
  if (c < channels) {                       // weights: asked for before the wait
    ssd_unpack(*reinterpret_cast<const float4*>(bias + c), bi);
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      float q[4];
      ssd_unpack(*reinterpret_cast<const float4*>(taps_w + (size_t)c * TAPS + 4 * i), q);
#pragma unroll
      for (int e = 0; e < 4; ++e) w[4 * i + e] = q[e];
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  int b, t0, n, strip;
  if (!ssd_find_piece(blockIdx.x, SSD_STRIP, seq_start, B, &b, &t0, &n, &strip) || c >= channels) return;
  float* mine = kept + (size_t)seq_slot[b] * (TAPS - 1) * channels + c;
  const int count = seq_start[b + 1] - seq_start[b];
  // the strip's inputs, and the TAPS - 1 ahead of it: inputs of the step, or, for the first strip, kept ones
  ssd_quad raw[SSD_STRIP + TAPS - 1];
  const act_t* zc = z + (size_t)t0 * ld + c;
#pragma unroll
  for (int i = 0; i < SSD_STRIP + TAPS - 1; ++i)
    if ((i >= TAPS - 1 || strip > 0) && i < n + TAPS - 1)
      raw[i] = *reinterpret_cast<const ssd_quad*>(zc + (ptrdiff_t)(i - (TAPS - 1)) * ld);
  float before[TAPS - 1][4];
#pragma unroll
  for (int i = 0; i < TAPS - 1; ++i) {
    if (strip > 0) ssd_unpack(raw[i], before[i]);
    else ssd_unpack(*reinterpret_cast<const float4*>(mine + (size_t)i * channels), before[i]);
  }
  if (strip == 0) {
    // this thread alone looks at the kept inputs, so it can replace them: the last TAPS - 1 of [kept | step]
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
      const int j = count - (TAPS - 1) + i;          // place in the step; negative: kept from before
      float v[4];
      if (j >= 0) ssd_unpack(*reinterpret_cast<const ssd_quad*>(zc + (size_t)j * ld), v);
      else {
#pragma unroll
        for (int q = 0; q < TAPS - 1; ++q)
          if (q == TAPS - 1 + j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = before[q][e];
          }
      }
      ssd_store4(mine + (size_t)i * channels, v);
    }
  }
#pragma unroll
  for (int j = 0; j < SSD_STRIP; ++j) {
    if (j >= n) break;
    float cur[4], o[4];
    ssd_unpack(raw[j + TAPS - 1], cur);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float acc = bi[e];
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i) acc = fmaf(w[e * TAPS + i], before[i][e], acc);
      o[e] = ssd_fast_silu(fmaf(w[e * TAPS + TAPS - 1], cur[e], acc));
    }
    ssd_store4(out + (size_t)(t0 + j) * channels + c, o);
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) before[i][e] = i + 1 < TAPS - 1 ? before[i + 1 < TAPS - 1 ? i + 1 : 0][e] : cur[e];
  }
}

// The convolution alone: out [T, channels] = silu(conv(z[:, col_x:]) + bias), z in the activation type.
extern "C" int TL_NAME(tl_conv_silu)(const void* z, int ld, int col_x, const float* taps_w, const float* bias, int taps,
                                     float* kept, void* out, const int* seq_start, const int* seq_slot, int T, int B,
                                     int channels, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  const uintptr_t at = (uintptr_t)z | (uintptr_t)kept | (uintptr_t)out | (uintptr_t)bias | (uintptr_t)taps_w;
  if (taps >= 2 && taps <= 4 && channels > 0 && channels % 4 == 0 && ld % 4 == 0 && col_x % 4 == 0 && (at & 15) == 0) {
    const dim3 grid(T / SSD_STRIP + B, (channels / 4 + 127) / 128);
#define CONV(TAPS_)                                                                                                  \
    return tl_launch(conv_silu_vec_kernel<TAPS_>, grid, dim3(128), 0, stream, (const act_t*)z + col_x, ld, taps_w,  \
                     bias, kept, (act_t*)out, seq_start, seq_slot, B, channels)
    if (taps == 2) CONV(2);
    if (taps == 3) CONV(3);
    CONV(4);
#undef CONV
  }
  return ssd_prep_launch<act_t>((const act_t*)z, ld, col_x, 0, taps_w, bias, taps, kept, out, nullptr, nullptr, nullptr,
                                seq_start, seq_slot, T, B, channels, 0, stream);
}

// ---------------------------------------------------------------------------------------------------
// The walk.  A block owns (sequence, head, 64 columns of the state): 16 quads of columns x 16 groups of RP
// rows, the state in registers.  Tokens come through shared memory eight at a time; a token's output is summed
// over a warp's two row groups by a shuffle, and over the eight warps through shared memory, once per eight
// tokens.  VEC: columns are read and written four at a time.
// ---------------------------------------------------------------------------------------------------
#define SSD_TT 8
#define SSD_COLS 64
template <int RP, bool VEC>
__global__ void __launch_bounds__(256)
ssd_walk_kernel(const act_t* __restrict__ xbc, const float2* __restrict__ dtla, const float* __restrict__ D,
                float* __restrict__ state, float* __restrict__ y, const int* __restrict__ seq_start,
                const int* __restrict__ seq_slot, int H, int G, int N, int P, int channels) {
  extern __shared__ __align__(16) float ssd_sm[];
  const int NP = RP * 16;                                  // rows, padded
  float* Bs = ssd_sm;                                       // [TT][NP]
  float* Cs = Bs + SSD_TT * NP;                             // [TT][NP]
  float* xs = Cs + SSD_TT * NP;                             // [TT][COLS]
  float* red = xs + SSD_TT * SSD_COLS;                      // [TT][8 warps][COLS]
  float* ad = red + SSD_TT * 8 * SSD_COLS;                  // [TT][2]: decay, dt
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * SSD_COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int quad = lane & 15, rg = warp * 2 + (lane >> 4);
  const int col = p0 + quad * 4;
  const int g = h / (H / G);
  const int t0 = seq_start[b], t1 = seq_start[b + 1];
  float* S = state + (((size_t)seq_slot[b] * H + h) * N) * P;
  float s[RP][4];
#pragma unroll
  for (int r = 0; r < RP; ++r) {
    const int row = rg + 16 * r;
    s[r][0] = s[r][1] = s[r][2] = s[r][3] = 0.0f;
    if (row < N) {
      if (VEC) {
        if (col < P) {
          const float4 v = *reinterpret_cast<const float4*>(S + (size_t)row * P + col);
          s[r][0] = v.x; s[r][1] = v.y; s[r][2] = v.z; s[r][3] = v.w;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (col + e < P) s[r][e] = S[(size_t)row * P + col + e];
      }
    }
  }
  const float Dh = D[h];
  const int off_b = H * P + g * N, off_c = H * P + G * N + g * N;
  for (int tb = t0; tb < t1; tb += SSD_TT) {
    const int cnt = t1 - tb < SSD_TT ? t1 - tb : SSD_TT;
    for (int i = tid; i < cnt * NP; i += 256) {
      const int p = i / NP, r = i - p * NP;
      const act_t* row = xbc + (size_t)(tb + p) * channels;
      Bs[i] = r < N ? to_f32(row[off_b + r]) : 0.0f;
      Cs[i] = r < N ? to_f32(row[off_c + r]) : 0.0f;
    }
    for (int i = tid; i < cnt * SSD_COLS; i += 256) {
      const int p = i / SSD_COLS, c = i - p * SSD_COLS;
      xs[i] = p0 + c < P ? to_f32(xbc[(size_t)(tb + p) * channels + h * P + p0 + c]) : 0.0f;
    }
    if (tid < cnt) {
      const float2 v = dtla[(size_t)(tb + tid) * H + h];
      ad[2 * tid] = expf(v.y);
      ad[2 * tid + 1] = v.x;
    }
    __syncthreads();
    for (int p = 0; p < cnt; ++p) {
      const float a = ad[2 * p], dt = ad[2 * p + 1];
      const float4 xv = *reinterpret_cast<const float4*>(xs + p * SSD_COLS + quad * 4);
      const float dx[4] = {dt * xv.x, dt * xv.y, dt * xv.z, dt * xv.w};
      float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int r = 0; r < RP; ++r) {
        const float bv = Bs[p * NP + rg + 16 * r], cv = Cs[p * NP + rg + 16 * r];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[r][e] = fmaf(a, s[r][e], dx[e] * bv);
          acc[e] = fmaf(s[r][e], cv, acc[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
      if (lane < 16)
        *reinterpret_cast<float4*>(red + (p * 8 + warp) * SSD_COLS + quad * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    }
    __syncthreads();
    for (int i = tid; i < cnt * SSD_COLS; i += 256) {
      const int p = i / SSD_COLS, c = i - p * SSD_COLS;
      if (p0 + c < P) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += red[(p * 8 + w) * SSD_COLS + c];
        y[(size_t)(tb + p) * H * P + h * P + p0 + c] = fmaf(Dh, xs[i], v);
      }
    }
    __syncthreads();      // the next tokens overwrite what was just read
  }
  pdl_launch_dependents();
#pragma unroll
  for (int r = 0; r < RP; ++r) {
    const int row = rg + 16 * r;
    if (row < N) {
      if (VEC) {
        if (col < P) *reinterpret_cast<float4*>(S + (size_t)row * P + col) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (col + e < P) S[(size_t)row * P + col + e] = s[r][e];
      }
    }
  }
}

template <int RP>
static int ssd_walk_launch(const act_t* xbc, const float2* dtla, const float* D, float* state, float* y,
                           const int* seq_start, const int* seq_slot, int B, int H, int G, int N, int P, int channels,
                           cudaStream_t stream) {
  dim3 grid(B, H, (P + SSD_COLS - 1) / SSD_COLS);
  const size_t smem = (size_t)(SSD_TT * (2 * RP * 16 + SSD_COLS + 8 * SSD_COLS + 2)) * sizeof(float);
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ssd_walk_kernel<RP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||
        cudaFuncSetAttribute(ssd_walk_kernel<RP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return TL_ERR_UNSUPPORTED;
    set = true;
  }
  if (P % 4 == 0)
    return tl_launch(ssd_walk_kernel<RP, true>, grid, dim3(256), smem, stream, xbc, dtla, D, state, y, seq_start,
                     seq_slot, H, G, N, P, channels);
  return tl_launch(ssd_walk_kernel<RP, false>, grid, dim3(256), smem, stream, xbc, dtla, D, state, y, seq_start,
                   seq_slot, H, G, N, P, channels);
}

extern "C" int TL_NAME(tl_ssd_walk)(const void* xbc, const float* dtla, const float* D, float* state, float* y,
                                    const int* seq_start, const int* seq_slot, int B, int H, int G, int N, int P,
                                    int channels, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H < 1 || G < 1 || H % G || N < 1 || P < 1 || channels < H * P + 2 * G * N) return TL_ERR_BAD_ARG;
  if (H > 65535 || N > 512 || (P + SSD_COLS - 1) / SSD_COLS > 65535) return TL_ERR_UNSUPPORTED;
#define WALK(RP_)                                                                                           \
  return ssd_walk_launch<RP_>((const act_t*)xbc, (const float2*)dtla, D, state, y, seq_start, seq_slot, B, H, \
                              G, N, P, channels, stream)
  if (N <= 16) WALK(1);
  if (N <= 32) WALK(2);
  if (N <= 64) WALK(4);
  if (N <= 128) WALK(8);
  if (N <= 256) WALK(16);
  WALK(32);
#undef WALK
}

// ---------------------------------------------------------------------------------------------------
// out = y silu(z) / rms(y silu(z)) * w, the root mean square over each of `parts` equal parts of a row.
// One block per (row, part).
// ---------------------------------------------------------------------------------------------------
#define SSD_GN_KEEP 4
template <int V>      // 4: rows in 16-byte pieces; 1: any size
__global__ void __launch_bounds__(1024)
ssd_gate_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, int ldz, const float* __restrict__ w,
                     float eps, act_t* __restrict__ out, int part, int inner) {
  __shared__ float scratch[33];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const int off = blockIdx.y * part;
  const float* yr = y + t * inner + off;
  const float* zr = z + t * ldz + off;
  act_t* o = out + t * inner + off;
  w += off;
  const bool fits = part <= (int)blockDim.x * V * SSD_GN_KEEP;
  float keep[SSD_GN_KEEP][V];
  float ss = 0.0f;
  auto gated = [&](int i, float (&v)[V]) {
    if (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(yr + i), b = *reinterpret_cast<const float4*>(zr + i);
      v[0] = a.x * ssd_silu(b.x);
      if (V > 1) { v[V > 1 ? 1 : 0] = a.y * ssd_silu(b.y); v[V > 2 ? 2 : 0] = a.z * ssd_silu(b.z); v[V > 3 ? 3 : 0] = a.w * ssd_silu(b.w); }
    } else {
      v[0] = yr[i] * ssd_silu(zr[i]);
    }
  };
  if (fits) {
#pragma unroll
    for (int j = 0; j < SSD_GN_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
#pragma unroll
      for (int e = 0; e < V; ++e) keep[j][e] = 0.0f;
      if (i < part) gated(i, keep[j]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(keep[j][e], keep[j][e], ss);
    }
  } else {
    for (int i = V * threadIdx.x; i < part; i += V * blockDim.x) {
      float v[V];
      gated(i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    }
  }
  ss = block_sum(ss, scratch);
  const float rms = sqrtf(ss / (float)part + eps);
  const float inv = 1.0f / rms;
  auto store = [&](int i, const float (&v)[V]) {
#pragma unroll
    for (int e = 0; e < V; ++e) o[i + e] = from_f32<act_t>(v[e] * inv * w[i + e]);
  };
  if (fits) {
#pragma unroll
    for (int j = 0; j < SSD_GN_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
      if (i < part) store(i, keep[j]);
    }
  } else {
    for (int i = V * threadIdx.x; i < part; i += V * blockDim.x) {
      float v[V];
      gated(i, v);
      store(i, v);
    }
  }
}

extern "C" int TL_NAME(tl_ssd_gate_norm)(const float* y, const float* z, int ldz, const float* w, float eps, void* out,
                                         int T, int inner, int parts, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (inner < 1 || parts < 1 || inner % parts) return TL_ERR_BAD_ARG;
  if (parts > 65535) return TL_ERR_UNSUPPORTED;
  const int part = inner / parts;
  const bool vec = part % 4 == 0 && inner % 4 == 0 && ldz % 4 == 0 && (((uintptr_t)y | (uintptr_t)z) & 15) == 0;
  const int per = vec ? 4 : 1;
  int threads = ((part + per * 2 - 1) / (per * 2) + 31) / 32 * 32;      // two pieces per thread
  threads = threads < 32 ? 32 : (threads > 1024 ? 1024 : threads);
  if (vec)
    return tl_launch(ssd_gate_norm_kernel<4>, dim3(T, parts), dim3(threads), 0, stream, y, z, ldz, w, eps,
                     (act_t*)out, part, inner);
  return tl_launch(ssd_gate_norm_kernel<1>, dim3(T, parts), dim3(threads), 0, stream, y, z, ldz, w, eps,
                   (act_t*)out, part, inner);
}

#if TL_DTYPE == 1
// ---------------------------------------------------------------------------------------------------
// Chunks on the tensor cores (what they compute: top of the file).  N and P are multiples of 16, N up to
// 256; a block takes up to 64 columns of P.  Rows in shared memory are padded by 16 bytes, so that the eight
// rows of an ldmatrix fall into eight different groups of banks.
// ---------------------------------------------------------------------------------------------------
#define SSD_Q 128
#define SSD_PT 64
#define SSD_PAD 8
typedef __nv_bfloat16 ssd_bf16;

__device__ __forceinline__ void ssd_cp16(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void ssd_ldm4(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s) : "memory");
}
__device__ __forceinline__ void ssd_ldm4t(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s) : "memory");
}
__device__ __forceinline__ void ssd_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// v0, v1 as sums of two bfloat16 numbers each: the larger parts packed in `hi`, what is left in `lo`
__device__ __forceinline__ void ssd_split2(float v0, float v1, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - back.x, v1 - back.y);
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = *reinterpret_cast<const unsigned*>(&l);
}

// The inclusive sums L of the decays' logarithms over the chunk's tokens and the step sizes, for one head,
// by the first 128 threads; two barriers inside.  Places past `n` get L of the last token and dt 0.
// Differences of L are what the weights are made of, and after a few strong decays L is large: the sums are
// taken in 64-bit and kept as a multiple of 1/16 (x, whose differences are exact) and a rest (y).
__device__ __forceinline__ float ssd_diff(float2 a, float2 b) { return (a.x - b.x) + (a.y - b.y); }
__device__ __forceinline__ void ssd_chunk_decays(const float2* __restrict__ dtla, int H, int h, int t0, int n,
                                                 float2* L, float* dts, double* warp_tot) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  double la = 0.0;
  float dt = 0.0f;
  if (tid < SSD_Q) {
    if (tid < n) {
      const float2 v = dtla[(size_t)(t0 + tid) * H + h];
      dt = v.x;
      la = v.y;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double u = __shfl_up_sync(0xffffffffu, la, o);
      if (lane >= o) la += u;
    }
    if (lane == 31) warp_tot[warp] = la;
  }
  __syncthreads();
  if (tid < SSD_Q) {
    for (int w = 0; w < warp; ++w) la += warp_tot[w];
    // (below -10^5 every weight is zero; the bound keeps the multiples of 1/16 exact)
    la = la < -1.0e5 ? -1.0e5 : la;
    const float coarse = rintf((float)la * 16.0f) * 0.0625f;
    L[tid] = make_float2(coarse, (float)(la - (double)coarse));
    dts[tid] = dt;
  }
  __syncthreads();
}

// E of every (chunk, head): ends [chunks][H][N][P]; total decay of the chunk: decs [chunks][H].
__global__ void __launch_bounds__(256)
ssd_chunk_state_kernel(const ssd_bf16* __restrict__ xbc, const float2* __restrict__ dtla, float* __restrict__ ends,
                       float* __restrict__ decs, const int* __restrict__ seq_start, int B, int H, int G, int N, int P,
                       int channels) {
  extern __shared__ __align__(16) unsigned char ssd_raw[];
  __shared__ float2 L[SSD_Q];
  __shared__ float dts[SSD_Q];
  __shared__ double wt[4];
  const int NS = N + SSD_PAD, PS = SSD_PT + SSD_PAD;
  ssd_bf16* Bs = reinterpret_cast<ssd_bf16*>(ssd_raw);        // [Q][NS]
  ssd_bf16* Xh = Bs + SSD_Q * NS;                              // [Q][PS]
  ssd_bf16* Xl = Xh + SSD_Q * PS;
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, p0 = blockIdx.z * SSD_PT;
  const int pt = P - p0 < SSD_PT ? P - p0 : SSD_PT;
  int b, t0, n, in_seq;
  if (!ssd_find_piece(blockIdx.x, SSD_Q, seq_start, B, &b, &t0, &n, &in_seq)) return;
  const int g = h / (H / G);
  const ssd_bf16* bsrc = xbc + (size_t)t0 * channels + H * P + g * N;
  const int nc = N / 8;
  for (int i = tid; i < SSD_Q * nc; i += 256) {
    const int row = i / nc, c = i - row * nc;
    ssd_bf16* dst = Bs + row * NS + c * 8;
    if (row < n) ssd_cp16(dst, bsrc + (size_t)row * channels + c * 8);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  ssd_chunk_decays(dtla, H, h, t0, n, L, dts, wt);
  const float2 Lend = L[SSD_Q - 1];
  if (blockIdx.z == 0 && tid == 0) decs[(size_t)blockIdx.x * H + h] = expf(Lend.x + Lend.y);
  const ssd_bf16* xsrc = xbc + (size_t)t0 * channels + h * P + p0;
  for (int i = tid; i < SSD_Q * (SSD_PT / 8); i += 256) {
    const int row = i / (SSD_PT / 8), c = (i - row * (SSD_PT / 8)) * 8;
    uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
    if (row < n && c < pt) {
      const uint4 v = *reinterpret_cast<const uint4*>(xsrc + (size_t)row * channels + c);
      const float wgt = expf(ssd_diff(Lend, L[row])) * dts[row];
      const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&v);
      const float2 a = __bfloat1622float2(q[0]), bb = __bfloat1622float2(q[1]), cc = __bfloat1622float2(q[2]),
                   d = __bfloat1622float2(q[3]);
      ssd_split2(a.x * wgt, a.y * wgt, hi.x, lo.x);
      ssd_split2(bb.x * wgt, bb.y * wgt, hi.y, lo.y);
      ssd_split2(cc.x * wgt, cc.y * wgt, hi.z, lo.z);
      ssd_split2(d.x * wgt, d.y * wgt, hi.w, lo.w);
    }
    *reinterpret_cast<uint4*>(Xh + row * PS + c) = hi;
    *reinterpret_cast<uint4*>(Xl + row * PS + c) = lo;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int ksteps = (n + 15) / 16;
  float* E = ends + (((size_t)blockIdx.x * H + h) * N) * P + p0;
  for (int mt = warp; mt < N / 16; mt += 8) {
    float acc[SSD_PT / 8][4];
#pragma unroll
    for (int i = 0; i < SSD_PT / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    for (int ks = 0; ks < ksteps; ++ks) {
      unsigned a[4];
      {
        const int i = lane >> 3, r = lane & 7;
        ssd_ldm4t(a, Bs + (ks * 16 + (i >> 1) * 8 + r) * NS + mt * 16 + (i & 1) * 8);
      }
#pragma unroll
      for (int np = 0; np < SSD_PT / 16; ++np) {
        if (np * 16 >= pt) continue;
        const int i = lane >> 3, r = lane & 7;
        const int at = (ks * 16 + (i & 1) * 8 + r) * PS + np * 16 + (i >> 1) * 8;
        unsigned f[4];
        ssd_ldm4t(f, Xh + at);
        ssd_mma(acc[2 * np], a, f[0], f[1]);
        ssd_mma(acc[2 * np + 1], a, f[2], f[3]);
        ssd_ldm4t(f, Xl + at);
        ssd_mma(acc[2 * np], a, f[0], f[1]);
        ssd_mma(acc[2 * np + 1], a, f[2], f[3]);
      }
    }
    const int r0 = mt * 16 + (lane >> 2);
#pragma unroll
    for (int i = 0; i < SSD_PT / 8; ++i) {
      const int c = i * 8 + (lane & 3) * 2;
      if (i * 8 < pt) {
        *reinterpret_cast<float2*>(E + (size_t)r0 * P + c) = make_float2(acc[i][0], acc[i][1]);
        *reinterpret_cast<float2*>(E + (size_t)(r0 + 8) * P + c) = make_float2(acc[i][2], acc[i][3]);
      }
    }
  }
  pdl_launch_dependents();
}

// The state at each chunk's start, as two bfloat16 parts [chunks][H][N * P] each; the state after the last
// chunk goes back to the slot.  A thread owns four numbers of a head's state.
__global__ void __launch_bounds__(256)
ssd_chunk_carry_kernel(const float* __restrict__ ends, const float* __restrict__ decs, ssd_bf16* __restrict__ hi,
                       ssd_bf16* __restrict__ lo, float* __restrict__ state, const int* __restrict__ seq_start,
                       const int* __restrict__ seq_slot, int H, int NP) {
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int i = (blockIdx.x * 256 + threadIdx.x) * 4;
  int chunk = 0;
  for (int k = 0; k < b; ++k) chunk += (seq_start[k + 1] - seq_start[k] + SSD_Q - 1) / SSD_Q;
  const int n_chunks = (seq_start[b + 1] - seq_start[b] + SSD_Q - 1) / SSD_Q;
  if (i < NP && n_chunks > 0) {
    float* S = state + ((size_t)seq_slot[b] * H + h) * NP + i;
    float4 s = *reinterpret_cast<const float4*>(S);
    constexpr int PF = 4;
    for (int c0 = 0; c0 < n_chunks; c0 += PF) {
      float4 e[PF];
      float d[PF];
#pragma unroll
      for (int k = 0; k < PF; ++k) {
        const int c = c0 + k < n_chunks ? c0 + k : n_chunks - 1;
        e[k] = *reinterpret_cast<const float4*>(ends + ((size_t)(chunk + c) * H + h) * NP + i);
        d[k] = decs[(size_t)(chunk + c) * H + h];
      }
#pragma unroll
      for (int k = 0; k < PF; ++k) {
        if (c0 + k >= n_chunks) continue;
        const size_t at = ((size_t)(chunk + c0 + k) * H + h) * NP + i;
        uint2 vh, vl;
        ssd_split2(s.x, s.y, vh.x, vl.x);
        ssd_split2(s.z, s.w, vh.y, vl.y);
        *reinterpret_cast<uint2*>(hi + at) = vh;
        *reinterpret_cast<uint2*>(lo + at) = vl;
        s.x = fmaf(d[k], s.x, e[k].x); s.y = fmaf(d[k], s.y, e[k].y);
        s.z = fmaf(d[k], s.z, e[k].z); s.w = fmaf(d[k], s.w, e[k].w);
      }
    }
    *reinterpret_cast<float4*>(S) = s;
  }
  pdl_launch_dependents();
}

// y of every (chunk, `hpb` heads of one group, 64 columns).  A warp owns 16 of the chunk's tokens; its
// products C_t . B_s stay in registers and serve every head of the block; a head's x and state parts come
// through `nbuf` buffers, the next head's on their way while this one is worked on.
__global__ void __launch_bounds__(256, 1)
ssd_chunk_out_kernel(const ssd_bf16* __restrict__ xbc, const float2* __restrict__ dtla, const float* __restrict__ D,
                     const ssd_bf16* __restrict__ hi, const ssd_bf16* __restrict__ lo, float* __restrict__ y,
                     const int* __restrict__ seq_start, int B, int H, int G, int N, int P, int channels, int hpb,
                     int nbuf) {
  extern __shared__ __align__(16) unsigned char ssd_raw[];
  __shared__ float2 L[2][SSD_Q];
  __shared__ float dts[2][SSD_Q];
  __shared__ double wt[4];
  const int NS = N + SSD_PAD, PS = SSD_PT + SSD_PAD;
  ssd_bf16* Cs = reinterpret_cast<ssd_bf16*>(ssd_raw);        // [Q][NS]
  ssd_bf16* Bs = Cs + SSD_Q * NS;                              // [Q][NS]
  ssd_bf16* bufs = Bs + SSD_Q * NS;                            // nbuf x { x [Q][PS], hi [N][PS], lo [N][PS] }
  const int buf_elems = (SSD_Q + 2 * N) * PS;
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h0 = blockIdx.y * hpb, p0 = blockIdx.z * SSD_PT;
  const int pt = P - p0 < SSD_PT ? P - p0 : SSD_PT;
  int b, t0, n, in_seq;
  if (!ssd_find_piece(blockIdx.x, SSD_Q, seq_start, B, &b, &t0, &n, &in_seq)) return;
  const int g = h0 / (H / G);
  const int nc = N / 8, pc = pt / 8;
  {
    const ssd_bf16* src = xbc + (size_t)t0 * channels + H * P + g * N;
    for (int i = tid; i < SSD_Q * nc; i += 256) {
      const int row = i / nc, c = i - row * nc;
      ssd_bf16 *db = Bs + row * NS + c * 8, *dc = Cs + row * NS + c * 8;
      if (row < n) {
        ssd_cp16(db, src + (size_t)row * channels + c * 8);
        ssd_cp16(dc, src + (size_t)row * channels + G * N + c * 8);
      } else {
        *reinterpret_cast<uint4*>(db) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(dc) = make_uint4(0, 0, 0, 0);
      }
    }
  }
  auto fetch = [&](int h, int buf) {
    ssd_bf16* X = bufs + buf * buf_elems;
    ssd_bf16 *Sh = X + SSD_Q * PS, *Sl = Sh + N * PS;
    const ssd_bf16* xsrc = xbc + (size_t)t0 * channels + h * P + p0;
    for (int i = tid; i < SSD_Q * pc; i += 256) {
      const int row = i / pc, c = (i - row * pc) * 8;
      if (row < n) ssd_cp16(X + row * PS + c, xsrc + (size_t)row * channels + c);
      else *reinterpret_cast<uint4*>(X + row * PS + c) = make_uint4(0, 0, 0, 0);
    }
    const size_t base = (((size_t)blockIdx.x * H + h) * N) * P + p0;
    for (int i = tid; i < N * pc; i += 256) {
      const int row = i / pc, c = (i - row * pc) * 8;
      ssd_cp16(Sh + row * PS + c, hi + base + (size_t)row * P + c);
      ssd_cp16(Sl + row * PS + c, lo + base + (size_t)row * P + c);
    }
  };
  fetch(h0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  ssd_chunk_decays(dtla, H, h0, t0, n, L[0], dts[0], wt);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  const int rows_here = n - warp * 16;           // of this warp's 16 tokens; a warp without tokens only helps to load
  float sc[SSD_Q / 8][4];
#pragma unroll
  for (int i = 0; i < SSD_Q / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.0f;
  if (rows_here > 0) {
    for (int kk = 0; kk < N / 16; ++kk) {
      unsigned a[4];
      ssd_ldm4(a, Cs + (warp * 16 + (lane & 15)) * NS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < SSD_Q / 16; ++np) {
        if (np > warp) continue;
        unsigned f[4];
        ssd_ldm4(f, Bs + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * NS + kk * 16 + ((lane >> 3) & 1) * 8);
        ssd_mma(sc[2 * np], a, f[0], f[1]);
        ssd_mma(sc[2 * np + 1], a, f[2], f[3]);
      }
    }
  }
  const int ta = warp * 16 + (lane >> 2), tb = ta + 8;      // this thread's two tokens of the chunk
  for (int k = 0; k < hpb; ++k) {
    const int h = h0 + k, buf = nbuf == 2 ? (k & 1) : 0;
    const float2* Lk = L[k & 1];
    const float* dk = dts[k & 1];
    if (nbuf == 2 && k + 1 < hpb) fetch(h + 1, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const ssd_bf16* X = bufs + buf * buf_elems;
    const ssd_bf16 *Sh = X + SSD_Q * PS, *Sl = Sh + N * PS;
    if (rows_here > 0) {
      float acc[SSD_PT / 8][4];
#pragma unroll
      for (int i = 0; i < SSD_PT / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
      // what the state at the chunk's start gives
      for (int kk = 0; kk < N / 16; ++kk) {
        unsigned a[4];
        ssd_ldm4(a, Cs + (warp * 16 + (lane & 15)) * NS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int np = 0; np < SSD_PT / 16; ++np) {
          if (np * 16 >= pt) continue;
          const int i = lane >> 3, r = lane & 7;
          const int at = (kk * 16 + (i & 1) * 8 + r) * PS + np * 16 + (i >> 1) * 8;
          unsigned f[4];
          ssd_ldm4t(f, Sh + at);
          ssd_mma(acc[2 * np], a, f[0], f[1]);
          ssd_mma(acc[2 * np + 1], a, f[2], f[3]);
          ssd_ldm4t(f, Sl + at);
          ssd_mma(acc[2 * np], a, f[0], f[1]);
          ssd_mma(acc[2 * np + 1], a, f[2], f[3]);
        }
      }
      const float2 La = Lk[ta], Lb = Lk[tb];
      const float ea = expf(La.x + La.y), eb = expf(Lb.x + Lb.y);
#pragma unroll
      for (int i = 0; i < SSD_PT / 8; ++i) {
        acc[i][0] *= ea; acc[i][1] *= ea;
        acc[i][2] *= eb; acc[i][3] *= eb;
      }
      // the chunk's own tokens up to each token
#pragma unroll
      for (int ks = 0; ks < SSD_Q / 16; ++ks) {
        if (ks > warp) continue;
        unsigned mh[4], ml[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int s0 = ks * 16 + half * 8 + (lane & 3) * 2, s1 = s0 + 1;
          const float2 L0 = Lk[s0], L1 = Lk[s1];
          const float d0 = dk[s0], d1 = dk[s1];
          const float (&v)[4] = sc[2 * ks + half];
          const float m00 = s0 <= ta ? v[0] * (expf(ssd_diff(La, L0)) * d0) : 0.0f;
          const float m01 = s1 <= ta ? v[1] * (expf(ssd_diff(La, L1)) * d1) : 0.0f;
          const float m10 = s0 <= tb ? v[2] * (expf(ssd_diff(Lb, L0)) * d0) : 0.0f;
          const float m11 = s1 <= tb ? v[3] * (expf(ssd_diff(Lb, L1)) * d1) : 0.0f;
          ssd_split2(m00, m01, mh[2 * half], ml[2 * half]);
          ssd_split2(m10, m11, mh[2 * half + 1], ml[2 * half + 1]);
        }
#pragma unroll
        for (int np = 0; np < SSD_PT / 16; ++np) {
          if (np * 16 >= pt) continue;
          const int i = lane >> 3, r = lane & 7;
          unsigned f[4];
          ssd_ldm4t(f, X + (ks * 16 + (i & 1) * 8 + r) * PS + np * 16 + (i >> 1) * 8);
          ssd_mma(acc[2 * np], mh, f[0], f[1]);
          ssd_mma(acc[2 * np + 1], mh, f[2], f[3]);
          ssd_mma(acc[2 * np], ml, f[0], f[1]);
          ssd_mma(acc[2 * np + 1], ml, f[2], f[3]);
        }
      }
      const float Dh = D[h];
#pragma unroll
      for (int i = 0; i < SSD_PT / 8; ++i) {
        const int c = i * 8 + (lane & 3) * 2;
        if (i * 8 >= pt) continue;
        if (ta < n) {
          const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(X + ta * PS + c));
          *reinterpret_cast<float2*>(y + (size_t)(t0 + ta) * H * P + h * P + p0 + c) =
              make_float2(fmaf(Dh, xv.x, acc[i][0]), fmaf(Dh, xv.y, acc[i][1]));
        }
        if (tb < n) {
          const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(X + tb * PS + c));
          *reinterpret_cast<float2*>(y + (size_t)(t0 + tb) * H * P + h * P + p0 + c) =
              make_float2(fmaf(Dh, xv.x, acc[i][2]), fmaf(Dh, xv.y, acc[i][3]));
        }
      }
    }
    if (k + 1 < hpb) {
      if (nbuf == 1) {
        __syncthreads();
        fetch(h + 1, 0);
        asm volatile("cp.async.commit_group;" ::: "memory");
      }
      ssd_chunk_decays(dtla, H, h + 1, t0, n, L[(k + 1) & 1], dts[(k + 1) & 1], wt);
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      __syncthreads();
    }
  }
  pdl_launch_dependents();
}

static bool ssd_chunk_takes(int N, int P) { return N % 16 == 0 && N >= 16 && N <= 256 && P % 16 == 0 && P >= 16; }

// Floats of scratch that the chunked form needs for a step of T tokens of B sequences (0: sizes it does not take).
extern "C" long long tl_ssd_chunk_scratch(int T, int B, int H, int N, int P) {
  if (!ssd_chunk_takes(N, P)) return 0;
  const long long chunks = T / SSD_Q + B;
  return 2 * chunks * H * N * P + (chunks * H + 3) / 4 * 4;
}

extern "C" int tl_ssd_chunked(const void* xbc, const float* dtla, const float* D, float* state, float* y,
                              const int* seq_start, const int* seq_slot, int T, int B, int H, int G, int N, int P,
                              int channels, float* scratch, int num_sms, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (H < 1 || G < 1 || H % G || channels < H * P + 2 * G * N || scratch == nullptr) return TL_ERR_BAD_ARG;
  if (!ssd_chunk_takes(N, P) || channels % 8 || ((uintptr_t)xbc & 15) || ((uintptr_t)scratch & 15) ||
      ((uintptr_t)state & 15) || H > 65535 || B > 65535)
    return TL_ERR_UNSUPPORTED;
  const int chunks = T / SSD_Q + B, ptiles = (P + SSD_PT - 1) / SSD_PT;
  if (ptiles > 65535) return TL_ERR_UNSUPPORTED;
  const size_t per = (size_t)chunks * H * N * P;
  float* ends = scratch;
  ssd_bf16 *hi = (ssd_bf16*)(scratch + per), *lo = hi + per;
  float* decs = scratch + 2 * per;
  const size_t NS = N + SSD_PAD, PS = SSD_PT + SSD_PAD;
  const size_t sm1 = (SSD_Q * NS + 2 * SSD_Q * PS) * 2;
  const size_t one = (2 * SSD_Q * NS + (SSD_Q + 2 * (size_t)N) * PS) * 2, more = (SSD_Q + 2 * (size_t)N) * PS * 2;
  const size_t most = 223 * 1024;       // and some 3 KB that are not dynamic
  if (one > most) return TL_ERR_UNSUPPORTED;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ssd_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(ssd_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most) != cudaSuccess)
      return TL_ERR_UNSUPPORTED;
    set = true;
  }
  // heads of a group that share a block: as many as still leave about two blocks per SM
  int hpb = 1;
  while (hpb < 8 && (H / G) % (2 * hpb) == 0 && (long long)chunks * (H / (2 * hpb)) * ptiles >= 2LL * num_sms) hpb *= 2;
  const int nbuf = (hpb > 1 && one + more <= most) ? 2 : 1;
  int rc = tl_launch(ssd_chunk_state_kernel, dim3(chunks, H, ptiles), dim3(256), sm1, stream, (const ssd_bf16*)xbc,
                     (const float2*)dtla, ends, decs, seq_start, B, H, G, N, P, channels);
  if (rc != 0) return rc;
  rc = tl_launch(ssd_chunk_carry_kernel, dim3((N * P / 4 + 255) / 256, H, B), dim3(256), 0, stream, (const float*)ends,
                 (const float*)decs, hi, lo, state, seq_start, seq_slot, H, N * P);
  if (rc != 0) return rc;
  return tl_launch(ssd_chunk_out_kernel, dim3(chunks, H / hpb, ptiles), dim3(256), one + (nbuf == 2 ? more : 0), stream,
                   (const ssd_bf16*)xbc, (const float2*)dtla, D, (const ssd_bf16*)hi, (const ssd_bf16*)lo, y, seq_start, B,
                   H, G, N, P, channels, hpb, nbuf);
}
#endif
