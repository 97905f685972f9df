// The selective scan of a state-space layer whose every channel c keeps `N` numbers, each with a decay rate of
// its own:
//   dt = softplus(zdt_c + b_c),   S_c,n <- exp(dt A_c,n) S_c,n + dt x_c B_n,
//   y_c = (sum_n S_c,n C_n + D_c x_c) * silu(z_c)                                    (A < 0, given)
// over each sequence's tokens of the step, from and into the state in the sequence's slot (32-bit).  Step sizes,
// decays, state, sums and the gate are 32-bit; x, z, B and C come in the activation type, y leaves in it.
//
// A block owns (sequence, a run of channels); a channel's states lie in the registers of LPC neighbouring lanes,
// NS each (padded with states that stay zero), so a token costs a thread NS exponentials, NS multiply-adds for the state and NS for the output, and
// the state crosses memory once per step whatever its tokens.  Tokens come through shared memory TT at a
// time; what the next ones need from memory is asked for while these are worked on.  The lanes' sums of a
// channel are added by shuffles, four tokens in one go (each lane ends with another token's sum).
#include "common.cuh"

#define SC_THREADS 128

__device__ __forceinline__ float sc_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sc_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

#if TL_DTYPE == 0
// e^x
#define SC_RATE 1.0f
__device__ __forceinline__ float sc_decay(float x) { return expf(x); }
#else
// 2^x by the hardware's approximation (relative error about 2^-22); the rates come times log2(e)
#define SC_RATE 1.4426950408889634f
__device__ __forceinline__ float sc_decay(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
#endif

// A lane's NS numbers of a channel's N (those past N: zero) times `f`, and back.
template <int NS>
__device__ __forceinline__ void sc_load(const float* row, int n0, int N, bool live, float f, float (&v)[NS]) {
  if (NS % 4 == 0 && N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
      float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (live && n0 + i < N) q = *reinterpret_cast<const float4*>(row + n0 + i);
      v[i] = q.x * f; v[i + 1] = q.y * f; v[i + 2] = q.z * f; v[i + 3] = q.w * f;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) v[i] = live && n0 + i < N ? row[n0 + i] * f : 0.0f;
  }
}
template <int NS>
__device__ __forceinline__ void sc_store(float* row, int n0, int N, bool live, const float (&v)[NS]) {
  if (!live) return;
  if (NS % 4 == 0 && N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 4)
      if (n0 + i < N) *reinterpret_cast<float4*>(row + n0 + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (n0 + i < N) row[n0 + i] = v[i];
  }
}

template <int NS>
__device__ __forceinline__ void sc_read(const float* p, float (&v)[NS]) {
  static_assert(NS % 4 == 0, "states per lane");
#pragma unroll
  for (int i = 0; i < NS; i += 4) {
    const float4 f = *reinterpret_cast<const float4*>(p + i);
    v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
  }
}

// x: [T, ldx]; zdt: [T, channels] 32-bit; bc: [T, ldbc] with B at column col_b and C at col_b + N; z: [T, ldz];
// A: [channels, N]; state: [slots, channels, N]; y: [T, channels].
template <int LPC, int NS, int TT>
__global__ void __launch_bounds__(SC_THREADS)
selective_scan_kernel(const act_t* __restrict__ x, int ldx, const float* __restrict__ zdt,
                      const float* __restrict__ dt_bias, const act_t* __restrict__ bc, int ldbc, int col_b,
                      const float* __restrict__ A, const float* __restrict__ D, const act_t* __restrict__ z, int ldz,
                      float* __restrict__ state, act_t* __restrict__ y, const int* __restrict__ seq_start,
                      const int* __restrict__ seq_slot, int channels, int N) {
  constexpr int CH = SC_THREADS / LPC;            // channels of a block
  constexpr int NP = LPC * NS;                    // states of a channel, padded
  constexpr int CP = CH + 1;
  constexpr int PER = (TT * CH + SC_THREADS - 1) / SC_THREADS;    // (token, channel) pairs per thread and tile
  constexpr int PBC = TT * NP * 2 / SC_THREADS;
  __shared__ __align__(16) float Bs[TT][NP], Cs[TT][NP];
  __shared__ float2 dx[TT][CP];                // (dt, dt x)
  __shared__ float ys[TT][CP];
  const int tid = threadIdx.x, l = tid % LPC, cl = tid / LPC;
  const int c0 = blockIdx.x * CH, c = c0 + cl, b = blockIdx.y;
  // rates, skip weights and biases are weights: asked for before the wait
  float a[NS], s[NS];
  sc_load<NS>(A + (size_t)c * N, l * NS, N, c < channels, SC_RATE, a);
  const int ec = tid % CH, et = tid / CH;         // this thread's channel, and first token, of a tile's pairs
  const bool live = c0 + ec < channels;
  const float bias = live ? dt_bias[c0 + ec] : 0.0f, Dc = live ? D[c0 + ec] : 0.0f;
  pdl_wait();
  const int t0 = seq_start[b], t1 = seq_start[b + 1];
  if (t0 >= t1) return;
  float* S = state + ((size_t)seq_slot[b] * channels + c) * N;
  sc_load<NS>(S, l * NS, N, c < channels, 1.0f, s);
  constexpr int ET = SC_THREADS / CH;             // tokens between a thread's pairs
  float rdt[PER], rx[PER], rz[PER], nz[PER], nx[PER];
  constexpr bool AHEAD = PBC <= 16;               // wide states: B and C are fetched when they are needed
  float rbc[AHEAD ? PBC : 1];
  auto fetch_bc = [&](int tb, int k) -> float {
    const int i = tid + k * SC_THREADS;
    const int p = i / (2 * NP), r = i - p * 2 * NP, n = r < NP ? r : r - NP;
    return tb + p < t1 && n < N ? to_f32(bc[(size_t)(tb + p) * ldbc + col_b + (r < NP ? 0 : N) + n]) : 0.0f;
  };
  auto fetch = [&](int tb) {
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int t = tb + et + k * ET;
      const bool ok = live && et + k * ET < TT && t < t1;
      rdt[k] = ok ? zdt[(size_t)t * channels + c0 + ec] : 0.0f;
      nx[k] = ok ? to_f32(x[(size_t)t * ldx + c0 + ec]) : 0.0f;
      nz[k] = ok ? to_f32(z[(size_t)t * ldz + c0 + ec]) : 0.0f;
    }
    if (AHEAD) {
#pragma unroll
      for (int k = 0; k < (AHEAD ? PBC : 1); ++k) rbc[k] = fetch_bc(tb, k);
    }
  };
  fetch(t0);
  for (int tb = t0; tb < t1; tb += TT) {
    const int cnt = t1 - tb < TT ? t1 - tb : TT;
    // the tile that was fetched goes to shared memory
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      if (et + k * ET >= TT) continue;
      const float dt = sc_softplus(rdt[k] + bias);
      rx[k] = nx[k];
      rz[k] = nz[k];
      dx[et + k * ET][ec] = make_float2(dt, dt * rx[k]);
    }
#pragma unroll
    for (int k = 0; k < PBC; ++k) {
      const int i = tid + k * SC_THREADS;
      const int p = i / (2 * NP), r = i - p * 2 * NP;
      const float v = AHEAD ? rbc[AHEAD ? k : 0] : fetch_bc(tb, k);
      if (r < NP) Bs[p][r] = v;
      else Cs[p][r - NP] = v;
    }
    __syncthreads();
    if (tb + TT < t1) fetch(tb + TT);
#pragma unroll 1
    for (int p0 = 0; p0 < cnt; p0 += 4) {
      float part[4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        part[p] = 0.0f;
        if (p0 + p < cnt) {
          const float2 d = dx[p0 + p][cl];
          float bv[NS], cv[NS];
          sc_read<NS>(&Bs[p0 + p][l * NS], bv);
          sc_read<NS>(&Cs[p0 + p][l * NS], cv);
#pragma unroll
          for (int i = 0; i < NS; ++i) {
            s[i] = fmaf(sc_decay(d.x * a[i]), s[i], d.y * bv[i]);
            part[p] = fmaf(s[i], cv[i], part[p]);
          }
        }
      }
      if (LPC >= 4) {
        // four tokens' sums over the channel's lanes: two exchanges leave lane j of a quad with token j's
        const bool hi2 = (l & 2) != 0, hi1 = (l & 1) != 0;
        const float u0 = __shfl_xor_sync(0xffffffffu, hi2 ? part[0] : part[2], 2);
        const float u1 = __shfl_xor_sync(0xffffffffu, hi2 ? part[1] : part[3], 2);
        const float v0 = (hi2 ? part[2] : part[0]) + u0, v1 = (hi2 ? part[3] : part[1]) + u1;
        const float w = __shfl_xor_sync(0xffffffffu, hi1 ? v0 : v1, 1);
        float v = (hi1 ? v1 : v0) + w;
#pragma unroll
        for (int o = 4; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (l < 4) ys[p0 + l][cl] = v;
      } else {
#pragma unroll
        for (int p = 0; p < 4; ++p) {
          float v = part[p];
#pragma unroll
          for (int o = 1; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (l == 0) ys[p0 + p][cl] = v;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int p = et + k * ET;
      if (live && p < cnt)
        y[(size_t)(tb + p) * channels + c0 + ec] = from_f32<act_t>(fmaf(Dc, rx[k], ys[p][ec]) * sc_silu(rz[k]));
    }
    // (the next tile's stores to ys come after the barrier that follows its staging)
  }
  pdl_launch_dependents();
  sc_store<NS>(S, l * NS, N, c < channels, s);
}

extern "C" int TL_NAME(tl_selective_scan)(const void* x, int ldx, const float* zdt, const float* dt_bias,
                                          const void* bc, int ldbc, int col_b, const float* A, const float* D,
                                          const void* z, int ldz, float* state, void* y, const int* seq_start,
                                          const int* seq_slot, int B, int channels, int N, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (channels < 1 || N < 1 || col_b < 0) return TL_ERR_BAD_ARG;
  if (N > 512 || B > 65535) return TL_ERR_UNSUPPORTED;
#define SCAN(LPC_, NS_, TT_)                                                                                         \
  return tl_launch(selective_scan_kernel<LPC_, NS_, TT_>, dim3((channels + SC_THREADS / LPC_ - 1) / (SC_THREADS / LPC_), B), \
                   dim3(SC_THREADS), 0, stream, (const act_t*)x, ldx, zdt, dt_bias, (const act_t*)bc, ldbc, col_b, A,  \
                   D, (const act_t*)z, ldz, state, (act_t*)y, seq_start, seq_slot, channels, N)
  if (N <= 4) SCAN(1, 4, 16);
  if (N <= 8) SCAN(2, 4, 16);
  if (N <= 16) SCAN(4, 4, 16);
  if (N <= 32) SCAN(4, 8, 16);
  if (N <= 64) SCAN(8, 8, 16);
  if (N <= 128) SCAN(16, 8, 16);
  if (N <= 256) SCAN(32, 8, 16);
  SCAN(32, 16, 8);
#undef SCAN
}
