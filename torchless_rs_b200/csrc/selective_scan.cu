// The selective scan of a state-space layer whose every channel c keeps `N` numbers, each with a decay rate of
// its own:
//   dt = softplus(zdt_c + b_c),   S_c,n <- exp(dt A_c,n) S_c,n + dt x_c B_n,
//   y_c = (sum_n S_c,n C_n + D_c x_c) * silu(z_c)                                    (A < 0, given)
// over each sequence's tokens of the step, from and into the state in the sequence's slot (32-bit).  Step sizes,
// decays, state, sums and the gate are 32-bit; x, z, B and C come in the activation type, y leaves in it.
//
// A block owns (sequence, a run of channels) and has two halves that work at the same time on neighbouring tiles of
// TT tokens.  The first half runs the recurrence: a channel's states lie in the registers of LPC neighbouring lanes,
// NS each (padded with states that stay zero), so a token costs a thread NS exponentials, NS multiply-adds for the
// state and NS for the output, and the state crosses memory once per step whatever its tokens; the lanes' sums of a
// channel are added by shuffles, four tokens in one go (each lane ends with another token's sum).  The second half
// copies what the tiles ahead need into a ring in shared memory (asynchronously, `AHEAD` tiles before they are used),
// turns step sizes into (dt, dt x) for the tile that comes next, and gates and writes the outputs of the tile before;
// each of its threads reads from the ring only what it copied there itself.
#include "common.cuh"

#define SC_HALF 128       // threads of each half
template <int U> struct ScInt { static constexpr int value = U; };

#if TL_DTYPE == 0
__device__ __forceinline__ float sc_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sc_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
// e^x
#define SC_RATE 1.0f
__device__ __forceinline__ float sc_decay(float x) { return expf(x); }
#else
__device__ __forceinline__ float sc_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
// log(1 + u) = 2 atanh(r), r = u / (2 + u) <= 1/3 for u = e^-|x| <= 1: the series 2 r (1 + r^2/3 + r^4/5 + ...), whose
// terms past r^14/15 are below 4e-9 of it
__device__ __forceinline__ float sc_softplus(float x) {
  const float u = __expf(-fabsf(x)), r = __fdividef(u, 2.0f + u), q = r * r;
  float p = fmaf(q, 1.0f / 15.0f, 1.0f / 13.0f);
  p = fmaf(p, q, 1.0f / 11.0f);
  p = fmaf(p, q, 1.0f / 9.0f);
  p = fmaf(p, q, 1.0f / 7.0f);
  p = fmaf(p, q, 1.0f / 5.0f);
  p = fmaf(p, q, 1.0f / 3.0f);
  p = fmaf(p, q, 1.0f);
  return fmaxf(x, 0.0f) + 2.0f * r * p;
}
// 2^x by the hardware's approximation (relative error about 2^-22); the rates come times log2(e)
#define SC_RATE 1.4426950408889634f
__device__ __forceinline__ float sc_decay(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
#endif

// V neighbouring numbers as 32-bit.
template <int V, typename T>
__device__ __forceinline__ void sc_get(const T* p, float (&v)[V]) {
  if (V == 1) {
    v[0] = to_f32(*p);
  } else if (sizeof(T) == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[V > 1 ? 1 : 0] = f.y; v[V > 2 ? 2 : 0] = f.z; v[V > 3 ? 3 : 0] = f.w;
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    v[0] = a.x; v[V > 1 ? 1 : 0] = a.y; v[V > 2 ? 2 : 0] = b.x; v[V > 3 ? 3 : 0] = b.y;
  }
}
// V neighbouring numbers into shared memory, asynchronously where V is 4.
template <int V, typename T>
__device__ __forceinline__ void sc_copy(T* dst, const T* src) {
  if (V == 4) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(d), "l"(src), "n"(4 * (int)sizeof(T)) : "memory");
  } else {
    *dst = *src;
  }
}
template <int V>
__device__ __forceinline__ void sc_put(act_t* p, const float (&v)[V]) {
  if (V == 1) {
    *p = from_f32<act_t>(v[0]);
  } else if (sizeof(act_t) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[V > 1 ? 1 : 0], v[V > 2 ? 2 : 0], v[V > 3 ? 3 : 0]);
  } else {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[V > 1 ? 1 : 0]);
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[V > 2 ? 2 : 0], v[V > 3 ? 3 : 0]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  }
}

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
  if (NS == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[NS > 1 ? 1 : 0] = f.y;
    return;
  }
#pragma unroll
  for (int i = 0; i + 3 < NS; i += 4) {
    const float4 f = *reinterpret_cast<const float4*>(p + i);
    v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
  }
}

// x: [T, ldx]; zdt: [T, channels] 32-bit; bc: [T, ldbc] with B at column col_b and C at col_b + N; z: [T, ldz];
// A: [channels, N]; state: [slots, channels, N]; y: [T, channels].  V: channels a thread of the second half takes at
// a time (4: 16- and 8-byte accesses).
template <int LPC, int NS, int TT>
struct ScSizes {
  static constexpr int CH = SC_HALF / LPC;             // channels of a block
  static constexpr int NP = LPC * NS;                  // states of a channel, padded
  static constexpr int YP = CH + (CH >= 32 ? 8 : 4);   // (the four tokens a quad of lanes writes fall into other banks)
  static constexpr int AHEAD = NP <= 64 ? 3 : 1;
  static constexpr int GROUP = NS > 4 && TT > 8 ? 8 : TT;   // tokens whose operands a thread of the first half reads in one go
  static constexpr int RING = AHEAD + 3;               // from the tile before to the one fetched last
  // offsets in shared memory, bytes
  static constexpr int B = 0, C = B + 2 * TT * NP * 4, DX = C + 2 * TT * NP * 4, Y = DX + 2 * TT * CH * 8;
  static constexpr int R_DT = Y + 2 * TT * YP * 4, R_X = R_DT + RING * TT * CH * 4;
  static constexpr int R_Z = R_X + RING * TT * CH * (int)sizeof(act_t);
  static constexpr int R_BC = R_Z + RING * TT * CH * (int)sizeof(act_t);
  static constexpr int BYTES = R_BC + RING * TT * 2 * NP * (int)sizeof(act_t);
};

template <int LPC, int NS, int TT, int V>
__global__ void __launch_bounds__(2 * SC_HALF)
selective_scan_kernel(const act_t* __restrict__ x, int ldx, const float* __restrict__ zdt,
                      const float* __restrict__ dt_bias, const act_t* __restrict__ bc, int ldbc, int col_b,
                      const float* __restrict__ A, const float* __restrict__ D, const act_t* __restrict__ z, int ldz,
                      float* __restrict__ state, act_t* __restrict__ y, const int* __restrict__ seq_start,
                      const int* __restrict__ seq_slot, int channels, int N) {
  using Z = ScSizes<LPC, NS, TT>;
  constexpr int CH = Z::CH, NP = Z::NP, YP = Z::YP, RING = Z::RING, AHEAD = Z::AHEAD;
  extern __shared__ __align__(16) unsigned char sc_smem[];
  float(*Bs)[TT][NP] = reinterpret_cast<float(*)[TT][NP]>(sc_smem + Z::B);
  float(*Cs)[TT][NP] = reinterpret_cast<float(*)[TT][NP]>(sc_smem + Z::C);
  float2(*dx)[TT][CH] = reinterpret_cast<float2(*)[TT][CH]>(sc_smem + Z::DX);      // (dt, dt x)
  float(*ys)[TT][YP] = reinterpret_cast<float(*)[TT][YP]>(sc_smem + Z::Y);
  const bool second = threadIdx.x >= SC_HALF;
  const int tid = threadIdx.x % SC_HALF;
  const int c0 = blockIdx.x * CH, b = blockIdx.y;
  if (!second) {
    // ---- the recurrence
    const int l = tid % LPC, cl = tid / LPC, c = c0 + cl;
    float a[NS], s[NS];
    sc_load<NS>(A + (size_t)c * N, l * NS, N, c < channels, SC_RATE, a);     // a weight: before the wait
    pdl_wait();
    const int n_tok = seq_start[b + 1] - seq_start[b];
    if (n_tok <= 0) return;
    float* S = state + ((size_t)seq_slot[b] * channels + c) * N;
    sc_load<NS>(S, l * NS, N, c < channels, 1.0f, s);
    __syncthreads();
    // U tokens from place p0 of a tile on (a place past the sequence's end has a step size of zero, which leaves
    // the state as it is)
    auto run = [&](auto u_tag, int buf, int p0) {
      constexpr int U = decltype(u_tag)::value;
      float part[U];
      float2 d[U];
      float bv[U][NS], cv[U][NS];
#pragma unroll
      for (int p = 0; p < U; ++p) {
        d[p] = dx[buf][p0 + p][cl];
        sc_read<NS>(&Bs[buf][p0 + p][l * NS], bv[p]);
        sc_read<NS>(&Cs[buf][p0 + p][l * NS], cv[p]);
      }
#pragma unroll
      for (int p = 0; p < U; ++p) {
        part[p] = 0.0f;
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          s[i] = fmaf(sc_decay(d[p].x * a[i]), s[i], d[p].y * bv[p][i]);
          part[p] = fmaf(s[i], cv[p][i], part[p]);
        }
      }
#pragma unroll
      for (int q = 0; q < U; q += 4) {
        if (LPC >= 4) {
          // four tokens' sums over the channel's lanes: two exchanges leave lane j of a quad with token j's
          const bool hi2 = (l & 2) != 0, hi1 = (l & 1) != 0;
          const float u0 = __shfl_xor_sync(0xffffffffu, hi2 ? part[q] : part[q + 2], 2);
          const float u1 = __shfl_xor_sync(0xffffffffu, hi2 ? part[q + 1] : part[q + 3], 2);
          const float v0 = (hi2 ? part[q + 2] : part[q]) + u0, v1 = (hi2 ? part[q + 3] : part[q + 1]) + u1;
          const float w = __shfl_xor_sync(0xffffffffu, hi1 ? v0 : v1, 1);
          float v = (hi1 ? v1 : v0) + w;
#pragma unroll
          for (int o = 4; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (l < 4) ys[buf][p0 + q + l][cl] = v;
        } else {
#pragma unroll
          for (int p = 0; p < 4; ++p) {
            float v = part[q + p];
#pragma unroll
            for (int o = 1; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (l == 0) ys[buf][p0 + q + p][cl] = v;
          }
        }
      }
    };
    for (int tb = 0, buf = 0; tb < n_tok; tb += TT, buf ^= 1) {
      const int cnt = n_tok - tb < TT ? n_tok - tb : TT;
      if (cnt <= 4) {
        run(ScInt<4>(), buf, 0);
      } else {
#pragma unroll 1
        for (int p0 = 0; p0 < cnt; p0 += Z::GROUP) run(ScInt<Z::GROUP>(), buf, p0);
      }
      __syncthreads();
    }
    pdl_launch_dependents();
    sc_store<NS>(S, l * NS, N, c < channels, s);
    return;
  }
  // ---- what goes in and what comes out
  constexpr int PER = (TT * CH / V + SC_HALF - 1) / SC_HALF;            // pieces (token, V channels) per thread and tile
  constexpr int PBC = (TT * 2 * NP / V + SC_HALF - 1) / SC_HALF;        // pieces of B and C
  constexpr int CV = CH / V, ET = SC_HALF / CV;   // pieces of a token, tokens between a thread's pieces
  const int ec = (tid % CV) * V, et = tid / CV;
  const bool live = c0 + ec < channels;
  float(*r_dt)[TT][CH] = reinterpret_cast<float(*)[TT][CH]>(sc_smem + Z::R_DT);
  act_t(*r_x)[TT][CH] = reinterpret_cast<act_t(*)[TT][CH]>(sc_smem + Z::R_X);
  act_t(*r_z)[TT][CH] = reinterpret_cast<act_t(*)[TT][CH]>(sc_smem + Z::R_Z);
  act_t(*r_bc)[TT][2 * NP] = reinterpret_cast<act_t(*)[TT][2 * NP]>(sc_smem + Z::R_BC);
  float bias[V], Dc[V];
#pragma unroll
  for (int e = 0; e < V; ++e) bias[e] = Dc[e] = 0.0f;
  if (live) { sc_get<V>(dt_bias + c0 + ec, bias); sc_get<V>(D + c0 + ec, Dc); }
  pdl_wait();
  const int t0 = seq_start[b], t1 = seq_start[b + 1];
  if (t0 >= t1) return;
  const int tiles = (t1 - t0 + TT - 1) / TT;
  auto fetch = [&](int i) {                       // tile i into its place of the ring
    const int tb = t0 + i * TT, slot = i % RING;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int p = et + k * ET, t = tb + p;
      if (live && p < TT && t < t1) {
        sc_copy<V>(&r_dt[slot][p][ec], zdt + (size_t)t * channels + c0 + ec);
        sc_copy<V>(&r_x[slot][p][ec], x + (size_t)t * ldx + c0 + ec);
        sc_copy<V>(&r_z[slot][p][ec], z + (size_t)t * ldz + c0 + ec);
      }
    }
#pragma unroll
    for (int k = 0; k < PBC; ++k) {
      const int q = (tid + k * SC_HALF) * V;
      const int p = q / (2 * NP), r = q - p * 2 * NP, n = r < NP ? r : r - NP;
      if (p < TT && tb + p < t1 && n < N)
        sc_copy<V>(&r_bc[slot][p][r], bc + (size_t)(tb + p) * ldbc + col_b + (r < NP ? 0 : N) + n);
    }
    if (V == 4) asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto stage = [&](int i) {                       // tile i, which has arrived, for the first half
    const int tb = t0 + i * TT, slot = i % RING, buf = i & 1;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int p = et + k * ET;
      if (p >= TT) continue;
      float dt[V], xv[V];
#pragma unroll
      for (int e = 0; e < V; ++e) dt[e] = xv[e] = 0.0f;
      if (live && tb + p < t1) {
        sc_get<V>(&r_dt[slot][p][ec], dt);
        sc_get<V>(&r_x[slot][p][ec], xv);
#pragma unroll
        for (int e = 0; e < V; ++e) dt[e] = sc_softplus(dt[e] + bias[e]);
      }
      if (V == 4) {
        float4* q = reinterpret_cast<float4*>(&dx[buf][p][ec]);
        constexpr int e1 = V > 1 ? 1 : 0, e2 = V > 2 ? 2 : 0, e3 = V > 3 ? 3 : 0;
        q[0] = make_float4(dt[0], dt[0] * xv[0], dt[e1], dt[e1] * xv[e1]);
        q[1] = make_float4(dt[e2], dt[e2] * xv[e2], dt[e3], dt[e3] * xv[e3]);
      } else {
        dx[buf][p][ec] = make_float2(dt[0], dt[0] * xv[0]);
      }
    }
#pragma unroll
    for (int k = 0; k < PBC; ++k) {
      const int q = (tid + k * SC_HALF) * V;
      const int p = q / (2 * NP), r = q - p * 2 * NP, n = r < NP ? r : r - NP;
      if (p >= TT) continue;
      float v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.0f;
      if (tb + p < t1 && n < N) sc_get<V>(&r_bc[slot][p][r], v);
      float* dst = r < NP ? &Bs[buf][p][r] : &Cs[buf][p][r - NP];
      if (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[V > 1 ? 1 : 0], v[V > 2 ? 2 : 0], v[V > 3 ? 3 : 0]);
      else *dst = v[0];
    }
  };
  auto finish = [&](int i) {                      // the outputs of tile i
    const int tb = t0 + i * TT, slot = i % RING, buf = i & 1;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int p = et + k * ET;
      if (!live || p >= TT || tb + p >= t1) continue;
      float xv[V], zv[V], o[V];
      sc_get<V>(&r_x[slot][p][ec], xv);
      sc_get<V>(&r_z[slot][p][ec], zv);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = fmaf(Dc[e], xv[e], ys[buf][p][ec + e]) * sc_silu(zv[e]);
      sc_put<V>(y + (size_t)(tb + p) * channels + c0 + ec, o);
    }
  };
#pragma unroll
  for (int i = 0; i <= AHEAD; ++i) fetch(i);      // (a tile past the end copies nothing)
  if (V == 4) asm volatile("cp.async.wait_group %0;" ::"n"(AHEAD) : "memory");
  stage(0);
  __syncthreads();
  for (int i = 0; i < tiles; ++i) {
    fetch(i + AHEAD + 1);
    if (i > 0) finish(i - 1);
    if (i + 1 < tiles) {
      if (V == 4) asm volatile("cp.async.wait_group %0;" ::"n"(AHEAD) : "memory");
      stage(i + 1);
    }
    __syncthreads();
  }
  pdl_launch_dependents();
  finish(tiles - 1);
}

template <int LPC, int NS, int TT>
static int sc_launch(const act_t* x, int ldx, const float* zdt, const float* dt_bias, const act_t* bc, int ldbc,
                     int col_b, const float* A, const float* D, const act_t* z, int ldz, float* state, act_t* y,
                     const int* seq_start, const int* seq_slot, int B, int channels, int N, cudaStream_t stream) {
  const dim3 grid((channels + SC_HALF / LPC - 1) / (SC_HALF / LPC), B);
  const uintptr_t at = (uintptr_t)x | (uintptr_t)zdt | (uintptr_t)dt_bias | (uintptr_t)D | (uintptr_t)z | (uintptr_t)y;
  const bool quads = channels % 4 == 0 && N % 4 == 0 && ldx % 4 == 0 && ldz % 4 == 0 && ldbc % 4 == 0 && col_b % 4 == 0 &&
                     ((at | (uintptr_t)bc) & 15) == 0;
  constexpr int smem = ScSizes<LPC, NS, TT>::BYTES;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(selective_scan_kernel<LPC, NS, TT, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
        cudaFuncSetAttribute(selective_scan_kernel<LPC, NS, TT, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return TL_ERR_UNSUPPORTED;
    set = true;
  }
  return tl_launch(quads ? selective_scan_kernel<LPC, NS, TT, 4> : selective_scan_kernel<LPC, NS, TT, 1>, grid,
                   dim3(2 * SC_HALF), smem, stream, x, ldx, zdt, dt_bias, bc, ldbc, col_b, A, D, z, ldz, state, y,
                   seq_start, seq_slot, channels, N);
}

extern "C" int TL_NAME(tl_selective_scan)(const void* x, int ldx, const float* zdt, const float* dt_bias,
                                          const void* bc, int ldbc, int col_b, const float* A, const float* D,
                                          const void* z, int ldz, float* state, void* y, const int* seq_start,
                                          const int* seq_slot, int T, int B, int channels, int N, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (channels < 1 || N < 1 || col_b < 0) return TL_ERR_BAD_ARG;
  if (N > 512 || B > 65535) return TL_ERR_UNSUPPORTED;
#define SCAN(LPC_, NS_, TT_)                                                                                          \
  return sc_launch<LPC_, NS_, TT_>((const act_t*)x, ldx, zdt, dt_bias, (const act_t*)bc, ldbc, col_b, A, D,           \
                                   (const act_t*)z, ldz, state, (act_t*)y, seq_start, seq_slot, B, channels, N, stream)
  if (T <= 4 * B) {            // decode steps and the like: small blocks
    if (N <= 4) SCAN(2, 2, 4);
    if (N <= 8) SCAN(2, 4, 4);
    if (N <= 16) SCAN(4, 4, 4);
    if (N <= 32) SCAN(4, 8, 4);
    if (N <= 64) SCAN(8, 8, 4);
    if (N <= 128) SCAN(16, 8, 4);
  }
  if (N <= 4) SCAN(2, 2, 16);
  if (N <= 8) SCAN(2, 4, 16);
  if (N <= 16) SCAN(4, 4, 16);
  if (N <= 32) SCAN(4, 8, 16);
  if (N <= 64) SCAN(8, 8, 16);
  if (N <= 128) SCAN(16, 8, 16);
  if (N <= 256) SCAN(32, 8, 8);
  SCAN(32, 16, 4);
#undef SCAN
}
