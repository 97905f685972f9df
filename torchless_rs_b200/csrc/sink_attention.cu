// Softmax attention with grouped key/value heads whose scores are capped, whose window keeps the
// sequence's first keys, and whose denominator holds a learned "sink" logit per head; queries and
// keys are RMS-normed per head, the key and value sizes may differ, and every head's output is
// multiplied by a sigmoid gate.  CUDA cores; serves the true 32-bit path and every size.
//
//   score(i, j) = cap * tanh((q_i . k_j) * scale / cap)            (cap 0: no cap)
//   j is visible to i  iff  j <= i and (i - j < window or j < keep_first)   (window 0: every j <= i)
//   p(i, j) = exp(score) / (sum over visible j' of exp(score(i, j')) + exp(sink_h))
//   out_i = gate_i * sum_j p(i, j) v_j
//
// Keys and values come from the paged cache only (keys [page][kv head][TL_PAGE][dim], values
// transposed [page][kv head][vdim][TL_PAGE]); the step's own keys are written there first, so a
// position's result does not depend on the step or batch that computes it.
#include "common.cuh"

#define SA_THREADS 128
#define SA_MAX_DIM 512
#define SA_MAX_V 4          // value entries per thread: value sizes up to 512

// The step's projections (32-bit, one row per token: q heads, k heads, v heads side by side) get
// their biases; q and k are divided by their root mean square per head and multiplied by a weight
// vector shared by the heads; q goes to `q_out` (act_t), k and v into the token's place in the pages.
__global__ void __launch_bounds__(256)
qk_norm_cache_write_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ bias,
                           const float* __restrict__ qw, const float* __restrict__ kw, float eps,
                           act_t* __restrict__ q_out, act_t* __restrict__ k_pages, act_t* __restrict__ v_pages,
                           const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                           const int* __restrict__ seq_slot, const int* __restrict__ page_table,
                           int table_stride, int nh, int nkv, int dim, int vdim) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int pos = token_pos[t];
  const int slot = seq_slot[token_seq[t]];
  const int page = page_table[(size_t)slot * table_stride + pos / TL_PAGE];
  const int in_page = pos % TL_PAGE;
  const float* row = z + (size_t)t * ldz;
  const int k_off = nh * dim, v_off = (nh + nkv) * dim;
  // a warp per head; the heads of a token are spread over the blocks of a grid row
  for (int head = blockIdx.y * nwarps + warp; head < nh + 2 * nkv; head += gridDim.y * nwarps) {
    if (head < nh + nkv) {
      const bool is_q = head < nh;
      const int off = head * dim;                      // q heads, then k heads
      const float* w = is_q ? qw : kw;
      float ss = 0.0f;
      for (int d = lane; d < dim; d += 32) {
        const float v = row[off + d] + (bias != nullptr ? bias[off + d] : 0.0f);
        ss = fmaf(v, v, ss);
      }
      ss = warp_sum(ss);
      const float inv = w != nullptr ? 1.0f / sqrtf(ss / (float)dim + eps) : 1.0f;
      act_t* dst = is_q ? q_out + (size_t)t * nh * dim + (size_t)head * dim
                        : k_pages + (((size_t)page * nkv + (head - nh)) * TL_PAGE + in_page) * dim;
      for (int d = lane; d < dim; d += 32) {
        const float v = row[off + d] + (bias != nullptr ? bias[off + d] : 0.0f);
        dst[d] = from_f32<act_t>(w != nullptr ? v * inv * w[d] : v);
      }
    } else {
      const int g = head - nh - nkv;
      const int off = v_off + g * vdim;
      act_t* dst = v_pages + ((size_t)page * nkv + g) * vdim * TL_PAGE + in_page;
      for (int d = lane; d < vdim; d += 32)
        dst[(size_t)d * TL_PAGE] = from_f32<act_t>(row[off + d] + (bias != nullptr ? bias[off + d] : 0.0f));
    }
  }
  (void)k_off;
}

extern "C" int TL_NAME(tl_qk_norm_cache_write)(const float* z, int ldz, const float* bias, const float* qw,
                                               const float* kw, float eps, void* q_out, void* k_pages,
                                               void* v_pages, const int* token_pos, const int* token_seq,
                                               const int* seq_slot, const int* page_table, int table_stride,
                                               int T, int nh, int nkv, int dim, int vdim, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nh < 1 || nkv < 1 || dim < 1 || vdim < 1) return TL_ERR_BAD_ARG;
  // few tokens: a block of four warps per four heads, so that a token's heads are worked on at once; many
  // tokens: a block per token
  const int heads = nh + 2 * nkv;
  const bool few = T < 512;
  const dim3 grid(T, few ? (heads + 3) / 4 : 1);
  return tl_launch(qk_norm_cache_write_kernel, grid, dim3(few ? 128 : 256), 0, stream, z, ldz, bias, qw, kw, eps,
                   (act_t*)q_out, (act_t*)k_pages, (act_t*)v_pages, token_pos, token_seq, seq_slot, page_table,
                   table_stride, nh, nkv, dim, vdim);
}

// The same with one norm over all query heads and one over all key heads (weights of the whole projection).
// Two kinds of block in one launch: the first T take a token each (its q and k, read once and kept in
// registers where the row fits), the others take 32 consecutive tokens of one value head, turned in shared
// memory, so that the transposed value pages are written in runs of positions.
#define WN_KEEP 8
template <int V>      // 4: q and k in 16-byte pieces; 1: any size
__global__ void __launch_bounds__(512)
qk_whole_norm_cache_write_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ bias,
                                 const float* __restrict__ qw, const float* __restrict__ kw, float eps,
                                 act_t* __restrict__ q_out, act_t* __restrict__ k_pages, act_t* __restrict__ v_pages,
                                 const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                                 const int* __restrict__ seq_slot, const int* __restrict__ page_table,
                                 int table_stride, int T, int nh, int nkv, int dim, int vdim, int vd_blocks) {
  __shared__ float scratch[33];
  __shared__ float vt[32][33];
  pdl_wait();
  pdl_launch_dependents();
  const int nq = nh * dim, nk = nkv * dim, v_off = nq + nk;
  if ((int)blockIdx.x >= T) {
    // 32 tokens x 32 entries of one value head
    int id = (int)blockIdx.x - T;
    const int d0 = (id % vd_blocks) * 32;
    id /= vd_blocks;
    const int g = id % nkv, tt0 = (id / nkv) * 32;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int r = warp; r < 32; r += nw) {
      const int t = tt0 + r, d = d0 + lane;
      float v = 0.0f;
      if (t < T && d < vdim) {
        const int c = v_off + g * vdim + d;
        v = z[(size_t)t * ldz + c] + (bias != nullptr ? bias[c] : 0.0f);
      }
      vt[r][lane] = v;
    }
    __syncthreads();
    const int t = tt0 + lane;
    if (t < T) {
      const int pos = token_pos[t];
      const int page = page_table[(size_t)seq_slot[token_seq[t]] * table_stride + pos / TL_PAGE];
      act_t* dst = v_pages + ((size_t)page * nkv + g) * vdim * TL_PAGE + pos % TL_PAGE;
      for (int r = warp; r < 32; r += nw)
        if (d0 + r < vdim) dst[(size_t)(d0 + r) * TL_PAGE] = from_f32<act_t>(vt[lane][r]);
    }
    return;
  }
  const int t = blockIdx.x;
  const float* row = z + (size_t)t * ldz;
  const int total = nq + nk;
  auto load = [&](int i, float (&v)[V]) {
    if (V == 4) {
      const float4 f = *reinterpret_cast<const float4*>(row + i);
      v[0] = f.x; v[V > 1 ? 1 : 0] = f.y; v[V > 2 ? 2 : 0] = f.z; v[V > 3 ? 3 : 0] = f.w;
    } else {
      v[0] = row[i];
    }
    if (bias != nullptr) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += bias[i + e];
    }
  };
  const bool fits = total <= (int)blockDim.x * V * WN_KEEP;
  float keep[WN_KEEP][V];
  float sq = 0.0f, sk = 0.0f;
  if (fits) {
#pragma unroll
    for (int j = 0; j < WN_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
#pragma unroll
      for (int e = 0; e < V; ++e) keep[j][e] = 0.0f;
      if (i < total) load(i, keep[j]);
      float s = 0.0f;
#pragma unroll
      for (int e = 0; e < V; ++e) s = fmaf(keep[j][e], keep[j][e], s);
      if (i < nq) sq += s; else sk += s;
    }
  } else {
    for (int i = V * threadIdx.x; i < total; i += V * blockDim.x) {
      float v[V], s = 0.0f;
      load(i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) s = fmaf(v[e], v[e], s);
      if (i < nq) sq += s; else sk += s;
    }
  }
  sq = block_sum(sq, scratch);
  sk = block_sum(sk, scratch);
  const float iq = 1.0f / sqrtf(sq / (float)nq + eps), ik = 1.0f / sqrtf(sk / (float)nk + eps);
  const int pos = token_pos[t];
  const int page = page_table[(size_t)seq_slot[token_seq[t]] * table_stride + pos / TL_PAGE];
  act_t* qd = q_out + (size_t)t * nq;
  act_t* kd = k_pages + (size_t)page * nkv * TL_PAGE * dim + (size_t)(pos % TL_PAGE) * dim;
  auto store = [&](int i, const float (&v)[V]) {
    if (i < nq) {
#pragma unroll
      for (int e = 0; e < V; ++e) qd[i + e] = from_f32<act_t>(v[e] * iq * qw[i + e]);
    } else {
      const int c = i - nq, g = c / dim, d = c - g * dim;
#pragma unroll
      for (int e = 0; e < V; ++e) kd[(size_t)g * TL_PAGE * dim + d + e] = from_f32<act_t>(v[e] * ik * kw[c + e]);
    }
  };
  if (fits) {
#pragma unroll
    for (int j = 0; j < WN_KEEP; ++j) {
      const int i = V * (threadIdx.x + j * blockDim.x);
      if (i < total) store(i, keep[j]);
    }
  } else {
    for (int i = V * threadIdx.x; i < total; i += V * blockDim.x) {
      float v[V];
      load(i, v);
      store(i, v);
    }
  }
}

extern "C" int TL_NAME(tl_qk_whole_norm_cache_write)(const float* z, int ldz, const float* bias, const float* qw,
                                                     const float* kw, float eps, void* q_out, void* k_pages,
                                                     void* v_pages, const int* token_pos, const int* token_seq,
                                                     const int* seq_slot, const int* page_table, int table_stride,
                                                     int T, int nh, int nkv, int dim, int vdim, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nh < 1 || nkv < 1 || dim < 1 || vdim < 1) return TL_ERR_BAD_ARG;
  const int vd_blocks = (vdim + 31) / 32;
  const long long blocks = T + (long long)((T + 31) / 32) * nkv * vd_blocks;
  if (blocks > 0x7fffffffLL) return TL_ERR_UNSUPPORTED;
  const bool vec = dim % 4 == 0 && ldz % 4 == 0 && ((uintptr_t)z & 15) == 0;
  const int total = (nh + nkv) * dim, per = vec ? 4 : 1;
  int threads = ((total + 2 * per - 1) / (2 * per) + 31) / 32 * 32;       // two pieces per thread
  threads = threads < 128 ? 128 : (threads > 512 ? 512 : threads);
  if (vec)
    return tl_launch(qk_whole_norm_cache_write_kernel<4>, dim3((unsigned)blocks), dim3(threads), 0, stream, z, ldz, bias,
                     qw, kw, eps, (act_t*)q_out, (act_t*)k_pages, (act_t*)v_pages, token_pos, token_seq, seq_slot,
                     page_table, table_stride, T, nh, nkv, dim, vdim, vd_blocks);
  return tl_launch(qk_whole_norm_cache_write_kernel<1>, dim3((unsigned)blocks), dim3(threads), 0, stream, z, ldz, bias, qw,
                   kw, eps, (act_t*)q_out, (act_t*)k_pages, (act_t*)v_pages, token_pos, token_seq, seq_slot, page_table,
                   table_stride, T, nh, nkv, dim, vdim, vd_blocks);
}

// One block per (token, query head).  The visible keys are walked as one run of n1 + n2 places:
// the n1 kept first keys that lie before the window, then the n2 keys of the window; 128 at a
// time with a running maximum and sum in 32-bit.  The sink opens the running maximum and the
// sum (as a key with score `sink` and no value), so it is counted once whatever the chunks.
__global__ void __launch_bounds__(SA_THREADS)
sink_attn_kernel(const act_t* __restrict__ q, const act_t* __restrict__ k_pages, const act_t* __restrict__ v_pages,
                 const float* __restrict__ gate, int ldg, const float* __restrict__ sink,
                 act_t* __restrict__ out, const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                 const int* __restrict__ seq_slot, const int* __restrict__ page_table, int table_stride, int nh,
                 int nkv, int dim, int vdim, int window, int keep_first, float scale, float cap) {
  __shared__ float qs[SA_MAX_DIM];
  __shared__ float ps[SA_THREADS];
  __shared__ int pg[SA_THREADS];   // page of each key of the chunk
  __shared__ int ky[SA_THREADS];   // its place in the page
  __shared__ float scratch[33];
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int kvh = h / (nh / nkv);
  const int pos = token_pos[t];
  const int slot = seq_slot[token_seq[t]];
  const int* table = page_table + (size_t)slot * table_stride;
  const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
  const int n1 = keep_first < lo ? keep_first : lo;
  const int total = n1 + (pos - lo + 1);
  const size_t kpage = (size_t)nkv * TL_PAGE * dim, vpage = (size_t)nkv * TL_PAGE * vdim;
  const size_t khead = (size_t)kvh * TL_PAGE * dim, vhead = (size_t)kvh * TL_PAGE * vdim;
  const float inv_cap = cap > 0.0f ? 1.0f / cap : 0.0f;

  for (int d = tid; d < dim; d += SA_THREADS) qs[d] = to_f32(q[(size_t)t * nh * dim + (size_t)h * dim + d]);
  __syncthreads();

  float m_run = sink != nullptr ? sink[h] : -INFINITY;
  float l_run = sink != nullptr ? 1.0f : 0.0f;
  float acc[SA_MAX_V] = {};         // value entries tid, tid + 128, ...
  for (int base = 0; base < total; base += SA_THREADS) {
    const int place = base + tid;
    const bool valid = place < total;
    float s = -INFINITY;
    int page = -1, in_page = 0;
    if (valid) {
      const int key = place < n1 ? place : lo + (place - n1);
      page = table[key / TL_PAGE];
      in_page = key % TL_PAGE;
      const act_t* krow = k_pages + (size_t)page * kpage + khead + (size_t)in_page * dim;
      float dot = 0.0f;
      for (int d = 0; d < dim; ++d) dot = fmaf(qs[d], to_f32(krow[d]), dot);
      s = dot * scale;
      if (cap > 0.0f) s = cap * tanhf(s * inv_cap);
    }
    const float cmax = block_max(s, scratch);
    const float m_new = fmaxf(m_run, cmax);
    const float p = valid ? expf(s - m_new) : 0.0f;
    ps[tid] = p;
    pg[tid] = page;
    ky[tid] = in_page;
    const float csum = block_sum(p, scratch);  // has the barriers that publish ps, pg and ky
    const float alpha = expf(m_run - m_new);   // 0 at the first chunk if there is no sink
    l_run = l_run * alpha + csum;
    m_run = m_new;
    const int cnt = total - base < SA_THREADS ? total - base : SA_THREADS;
    if (tid < vdim) {
#pragma unroll
      for (int i = 0; i < SA_MAX_V; ++i) acc[i] *= alpha;
      for (int j = 0; j < cnt; ++j) {
        const act_t* vcol = v_pages + (size_t)pg[j] * vpage + vhead + ky[j];
        const float pj = ps[j];
#pragma unroll
        for (int i = 0; i < SA_MAX_V; ++i)
          if (tid + i * SA_THREADS < vdim) acc[i] = fmaf(pj, to_f32(vcol[(size_t)(tid + i * SA_THREADS) * TL_PAGE]), acc[i]);
      }
    }
    __syncthreads();  // ps, pg and ky are rewritten by the next chunk
  }
  pdl_launch_dependents();   // only now: a grid let go earlier would sit on the SMs and take issue slots
  float gv = 1.0f;
  if (gate != nullptr) gv = 1.0f / (1.0f + expf(-gate[(size_t)t * ldg + h]));
  const float f = gv / l_run;
  act_t* o = out + (size_t)t * nh * vdim + (size_t)h * vdim;
#pragma unroll
  for (int i = 0; i < SA_MAX_V; ++i)
    if (tid + i * SA_THREADS < vdim) o[tid + i * SA_THREADS] = from_f32<act_t>(acc[i] * f);
}

extern "C" int TL_NAME(tl_sink_attn)(const void* q, const void* k_pages, const void* v_pages, const float* gate,
                                     int ldg, const float* sink, void* out, const int* token_pos,
                                     const int* token_seq, const int* seq_slot, const int* page_table,
                                     int table_stride, int T, int nh, int nkv, int dim, int vdim, int window,
                                     int keep_first, float scale, float cap, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dim < 1 || dim > SA_MAX_DIM || vdim < 1 || vdim > SA_MAX_V * SA_THREADS || nkv <= 0 || nh % nkv != 0 ||
      nh > 65535 || window < 0 || keep_first < 0)
    return TL_ERR_UNSUPPORTED;
  dim3 grid(T, nh);
  return tl_launch(sink_attn_kernel, grid, dim3(SA_THREADS), 0, stream, (const act_t*)q, (const act_t*)k_pages,
                   (const act_t*)v_pages, gate, ldg, sink, (act_t*)out, token_pos, token_seq, seq_slot,
                   page_table, table_stride, nh, nkv, dim, vdim, window, keep_first, scale, cap);
}
