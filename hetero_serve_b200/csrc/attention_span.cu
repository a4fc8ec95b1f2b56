// Grouped softmax attention over the paged cache with a linear bias of the distance, a sliding
// window that keeps the first tokens, capped scores and a sink, on the CUDA cores.
//
// The cache keeps one row [key (D) | value (V)] per token and key/value head (pool
// [pages][kv_heads][page_size][D + V]).
//
//   span_prepare    from the float32 projection: q (and k) divided by their root mean square per
//                   head when asked (no weight), or both over their whole projections (with
//                   weights), then turned by the token's position on each head's first rot_dims
//                   numbers (number i pairs with i + rot_dims/2); q to a float32 buffer, the row [k | v] straight
//                   into the token's page; the values are columns of their own or the keys as
//                   projected.  A layer that only reads another's rows writes nothing and has
//                   no key or value columns.
//   span_attention  a block per (token, query head).  Query i sees j <= i with i - j < window
//                   (window 0: all) or j < keep_first; score = q . k * scale - slope_h * (i - j),
//                   then softcap * tanh(score / softcap) when there is a cap; a sink (one logit a
//                   head, as it stands) enters the denominator alone;
//                   its eight warps take rounds of 32 keys in turn (a key per lane for the
//                   scores, a column per lane for the values, four value rows in flight), each
//                   with a running softmax of its own, joined under one maximum at the end; the
//                   output may be multiplied element by element by the sigmoid of gate columns
//                   and by a scale before it is rounded.  With a list of tokens (the
//                   single-query section of a step's work lists) only those are served.
//
// Scores, softmax state and accumulators are float32.  A row's result depends on its own
// request only: the keys are dealt to the warps in an order fixed by the position.
#include "common.cuh"
#include "rotary.cuh"

namespace hs {

constexpr int SA_WARPS = 8;

template <typename TC>
__global__ void __launch_bounds__(SA_WARPS * 32)
span_prepare_kernel(float* __restrict__ q_out, TC* __restrict__ pool,
                    const float* __restrict__ proj, int proj_stride, int q_off, int k_off,
                    int v_off, const int* __restrict__ table, int max_pages, int num_pages,
                    const int* __restrict__ tok_pos, const int* __restrict__ tok_req, int H, int G,
                    int D, int V, int qk_norm, float eps, int page_size, int writes,
                    const float* __restrict__ wq, const float* __restrict__ wk,
                    const float* __restrict__ freq, int rot_dims, int* __restrict__ status) {
  extern __shared__ float2 s_turn[];               // cosine and sine per turned pair
  __shared__ float s_sq[2][SA_WARPS];
  pdl_trigger();
  const int t = blockIdx.x;
  const int r = tok_req[t];
  if (r < 0) return;
  const int pos = tok_pos[t];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = rot_dims >> 1;
  for (int i = threadIdx.x; i < half; i += SA_WARPS * 32)
    pair_angle(pos, freq[i], &s_turn[i].x, &s_turn[i].y);
  pdl_wait();
  TC* row = nullptr;
  if (writes) {
    const int pi = pos / page_size;
    const int page = (pos >= 0 && pi < max_pages) ? table[(size_t)r * max_pages + pi] : -1;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, HS_STATUS_BAD_PAGE);
    } else {
      row = pool + ((size_t)page * G * page_size + (pos % page_size)) * (size_t)(D + V);
    }
  }
  const float* pr = proj + (size_t)t * proj_stride;
  float rq = 1.0f, rk = 1.0f;                      // of the whole projections
  if (wq) {
    float sq = 0.f, sk = 0.f;
    for (int e = threadIdx.x; e < H * D; e += SA_WARPS * 32) sq = fmaf(pr[q_off + e], pr[q_off + e], sq);
    if (row)
      for (int e = threadIdx.x; e < G * D; e += SA_WARPS * 32)
        sk = fmaf(pr[k_off + e], pr[k_off + e], sk);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      s_sq[0][warp] = sq;
      s_sq[1][warp] = sk;
    }
  }
  __syncthreads();                                 // the sums, and the pairs' angles
  if (wq) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int w = 0; w < SA_WARPS; ++w) {
      sq += s_sq[0][w];
      sk += s_sq[1][w];
    }
    rq = 1.0f / sqrtf(sq / (float)(H * D) + eps);
    rk = 1.0f / sqrtf(sk / (float)(G * D) + eps);
  }
  const int jobs = row ? H + 2 * G : H;            // query heads, key heads, value heads
  for (int job = warp; job < jobs; job += SA_WARPS) {
    const bool is_q = job < H, is_k = !is_q && job < H + G;
    const int g = is_q ? 0 : (is_k ? job - H : job - H - G);
    const int n = (is_q || is_k) ? D : V;
    // the values: columns of their own, or the keys as projected (before any norm)
    const float* src = is_q ? pr + q_off + (size_t)job * D
                     : (is_k || v_off < 0) ? pr + k_off + (size_t)g * D
                                           : pr + v_off + (size_t)g * V;
    float rn = 1.0f;
    if (qk_norm && (is_q || is_k)) {
      float ss = 0.f;
      for (int e = lane; e < n; e += 32) ss = fmaf(src[e], src[e], ss);
      ss = warp_sum(ss);
      rn = 1.0f / sqrtf(ss / (float)n + eps);
    }
    const float* wt = nullptr;
    if (wq && (is_q || is_k)) {
      rn = is_q ? rq : rk;
      wt = is_q ? wq + (size_t)job * D : wk + (size_t)g * D;
    }
    const int turned = (is_q || is_k) ? rot_dims : 0;
    float* qdst = is_q ? q_out + (size_t)t * H * D + (size_t)job * D : nullptr;
    TC* cdst = is_q ? nullptr : row + (size_t)g * page_size * (D + V) + (is_k ? 0 : D);
    for (int e = lane; e < n; e += 32) {
      float val = src[e] * rn;
      if (wt) val *= wt[e];
      if (e < turned) {
        const bool low = e < half;
        const int pe = low ? e + half : e - half;
        float other = src[pe] * rn;
        if (wt) other *= wt[pe];
        const float2 cs = s_turn[low ? e : pe];
        val = low ? val * cs.x - other * cs.y : val * cs.x + other * cs.y;
      }
      if (qdst) qdst[e] = val;
      else cdst[e] = from_f<TC>(val);
    }
  }
}

// The same for norms over the whole projections (or none), four numbers a thread: sizes, offsets and
// half the turned extent in whole 16-byte pieces.
template <typename TC>
__global__ void __launch_bounds__(SA_WARPS * 32)
span_prepare_wide_kernel(float* __restrict__ q_out, TC* __restrict__ pool,
                         const float* __restrict__ proj, int proj_stride, int q_off, int k_off,
                         int v_off, const int* __restrict__ table, int max_pages, int num_pages,
                         const int* __restrict__ tok_pos, const int* __restrict__ tok_req, int H,
                         int G, int D, int V, float eps, int page_size, int writes,
                         const float* __restrict__ wq, const float* __restrict__ wk,
                         const float* __restrict__ freq, int rot_dims, int* __restrict__ status) {
  extern __shared__ __align__(16) float s_wide[];  // q [H*D] | k [G*D] | cosines, sines [rot_dims]
  __shared__ float s_sq[2][SA_WARPS];
  pdl_trigger();
  const int t = blockIdx.x;
  const int r = tok_req[t];
  if (r < 0) return;
  const int pos = tok_pos[t], half = rot_dims >> 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nq = H * D, nk = writes ? G * D : 0;
  float* s_cos = s_wide + nq + nk;
  float* s_sin = s_cos + half;
  for (int i = threadIdx.x; i < half; i += SA_WARPS * 32) pair_angle(pos, freq[i], &s_cos[i], &s_sin[i]);
  TC* row = nullptr;
  if (writes) {
    const int pi = pos / page_size;
    const int page = (pos >= 0 && pi < max_pages) ? table[(size_t)r * max_pages + pi] : -1;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, HS_STATUS_BAD_PAGE);
    } else {
      row = pool + ((size_t)page * G * page_size + (pos % page_size)) * (size_t)(D + V);
    }
  }
  pdl_wait();
  const float* pr = proj + (size_t)t * proj_stride;
  auto put = [&](TC* dst, float4 v) {
    if constexpr (sizeof(TC) == 4) {
      *(float4*)dst = v;
    } else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
      *(uint2*)dst = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
    }
  };
  float sq = 0.f, sk = 0.f;
  for (int e = 4 * threadIdx.x; e < nq + nk; e += 4 * SA_WARPS * 32) {
    const float4 v = *(const float4*)(pr + (e < nq ? q_off + e : k_off + e - nq));
    *(float4*)(s_wide + e) = v;
    const float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
    if (e < nq) sq += ss;
    else sk += ss;
  }
  if (row) {                                       // values go as they are
    const float* src = pr + (v_off < 0 ? k_off : v_off);
    for (int e = 4 * threadIdx.x; e < G * V; e += 4 * SA_WARPS * 32) {
      const int g = e / V, c = e - g * V;
      put(row + (size_t)g * page_size * (D + V) + D + c, *(const float4*)(src + e));
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    s_sq[0][warp] = sq;
    s_sq[1][warp] = sk;
  }
  __syncthreads();
  float rq = 1.0f, rk = 1.0f;
  if (wq) {
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < SA_WARPS; ++w) {
      sq += s_sq[0][w];
      sk += s_sq[1][w];
    }
    rq = 1.0f / sqrtf(sq / (float)(H * D) + eps);
    rk = 1.0f / sqrtf(sk / (float)(G * D) + eps);
  }
  for (int e = 4 * threadIdx.x; e < nq + nk; e += 4 * SA_WARPS * 32) {
    const bool is_q = e < nq;
    const int at = is_q ? e : e - nq, g = at / D, c = at - g * D;
    if (!is_q && !row) break;
    const float rn = is_q ? rq : rk;
    const float* wt = is_q ? wq : wk;
    auto normed = [&](int i) {                     // the piece at i numbers from this one
      float4 v = *(const float4*)(s_wide + e + i);
      v = make_float4(v.x * rn, v.y * rn, v.z * rn, v.w * rn);
      if (wt) {
        const float4 w = *(const float4*)(wt + at + i);
        v = make_float4(v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w);
      }
      return v;
    };
    float4 v = normed(0);
    if (c < rot_dims) {
      const bool low = c < half;
      const float4 o = normed(low ? half : -half);
      const float4 cs = *(const float4*)(s_cos + (low ? c : c - half));
      float4 sn = *(const float4*)(s_sin + (low ? c : c - half));
      if (low) sn = make_float4(-sn.x, -sn.y, -sn.z, -sn.w);
      v = make_float4(v.x * cs.x + o.x * sn.x, v.y * cs.y + o.y * sn.y, v.z * cs.z + o.z * sn.z,
                      v.w * cs.w + o.w * sn.w);
    }
    if (is_q) *(float4*)(q_out + (size_t)t * nq + e) = v;
    else put(row + (size_t)g * page_size * (D + V) + c, v);
  }
}

__device__ __forceinline__ float sa_dot(const float* __restrict__ k, const float* q, int D,
                                        bool vec) {
  float s = 0.f;
  if (vec) {
    const float4* k4 = reinterpret_cast<const float4*>(k);
    for (int i = 0; i < D / 4; ++i) {
      const float4 a = k4[i];
      s = fmaf(a.x, q[4 * i], s); s = fmaf(a.y, q[4 * i + 1], s);
      s = fmaf(a.z, q[4 * i + 2], s); s = fmaf(a.w, q[4 * i + 3], s);
    }
  } else {
    for (int i = 0; i < D; ++i) s = fmaf(k[i], q[i], s);
  }
  return s;
}
__device__ __forceinline__ float sa_dot(const __nv_bfloat16* __restrict__ k, const float* q,
                                        int D, bool vec) {
  float s = 0.f;
  if (vec) {
    const uint4* k8 = reinterpret_cast<const uint4*>(k);
    for (int i = 0; i < D / 8; ++i) {
      const uint4 a = k8[i];
      const unsigned w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        // a bfloat16 is the upper half of a float
        s = fmaf(__uint_as_float(w[j] << 16), q[8 * i + 2 * j], s);
        s = fmaf(__uint_as_float(w[j] & 0xffff0000u), q[8 * i + 2 * j + 1], s);
      }
    }
  } else {
    for (int i = 0; i < D; ++i) s = fmaf(__bfloat162float(k[i]), q[i], s);
  }
  return s;
}

// SA_MAXC: value columns a lane owns (V <= 32 * SA_MAXC); the launcher picks 2, 8 or 32.
template <typename TC, typename TO, int SA_MAXC>
__global__ void __launch_bounds__(SA_WARPS * 32)
span_attention_kernel(TO* __restrict__ out, const float* __restrict__ q,
                      const TC* __restrict__ pool, const int* __restrict__ table, int max_pages,
                      int num_pages, const int* __restrict__ tok_pos,
                      const int* __restrict__ tok_req, const float* __restrict__ slopes,
                      const float* __restrict__ gate, int gate_stride, int gate_offset,
                      float out_scale, int n_tokens, int H, int G, int D, int V, int window,
                      int keep_first, float scale, int page_size, int vec,
                      const int* __restrict__ listed, const int* __restrict__ plan_head,
                      float softcap, const float* __restrict__ sinks, int* __restrict__ status) {
  extern __shared__ float s_sa[];                  // q [D] | acc [SA_WARPS][V] | m, l [2 SA_WARPS]
  float* sq = s_sa;
  float* s_acc = s_sa + D;
  float* s_ml = s_acc + (size_t)SA_WARPS * V;
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = blockIdx.x;
  // with a list only the listed tokens are served, as many as the list's head says
  const int n_here = listed ? min(n_tokens, plan_head[0]) : n_tokens;
  if (item >= (long long)n_here * H) return;
  // consecutive tokens of one head are neighbours in the grid: their keys overlap in the L2
  const int h = (int)(item / n_here), entry = (int)(item - (long long)h * n_here);
  const int t = listed ? listed[3 * entry] : entry;
  const int r = tok_req[t];
  if (r < 0) return;
  const int pos = tok_pos[t];
  const int g = h / (H / G);
  const float* qr = q + (size_t)t * H * D + (size_t)h * D;
  for (int e = threadIdx.x; e < D; e += SA_WARPS * 32) sq[e] = qr[e] * scale;
  __syncthreads();
  const int row_len = D + V;
  const int first = window > 0 ? max(0, pos - window + 1) : 0;
  const int kept = min(keep_first, first);          // first tokens that lie behind the window
  const int n_keys = kept + (pos - first + 1);
  const float slope = slopes ? slopes[h] : 0.f;
  const int* tab = table + (size_t)r * max_pages;
  float m = -INFINITY, l = 0.f;
  float acc[SA_MAXC];
#pragma unroll
  for (int c = 0; c < SA_MAXC; ++c) acc[c] = 0.f;
  bool bad = false;
  for (int base = warp * 32; base < n_keys; base += SA_WARPS * 32) {
    const int kk = base + lane;
    const TC* krow = nullptr;
    int j = 0;
    if (kk < n_keys) {
      j = kk < kept ? kk : first + (kk - kept);
      const int pi = j / page_size;
      const int page = pi < max_pages ? tab[pi] : -1;
      if (page < 0 || page >= num_pages) bad = true;
      else krow = pool + (((size_t)page * G + g) * page_size + (j % page_size)) * (size_t)row_len;
    }
    // the bias of the distance is taken off the scaled score
    float s = krow ? sa_dot(krow, sq, D, vec != 0) - slope * (float)(pos - j) : -INFINITY;
    if (softcap > 0.f && krow) s = softcap * tanhf(s / softcap);
    const float m_new = fmaxf(m, warp_max(s));
    if (m_new == -INFINITY) continue;               // no valid key in this round
    const float corr = expf(m - m_new);             // m = -inf: 0
    const float p = krow ? expf(s - m_new) : 0.f;
    l = fmaf(l, corr, warp_sum(p));
    m = m_new;
#pragma unroll
    for (int c = 0; c < SA_MAXC; ++c) acc[c] *= corr;
    const int n_round = min(32, n_keys - base);
    // four value rows in flight: their loads are issued before the first is used
    for (int jj = 0; jj < n_round; jj += 4) {
      float pj[4];
      const TC* vr[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int src = (jj + u) & 31;
        pj[u] = __shfl_sync(0xffffffffu, p, src);
        const unsigned long long ptr =
            __shfl_sync(0xffffffffu, (unsigned long long)(uintptr_t)krow, src);
        vr[u] = jj + u < n_round && ptr != 0ull ? reinterpret_cast<const TC*>((uintptr_t)ptr) + D
                                                : nullptr;
      }
#pragma unroll
      for (int c = 0; c < SA_MAXC; ++c) {
        const int e = c * 32 + lane;
        if (e < V) {
          float v[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) v[u] = vr[u] ? to_f(vr[u][e]) : 0.f;
#pragma unroll
          for (int u = 0; u < 4; ++u)
            if (vr[u]) acc[c] = fmaf(pj[u], v[u], acc[c]);
        }
      }
    }
  }
  if (__any_sync(0xffffffffu, bad) && lane == 0) atomicOr(status, HS_STATUS_BAD_PAGE);
  // the warps' shares joined under one maximum, in the order of the warps
  if (lane == 0) {
    s_ml[warp] = m;
    s_ml[SA_WARPS + warp] = l;
  }
#pragma unroll
  for (int c = 0; c < SA_MAXC; ++c) {
    const int e = c * 32 + lane;
    if (e < V) s_acc[(size_t)warp * V + e] = acc[c];
  }
  __syncthreads();
  float top = -INFINITY;
#pragma unroll
  for (int w = 0; w < SA_WARPS; ++w) top = fmaxf(top, s_ml[w]);
  if (sinks) top = fmaxf(top, sinks[h]);
  float total = sinks ? expf(sinks[h] - top) : 0.f, share[SA_WARPS];
#pragma unroll
  for (int w = 0; w < SA_WARPS; ++w) {
    share[w] = s_ml[w] == -INFINITY ? 0.f : expf(s_ml[w] - top);
    total = fmaf(s_ml[SA_WARPS + w], share[w], total);
  }
  const float inv = total > 0.f ? 1.0f / total : 0.f;
  TO* orow = out + (size_t)t * H * V + (size_t)h * V;
  const float* grow = gate ? gate + (size_t)t * gate_stride + gate_offset + (size_t)h * V : nullptr;
  for (int e = threadIdx.x; e < V; e += SA_WARPS * 32) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < SA_WARPS; ++w) o = fmaf(s_acc[(size_t)w * V + e], share[w], o);
    o *= inv;
    if (grow) o *= 1.0f / (1.0f + expf(-grow[e]));
    orow[e] = from_f<TO>(o * out_scale);
  }
}

}  // namespace hs

// proj: float32 rows of `proj_stride` columns with q (H*D) at q_off, k (G*D) at k_off and v (G*V)
// at v_off (v_off < 0: the values are the keys as projected; V must equal D); without `writes`
// only the q columns are read.
HS_EXPORT int hs_span_prepare(float* q_out, void* pool, const float* proj, int proj_stride,
                              int q_off, int k_off, int v_off, const int* table, int max_pages,
                              int num_pages, const int* tok_pos, const int* tok_req,
                              int n_tokens, int H, int G, int D, int V, int qk_norm, float eps,
                              int page_size, int writes, const float* wq, const float* wk,
                              const float* freq, int rot_dims, int cache_dtype, int* status,
                              void* stream) {
  if (!q_out || !pool || !proj || !table || !tok_pos || !tok_req || !status)
    return HS_ERR_ARGUMENT;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || page_size <= 0 || q_off < 0 ||
      q_off + H * D > proj_stride)
    return HS_ERR_UNSUPPORTED;
  if (writes && (k_off < 0 || k_off + G * D > proj_stride || (v_off < 0 && V != D) ||
                 (v_off >= 0 && v_off + G * V > proj_stride)))
    return HS_ERR_UNSUPPORTED;
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > D || (rot_dims && !freq) || (wq && qk_norm) ||
      (wq && writes && !wk))
    return HS_ERR_ARGUMENT;
  if (n_tokens <= 0) return HS_OK;
  const size_t smem = (size_t)(rot_dims / 2) * sizeof(float2);
  if (smem > 40 * 1024) return HS_ERR_UNSUPPORTED;
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e;
  const size_t wide = ((size_t)(H + (writes ? G : 0)) * D + rot_dims) * sizeof(float);
  if (!qk_norm && D % 4 == 0 && V % 4 == 0 && rot_dims % 8 == 0 && q_off % 4 == 0 &&
      (!writes || (k_off % 4 == 0 && (v_off < 0 || v_off % 4 == 0))) && proj_stride % 4 == 0 &&
      wide <= 47 * 1024 &&
      !(((uintptr_t)q_out | (uintptr_t)pool | (uintptr_t)proj | (uintptr_t)wq | (uintptr_t)wk) & 15)) {
#define HS_SPW(TC)                                                                                 \
  e = hs_launch(hs::span_prepare_wide_kernel<TC>, dim3(n_tokens), dim3(hs::SA_WARPS * 32), wide, st, \
                hs_pdl_enabled(), q_out, (TC*)pool, proj, proj_stride, q_off, k_off, v_off, table, \
                max_pages, num_pages, tok_pos, tok_req, H, G, D, V, eps, page_size, writes, wq, wk, \
                freq, rot_dims, status)
    if (cache_dtype == HS_DT_BF16) HS_SPW(__nv_bfloat16);
    else if (cache_dtype == HS_DT_F32) HS_SPW(float);
    else return HS_ERR_UNSUPPORTED;
#undef HS_SPW
    return e == cudaSuccess ? HS_OK : (int)e;
  }
  if (cache_dtype == HS_DT_BF16)
    e = hs_launch(hs::span_prepare_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(hs::SA_WARPS * 32),
                  smem, st, hs_pdl_enabled(), q_out, (__nv_bfloat16*)pool, proj, proj_stride, q_off,
                  k_off, v_off, table, max_pages, num_pages, tok_pos, tok_req, H, G, D, V, qk_norm,
                  eps, page_size, writes, wq, wk, freq, rot_dims, status);
  else if (cache_dtype == HS_DT_F32)
    e = hs_launch(hs::span_prepare_kernel<float>, dim3(n_tokens), dim3(hs::SA_WARPS * 32), smem, st,
                  hs_pdl_enabled(), q_out, (float*)pool, proj, proj_stride, q_off, k_off, v_off,
                  table, max_pages, num_pages, tok_pos, tok_req, H, G, D, V, qk_norm, eps,
                  page_size, writes, wq, wk, freq, rot_dims, status);
  else
    return HS_ERR_UNSUPPORTED;
  return e == cudaSuccess ? HS_OK : (int)e;
}

HS_EXPORT int hs_span_attention(void* out, const float* q, const void* pool, const int* table,
                                int max_pages, int num_pages, const int* tok_pos,
                                const int* tok_req, const float* slopes, const float* gate,
                                int gate_stride, int gate_offset, float out_scale, int n_tokens,
                                int H, int G, int D, int V, int window, int keep_first,
                                float scale, int page_size, int cache_dtype, int out_dtype,
                                const int* listed, const int* plan_head, float softcap,
                                const float* sinks, int* status, void* stream) {
  if (!out || !q || !pool || !table || !tok_pos || !tok_req || !status || (listed && !plan_head))
    return HS_ERR_ARGUMENT;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || V > 1024 || window < 0 ||
      keep_first < 0 || page_size <= 0 ||
      (gate && (gate_offset < 0 || gate_offset + H * V > gate_stride)))
    return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  const size_t smem = ((size_t)D + (size_t)hs::SA_WARPS * (V + 2)) * sizeof(float);
  if (smem > 48 * 1024) return HS_ERR_UNSUPPORTED;
  const long long items = (long long)n_tokens * H;
  if (items > 0x7fffffffLL) return HS_ERR_TOO_LARGE;
  const dim3 grid((unsigned)items), blk(hs::SA_WARPS * 32);
  cudaStream_t st = (cudaStream_t)stream;
  const bool pdl = hs_pdl_enabled();
  // 16-byte reads of a key row need rows that start and end on 16 bytes
  const int per16 = cache_dtype == HS_DT_BF16 ? 8 : 4;
  const int vec = (D % per16 == 0 && V % per16 == 0) ? 1 : 0;
  cudaError_t e;
#define HS_SA_LAUNCH_C(TC, TO, C)                                                                \
  e = hs_launch(hs::span_attention_kernel<TC, TO, C>, grid, blk, smem, st, pdl, (TO*)out, q,     \
                (const TC*)pool, table, max_pages, num_pages, tok_pos, tok_req, slopes, gate,    \
                gate_stride, gate_offset, out_scale, n_tokens, H, G, D, V, window, keep_first,   \
                scale, page_size, vec, listed, plan_head, softcap, sinks, status)
#define HS_SA_LAUNCH(TC, TO)                                                                     \
  do {                                                                                           \
    if (V <= 64) HS_SA_LAUNCH_C(TC, TO, 2);                                                      \
    else if (V <= 256) HS_SA_LAUNCH_C(TC, TO, 8);                                                \
    else HS_SA_LAUNCH_C(TC, TO, 32);                                                             \
  } while (0)
  if (cache_dtype == HS_DT_BF16 && out_dtype == HS_DT_BF16) HS_SA_LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (cache_dtype == HS_DT_F32 && out_dtype == HS_DT_F32) HS_SA_LAUNCH(float, float);
  else return HS_ERR_UNSUPPORTED;
#undef HS_SA_LAUNCH
#undef HS_SA_LAUNCH_C
  return e == cudaSuccess ? HS_OK : (int)e;
}
