// The state-space recurrence of ssm.cu over prompt portions on the tensor cores (mma.sync m16n8k16,
// bfloat16 operands, float32 accumulators), for activated rows kept in bfloat16.
//
// A portion is cut into chunks of 128 tokens.  With cs_t = la_1 + .. + la_t inside a chunk (la: the
// decay's logarithm), S the state in front of it and S' the state behind it,
//
//     y_t = D x_t + sum_{j <= t} exp(cs_t - cs_j) dt_j (C_t . B_j) x_j + exp(cs_t) S^T C_t
//     S'  = exp(cs_n) S + sum_j B_j (exp(cs_n - cs_j) dt_j x_j)^T
//
// so that everything but the chain of states is parallel over chunks, requests and heads:
//
//   chunk_state   the chunk's own contribution to S' and its whole decay
//   chunk_chain   S from chunk to chunk, element by element, in place of the contributions; the
//                 request's slot receives the last state, and its newest inputs
//   chunk_out     y
//
// B, C and x are bfloat16 numbers; what multiplies them and is not (weighted rows, weights, states)
// enters a product as the sum of three bfloat16 terms, a float32's whole mantissa, so the products
// keep what float32 products keep.  Decays, their sums and exponentials and the chain of states are
// float32.  A row's arithmetic depends on its own request and the place in its portion alone.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace hs {

constexpr int CK_LEN = 128;          // tokens of a chunk
constexpr int CK_TERMS = 3;
constexpr int CK_THREADS = 256;
constexpr int CK_PAD = 8;            // bfloat16 numbers behind a row in shared memory

struct ChunkShape {
  int H, G, N, V, taps;
  int channels;                      // floats in an activated row: x [H*V] | B [G*N] | C [G*N]
  int stride, x_off, state_stride;   // of the projection and the slots (for the kept inputs)
  int n_requests;
};

__device__ __forceinline__ void ck_ldsm_t(uint32_t* r, const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ck_copy16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(
                   (uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
// the next bfloat16 term of a pair; what it leaves stays in v (exact)
__device__ __forceinline__ uint32_t ck_term(float2& v) {
  const __nv_bfloat162 b = __floats2bfloat162_rn(v.x, v.y);
  v.x -= __bfloat162float(b.x);
  v.y -= __bfloat162float(b.y);
  return *(const uint32_t*)&b;
}

// chunk number `slot` of the step: which request's, and which of its chunks
__device__ __forceinline__ bool ck_find(const int* __restrict__ req_len, int n_requests, int slot,
                                        int& r, int& c) {
  for (r = 0; r < n_requests; ++r) {
    const int k = (req_len[r] + CK_LEN - 1) / CK_LEN;
    if (slot < k) {
      c = slot;
      return true;
    }
    slot -= k;
  }
  return false;
}

// s_cs[t] = sum of the chunk's first t + 1 logarithms, s_dt[t] = dt; tokens from n on add nothing
__device__ __forceinline__ void ck_sums(float* s_cs, float* s_dt, const float* __restrict__ step,
                                        int t0, int n, int H, int h) {
  if (threadIdx.x < 32) {
    float v[CK_LEN / 32], sum = 0.f;
#pragma unroll
    for (int i = 0; i < CK_LEN / 32; ++i) {
      const int t = threadIdx.x * (CK_LEN / 32) + i;
      float la = 0.f, dt = 0.f;
      if (t < n) {
        dt = step[(size_t)(t0 + t) * 2 * H + h];
        la = step[(size_t)(t0 + t) * 2 * H + H + h];
      }
      s_dt[t] = dt;
      sum += la;
      v[i] = sum;
    }
    float before = sum;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float w = __shfl_up_sync(0xffffffffu, before, o);
      if ((int)threadIdx.x >= o) before += w;
    }
    before -= sum;
#pragma unroll
    for (int i = 0; i < CK_LEN / 32; ++i) s_cs[threadIdx.x * (CK_LEN / 32) + i] = before + v[i];
  }
}

// ---- the chunks' contributions ------------------------------------------------------------------
__global__ void __launch_bounds__(CK_THREADS)
ssm_chunk_state_kernel(float* __restrict__ dS, float* __restrict__ whole,
                       const __nv_bfloat16* __restrict__ rows, const float* __restrict__ step,
                       const int* __restrict__ req_start, const int* __restrict__ req_len,
                       ChunkShape s) {
  extern __shared__ __align__(16) uint8_t ck_smem[];
  __shared__ float s_cs[CK_LEN], s_dt[CK_LEN];
  pdl_trigger();
  pdl_wait();
  const int slot = blockIdx.x, h = blockIdx.y, g = h / (s.H / s.G);
  int r, c;
  if (!ck_find(req_len, s.n_requests, slot, r, c)) return;
  const int N = s.N, V = s.V, NS = N + CK_PAD, VS = V + CK_PAD;
  const int n = min(CK_LEN, req_len[r] - c * CK_LEN), t0 = req_start[r] + c * CK_LEN;
  __nv_bfloat16* sB = (__nv_bfloat16*)ck_smem;            // [CK_LEN][NS]
  __nv_bfloat16* sX = sB + CK_LEN * NS;                   // [terms][CK_LEN][VS]
  const __nv_bfloat16* base = rows + (size_t)t0 * s.channels;
  const int b_off = s.H * V + g * N, nq = N / 8;
  for (int i = threadIdx.x; i < CK_LEN * nq; i += CK_THREADS) {
    const int t = i / nq, q = (i - t * nq) * 8;
    ck_copy16(sB + t * NS + q, base + (size_t)(t < n ? t : 0) * s.channels + b_off + q, t < n);
  }
  asm volatile("cp.async.commit_group;");
  // the x rows, eight numbers a piece, on their way while the decays are summed up
  constexpr int XP = 128 / 8 * CK_LEN / CK_THREADS;       // pieces of a thread at most (V <= 128)
  const int vq = V / 8;
  uint4 xr[XP];
#pragma unroll
  for (int k = 0; k < XP; ++k) {
    const int i = threadIdx.x + k * CK_THREADS;
    const int t = i / vq, q = (i - t * vq) * 8;
    if (t < n) xr[k] = *(const uint4*)(base + (size_t)t * s.channels + h * V + q);
  }
  ck_sums(s_cs, s_dt, step, t0, n, s.H, h);
  __syncthreads();
  const float end = s_cs[CK_LEN - 1];                     // tokens from n on added nothing
#pragma unroll
  for (int k = 0; k < XP; ++k) {
    const int i = threadIdx.x + k * CK_THREADS;
    const int t = i / vq, q = (i - t * vq) * 8;
    if (t >= CK_LEN) continue;
    const float w = t < n ? expf(end - s_cs[t]) * s_dt[t] : 0.f;
    const uint32_t u[4] = {xr[k].x, xr[k].y, xr[k].z, xr[k].w};
    uint32_t o[CK_TERMS][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {                         // a bfloat16 is the upper half of a float
      float2 x = make_float2(0.f, 0.f);
      if (t < n) x = make_float2(__uint_as_float(u[j] << 16) * w, __uint_as_float(u[j] & 0xffff0000u) * w);
#pragma unroll
      for (int m = 0; m < CK_TERMS; ++m) o[m][j] = ck_term(x);
    }
#pragma unroll
    for (int m = 0; m < CK_TERMS; ++m)
      *(uint4*)(sX + (m * CK_LEN + t) * VS + q) = make_uint4(o[m][0], o[m][1], o[m][2], o[m][3]);
  }
  asm volatile("cp.async.wait_group 0;");
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3;
  const int m_tiles = N / 16, n_pairs = V / 16;
  const int steps = (n + 15) / 16;
  float* out = dS + ((size_t)slot * s.H + h) * N * V;
  for (int item = warp; item < m_tiles * n_pairs; item += CK_THREADS / 32) {
    const int m0 = item / n_pairs * 16, v0 = item % n_pairs * 16;
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int kk = 0; kk < steps; ++kk) {
      uint32_t a[4], b[4];
      ck_ldsm_t(a, sB + (kk * 16 + (mi >> 1) * 8 + (lane & 7)) * NS + m0 + (mi & 1) * 8);
#pragma unroll
      for (int k = CK_TERMS - 1; k >= 0; --k) {           // the small terms first
        ck_ldsm_t(b, sX + (k * CK_LEN + kk * 16 + (mi & 1) * 8 + (lane & 7)) * VS + v0 + (mi >> 1) * 8);
        mma_bf16(acc[0], a, b);
        mma_bf16(acc[1], a, b + 2);
      }
    }
    const int row = m0 + (lane >> 2), col = v0 + 2 * (lane & 3);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      *(float2*)(out + (size_t)row * V + col + 8 * i) = make_float2(acc[i][0], acc[i][1]);
      *(float2*)(out + (size_t)(row + 8) * V + col + 8 * i) = make_float2(acc[i][2], acc[i][3]);
    }
  }
  if (threadIdx.x == 0) whole[(size_t)slot * s.H + h] = expf(end);
}

// ---- the chain of states ------------------------------------------------------------------------
__global__ void __launch_bounds__(CK_THREADS)
ssm_chunk_chain_kernel(float* __restrict__ dS, const float* __restrict__ whole,
                       float* __restrict__ state, const float* __restrict__ proj,
                       const int* __restrict__ tok_pos, const int* __restrict__ req_start,
                       const int* __restrict__ req_len, const int* __restrict__ req_slot,
                       ChunkShape s) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.z, h = blockIdx.y;
  const int n = req_len[r];
  if (n <= 0) return;
  int first = 0;
  for (int i = 0; i < r; ++i) first += (req_len[i] + CK_LEN - 1) / CK_LEN;
  const int chunks = (n + CK_LEN - 1) / CK_LEN, NV = s.N * s.V;
  float* slot = state + (size_t)req_slot[r] * s.state_stride;
  const int at = (blockIdx.x * CK_THREADS + threadIdx.x) * 4;
  if (at < NV) {
    float* own = slot + (size_t)h * NV + at;
    float4 st = *(const float4*)own;
    float* d = dS + ((size_t)first * s.H + h) * NV + at;
    const size_t hop = (size_t)s.H * NV;
    const float* w = whole + (size_t)first * s.H + h;
    constexpr int AHEAD = 8;                              // contributions in flight
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
      float4 add[AHEAD];
      float a[AHEAD];
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if (c0 + i < chunks) {
          add[i] = *(const float4*)(d + (c0 + i) * hop);
          a[i] = w[(size_t)(c0 + i) * s.H];
        }
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if (c0 + i < chunks) {
          *(float4*)(d + (c0 + i) * hop) = st;            // the state in front of the chunk
          st.x = fmaf(a[i], st.x, add[i].x); st.y = fmaf(a[i], st.y, add[i].y);
          st.z = fmaf(a[i], st.z, add[i].z); st.w = fmaf(a[i], st.w, add[i].w);
        }
    }
    *(float4*)own = st;
  }
  if (blockIdx.x == 0) {                                  // each head keeps a share of the inputs
    const int C = s.channels, k = min(n, s.taps), t0 = req_start[r], pos0 = tok_pos[t0];
    const int c_lo = (int)((long long)C * h / s.H), span = (int)((long long)C * (h + 1) / s.H) - c_lo;
    float* ring = slot + (size_t)s.H * NV;
    for (int i = threadIdx.x; i < k * span; i += CK_THREADS) {
      const int j = n - k + i / span, c = c_lo + i % span;
      ring[(size_t)((pos0 + j) % s.taps) * C + c] = proj[(size_t)(t0 + j) * s.stride + s.x_off + c];
    }
  }
}

// ---- the outputs --------------------------------------------------------------------------------
// VT: output tiles of 8 columns a warp keeps at most (V <= 8 * VT).  A warp owns 16 tokens.
template <int VT>
__global__ void __launch_bounds__(CK_THREADS)
ssm_chunk_out_kernel(float* __restrict__ y, const float* __restrict__ S_in,
                     const __nv_bfloat16* __restrict__ rows, const float* __restrict__ step,
                     const float* __restrict__ skip, const int* __restrict__ req_start,
                     const int* __restrict__ req_len, ChunkShape s) {
  extern __shared__ __align__(16) uint8_t ck_smem[];
  __shared__ float s_cs[CK_LEN], s_dt[CK_LEN];
  pdl_trigger();
  pdl_wait();
  const int slot = blockIdx.x, h = blockIdx.y, g = h / (s.H / s.G);
  int r, c;
  if (!ck_find(req_len, s.n_requests, slot, r, c)) return;
  const int N = s.N, V = s.V, NS = N + CK_PAD, VS = V + CK_PAD;
  const int n = min(CK_LEN, req_len[r] - c * CK_LEN), t0 = req_start[r] + c * CK_LEN;
  __nv_bfloat16* sC = (__nv_bfloat16*)ck_smem;            // [CK_LEN][NS]
  __nv_bfloat16* sX = sC + CK_LEN * NS;                   // [CK_LEN][VS]
  __nv_bfloat16* sS = sX + CK_LEN * VS;                   // [terms][N][VS]
  __nv_bfloat16* sB = sS;                                 // [CK_LEN][NS], once S has been used
  const __nv_bfloat16* base = rows + (size_t)t0 * s.channels;
  const int b_off = s.H * V + g * N, c_off = b_off + s.G * N, nq = N / 8, vq = V / 8;
  for (int i = threadIdx.x; i < CK_LEN * nq; i += CK_THREADS) {
    const int t = i / nq, q = (i - t * nq) * 8;
    const __nv_bfloat16* row = base + (size_t)(t < n ? t : 0) * s.channels;
    ck_copy16(sC + t * NS + q, row + c_off + q, t < n);
  }
  for (int i = threadIdx.x; i < CK_LEN * vq; i += CK_THREADS) {
    const int t = i / vq, q = (i - t * vq) * 8;
    ck_copy16(sX + t * VS + q, base + (size_t)(t < n ? t : 0) * s.channels + h * V + q, t < n);
  }
  asm volatile("cp.async.commit_group;");
  const float* S = S_in + ((size_t)slot * s.H + h) * N * V;
  const int v4 = V / 4, s_pieces = N * v4;
  constexpr int AHEAD = 8;
  float4 sr[AHEAD];
  auto fetch_s = [&](int i0) {
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      const int i = i0 + k * CK_THREADS + threadIdx.x;
      if (i < s_pieces) sr[k] = *(const float4*)(S + (size_t)i * 4);
    }
  };
  fetch_s(0);                                             // on its way while the decays are summed
  ck_sums(s_cs, s_dt, step, t0, n, s.H, h);
  for (int i0 = 0; i0 < s_pieces; i0 += AHEAD * CK_THREADS) {
    if (i0 > 0) fetch_s(i0);
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      const int i = i0 + k * CK_THREADS + threadIdx.x;
      if (i >= s_pieces) continue;
      const int d = i / v4, q = 4 * (i - d * v4);
      float2 lo = make_float2(sr[k].x, sr[k].y), hi = make_float2(sr[k].z, sr[k].w);
#pragma unroll
      for (int m = 0; m < CK_TERMS; ++m) {
        const uint32_t a = ck_term(lo), b = ck_term(hi);
        *(uint2*)(sS + (m * N + d) * VS + q) = make_uint2(a, b);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;");
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3;
  const int gq = lane >> 2, tq = lane & 3;
  const bool live = warp * 16 < n;
  const int row_a = warp * 16 + gq, row_b = row_a + 8, nt_all = V / 8;
  const float cs_a = s_cs[row_a], cs_b = s_cs[row_b];
  float acc[VT][4];
#pragma unroll
  for (int i = 0; i < VT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const __nv_bfloat16* cp = sC + (warp * 16 + (lane & 15)) * NS + (lane >> 4) * 8;
  // what came before the chunk
  for (int kk = 0; kk < N / 16 && live; ++kk) {
    uint32_t a[4];
    ldmatrix_x4(a, cp + kk * 16);
#pragma unroll
    for (int k = CK_TERMS - 1; k >= 0; --k)
#pragma unroll
      for (int dp = 0; dp < VT / 2; ++dp) {
        if (2 * dp >= nt_all) continue;
        uint32_t b[4];
        ck_ldsm_t(b, sS + (k * N + kk * 16 + (mi & 1) * 8 + (lane & 7)) * VS + dp * 16 + (mi >> 1) * 8);
        mma_bf16(acc[2 * dp], a, b);
        mma_bf16(acc[2 * dp + 1], a, b + 2);
      }
  }
  __syncthreads();                                        // S has been used: B takes its place
  for (int i = threadIdx.x; i < CK_LEN * nq; i += CK_THREADS) {
    const int t = i / nq, q = (i - t * nq) * 8;
    ck_copy16(sB + t * NS + q, base + (size_t)(t < n ? t : 0) * s.channels + b_off + q, t < n);
  }
  asm volatile("cp.async.commit_group;");
  const float ea = expf(cs_a), eb = expf(cs_b);
#pragma unroll
  for (int i = 0; i < VT; ++i) {
    acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb;
  }
  asm volatile("cp.async.wait_group 0;");
  __syncthreads();
  if (!live) return;                                      // no block barrier from here on
  // the chunk's own tokens, 32 at a time
  for (int j0 = 0; j0 <= warp * 16 + 15 && j0 < n; j0 += 32) {
    float p[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f;
    for (int ks = 0; ks < N / 16; ++ks) {
      uint32_t a[4], b[4];
      ldmatrix_x4(a, cp + ks * 16);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        ldmatrix_x4(b, sB + (j0 + np * 16 + (mi >> 1) * 8 + (lane & 7)) * NS + ks * 16 + (mi & 1) * 8);
        mma_bf16(p[2 * np], a, b);
        mma_bf16(p[2 * np + 1], a, b + 2);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int j = j0 + nt * 8 + tq * 2 + (q & 1), i = q < 2 ? row_a : row_b;
        p[nt][q] = j <= i ? p[nt][q] * expf((q < 2 ? cs_a : cs_b) - s_cs[j]) * s_dt[j] : 0.f;
      }
#pragma unroll
    for (int kk = 0; kk < 2; ++kk) {
      uint32_t a[CK_TERMS][4];
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const int nt = 2 * kk + (w >> 1), q = (w & 1) * 2;
        float2 v = make_float2(p[nt][q], p[nt][q + 1]);
#pragma unroll
        for (int k = 0; k < CK_TERMS; ++k) a[k][w] = ck_term(v);
      }
#pragma unroll
      for (int dp = 0; dp < VT / 2; ++dp) {
        if (2 * dp >= nt_all) continue;
        uint32_t b[4];
        ck_ldsm_t(b, sX + (j0 + kk * 16 + (mi & 1) * 8 + (lane & 7)) * VS + dp * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int k = CK_TERMS - 1; k >= 0; --k) {
          mma_bf16(acc[2 * dp], a[k], b);
          mma_bf16(acc[2 * dp + 1], a[k], b + 2);
        }
      }
    }
  }
  const float dh = skip[h];
  const size_t yw = (size_t)s.H * V;
  float* yo = y + (size_t)t0 * yw + (size_t)h * V;
#pragma unroll
  for (int i = 0; i < VT; ++i) {
    if (i >= nt_all) continue;
    const int e = i * 8 + tq * 2;
    if (row_a < n) {
      const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)(sX + row_a * VS + e));
      *(float2*)(yo + (size_t)row_a * yw + e) = make_float2(fmaf(dh, x.x, acc[i][0]), fmaf(dh, x.y, acc[i][1]));
    }
    if (row_b < n) {
      const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)(sX + row_b * VS + e));
      *(float2*)(yo + (size_t)row_b * yw + e) = make_float2(fmaf(dh, x.x, acc[i][2]), fmaf(dh, x.y, acc[i][3]));
    }
  }
}

static inline size_t ck_state_smem(int N, int V) {
  return (size_t)CK_LEN * 2 * ((N + CK_PAD) + CK_TERMS * (V + CK_PAD));
}
static inline size_t ck_out_smem(int N, int V) {
  const size_t states = (size_t)CK_TERMS * N * (V + CK_PAD), keys = (size_t)CK_LEN * (N + CK_PAD);
  return 2 * (keys + (size_t)CK_LEN * (V + CK_PAD) + (states > keys ? states : keys));
}

}  // namespace hs

// Whether the chunked form takes these sizes.
HS_EXPORT int hs_ssm_chunk_takes(int H, int G, int N, int V) {
  return H > 0 && G > 0 && H % G == 0 && N > 0 && N % 16 == 0 && V > 0 && V % 16 == 0 && V <= 128 &&
                 hs::ck_out_smem(N, V) <= 220 * 1024
             ? 1
             : 0;
}

// Chunks a step of n_tokens tokens and n_requests requests can have.
HS_EXPORT int hs_ssm_chunk_slots(int n_tokens, int n_requests) {
  return n_tokens / hs::CK_LEN + n_requests;
}

// y [tokens, H*V] float32; rows [tokens, channels] bfloat16 and step as ssm_prepare left them; dS
// [slots, H, N, V] and whole [slots, H] float32 scratch.
HS_EXPORT int hs_ssm_chunked(float* y, float* state, const void* rows, const float* step,
                             const float* proj, const float* skip, const int* tok_pos,
                             const int* req_start, const int* req_len, const int* req_slot,
                             int n_requests, int n_tokens, int H, int G, int N, int V, int taps,
                             int stride, int x_off, int state_stride, float* dS, float* whole,
                             void* stream) {
  using namespace hs;
  if (!y || !state || !rows || !step || !proj || !skip || !tok_pos || !req_start || !req_len ||
      !req_slot || !dS || !whole)
    return HS_ERR_ARGUMENT;
  const int C = H * V + 2 * G * N;
  if (!hs_ssm_chunk_takes(H, G, N, V) || taps <= 0 || x_off < 0 || x_off + C > stride ||
      state_stride % 4 || H * N * V + taps * C > state_stride)
    return HS_ERR_UNSUPPORTED;
  if (((uintptr_t)rows | (uintptr_t)state | (uintptr_t)dS | (uintptr_t)y) & 15) return HS_ERR_UNSUPPORTED;
  if (n_requests <= 0 || n_tokens <= 0) return HS_OK;
  if (n_requests > 65535 || H > 65535) return HS_ERR_TOO_LARGE;
  const ChunkShape s = {H, G, N, V, taps, C, stride, x_off, state_stride, n_requests};
  const int slots = hs_ssm_chunk_slots(n_tokens, n_requests);
  cudaStream_t st = (cudaStream_t)stream;
  const bool pdl = hs_pdl_enabled();
  const __nv_bfloat16* rw = (const __nv_bfloat16*)rows;
  const size_t sm1 = ck_state_smem(N, V), sm2 = ck_out_smem(N, V);
  cudaError_t e = cudaFuncSetAttribute(ssm_chunk_state_kernel,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1);
  if (e != cudaSuccess) return (int)e;
  e = hs_launch(ssm_chunk_state_kernel, dim3(slots, H), dim3(CK_THREADS), sm1, st, pdl, dS, whole, rw,
                step, req_start, req_len, s);
  if (e != cudaSuccess) return (int)e;
  e = hs_launch(ssm_chunk_chain_kernel, dim3((N * V / 4 + CK_THREADS - 1) / CK_THREADS, H, n_requests),
                dim3(CK_THREADS), 0, st, pdl, dS, (const float*)whole, state, proj, tok_pos, req_start,
                req_len, req_slot, s);
  if (e != cudaSuccess) return (int)e;
#define HS_CK(VT)                                                                                  \
  do {                                                                                             \
    auto k = ssm_chunk_out_kernel<VT>;                                                             \
    e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm2);            \
    if (e == cudaSuccess)                                                                          \
      e = hs_launch(k, dim3(slots, H), dim3(CK_THREADS), sm2, st, pdl, y, (const float*)dS, rw, step, \
                    skip, req_start, req_len, s);                                                  \
  } while (0)
  if (V <= 32) HS_CK(4);
  else if (V <= 64) HS_CK(8);
  else HS_CK(16);
#undef HS_CK
  return e == cudaSuccess ? HS_OK : (int)e;
}
