// The residual stream at the places where blocks touch it, each with the norm of what comes next in
// the same launch:
//
//   embed_norm     x  = norm(table[id])                            (weight, optional bias)
//                  x0 = x                                          (optional copy, kept for `again`)
//   residual_mix   x += s1 * y1 (+ s2 * y2) (+ again)              (s1, s2: one factor per column)
//
//   then, optional in both:  out = norm2(x), float32 or bfloat16
//
//   hyper_mix      several copies of the stream behind a sublayer (a token's copies are neighbours
//                  in one row):  x_t <- sum_s mix[s][t] x_s + write[t] y;
//                  u = sum_t read[t] x_t;  out = u / sqrt(mean(u^2) + eps) * weight
//
// The norms of the first two are (v - mean) / sqrt(variance + eps) * weight (+ bias), the variance being the mean of
// the squared deviations.  One block per row.  All sums are float32, formed in an order fixed by
// the width, so a row's result does not depend on its neighbours in the batch.
#include "common.cuh"

namespace hs {

constexpr int SM_THREADS = 256;
constexpr int SM_V4 = 4;              // float4 a thread keeps: rows of up to 4,096 floats

__device__ __forceinline__ float sm_block_sum(float v, float* s_part) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockDim.x >> 5;
  __syncthreads();                    // the partial sums of the round before have been read
  if (lane == 0) s_part[warp] = v;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < n; ++i) total += s_part[i];
  return total;
}

// A row held by its block: in registers, four columns a piece (VEC; the width is a multiple of 4
// and every pointer 16-byte aligned), or in shared memory, any width.
template <bool VEC>
struct Row {
  float4 v[VEC ? SM_V4 : 1];
  float* s;
  int width;

  template <typename F>               // f(column of the piece, the piece's values): VEC pieces
  __device__ __forceinline__ void each(F f) {
    if constexpr (VEC) {
#pragma unroll
      for (int i = 0; i < SM_V4; ++i) {
        const int c = 4 * (threadIdx.x + i * blockDim.x);
        if (c < width) f(c, &v[i].x);
      }
    } else {
      for (int c = threadIdx.x; c < width; c += blockDim.x) f(c, s + c);
    }
  }
};
template <bool VEC> constexpr int PIECE = VEC ? 4 : 1;

template <bool VEC>
__device__ __forceinline__ void load_piece(float* d, const float* p) {
  if constexpr (VEC) *(float4*)d = *(const float4*)p;
  else *d = *p;
}
template <bool VEC>
__device__ __forceinline__ void load_piece(float* d, const __nv_bfloat16* p) {
  if constexpr (VEC) {
    const uint2 u = *(const uint2*)p;
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&u.x);
    const float2 b = __bfloat1622float2(*(const __nv_bfloat162*)&u.y);
    d[0] = a.x; d[1] = a.y; d[2] = b.x; d[3] = b.y;
  } else {
    *d = to_f(*p);
  }
}
template <bool VEC>
__device__ __forceinline__ void store_piece(float* p, const float* d) {
  if constexpr (VEC) *(float4*)p = *(const float4*)d;
  else *p = *d;
}
template <bool VEC>
__device__ __forceinline__ void store_piece(__nv_bfloat16* p, const float* d) {
  if constexpr (VEC) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(d[0], d[1]), b = __floats2bfloat162_rn(d[2], d[3]);
    uint2 u;
    u.x = *(const uint32_t*)&a; u.y = *(const uint32_t*)&b;
    *(uint2*)p = u;
  } else {
    *p = __float2bfloat16_rn(*d);
  }
}

// mean and 1 / sqrt(variance + eps) of the row
template <bool VEC>
__device__ __forceinline__ float2 row_stats(Row<VEC>& row, float eps, float* s_part) {
  float s = 0.f;
  row.each([&](int, float* d) {
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) s += d[i];
  });
  const float mean = sm_block_sum(s, s_part) / (float)row.width;
  float q = 0.f;
  row.each([&](int, float* d) {
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) q = fmaf(d[i] - mean, d[i] - mean, q);
  });
  const float var = sm_block_sum(q, s_part) / (float)row.width;
  return make_float2(mean, 1.0f / sqrtf(var + eps));
}

template <bool VEC>
__device__ __forceinline__ void normed_piece(float* o, const float* d, int c, float2 st,
                                             const float* g, const float* b) {
  float w[PIECE<VEC>], a[PIECE<VEC>];
  load_piece<VEC>(w, g + c);
  if (b) load_piece<VEC>(a, b + c);
#pragma unroll
  for (int i = 0; i < PIECE<VEC>; ++i)
    o[i] = (d[i] - st.x) * st.y * w[i] + (b ? a[i] : 0.f);
}

template <bool VEC, typename TO>
__device__ __forceinline__ void row_norm_out(Row<VEC>& row, TO* out, const float* g, const float* b,
                                             float eps, float* s_part) {
  const float2 st = row_stats<VEC>(row, eps, s_part);
  row.each([&](int c, float* d) {
    __align__(16) float o[PIECE<VEC>];
    normed_piece<VEC>(o, d, c, st, g, b);
    store_piece<VEC>(out + c, o);
  });
}

template <bool VEC, typename T, typename TO>
__global__ void __launch_bounds__(SM_THREADS)
embed_norm_kernel(float* __restrict__ x, float* __restrict__ x0, const int* __restrict__ ids,
                  const int* __restrict__ req, const T* __restrict__ table, int width, int vocab,
                  const int* __restrict__ feedback, int n_feedback, const float* __restrict__ g,
                  const float* __restrict__ b, float eps, TO* __restrict__ out,
                  const float* __restrict__ g2, const float* __restrict__ b2, float eps2,
                  int* status) {
  extern __shared__ __align__(16) float s_row[];
  __shared__ float s_part[SM_THREADS / 32];
  pdl_trigger();
  const int t = blockIdx.x;
  int id = ids[t];
  bool ok = req[t] >= 0;
  // id = -(s + 1): the token that the latest sampling step left in feedback[s]
  if (ok && id < 0 && feedback != nullptr && -(id + 1) < n_feedback) id = feedback[-(id + 1)];
  if (ok && (id < 0 || id >= vocab)) {
    if (threadIdx.x == 0) atomicOr(status, HS_STATUS_BAD_TOKEN);
    ok = false;
  }
  Row<VEC> row;
  row.s = s_row;
  row.width = width;
  const size_t at = (size_t)t * width;
  if (!ok) {                          // padding rows, or a refused id: defined, finite rows
    __align__(16) const float zero[4] = {0.f, 0.f, 0.f, 0.f};
    row.each([&](int c, float*) {
      store_piece<VEC>(x + at + c, zero);
      if (x0) store_piece<VEC>(x0 + at + c, zero);
      if (out) store_piece<VEC>(out + at + c, zero);
    });
    return;
  }
  row.each([&](int c, float* d) { load_piece<VEC>(d, table + (size_t)id * width + c); });
  const float2 st = row_stats<VEC>(row, eps, s_part);
  row.each([&](int c, float* d) {
    __align__(16) float o[PIECE<VEC>];
    normed_piece<VEC>(o, d, c, st, g, b);
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) d[i] = o[i];
    store_piece<VEC>(x + at + c, d);
    if (x0) store_piece<VEC>(x0 + at + c, d);
  });
  if (out) row_norm_out<VEC>(row, out + at, g2, b2, eps2, s_part);
}

constexpr int HM_MAX = 16;            // copies of the stream at most

// SM: copies a thread holds (exactly n_streams for SM <= 4).  src holds src_streams rows a token, or
// one row that stands for all copies; dst may be src.  y, dst, u, out may be null; without y the
// copies stay as they are; without rd every copy counts once in u.
template <bool VEC, int SM, typename TO>
__global__ void __launch_bounds__(SM_THREADS)
hyper_mix_kernel(float* dst, const float* src, int src_streams, const float* __restrict__ y,
                 int n_streams, const float* __restrict__ mix, const float* __restrict__ wr,
                 const float* __restrict__ rd, int width, float* __restrict__ u,
                 TO* __restrict__ out, const float* __restrict__ g, float eps) {
  extern __shared__ __align__(16) float s_row[];
  __shared__ float s_part[SM_THREADS / 32];
  __shared__ float s_mix[HM_MAX * HM_MAX], s_wr[HM_MAX], s_rd[HM_MAX];
  pdl_trigger();
  const int n = SM <= 4 ? SM : n_streams;
  // the tables are weights: fetched ahead of the wait
  if (y)
    for (int i = threadIdx.x; i < n * n; i += blockDim.x) s_mix[i] = mix[i];
  if ((int)threadIdx.x < n) {
    s_wr[threadIdx.x] = y ? wr[threadIdx.x] : 0.f;
    s_rd[threadIdx.x] = rd ? rd[threadIdx.x] : 1.f;
  }
  __syncthreads();
  pdl_wait();
  Row<VEC> row;
  row.s = s_row;
  row.width = width;
  const size_t t = blockIdx.x;
  const float* sr = src + t * src_streams * width;
  const size_t step = src_streams > 1 ? width : 0;
  float* dr = dst ? dst + t * n * width : nullptr;
  row.each([&](int c, float* d) {
    __align__(16) float xs[SM][PIECE<VEC>], yv[PIECE<VEC>], acc[PIECE<VEC>];
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < n) load_piece<VEC>(xs[s], sr + s * step + c);
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) acc[i] = 0.f;
    if (y) load_piece<VEC>(yv, y + t * width + c);
#pragma unroll
    for (int to = 0; to < SM; ++to) {
      if (to >= n) continue;
      __align__(16) float v[PIECE<VEC>];
      if (y) {
        const float w = s_wr[to];
#pragma unroll
        for (int i = 0; i < PIECE<VEC>; ++i) v[i] = w * yv[i];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (s >= n) continue;
          const float m = s_mix[s * n + to];
#pragma unroll
          for (int i = 0; i < PIECE<VEC>; ++i) v[i] = fmaf(m, xs[s][i], v[i]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < PIECE<VEC>; ++i) v[i] = xs[to][i];
      }
      if (dr) store_piece<VEC>(dr + (size_t)to * width + c, v);
      const float r = s_rd[to];
#pragma unroll
      for (int i = 0; i < PIECE<VEC>; ++i) acc[i] = fmaf(r, v[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) d[i] = acc[i];
    if (u) store_piece<VEC>(u + t * width + c, d);
  });
  if (!out) return;
  float q = 0.f;
  row.each([&](int, float* d) {
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) q = fmaf(d[i], d[i], q);
  });
  const float r = 1.0f / sqrtf(sm_block_sum(q, s_part) / (float)width + eps);
  row.each([&](int c, float* d) {
    __align__(16) float o[PIECE<VEC>], w[PIECE<VEC>];
    load_piece<VEC>(w, g + c);
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) o[i] = d[i] * r * w[i];
    store_piece<VEC>(out + t * width + c, o);
  });
}

template <bool VEC, typename TO>
__global__ void __launch_bounds__(SM_THREADS)
residual_mix_kernel(float* __restrict__ x, const float* __restrict__ y1,
                    const float* __restrict__ s1, const float* __restrict__ y2,
                    const float* __restrict__ s2, const float* __restrict__ again, int width,
                    TO* __restrict__ out, const float* __restrict__ g, const float* __restrict__ b,
                    float eps) {
  extern __shared__ __align__(16) float s_row[];
  __shared__ float s_part[SM_THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const size_t at = (size_t)blockIdx.x * width;
  Row<VEC> row;
  row.s = s_row;
  row.width = width;
  row.each([&](int c, float* d) {
    __align__(16) float a[PIECE<VEC>], f[PIECE<VEC>], sum[PIECE<VEC>];
    load_piece<VEC>(d, x + at + c);
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) sum[i] = 0.f;
    if (y1) {
      load_piece<VEC>(a, y1 + at + c);
      load_piece<VEC>(f, s1 + c);
#pragma unroll
      for (int i = 0; i < PIECE<VEC>; ++i) sum[i] = a[i] * f[i];
    }
    if (y2) {
      load_piece<VEC>(a, y2 + at + c);
      load_piece<VEC>(f, s2 + c);
#pragma unroll
      for (int i = 0; i < PIECE<VEC>; ++i) sum[i] = fmaf(a[i], f[i], sum[i]);
    }
#pragma unroll
    for (int i = 0; i < PIECE<VEC>; ++i) d[i] += sum[i];
    if (again) {
      load_piece<VEC>(a, again + at + c);
#pragma unroll
      for (int i = 0; i < PIECE<VEC>; ++i) d[i] += a[i];
    }
    store_piece<VEC>(x + at + c, d);
  });
  if (out) row_norm_out<VEC>(row, out + at, g, b, eps, s_part);
}

static inline bool sm_vec(int width, const void* const* ptrs, int n) {
  if (width % 4 || width > SM_THREADS * 4 * SM_V4) return false;
  for (int i = 0; i < n; ++i)
    if ((uintptr_t)ptrs[i] & 15) return false;
  return true;
}
static inline int sm_threads(int width, bool vec) {
  const int pieces = vec ? width / 4 : width;
  const int n = (pieces + 31) / 32 * 32;
  return n < SM_THREADS ? n : SM_THREADS;
}

}  // namespace hs

// out (with g2): the norm of the new rows, of type out_dtype; x0: a copy of x; both may be null.
HS_EXPORT int hs_embed_norm(float* x, float* x0, const int* ids, const int* req, const void* table,
                            int n_tokens, int width, int vocab, int table_dtype,
                            const int* feedback, int n_feedback, const float* g, const float* b,
                            float eps, void* out, const float* g2, const float* b2, float eps2,
                            int out_dtype, int* status, void* stream) {
  if (!x || !ids || !req || !table || !g || !status || (out && !g2)) return HS_ERR_ARGUMENT;
  if (width <= 0) return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  const void* ptrs[] = {x, x0, table, g, b, out, g2, b2};
  const bool vec = hs::sm_vec(width, ptrs, 8);
  const size_t smem = vec ? 0 : (size_t)width * sizeof(float);
  if (smem > 47 * 1024) return HS_ERR_UNSUPPORTED;
  const dim3 grid(n_tokens), block(hs::sm_threads(width, vec));
  cudaStream_t st = (cudaStream_t)stream;
#define HS_EN(VEC, T, TO)                                                                        \
  hs::embed_norm_kernel<VEC, T, TO><<<grid, block, smem, st>>>(                                  \
      x, x0, ids, req, (const T*)table, width, vocab, feedback, n_feedback, g, b, eps, (TO*)out, \
      g2, b2, eps2, status)
#define HS_EN_T(T)                                                               \
  do {                                                                           \
    if (out_dtype == HS_DT_BF16) { if (vec) HS_EN(true, T, __nv_bfloat16); else HS_EN(false, T, __nv_bfloat16); } \
    else if (out_dtype == HS_DT_F32) { if (vec) HS_EN(true, T, float); else HS_EN(false, T, float); } \
    else return HS_ERR_UNSUPPORTED;                                              \
  } while (0)
  if (table_dtype == HS_DT_F32) HS_EN_T(float);
  else if (table_dtype == HS_DT_BF16) HS_EN_T(__nv_bfloat16);
  else return HS_ERR_UNSUPPORTED;
#undef HS_EN_T
#undef HS_EN
  HS_LAUNCH_CHECK();
  return HS_OK;
}

// y1 / y2 / again / out may each be null (at least one of the first three is there).
HS_EXPORT int hs_residual_mix(float* x, const float* y1, const float* s1, const float* y2,
                              const float* s2, const float* again, int n_rows, int width, void* out,
                              const float* g, const float* b, float eps, int out_dtype,
                              void* stream) {
  if (!x || (y1 && !s1) || (y2 && !s2) || (!y1 && !y2 && !again) || (out && !g))
    return HS_ERR_ARGUMENT;
  if (width <= 0) return HS_ERR_UNSUPPORTED;
  if (n_rows <= 0) return HS_OK;
  const void* ptrs[] = {x, y1, s1, y2, s2, again, out, g, b};
  const bool vec = hs::sm_vec(width, ptrs, 9);
  const size_t smem = vec ? 0 : (size_t)width * sizeof(float);
  if (smem > 47 * 1024) return HS_ERR_UNSUPPORTED;
  const dim3 grid(n_rows), block(hs::sm_threads(width, vec));
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e = cudaSuccess;
#define HS_RM(VEC, TO)                                                                          \
  e = hs_launch(hs::residual_mix_kernel<VEC, TO>, grid, block, smem, st, hs_pdl_enabled(), x,   \
                y1, s1, y2, s2, again, width, (TO*)out, g, b, eps)
  if (out && out_dtype == HS_DT_BF16) { if (vec) HS_RM(true, __nv_bfloat16); else HS_RM(false, __nv_bfloat16); }
  else if (!out || out_dtype == HS_DT_F32) { if (vec) HS_RM(true, float); else HS_RM(false, float); }
  else return HS_ERR_UNSUPPORTED;
#undef HS_RM
  return e == cudaSuccess ? HS_OK : (int)e;
}

// See hyper_mix_kernel.  src_streams: 1 or n_streams rows a token in src.
HS_EXPORT int hs_hyper_mix(float* dst, const float* src, int src_streams, const float* y,
                           int n_streams, const float* mix, const float* wr, const float* rd,
                           int n_rows, int width, float* u, void* out, const float* g, float eps,
                           int out_dtype, void* stream) {
  if (!src || (y && (!mix || !wr)) || (!dst && !u && !out) || (out && !g)) return HS_ERR_ARGUMENT;
  if (width <= 0 || n_streams <= 0 || n_streams > hs::HM_MAX ||
      (src_streams != 1 && src_streams != n_streams))
    return HS_ERR_UNSUPPORTED;
  if (n_rows <= 0) return HS_OK;
  const void* ptrs[] = {dst, src, y, u, out, g};
  const bool vec = hs::sm_vec(width, ptrs, 6);
  const size_t smem = vec ? 0 : (size_t)width * sizeof(float);
  if (smem > 40 * 1024) return HS_ERR_UNSUPPORTED;
  const dim3 grid(n_rows), block(hs::sm_threads(width, vec));
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e = cudaSuccess;
#define HS_HM(VEC, SM, TO)                                                                      \
  e = hs_launch(hs::hyper_mix_kernel<VEC, SM, TO>, grid, block, smem, st, hs_pdl_enabled(), dst, \
                src, src_streams, y, n_streams, mix, wr, rd, width, u, (TO*)out, g, eps)
#define HS_HM_S(VEC, TO)                      \
  do {                                        \
    switch (n_streams) {                      \
      case 1: HS_HM(VEC, 1, TO); break;       \
      case 2: HS_HM(VEC, 2, TO); break;       \
      case 3: HS_HM(VEC, 3, TO); break;       \
      case 4: HS_HM(VEC, 4, TO); break;       \
      default: HS_HM(VEC, hs::HM_MAX, TO);    \
    }                                         \
  } while (0)
  if (out && out_dtype == HS_DT_BF16) { if (vec) HS_HM_S(true, __nv_bfloat16); else HS_HM_S(false, __nv_bfloat16); }
  else if (!out || out_dtype == HS_DT_F32) { if (vec) HS_HM_S(true, float); else HS_HM_S(false, float); }
  else return HS_ERR_UNSUPPORTED;
#undef HS_HM_S
#undef HS_HM
  return e == cudaSuccess ? HS_OK : (int)e;
}
