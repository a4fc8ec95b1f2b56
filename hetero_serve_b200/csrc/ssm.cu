// State-space duality (Mamba-2) as a recurrence on a float32 state S [N, V] per head and request.
//
// A token's row of the fused input projection holds [z | x: H*V | B: G*N | C: G*N | dt: H]; head h
// uses group g = h / (H / G).  x, B and C (the "channels", neighbours in the row from x_off on) pass
// a causal convolution per channel with a bias, and silu; then
//
//     dt_h = softplus(dt_h + dt_bias_h);  la_h = -exp(A_log_h) * dt_h          (the decay's logarithm)
//     S_h <- exp(la_h) S_h + dt_h B x_h^T;   y_h = S_h^T C + D_h x_h
//
//   ssm_prepare     per token: the activated channels as one row, and [dt | la]
//   ssm_recurrence  token after token: a block per (request, head, group of value columns), a thread
//                   keeps 16 state rows of a column in registers, the parts of a column are lanes of
//                   one warp; tokens' rows through two buffers of shared memory
//   ssm_step        both in one launch for a step in which every request brings one token
//
// State of a slot: [H, N, V] floats, then the convolutions' newest inputs as a ring of `taps` rows
// of `channels` floats: the input of position p lies in row p % taps.  A step of single tokens writes
// row p % taps while every block reads the taps - 1 other rows, so no block can disturb another; for
// prompt portions ssm_recurrence writes the rows, behind the launch that read them.
#include "common.cuh"

namespace hs {

struct SsmShape {
  int H, G, N, V, taps;
  int stride;                    // floats in a projection row
  int x_off;                     // column of x in it
  int state_stride;              // floats in a slot
};
__host__ __device__ inline int ssm_channels(const SsmShape& s) { return s.H * s.V + 2 * s.G * s.N; }

__device__ __forceinline__ float ssm_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ssm_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// channel c of the token at position pos whose portion began `back` tokens ago (0: it is the first):
// convolved and activated.  `own` points at the channel in the token's own projection row.
__device__ __forceinline__ float ssm_conv(const float* __restrict__ own, int stride,
                                          const float* __restrict__ ring, int C, int c, int pos,
                                          int back, int taps, const float* __restrict__ w,
                                          const float* __restrict__ bias) {
  float acc = bias[c];
#pragma unroll 4
  for (int j = 0; j < taps; ++j) {
    const int ago = taps - 1 - j;
    if (pos < ago) continue;                               // before the sequence: zero
    const float in = ago <= back ? own[-(ptrdiff_t)ago * stride]
                                 : ring[(size_t)((pos - ago) % taps) * C + c];
    acc = fmaf(w[(size_t)j * C + c], in, acc);
  }
  return ssm_silu(acc);
}

constexpr int SP_TOK = 2;        // tokens a block of ssm_prepare walks

// VEC: four channels a thread (every row and offset in whole 16-byte pieces)
template <bool VEC, typename TR>
__global__ void __launch_bounds__(256)
ssm_prepare_kernel(TR* __restrict__ rows, float* __restrict__ step, const float* __restrict__ proj,
                   const float* __restrict__ state, const int* __restrict__ tok_req,
                   const int* __restrict__ tok_pos, const int* __restrict__ req_start,
                   const int* __restrict__ req_slot, const float* __restrict__ conv_w,
                   const float* __restrict__ conv_b, const float* __restrict__ dt_bias,
                   const float* __restrict__ a_log, SsmShape s, int n_tokens) {
  pdl_trigger();
  pdl_wait();
  const int C = ssm_channels(s), t0 = blockIdx.x * SP_TOK, t1 = min(n_tokens, t0 + SP_TOK);
  if (blockIdx.y == gridDim.y - 1) {                       // dt and the decay's logarithm
    for (int i = threadIdx.x; i < (t1 - t0) * s.H; i += 256) {
      const int t = t0 + i / s.H, h = i % s.H;
      if (tok_req[t] < 0) continue;
      const float dt = ssm_softplus(proj[(size_t)t * s.stride + s.x_off + C + h] + dt_bias[h]);
      step[(size_t)t * 2 * s.H + h] = dt;
      step[(size_t)t * 2 * s.H + s.H + h] = -expf(a_log[h]) * dt;
    }
    return;
  }
  constexpr int P = VEC ? 4 : 1;
  const int c = (blockIdx.y * 256 + threadIdx.x) * P;
  if (c >= C) return;
  for (int t = t0; t < t1; ++t) {
    const int r = tok_req[t];
    if (r < 0) continue;
    const int pos = tok_pos[t], back = t - req_start[r];
    const float* ring = state + (size_t)req_slot[r] * s.state_stride + (size_t)s.H * s.N * s.V;
    const float* own = proj + (size_t)t * s.stride + s.x_off + c;
    if constexpr (VEC) {
      float4 acc = *(const float4*)(conv_b + c);
#pragma unroll 4
      for (int j = 0; j < s.taps; ++j) {
        const int ago = s.taps - 1 - j;
        if (pos < ago) continue;
        const float4 in = ago <= back
                              ? *(const float4*)(own - (ptrdiff_t)ago * s.stride)
                              : *(const float4*)(ring + (size_t)((pos - ago) % s.taps) * C + c);
        const float4 w = *(const float4*)(conv_w + (size_t)j * C + c);
        acc.x = fmaf(w.x, in.x, acc.x); acc.y = fmaf(w.y, in.y, acc.y);
        acc.z = fmaf(w.z, in.z, acc.z); acc.w = fmaf(w.w, in.w, acc.w);
      }
      acc = make_float4(ssm_silu(acc.x), ssm_silu(acc.y), ssm_silu(acc.z), ssm_silu(acc.w));
      if constexpr (sizeof(TR) == 4) {
        *(float4*)(rows + (size_t)t * C + c) = acc;
      } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(acc.x, acc.y);
        const __nv_bfloat162 hi = __floats2bfloat162_rn(acc.z, acc.w);
        *(uint2*)(rows + (size_t)t * C + c) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
      }
    } else {
      rows[(size_t)t * C + c] =
          from_f<TR>(ssm_conv(own, s.stride, ring, C, c, pos, back, s.taps, conv_w, conv_b));
    }
  }
}

// the inputs of the portion's last tokens into their rows of the ring: channels c_lo .. c_hi - 1
__device__ __forceinline__ void ssm_keep_inputs(float* __restrict__ ring,
                                                const float* __restrict__ proj, const SsmShape& s,
                                                int t0, int n, int pos0, int c_lo, int c_hi) {
  const int C = ssm_channels(s), span = c_hi - c_lo, k = min(n, s.taps);
  for (int i = threadIdx.x; i < k * span; i += blockDim.x) {
    const int j = n - k + i / span, c = c_lo + i % span;
    ring[(size_t)((pos0 + j) % s.taps) * C + c] = proj[(size_t)(t0 + j) * s.stride + s.x_off + c];
  }
}

// ---- the recurrence over portions -------------------------------------------------------------
constexpr int SR_THREADS = 128;
constexpr int SR_ROWS = 16;          // state rows a thread keeps
constexpr int SR_PART = SR_ROWS + 4; // floats between two parts' rows of a token: distinct banks
constexpr int SR_TOK = 16;           // tokens staged at a time (8 when N is above 128, 4 above 256)

__device__ __forceinline__ void sr_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(
                   (uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// up to `here` tokens from `tok` on into one buffer: B [ntok][Np], C [ntok][Np], x [ntok][cols],
// [decay | dt] [ntok][2]
__device__ __forceinline__ void sr_stage(float* buf, const float* __restrict__ rows,
                                         const float* __restrict__ step, int tok, int here,
                                         const SsmShape& s, int h, int g, int Np, int cols, int v0,
                                         int ntok, int vec) {
  const int C = ssm_channels(s), b_off = s.H * s.V + g * s.N, c_off = b_off + s.G * s.N;
  float* s_b = buf;
  float* s_c = s_b + ntok * Np;
  float* s_x = s_c + ntok * Np;
  float* s_d = s_x + ntok * cols;
  if (vec) {
    const int nq = s.N / 4, cq = cols / 4;
    for (int e = threadIdx.x; e < here * nq; e += SR_THREADS) {
      const int tt = e / nq, c = 4 * (e - tt * nq);
      const float* row = rows + (size_t)(tok + tt) * C;
      const int at = tt * Np + c / SR_ROWS * SR_PART + c % SR_ROWS;
      sr_cp16(s_b + at, row + b_off + c);
      sr_cp16(s_c + at, row + c_off + c);
    }
    for (int e = threadIdx.x; e < here * cq; e += SR_THREADS) {
      const int tt = e / cq, c = 4 * (e - tt * cq);
      if (v0 + c < s.V)
        sr_cp16(s_x + tt * cols + c, rows + (size_t)(tok + tt) * C + (size_t)h * s.V + v0 + c);
    }
  } else {
    for (int e = threadIdx.x; e < here * s.N; e += SR_THREADS) {
      const int tt = e / s.N, c = e - tt * s.N;
      const float* row = rows + (size_t)(tok + tt) * C;
      const int at = tt * Np + c / SR_ROWS * SR_PART + c % SR_ROWS;
      s_b[at] = row[b_off + c];
      s_c[at] = row[c_off + c];
    }
    for (int e = threadIdx.x; e < here * cols; e += SR_THREADS) {
      const int tt = e / cols, c = e - tt * cols;
      if (v0 + c < s.V) s_x[e] = rows[(size_t)(tok + tt) * C + (size_t)h * s.V + v0 + c];
    }
  }
  if ((int)threadIdx.x < here) {
    const float* st = step + (size_t)(tok + threadIdx.x) * 2 * s.H;
    s_d[2 * threadIdx.x] = expf(st[s.H + h]);
    s_d[2 * threadIdx.x + 1] = st[h];
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}

__device__ __forceinline__ float sr_token(float (&st)[SR_ROWS], const float* bp, const float* cp,
                                          float xdt, float decay) {
  float part[SR_ROWS / 4];
#pragma unroll
  for (int i = 0; i < SR_ROWS / 4; ++i) {
    const float4 b = *(const float4*)(bp + 4 * i), c = *(const float4*)(cp + 4 * i);
    st[4 * i + 0] = fmaf(b.x, xdt, decay * st[4 * i + 0]);
    st[4 * i + 1] = fmaf(b.y, xdt, decay * st[4 * i + 1]);
    st[4 * i + 2] = fmaf(b.z, xdt, decay * st[4 * i + 2]);
    st[4 * i + 3] = fmaf(b.w, xdt, decay * st[4 * i + 3]);
    float a = st[4 * i + 0] * c.x;
    a = fmaf(st[4 * i + 1], c.y, a);
    a = fmaf(st[4 * i + 2], c.z, a);
    part[i] = fmaf(st[4 * i + 3], c.w, a);
  }
  return (part[0] + part[1]) + (part[2] + part[3]);
}

__global__ void __launch_bounds__(SR_THREADS, 1)
ssm_recurrence_kernel(float* __restrict__ y, float* __restrict__ state,
                      const float* __restrict__ rows, const float* __restrict__ step,
                      const float* __restrict__ proj, const float* __restrict__ skip,
                      const int* __restrict__ tok_pos, const int* __restrict__ req_start,
                      const int* __restrict__ req_len, const int* __restrict__ req_slot, SsmShape s,
                      int P, int ntok, int vec) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  const int Np = P * SR_PART, cols = SR_THREADS / P;
  const int per_buf = ntok * (2 * Np + cols + 2);
  const int r = blockIdx.z, h = blockIdx.y, g = h / (s.H / s.G);
  const int n = req_len[r];
  if (n <= 0) return;
  const int t0 = req_start[r];
  float* slot = state + (size_t)req_slot[r] * s.state_stride;
  if (blockIdx.x == 0) {                            // each head keeps a share of the inputs
    const int C = ssm_channels(s);
    ssm_keep_inputs(slot + (size_t)s.H * s.N * s.V, proj, s, t0, n, tok_pos[t0],
                    (int)((long long)C * h / s.H), (int)((long long)C * (h + 1) / s.H));
  }
  const int part = threadIdx.x % P, col = threadIdx.x / P;
  const int v0 = blockIdx.x * cols, v = v0 + col;
  const bool ok = v < s.V;
  const float dh = skip[h];
  float* S = slot + (size_t)h * s.N * s.V;
  float st[SR_ROWS];
#pragma unroll
  for (int i = 0; i < SR_ROWS; ++i) {
    const int d = part * SR_ROWS + i;
    st[i] = (ok && d < s.N) ? S[(size_t)d * s.V + v] : 0.f;
  }
  if (s.N != P * SR_ROWS || s.V % cols) {           // rows or columns past the sizes read as zero
    for (int e = threadIdx.x; e < 2 * per_buf; e += SR_THREADS) smem[e] = 0.f;
    __syncthreads();
  }
  sr_stage(smem, rows, step, t0, min(ntok, n), s, h, g, Np, cols, v0, ntok, vec);
  int buf = 0;
  const size_t yw = (size_t)s.H * s.V;
  for (int base = 0; base < n; base += ntok, buf ^= 1) {
    const int here = min(ntok, n - base);
    if (base + ntok < n) {
      sr_stage(smem + (buf ^ 1) * per_buf, rows, step, t0 + base + ntok, min(ntok, n - base - ntok), s,
               h, g, Np, cols, v0, ntok, vec);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* s_b = smem + buf * per_buf;
    const float* s_c = s_b + ntok * Np;
    const float* s_x = s_c + ntok * Np;
    const float* s_d = s_x + ntok * cols;
    float* yo = y + (size_t)(t0 + base) * yw + (size_t)h * s.V + v;
    auto one = [&](int tt) {
      const float x = s_x[tt * cols + col];
      return sr_token(st, s_b + tt * Np + part * SR_PART, s_c + tt * Np + part * SR_PART,
                      x * s_d[2 * tt + 1], s_d[2 * tt]);
    };
    int tt = 0;
    for (; tt + 4 <= here; tt += 4) {               // four tokens: their sums and folds overlap
      float acc[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[q] = one(tt + q);
      for (int off = 1; off < P; off <<= 1) {
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[q] += __shfl_xor_sync(0xffffffffu, acc[q], off);
      }
      if (part == 0 && ok) {
#pragma unroll
        for (int q = 0; q < 4; ++q)
          yo[(size_t)(tt + q) * yw] = fmaf(dh, s_x[(tt + q) * cols + col], acc[q]);
      }
    }
    for (; tt < here; ++tt) {
      float acc = one(tt);
      for (int off = 1; off < P; off <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
      if (part == 0 && ok) yo[(size_t)tt * yw] = fmaf(dh, s_x[tt * cols + col], acc);
    }
    __syncthreads();                                // this buffer is staged into again next turn
  }
#pragma unroll
  for (int i = 0; i < SR_ROWS; ++i) {
    const int d = part * SR_ROWS + i;
    if (ok && d < s.N) S[(size_t)d * s.V + v] = st[i];
  }
}

// ---- single tokens ----------------------------------------------------------------------------
constexpr int SS_THREADS = 256;
constexpr int SS_COLS = 64;          // value columns of a block at most
constexpr int SS_BATCH = 8;          // state rows a thread has in flight

// A block per (token, head, 64 value columns).  PC: columns a thread owns (4, or 1 for sizes that are
// no whole 16-byte pieces); the threads of a column share its state rows.
template <int PC>
__global__ void __launch_bounds__(SS_THREADS)
ssm_step_kernel(float* __restrict__ y, float* __restrict__ state, const float* __restrict__ proj,
                const float* __restrict__ skip, const int* __restrict__ tok_req,
                const int* __restrict__ tok_pos, const int* __restrict__ req_slot,
                const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                const float* __restrict__ dt_bias, const float* __restrict__ a_log, SsmShape s) {
  extern __shared__ __align__(16) float s_row[];          // B [N] | C [N] | x [SS_COLS] | shares
  __shared__ float s_dt[2];
  pdl_trigger();
  const int t = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SS_COLS;
  const int r = tok_req[t];
  if (r < 0) return;
  const int cols = min(SS_COLS, s.V - v0);
  const int lanes = (cols + PC - 1) / PC, groups = SS_THREADS / lanes;
  const int lane = threadIdx.x % lanes, grp = threadIdx.x / lanes;
  const bool work = grp < groups;
  const int C = ssm_channels(s), N = s.N, g = h / (s.H / s.G);
  float* slot = state + (size_t)req_slot[r] * s.state_stride;
  float* S = slot + (size_t)h * N * s.V + v0 + lane * PC;
  float* s_b = s_row;
  float* s_c = s_b + N;
  float* s_x = s_c + N;
  float* s_y = s_x + SS_COLS;                             // [groups][lanes * PC]
  __align__(16) float st[SS_BATCH][PC];
  auto fetch = [&](int base) {
#pragma unroll
    for (int i = 0; i < SS_BATCH; ++i) {
      const int d = base + i * groups + grp;
      if (!work || d >= N) continue;
      if constexpr (PC == 4) *(float4*)st[i] = *(const float4*)(S + (size_t)d * s.V);
      else st[i][0] = S[(size_t)d * s.V];
    }
  };
  fetch(0);              // an earlier step's numbers: nothing of this step writes them but this block
  pdl_wait();
  const int pos = tok_pos[t];
  float* ring = slot + (size_t)s.H * N * s.V;
  const float* own = proj + (size_t)t * s.stride + s.x_off;
  // the block that keeps a channel's input for later tokens: x by its own, B and C by the first of
  // the group's heads
  const bool keeps = h % (s.H / s.G) == 0 && blockIdx.z == 0;
  for (int i = threadIdx.x; i < 2 * N + cols; i += SS_THREADS) {
    const int c = i < N ? s.H * s.V + g * N + i
                : i < 2 * N ? s.H * s.V + (s.G + g) * N + i - N : h * s.V + v0 + i - 2 * N;
    s_row[i] = ssm_conv(own + c, s.stride, ring, C, c, pos, 0, s.taps, conv_w, conv_b);
    if (i >= 2 * N || keeps) ring[(size_t)(pos % s.taps) * C + c] = own[c];
  }
  if (threadIdx.x == 0) {
    const float dt = ssm_softplus(own[C + h] + dt_bias[h]);
    s_dt[0] = dt;
    s_dt[1] = expf(-expf(a_log[h]) * dt);
  }
  __syncthreads();
  const float dt = s_dt[0], decay = s_dt[1];
  float xd[PC], acc[PC];
#pragma unroll
  for (int c = 0; c < PC; ++c) {
    xd[c] = work && lane * PC + c < cols ? s_x[lane * PC + c] * dt : 0.f;
    acc[c] = 0.f;
  }
  for (int base = 0; base < N; base += SS_BATCH * groups) {
    if (base > 0) fetch(base);
#pragma unroll
    for (int i = 0; i < SS_BATCH; ++i) {
      const int d = base + i * groups + grp;
      if (!work || d >= N) continue;
      const float b = s_b[d], cc = s_c[d];
#pragma unroll
      for (int c = 0; c < PC; ++c) {
        st[i][c] = fmaf(b, xd[c], decay * st[i][c]);
        acc[c] = fmaf(st[i][c], cc, acc[c]);
      }
      if constexpr (PC == 4) *(float4*)(S + (size_t)d * s.V) = *(const float4*)st[i];
      else S[(size_t)d * s.V] = st[i][0];
    }
  }
  if (work) {
#pragma unroll
    for (int c = 0; c < PC; ++c) s_y[(size_t)grp * lanes * PC + lane * PC + c] = acc[c];
  }
  __syncthreads();
  for (int c = threadIdx.x; c < cols; c += SS_THREADS) {
    float v = 0.f;
    for (int k = 0; k < groups; ++k) v += s_y[(size_t)k * lanes * PC + c];
    y[(size_t)t * s.H * s.V + (size_t)h * s.V + v0 + c] = fmaf(skip[h], s_x[c], v);
  }
}

static inline bool ssm_shape(SsmShape& s, int H, int G, int N, int V, int taps, int stride, int x_off,
                             int state_stride) {
  s = {H, G, N, V, taps, stride, x_off, state_stride};
  return H > 0 && G > 0 && H % G == 0 && N > 0 && V > 0 && taps > 0 && x_off >= 0 &&
         x_off + ssm_channels(s) + H <= stride && H * N * V + taps * ssm_channels(s) <= state_stride;
}

}  // namespace hs

// rows [n_tokens, channels] of rows_dtype, step [n_tokens, 2 H] float32; conv_w [taps, channels].
HS_EXPORT int hs_ssm_prepare(void* rows, float* step, const float* proj, const float* state,
                             const int* tok_req, const int* tok_pos, const int* req_start,
                             const int* req_slot, const float* conv_w, const float* conv_b,
                             const float* dt_bias, const float* a_log, int n_tokens, int H, int G,
                             int N, int V, int taps, int stride, int x_off, int state_stride,
                             int rows_dtype, void* stream) {
  using namespace hs;
  if (!rows || !step || !proj || !state || !tok_req || !tok_pos || !req_start || !req_slot ||
      !conv_w || !conv_b || !dt_bias || !a_log)
    return HS_ERR_ARGUMENT;
  SsmShape s;
  if (!ssm_shape(s, H, G, N, V, taps, stride, x_off, state_stride)) return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  const int C = ssm_channels(s);
  const bool vec = C % 4 == 0 && stride % 4 == 0 && x_off % 4 == 0 && state_stride % 4 == 0 &&
                   (H * N * V) % 4 == 0 &&
                   !(((uintptr_t)rows | (uintptr_t)proj | (uintptr_t)state | (uintptr_t)conv_w |
                      (uintptr_t)conv_b) & 15);
  const int per = vec ? 1024 : 256;
  const dim3 grid((n_tokens + SP_TOK - 1) / SP_TOK, (C + per - 1) / per + 1);
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e;
#define HS_SSM_P(VEC, TR)                                                                           \
  e = hs_launch(ssm_prepare_kernel<VEC, TR>, grid, dim3(256), 0, st, hs_pdl_enabled(), (TR*)rows, step, \
                proj, state, tok_req, tok_pos, req_start, req_slot, conv_w, conv_b, dt_bias, a_log, s, \
                n_tokens)
  if (rows_dtype == HS_DT_F32) { if (vec) HS_SSM_P(true, float); else HS_SSM_P(false, float); }
  else if (rows_dtype == HS_DT_BF16) { if (vec) HS_SSM_P(true, __nv_bfloat16); else HS_SSM_P(false, __nv_bfloat16); }
  else return HS_ERR_UNSUPPORTED;
#undef HS_SSM_P
  return e == cudaSuccess ? HS_OK : (int)e;
}

// y [tokens, H*V] float32; rows and step as ssm_prepare left them (rows float32).
HS_EXPORT int hs_ssm_recurrence(float* y, float* state, const float* rows, const float* step,
                                const float* proj, const float* skip, const int* tok_pos,
                                const int* req_start, const int* req_len, const int* req_slot,
                                int n_requests, int H, int G, int N, int V, int taps, int stride,
                                int x_off, int state_stride, void* stream) {
  using namespace hs;
  if (!y || !state || !rows || !step || !proj || !skip || !tok_pos || !req_start || !req_len ||
      !req_slot)
    return HS_ERR_ARGUMENT;
  SsmShape s;
  if (!ssm_shape(s, H, G, N, V, taps, stride, x_off, state_stride) || N > 32 * SR_ROWS)
    return HS_ERR_UNSUPPORTED;
  if (n_requests <= 0) return HS_OK;
  if (n_requests > 65535 || H > 65535) return HS_ERR_TOO_LARGE;
  int P = 1;
  while (P * SR_ROWS < N) P *= 2;
  const int cols = SR_THREADS / P, ntok = P <= 8 ? SR_TOK : P == 16 ? SR_TOK / 2 : SR_TOK / 4;
  const int vec = N % 4 == 0 && V % 4 == 0 && cols % 4 == 0 && !((uintptr_t)rows & 15) ? 1 : 0;
  const size_t smem = (size_t)2 * ntok * (2 * P * SR_PART + cols + 2) * sizeof(float);
  if (smem > 48 * 1024) return HS_ERR_UNSUPPORTED;
  cudaError_t e = hs_launch(ssm_recurrence_kernel, dim3((V + cols - 1) / cols, H, n_requests),
                            dim3(SR_THREADS), smem, (cudaStream_t)stream, hs_pdl_enabled(), y, state,
                            rows, step, proj, skip, tok_pos, req_start, req_len, req_slot, s, P, ntok,
                            vec);
  return e == cudaSuccess ? HS_OK : (int)e;
}

// Every request of the step brings one token: tokens are told apart by tok_req alone.
HS_EXPORT int hs_ssm_step(float* y, float* state, const float* proj, const float* skip,
                          const int* tok_req, const int* tok_pos, const int* req_slot,
                          const float* conv_w, const float* conv_b, const float* dt_bias,
                          const float* a_log, int n_tokens, int H, int G, int N, int V, int taps,
                          int stride, int x_off, int state_stride, void* stream) {
  using namespace hs;
  if (!y || !state || !proj || !skip || !tok_req || !tok_pos || !req_slot || !conv_w || !conv_b ||
      !dt_bias || !a_log)
    return HS_ERR_ARGUMENT;
  SsmShape s;
  if (!ssm_shape(s, H, G, N, V, taps, stride, x_off, state_stride)) return HS_ERR_UNSUPPORTED;
  const size_t smem = (size_t)(2 * N + SS_COLS + SS_THREADS * 4) * sizeof(float);
  if (smem > 47 * 1024) return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  if (H > 65535) return HS_ERR_TOO_LARGE;
  const bool vec = V % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
  const dim3 grid(n_tokens, H, (V + SS_COLS - 1) / SS_COLS);
  cudaStream_t st = (cudaStream_t)stream;
  const cudaError_t e =
      vec ? hs_launch(ssm_step_kernel<4>, grid, dim3(SS_THREADS), smem, st, hs_pdl_enabled(), y, state,
                      proj, skip, tok_req, tok_pos, req_slot, conv_w, conv_b, dt_bias, a_log, s)
          : hs_launch(ssm_step_kernel<1>, grid, dim3(SS_THREADS), smem, st, hs_pdl_enabled(), y, state,
                      proj, skip, tok_req, tok_pos, req_slot, conv_w, conv_b, dt_bias, a_log, s);
  return e == cudaSuccess ? HS_OK : (int)e;
}
