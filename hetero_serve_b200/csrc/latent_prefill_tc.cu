// Attention over a shared latent for prompt portions, with or without a window, on tcgen05 tensor
// cores (sm_100a), bfloat16 operands, float32 accumulators.  Same mathematics as latent_attention.cu,
// in the form that costs prompts least: keys and values are EXPANDED per head, once for every
// position the step's portions can see, instead of absorbing the expansions into the queries (a query
// and key meet in dim + rot_dim and vdim numbers here, in 2 * kv_rank + rot_dim there).
//
//   gather   the rows [latent | turned key part] of the positions a portion sees are brought from
//            their pages into a dense block (latents and key parts apart), and the portion's
//            queries are turned, rounded and padded to whole 64-number chunks, in one launch;
//   (linear  the dense latents times [W_uk; W_uv], the framework's own product)
//   attend   S = [q | q_rot] [k | k_rot]^T,  softmax over what is visible,  O = P V, optionally times
//            the sigmoid of gate columns.
//
// Dense rows: position p of request r lies in row base[r] + p.  A portion of n tokens from position
// s sees positions lo = max(0, s - window + 1) .. s + n - 1; with k requests that bring portions
// before r, its rows start at req_start[r] + k * (window - 1).  Without a window (0) it sees all
// positions 0 .. s + n - 1 and its rows follow those of the portions before r.  Rows nobody wrote
// hold zeros or an earlier step's numbers: finite, and always masked.
//
// The second and third step serve attention over keys and values of the cache itself as well
// (span_gather brings [all keys | all values] of a position into one dense row): query heads that
// share a key/value head, no turned part, capped scores, a sink in the denominator.
//
// A block works on up to 128 consecutive queries of one request x one head, 128 keys a tile:
//   warp 0      TMA producer: the queries once; per tile the key chunks of 64 numbers (the head's
//               columns of the expanded rows, then the shared turned part) into two stages, the
//               value chunks into one;
//   warp 1      one thread issues S = Q K^T into one of two TMEM buffers (S of the next tile while
//               the softmax of this one runs) and O_tile = P V (values N-contiguous);
//   warps 2..9  softmax, two threads a query row (a half of the tile's keys each, the maxima
//               exchanged through shared memory); P goes to shared memory as bfloat16 in the
//               swizzled operand layout, O_tile is added into float32 registers.
// Head sizes that are no multiple of 64 are padded: a key chunk then reads on into the next
// columns, which the padded queries' zeros cancel; surplus output columns are not stored.
//
// Every mbarrier wait is bounded (tcgen05.cuh); on a time-out the status word is set, the block
// leaves its loops, frees its TMEM and returns.
#include "rotary.cuh"
#include "tcgen05.cuh"

namespace hs {

constexpr int LP_BQ = 128, LP_BKV = 128;
constexpr int LP_THREADS = 320, LP_SOFTMAX_WARPS = 8;
constexpr int LP_CHUNK = 128 * 64 * 2;                 // 128 rows of 64 numbers: 16 KB
constexpr int LP_GATHER_BLOCKS = 48;                   // blocks that share a request's rows

// ---- gather --------------------------------------------------------------------------------
// blocks 0 .. n_requests * LP_GATHER_BLOCKS - 1: the dense rows; then one block a token: queries
template <int THREADS>
__global__ void __launch_bounds__(THREADS)
latent_gather_kernel(__nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rope,
                     __nv_bfloat16* __restrict__ q_out, int* __restrict__ base,
                     const float* __restrict__ q, const __nv_bfloat16* __restrict__ pool,
                     const int* __restrict__ table, const int* __restrict__ req_start,
                     const int* __restrict__ req_len, const int* __restrict__ tok_pos,
                     const int* __restrict__ tok_req, int n_requests, int n_tokens, int cap_rows,
                     int window, int max_single, int R, int P, int n_heads, int D, int q_pad_d,
                     int q_stride, int page_size, int num_pages, int max_pages,
                     const float* __restrict__ freq, int rot_dims, int* status) {
  pdl_trigger();
  pdl_wait();
  const int n_gather = n_requests * LP_GATHER_BLOCKS;
  if ((int)blockIdx.x < n_gather) {
    const int r = blockIdx.x / LP_GATHER_BLOCKS, part = blockIdx.x - r * LP_GATHER_BLOCKS;
    const int n = req_len[r];
    if (n <= max_single) {
      if (part == 0 && threadIdx.x == 0) base[r] = -1;
      return;
    }
    const int pos0 = tok_pos[req_start[r]];
    int lo = 0, row0 = 0;
    if (window > 0) {
      int before = 0;
      for (int i = 0; i < r; ++i) before += req_len[i] > max_single;
      lo = max(0, pos0 + 1 - window);
      row0 = req_start[r] + before * (window - 1);
    } else {
      for (int i = 0; i < r; ++i)
        if (req_len[i] > max_single) row0 += tok_pos[req_start[i]] + req_len[i];
    }
    const int rows = pos0 + n - lo;
    if (part == 0 && threadIdx.x == 0) base[r] = row0 - lo;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int W = R + P;
    const bool vec = (R & 7) == 0 && (P & 7) == 0;
    for (int i = part * (THREADS / 32) + warp; i < rows; i += LP_GATHER_BLOCKS * (THREADS / 32)) {
      const int row = row0 + i, p = lo + i, pi = p / page_size;
      if (row >= cap_rows) break;                       // the caller's blocks are too small
      const int page = pi < max_pages ? table[(size_t)r * max_pages + pi] : -1;
      if (page < 0 || page >= num_pages) {
        if (lane == 0) atomicOr(status, HS_STATUS_BAD_PAGE);
        continue;
      }
      const __nv_bfloat16* src = pool + ((size_t)page * page_size + (p - pi * page_size)) * W;
      __nv_bfloat16* dl = lat + (size_t)row * R;
      __nv_bfloat16* dr = rope + (size_t)row * 64;
      if (vec) {
        for (int e = lane * 8; e < R; e += 256) *(uint4*)(dl + e) = *(const uint4*)(src + e);
        if (lane < 8)
          *(uint4*)(dr + lane * 8) = lane * 8 < P ? *(const uint4*)(src + R + lane * 8)
                                                  : make_uint4(0, 0, 0, 0);
      } else {
        for (int e = lane; e < R; e += 32) dl[e] = src[e];
        for (int e = lane; e < 64; e += 32) dr[e] = e < P ? src[R + e] : __float2bfloat16_rn(0.f);
      }
    }
    return;
  }
  const int t = blockIdx.x - n_gather;
  const int r = tok_req[t];
  if (r < 0 || req_len[r] <= max_single) return;
  const int pos = tok_pos[t];
  __shared__ float2 s_cs[32];                            // cosine and sine of a turned pair
  if ((int)threadIdx.x < rot_dims / 2)
    pair_angle(pos, freq[threadIdx.x], &s_cs[threadIdx.x].x, &s_cs[threadIdx.x].y);
  __syncthreads();
  const int qw = q_pad_d + 64;                           // padded numbers a head
  const float* src = q + (size_t)t * q_stride;
  __nv_bfloat16* dst = q_out + (size_t)t * n_heads * qw;
  for (int i = threadIdx.x; i < n_heads * qw / 2; i += THREADS) {
    const int h = 2 * i / qw, e = 2 * i - h * qw;        // a pair of neighbours
    const float* s = src + (size_t)h * (D + P);
    float x = 0.f, y = 0.f;
    if (e < D) {                                         // D is even
      x = s[e];
      y = s[e + 1];
    } else if (e >= q_pad_d && e - q_pad_d < P) {
      const int k = e - q_pad_d;
      x = s[D + k];
      y = k + 1 < P ? s[D + k + 1] : 0.f;
      if (k < rot_dims) {
        const float2 cs = s_cs[k >> 1];
        const float a = x * cs.x - y * cs.y;
        y = y * cs.x + x * cs.y;
        x = a;
      }
    }
    *(__nv_bfloat162*)(dst + 2 * i) = __floats2bfloat162_rn(x, y);
  }
}

// The same for a cache of keys and values: dense rows [G keys of D | G values of V], queries padded.
__global__ void __launch_bounds__(256)
span_gather_kernel(__nv_bfloat16* __restrict__ kv, __nv_bfloat16* __restrict__ q_out,
                   int* __restrict__ base, const float* __restrict__ q,
                   const __nv_bfloat16* __restrict__ pool, const int* __restrict__ table,
                   const int* __restrict__ req_start, const int* __restrict__ req_len,
                   const int* __restrict__ tok_pos, const int* __restrict__ tok_req, int n_requests,
                   int cap_rows, int window, int max_single, int H, int G, int D, int V, int q_pad_d,
                   int page_size, int num_pages, int max_pages, int* status) {
  pdl_trigger();
  pdl_wait();
  const int n_gather = n_requests * LP_GATHER_BLOCKS;
  if ((int)blockIdx.x < n_gather) {
    const int r = blockIdx.x / LP_GATHER_BLOCKS, part = blockIdx.x - r * LP_GATHER_BLOCKS;
    const int n = req_len[r];
    if (n <= max_single) {
      if (part == 0 && threadIdx.x == 0) base[r] = -1;
      return;
    }
    const int pos0 = tok_pos[req_start[r]];
    int lo = 0, row0 = 0;
    if (window > 0) {
      int before = 0;
      for (int i = 0; i < r; ++i) before += req_len[i] > max_single;
      lo = max(0, pos0 + 1 - window);
      row0 = req_start[r] + before * (window - 1);
    } else {
      for (int i = 0; i < r; ++i)
        if (req_len[i] > max_single) row0 += tok_pos[req_start[i]] + req_len[i];
    }
    const int rows = pos0 + n - lo;
    if (part == 0 && threadIdx.x == 0) base[r] = row0 - lo;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int W = D + V, wq = W / 8, pieces = G * wq;
    for (int i = part * 8 + warp; i < rows; i += LP_GATHER_BLOCKS * 8) {
      const int row = row0 + i, p = lo + i, pi = p / page_size;
      if (row >= cap_rows) break;                         // the caller's block is too small
      const int page = pi < max_pages ? table[(size_t)r * max_pages + pi] : -1;
      if (page < 0 || page >= num_pages) {
        if (lane == 0) atomicOr(status, HS_STATUS_BAD_PAGE);
        continue;
      }
      const __nv_bfloat16* src =
          pool + ((size_t)page * G * page_size + (p - pi * page_size)) * (size_t)W;
      __nv_bfloat16* dst = kv + (size_t)row * G * W;
      for (int c = lane; c < pieces; c += 32) {
        const int g = c / wq, e = (c - g * wq) * 8;
        *(uint4*)(dst + (e < D ? g * D + e : G * D + g * V + e - D)) =
            *(const uint4*)(src + (size_t)g * page_size * W + e);
      }
    }
    return;
  }
  const int t = blockIdx.x - n_gather;
  const int r = tok_req[t];
  if (r < 0 || req_len[r] <= max_single) return;
  const float* src = q + (size_t)t * H * D;
  __nv_bfloat16* dst = q_out + (size_t)t * H * q_pad_d;
  for (int i = 4 * threadIdx.x; i < H * q_pad_d; i += 4 * 256) {
    const int h = i / q_pad_d, e = i - h * q_pad_d;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e < D) v = *(const float4*)(src + (size_t)h * D + e);       // D is a multiple of 8
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *(uint2*)(dst + i) = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
  }
}

// ---- attend --------------------------------------------------------------------------------
struct LatentTcParams {
  __nv_bfloat16* out;             // [tokens, heads * V]
  const int* plan;
  const int* base;
  int* status;
  int tiles_off, n_heads, D, V, window, cap_rows;     // window: huge when there is none
  float scale, softcap;           // softcap 0: none
  int kv_group, v_col;            // query heads of a key/value head; column of the first value
  const float* sinks;             // [n_heads] or null
  const float* gate;              // [tokens, gate_stride] or null: column gate_off + h * V + e
  int gate_stride, gate_off;
};

enum { LB_Q = 0, LB_K_FULL = 1, LB_K_EMPTY = 3, LB_V_FULL = 5, LB_V_EMPTY = 6, LB_S_FULL = 7,
       LB_S_EMPTY = 9, LB_P_FULL = 11, LB_PV_DONE = 12, LB_O_EMPTY = 13, LB_COUNT = 14 };

// the fast exponential of the other tcgen05 attention: 2^x
__device__ __forceinline__ float lp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// cap * tanh(s / cap) = cap * (1 - 2 / (1 + e^(2 s / cap))), the exponent as z * in
__device__ __forceinline__ float lp_cap(float z, float in, float cap) {
  return cap * (1.0f - __fdividef(2.0f, 1.0f + lp_ex2(z * in)));
}
// values, N-contiguous, more than one 64-number chunk wide: the chunks lie 16 KB apart
__device__ __forceinline__ uint64_t lp_value_desc(uint32_t saddr) {
  uint64_t d = make_smem_desc(saddr);
  d &= ~((uint64_t)0x3FFFu << 16);
  d |= (uint64_t)(LP_CHUNK >> 4) << 16;                 // leading byte offset: between chunks
  return d;
}

// NK: key chunks of 64 numbers (with TURNED, the shared turned part is the last); NV: value chunks
template <int NK, int NV, bool TURNED>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                         const __grid_constant__ CUtensorMap map_kv,
                         const __grid_constant__ CUtensorMap map_rope, const LatentTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;                                    // [NK][128 queries][128 B]
  uint8_t* sK = sQ + NK * LP_CHUNK;                      // [2 stages][NK][128 keys][128 B]
  uint8_t* sV = sK + 2 * NK * LP_CHUNK;                  // [NV][128 keys][128 B]
  uint8_t* sP = sV + NV * LP_CHUNK;                      // [2 k-blocks][128 rows][128 B]
  uint64_t* bars = (uint64_t*)(sP + 2 * LP_CHUNK);
  uint32_t* tmem_slot = (uint32_t*)(bars + LB_COUNT);
  __shared__ float s_max2[2][2][LP_BQ];                  // [tile parity][half][row]
  __shared__ float s_l[2][LP_BQ];

  if ((int)blockIdx.y >= p.plan[1]) return;
  const int4 ti = *(const int4*)(p.plan + p.tiles_off + 4 * blockIdx.y);
  const int tok0 = ti.x, nq = ti.y, r = ti.z, pos0 = ti.w;
  const int h = blockIdx.x, hk = h / p.kv_group;
  if (r < 0 || nq <= 0 || nq > LP_BQ || pos0 < 0) return;
  const int pos_last = pos0 + nq - 1;
  const int lo = max(0, pos0 + 1 - p.window);            // the oldest position a query here sees
  const int n_kv = (pos_last - lo) / LP_BKV + 1;
  const int row_lo = p.base[r] + lo;
  if (row_lo < 0 || row_lo + (pos_last - lo) >= p.cap_rows) {
    if (threadIdx.x == 0) atomicOr(p.status, HS_STATUS_BAD_POSITION);
    return;
  }

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr uint32_t S_COLS = LP_BKV, O_COL = 2 * S_COLS, TMEM_COLS = 512;
  if (threadIdx.x == 0) {
    for (int i = 0; i < LB_COUNT; ++i) {
      const bool many = i == LB_S_EMPTY || i == LB_S_EMPTY + 1 || i == LB_P_FULL || i == LB_O_EMPTY;
      mbar_init(&bars[i], many ? LP_SOFTMAX_WARPS : 1);
    }
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  // This kernel is launched without the programmatic attribute and lets the next one start only
  // now that every block has its tensor memory: a block that waits for tensor memory held by a
  // later kernel's block, which waits for this kernel, would wait for ever.
  pdl_trigger();
  bool ok = true;

  if (warp == 0) {
    if (lane == 0) {
      auto load_k = [&](int kt) -> bool {
        const int st = kt & 1, y = row_lo + kt * LP_BKV;
        if (kt >= 2 && !mbar_wait(&bars[LB_K_EMPTY + st], ((kt >> 1) - 1) & 1, p.status))
          return false;
        mbar_expect_tx(&bars[LB_K_FULL + st], NK * LP_CHUNK);
        uint8_t* dk = sK + st * NK * LP_CHUNK;
#pragma unroll
        for (int c = 0; c < (TURNED ? NK - 1 : NK); ++c)
          tma_load_2d(dk + c * LP_CHUNK, &map_kv, &bars[LB_K_FULL + st], hk * p.D + c * 64, y);
        if (TURNED) tma_load_2d(dk + (NK - 1) * LP_CHUNK, &map_rope, &bars[LB_K_FULL + st], 0, y);
        return true;
      };
      mbar_expect_tx(&bars[LB_Q], NK * LP_CHUNK);
#pragma unroll
      for (int c = 0; c < NK; ++c)
        tma_load_2d(sQ + c * LP_CHUNK, &map_q, &bars[LB_Q], (h * NK + c) * 64, tok0);
      ok = load_k(0);
      for (int kt = 0; kt < n_kv && ok; ++kt) {
        const int y = row_lo + kt * LP_BKV;
        if (kt + 1 < n_kv) ok = load_k(kt + 1);          // ahead of this tile's values
        if (!ok) break;
        if (kt >= 1) ok = mbar_wait(&bars[LB_V_EMPTY], (kt - 1) & 1, p.status);
        if (!ok) break;
        mbar_expect_tx(&bars[LB_V_FULL], NV * LP_CHUNK);
#pragma unroll
        for (int c = 0; c < NV; ++c)
          tma_load_2d(sV + c * LP_CHUNK, &map_kv, &bars[LB_V_FULL],
                      p.v_col + hk * p.V + c * 64, y);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(LP_BQ, LP_BKV, false);
      constexpr uint32_t idesc_o = make_idesc(LP_BQ, NV * 64, true);
      ok = mbar_wait(&bars[LB_Q], 0, p.status);
      auto issue_s = [&](int kt) -> bool {
        const int st = kt & 1;
        if (!mbar_wait(&bars[LB_K_FULL + st], (kt >> 1) & 1, p.status)) return false;
        if (kt >= 2 && !mbar_wait(&bars[LB_S_EMPTY + st], ((kt >> 1) - 1) & 1, p.status))
          return false;
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < NK; ++c) {
          const uint64_t qd = make_smem_desc(smem_u32(sQ + c * LP_CHUNK));
          const uint64_t kd = make_smem_desc(smem_u32(sK + (st * NK + c) * LP_CHUNK));
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16(tmem_base + st * S_COLS, qd + (uint64_t)(k * 2), kd + (uint64_t)(k * 2),
                      idesc_s, c + k > 0 ? 1u : 0u);
        }
        umma_commit(&bars[LB_S_FULL + st]);
        umma_commit(&bars[LB_K_EMPTY + st]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int kt = 0; kt < n_kv && ok; ++kt) {
        if (kt + 1 < n_kv) ok = issue_s(kt + 1);         // overlaps the softmax of tile kt
        if (ok) ok = mbar_wait(&bars[LB_P_FULL], kt & 1, p.status);
        if (ok) ok = mbar_wait(&bars[LB_V_FULL], kt & 1, p.status);
        if (ok && kt >= 1) ok = mbar_wait(&bars[LB_O_EMPTY], (kt - 1) & 1, p.status);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < LP_BKV / 16; ++k) {
          const uint64_t pd =
              make_smem_desc(smem_u32(sP) + (k >> 2) * LP_CHUNK) + (uint64_t)((k & 3) * 2);
          const uint64_t vd = lp_value_desc(smem_u32(sV) + k * 2048);
          umma_bf16(tmem_base + O_COL, pd, vd, idesc_o, k > 0 ? 1u : 0u);
        }
        umma_commit(&bars[LB_PV_DONE]);
        umma_commit(&bars[LB_V_EMPTY]);
      }
    }
  } else {
    const int qtr = warp & 3;                              // TMEM lane quarter of this warp
    const int half = (warp - 2) >> 2;                      // keys 0..63 or 64..127 of a tile
    const int row = qtr * 32 + lane;
    const int pos_r = min(pos0 + row, pos_last);           // rows past nq: finite, never stored
    const uint32_t lane_addr = tmem_base + ((uint32_t)(qtr * 32) << 16);
    const bool capped = p.softcap > 0.f;
    const float to2 = p.scale * 1.4426950408889634f;       // a score in units of log2(e)
    const float sl2 = capped ? 1.0f : to2;                 // capped scores are in those units already
    const float cap2 = p.softcap * 1.4426950408889634f;
    const float cap_in = capped ? 2.0f * to2 / p.softcap : 0.f;      // 2 log2(e) scale / cap
    float m = -INFINITY, l = 0.f, corr_pending = 1.f;
    constexpr int OC = NV * 32;                            // output columns of this thread
    float o[OC];
#pragma unroll
    for (int d = 0; d < OC; ++d) o[d] = 0.f;

    auto accumulate_o = [&](int kt) -> bool {              // O_tile of tile kt
      if (!mbar_wait(&bars[LB_PV_DONE], kt & 1, p.status)) return false;
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < NV; ++c) {
        uint32_t v[32];
        tmem_ld32(lane_addr + O_COL + half * OC + c * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j)
          o[c * 32 + j] = fmaf(o[c * 32 + j], corr_pending, __uint_as_float(v[j]));
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[LB_O_EMPTY]);
      return true;
    };

    for (int kt = 0; kt < n_kv && ok; ++kt) {
      const int sb = kt & 1;
      ok = mbar_wait(&bars[LB_S_FULL + sb], (kt >> 1) & 1, p.status);
      if (!ok) break;
      tc_fence_after();
      const int t_lo = lo + kt * LP_BKV;                   // the tile's first position
      const int j0 = t_lo + half * 64;                     // this thread's first position
      const int vis_hi = pos_r - j0, vis_lo = pos_r - p.window + 1 - j0;   // visible: lo .. hi
      const bool edge = t_lo + LP_BKV - 1 > pos0 || t_lo < pos_last - p.window + 1;
      const uint32_t s_addr = lane_addr + sb * S_COLS + half * 64;
      uint32_t va[32], vb[32];
      tmem_ld32(s_addr, va);
      tmem_ld32(s_addr + 32, vb);
      tmem_ld_wait();
      if (capped) {                                        // cap * tanh(s / cap)
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          va[j] = __float_as_uint(lp_cap(__uint_as_float(va[j]), cap_in, cap2));
          vb[j] = __float_as_uint(lp_cap(__uint_as_float(vb[j]), cap_in, cap2));
        }
      }
      if (edge) {
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          if (j > vis_hi || j < vis_lo) va[j] = 0xff800000u;            // -infinity
          if (j + 32 > vis_hi || j + 32 < vis_lo) vb[j] = 0xff800000u;
        }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < 32; ++j)
        mx4[j & 3] = fmaxf(mx4[j & 3], fmaxf(__uint_as_float(va[j]), __uint_as_float(vb[j])));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      s_max2[kt & 1][half][row] = mx;
      asm volatile("bar.sync %0, 64;" ::"r"(1 + qtr) : "memory");   // the two warps of the quarter
      mx = fmaxf(mx, s_max2[kt & 1][half ^ 1][row]);
      const float m_new = fmaxf(m, mx * sl2);
      const float corr = (m_new == -INFINITY) ? 1.f : lp_ex2(m - m_new);
      const float base = (m_new == -INFINITY) ? 0.f : m_new;
      uint32_t pk[32];
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 32; j += 2) {                    // a masked score gives 2^-inf = 0
        const float e0 = lp_ex2(fmaf(__uint_as_float(va[j]), sl2, -base));
        const float e1 = lp_ex2(fmaf(__uint_as_float(va[j + 1]), sl2, -base));
        sum += e0 + e1;
        const __nv_bfloat162 b2 = __floats2bfloat162_rn(e0, e1);
        pk[j >> 1] = *(const uint32_t*)&b2;
      }
#pragma unroll
      for (int j = 0; j < 32; j += 2) {
        const float e0 = lp_ex2(fmaf(__uint_as_float(vb[j]), sl2, -base));
        const float e1 = lp_ex2(fmaf(__uint_as_float(vb[j + 1]), sl2, -base));
        sum += e0 + e1;
        const __nv_bfloat162 b2 = __floats2bfloat162_rn(e0, e1);
        pk[16 + (j >> 1)] = *(const uint32_t*)&b2;
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[LB_S_EMPTY + sb]);  // S[sb] may be overwritten
      l = l * corr + sum;
      m = m_new;
      if (kt >= 1) {                       // the tile before: its P V is done (P is free)
        ok = accumulate_o(kt - 1);
        if (!ok) break;
      }
      corr_pending = corr;
      // this half row of P: k-block `half`, chunk c of 8 keys at
      //   half * 16 KB + (row / 8) * 1 KB + (row % 8) * 128 B + ((c ^ (row % 8)) * 16 B)
      uint8_t* prow = sP + half * LP_CHUNK + (row >> 3) * 1024 + (row & 7) * 128;
#pragma unroll
      for (int c = 0; c < 8; ++c)
        *(uint4*)(prow + ((c ^ (row & 7)) << 4)) =
            make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[LB_P_FULL]);
    }
    if (ok) ok = accumulate_o(n_kv - 1);
    s_l[half][row] = l;
    asm volatile("bar.sync %0, 64;" ::"r"(1 + qtr) : "memory");
    float l_all = l + s_l[half ^ 1][row], keep = 1.f;
    if (p.sinks) {
      const float sk = p.sinks[h] * 1.4426950408889634f, top = fmaxf(m, sk);
      keep = lp_ex2(m - top);
      l_all = l_all * keep + lp_ex2(sk - top);
    }
    if (ok && row < nq) {
      const float inv = l_all > 0.f ? keep / l_all : 0.f;
      __nv_bfloat16* orow = p.out + ((size_t)(tok0 + row) * p.n_heads + h) * p.V;
      const float* grow = p.gate ? p.gate + (size_t)(tok0 + row) * p.gate_stride + p.gate_off +
                                       (size_t)h * p.V + half * OC
                                 : nullptr;
      // this thread's columns are half * OC .. + OC - 1; V is a multiple of 8
#pragma unroll
      for (int c = 0; c < OC; c += 8) {
        if (half * OC + c >= p.V) continue;
        uint32_t u[4];
        float w[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
          w[i] = grow ? __fdividef(inv, 1.0f + __expf(-grow[c + i])) : inv;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const __nv_bfloat162 b2 =
              __floats2bfloat162_rn(o[c + 2 * i] * w[2 * i], o[c + 2 * i + 1] * w[2 * i + 1]);
          u[i] = *(const uint32_t*)&b2;
        }
        *(uint4*)(orow + half * OC + c) = make_uint4(u[0], u[1], u[2], u[3]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

typedef CUresult (*EncodeTiledFnL)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*,
                                   const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                   const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// [rows, cols] bfloat16, contiguous rows, boxes of 128 rows x 64 columns, 128-byte swizzle
static int lp_map(CUtensorMap* map, const void* base, long long rows, long long cols) {
  static EncodeTiledFnL fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) !=
            cudaSuccess ||
        q != cudaDriverEntryPointSuccess)
      return HS_ERR_UNSUPPORTED;
    fn = (EncodeTiledFnL)ptr;
  }
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
  cuuint32_t box[2] = {64u, 128u};
  cuuint32_t elem[2] = {1, 1};
  CUresult e = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides,
                  box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return e == CUDA_SUCCESS ? HS_OK : HS_ERR_ARGUMENT;
}

}  // namespace hs

// Whether the expanded form takes these sizes: head parts in whole 16-byte pieces, keys of up to
// 128 + 64 numbers, values of up to 128.
HS_EXPORT int hs_latent_prefill_tc_takes(int D, int P, int V, int R, int window, float scale) {
  return D > 0 && D <= 128 && D % 8 == 0 && P > 0 && P <= 64 && V > 0 && V <= 128 && V % 8 == 0 &&
                 R > 0 && R % 8 == 0 && window >= 0 && scale > 0.f
             ? 1
             : 0;
}

// lat [cap_rows, R], rope [cap_rows, 64], q_out [n_tokens, n_heads * (pad64(D) + 64)], base
// [n_requests]; q [n_tokens, n_heads * (D + P)] float32, rows q_stride numbers apart.  Requests of up to max_single tokens are
// not gathered (their base is -1).
HS_EXPORT int hs_latent_gather(void* lat, void* rope, void* q_out, int* base, const float* q,
                               const void* pool, const int* table, const int* req_start,
                               const int* req_len, const int* tok_pos, const int* tok_req,
                               int n_requests, int n_tokens, int cap_rows, int window,
                               int max_single, int R, int P, int n_heads, int D, int q_stride,
                               int page_size,
                               int num_pages, int max_pages, const float* freq, int rot_dims,
                               int* status, void* stream) {
  if (!lat || !rope || !q_out || !base || !q || !pool || !table || !req_start || !req_len ||
      !tok_pos || !tok_req || !status)
    return HS_ERR_ARGUMENT;
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > P || (rot_dims && !freq)) return HS_ERR_ARGUMENT;
  if (window < 0 || R <= 0 || P <= 0 || P > 64 || D <= 0 || D % 2 || n_heads <= 0 ||
      page_size <= 0 || q_stride < n_heads * (D + P))
    return HS_ERR_UNSUPPORTED;
  if (n_requests <= 0 || n_tokens <= 0) return HS_OK;
  const int pad = (D + 63) / 64 * 64;
  cudaError_t e = hs_launch(
      hs::latent_gather_kernel<256>, dim3(n_requests * hs::LP_GATHER_BLOCKS + n_tokens), dim3(256), 0,
      (cudaStream_t)stream, hs_pdl_enabled(), (__nv_bfloat16*)lat, (__nv_bfloat16*)rope,
      (__nv_bfloat16*)q_out, base, q, (const __nv_bfloat16*)pool, table, req_start, req_len,
      tok_pos, tok_req, n_requests, n_tokens, cap_rows, window, max_single, R, P, n_heads, D, pad,
      q_stride, page_size, num_pages, max_pages, freq, rot_dims, status);
  return e == cudaSuccess ? HS_OK : (int)e;
}

// Whether prompt portions over a cache of keys and values take these sizes: keys of up to 192
// numbers, values of up to 128, in whole 16-byte pieces.
HS_EXPORT int hs_span_prefill_tc_takes(int H, int G, int D, int V, int window, float scale) {
  return H > 0 && G > 0 && H % G == 0 && D > 0 && D <= 192 && D % 8 == 0 && V > 0 && V <= 128 &&
                 V % 8 == 0 && window >= 0 && scale > 0.f
             ? 1
             : 0;
}

// kv [cap_rows, G * (D + V)], q_out [n_tokens, H * pad64(D)], base [n_requests]; q [n_tokens, H * D]
// float32; pool [pages][G][page_size][D + V].
HS_EXPORT int hs_span_gather(void* kv, void* q_out, int* base, const float* q, const void* pool,
                             const int* table, const int* req_start, const int* req_len,
                             const int* tok_pos, const int* tok_req, int n_requests, int n_tokens,
                             int cap_rows, int window, int max_single, int H, int G, int D, int V,
                             int page_size, int num_pages, int max_pages, int* status, void* stream) {
  if (!kv || !q_out || !base || !q || !pool || !table || !req_start || !req_len || !tok_pos ||
      !tok_req || !status)
    return HS_ERR_ARGUMENT;
  if (!hs_span_prefill_tc_takes(H, G, D, V, window, 1.f) || page_size <= 0 ||
      (((uintptr_t)kv | (uintptr_t)q_out | (uintptr_t)q | (uintptr_t)pool) & 15))
    return HS_ERR_UNSUPPORTED;
  if (n_requests <= 0 || n_tokens <= 0) return HS_OK;
  cudaError_t e = hs_launch(
      hs::span_gather_kernel, dim3(n_requests * hs::LP_GATHER_BLOCKS + n_tokens), dim3(256), 0,
      (cudaStream_t)stream, hs_pdl_enabled(), (__nv_bfloat16*)kv, (__nv_bfloat16*)q_out, base, q,
      (const __nv_bfloat16*)pool, table, req_start, req_len, tok_pos, tok_req, n_requests, cap_rows,
      window, max_single, H, G, D, V, (D + 63) / 64 * 64, page_size, num_pages, max_pages, status);
  return e == cudaSuccess ? HS_OK : (int)e;
}

// kv [cap_rows, n_heads * (D + V)]: the expanded keys of all heads, then the values, and rope
// [cap_rows, 64]; or (rope null) [cap_rows, kv_heads * (D + V)]: keys and values as span_gather left
// them.  softcap 0 and sinks null: none.
HS_EXPORT int hs_latent_prefill_tc(void* out, const void* q, const void* kv, const void* rope,
                                   const int* base, const int* plan, int tiles_off, int tile_cap,
                                   int n_tokens, int cap_rows, int n_heads, int D, int P, int V,
                                   int R, int window, float scale, const float* gate,
                                   int gate_stride, int gate_off, int kv_heads, float softcap,
                                   const float* sinks, int* status, void* stream) {
  using namespace hs;
  if (gate && (gate_off < 0 || gate_off + n_heads * V > gate_stride)) return HS_ERR_ARGUMENT;
  if (!out || !q || !kv || !base || !plan || !status || softcap < 0.f) return HS_ERR_ARGUMENT;
  if (n_heads <= 0 || kv_heads <= 0 || n_heads % kv_heads ||
      (rope ? kv_heads != n_heads || !hs_latent_prefill_tc_takes(D, P, V, R, window, scale)
            : !hs_span_prefill_tc_takes(n_heads, kv_heads, D, V, window, scale)))
    return HS_ERR_UNSUPPORTED;
  if (((uintptr_t)out | (uintptr_t)q | (uintptr_t)kv | (uintptr_t)rope) & 15) return HS_ERR_UNSUPPORTED;
  if (tile_cap <= 0 || n_tokens <= 0) return HS_OK;
  const int nk = (D + 63) / 64 + (rope ? 1 : 0), nv = (V + 63) / 64;
  CUtensorMap mq, mkv, mr;
  if (int e = lp_map(&mq, q, n_tokens, (long long)n_heads * nk * 64)) return e;
  if (int e = lp_map(&mkv, kv, cap_rows, (long long)kv_heads * (D + V))) return e;
  if (int e = rope ? lp_map(&mr, rope, cap_rows, 64) : HS_OK) return e;
  if (!rope) mr = mkv;                                   // never used
  LatentTcParams p;
  p.out = (__nv_bfloat16*)out; p.plan = plan; p.base = base; p.status = status;
  p.tiles_off = tiles_off; p.n_heads = n_heads; p.D = D; p.V = V;
  p.window = window > 0 ? window : 1 << 28;
  p.kv_group = n_heads / kv_heads; p.v_col = kv_heads * D; p.softcap = softcap; p.sinks = sinks;
  p.gate = gate; p.gate_stride = gate_stride; p.gate_off = gate_off;
  p.cap_rows = cap_rows; p.scale = scale;
  const dim3 grid(n_heads, tile_cap), block(LP_THREADS);
  cudaError_t e = cudaSuccess;
#define HS_LP(NK, NV, T)                                                                          \
  do {                                                                                            \
    auto kern = latent_prefill_tc_kernel<NK, NV, T>;                                              \
    /* more than half of an SM's shared memory: two of these never share an SM, since each       \
       allocates all of its tensor memory */                                                      \
    const size_t need = (size_t)(3 * NK + NV + 2) * LP_CHUNK + 256 + 1024;                        \
    const size_t smem = need > 120 * 1024 ? need : 120 * 1024;                                    \
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);       \
    if (e == cudaSuccess)                                                                         \
      e = hs_launch(kern, grid, block, smem, (cudaStream_t)stream, false, mq, mkv, mr, p);        \
  } while (0)
  if (rope) {
    if (nk == 2 && nv == 1) HS_LP(2, 1, true);
    else if (nk == 2) HS_LP(2, 2, true);
    else if (nv == 1) HS_LP(3, 1, true);
    else HS_LP(3, 2, true);
  } else {
    if (nk == 1 && nv == 1) HS_LP(1, 1, false);
    else if (nk == 1) HS_LP(1, 2, false);
    else if (nk == 2 && nv == 1) HS_LP(2, 1, false);
    else if (nk == 2) HS_LP(2, 2, false);
    else if (nv == 1) HS_LP(3, 1, false);
    else HS_LP(3, 2, false);
  }
#undef HS_LP
  return e == cudaSuccess ? HS_OK : (int)e;
}
