// Attention over a shared latent for the single-query tokens of a step, on the tensor cores
// (mma.sync m16n8k16, bfloat16 operands, float32 accumulators).  Same mathematics as
// latent_attention.cu: absorbed queries against rows [latent (R) | turned key part (P)] of the
// pages, every visible position (with a window the last `window` ones), an optional sink.
//
// All heads of a token read the same rows, so 16 heads are the 16 rows of one product: a block
// works on one token and up to 16 heads, 32 keys a tile in two cp.async stages.  A token's keys are
// shared out over a cluster of up to eight blocks; their shares (maximum, sum, weighted rows) stay
// in shared memory and are joined across the cluster, each block finishing a part of the output.
// The split depends on the token's position and the window alone.
// The rows are bfloat16 numbers already; a query enters as the sum of three bfloat16 terms (its
// rounding, the rounding of what is left, and again: a float32's whole mantissa) and a weight as the
// sum of two, so scores and weights keep what a float32 product keeps.
//   S = Q K^T       a warp per 8 keys of the tile
//   softmax         running maximum per head, joined over the four warps through shared memory
//   O += P V        V is the first R columns of the same rows; a warp owns every fourth 8 columns
#include "mma_tiles.cuh"
#include "rotary.cuh"
#include "tcgen05.cuh"

namespace hs {

constexpr int LD_KEYS = 32, LD_HEADS = 16, LD_THREADS = 128, LD_MAX_SHARE = 8;
constexpr int LD_Q_TERMS = 3, LD_P_TERMS = 2;

struct LatentDecodeParams {
  float* out;
  const float* qa;
  const float* qr;
  const __nv_bfloat16* pool;
  const int* table;
  const float* sink;              // null: none
  const int* plan;
  const float* freq;
  int* status;
  int n_heads, R, P, qr_stride, qr_hstride, qr_off, page_size, num_pages, max_pages, rot_dims, window;
  float scale;
};

__device__ __forceinline__ float4 ld_cluster_f4(uint32_t a) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];"
               : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ float2 ld_cluster_f2(uint32_t a) {
  float2 v;
  asm volatile("ld.shared::cluster.v2.f32 {%0,%1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
  return v;
}

// NTW: output tiles of 8 columns a warp keeps at most (R <= 32 * NTW)
template <int NTW>
__global__ void __launch_bounds__(LD_THREADS)
latent_decode_mma_kernel(const LatentDecodeParams p) {
  extern __shared__ __align__(16) uint8_t ld_smem[];
  __shared__ __align__(16) __nv_bfloat16 s_p[LD_P_TERMS][LD_HEADS][LD_KEYS + 8];
  __shared__ float s_mx[4][LD_HEADS], s_l[4][LD_HEADS];
  __shared__ __align__(8) float2 s_ml[LD_HEADS];          // this block's share: maximum, sum
  __shared__ float2 s_all[LD_MAX_SHARE][LD_HEADS];
  __shared__ float s_w[LD_MAX_SHARE][LD_HEADS];
  __shared__ float2 s_cs[256];                            // cosine and sine of a rotated pair
  pdl_trigger();
  pdl_wait();
  if ((int)blockIdx.x >= p.plan[0]) return;               // the whole cluster
  const int t = p.plan[4 + 3 * blockIdx.x], req = p.plan[5 + 3 * blockIdx.x];
  const int pos = p.plan[6 + 3 * blockIdx.x];
  const int R = p.R, P = p.P, W = R + P, H = p.n_heads;
  const int W32 = (W + 31) & ~31, WS = W32 + 8;
  __nv_bfloat16* sQ = (__nv_bfloat16*)ld_smem;            // [3 terms][16][WS]
  __nv_bfloat16* sK = sQ + LD_Q_TERMS * LD_HEADS * WS;                 // [2][32][WS]
  float* sO = (float*)sK;                                 // [16][R], once the tiles are done
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int h0 = blockIdx.y * LD_HEADS;
  const int share = gridDim.z, rank = blockIdx.z;         // the cluster spans z
  const int first = p.window > 0 ? max(0, pos + 1 - p.window) : 0;
  const int n_keys = pos + 1 - first;
  const int n_tiles = (n_keys + LD_KEYS - 1) / LD_KEYS;
  const int per = (n_tiles + share - 1) / share;
  const int lo = rank * per, hi = min(n_tiles, lo + per);

  // a warp brings eight rows of a tile: the first eight lanes look their pages up
  auto fetch = [&](int tile, int st) {
    long long at = -1;
    const int kk = tile * LD_KEYS + warp * 8 + (lane & 7);
    if (kk < n_keys) {
      const int kp = first + kk, pi = kp / p.page_size;
      const int page = pi < p.max_pages ? p.table[(size_t)req * p.max_pages + pi] : -1;
      if (page < 0 || page >= p.num_pages) atomicOr(p.status, HS_STATUS_BAD_PAGE);
      else at = ((long long)page * p.page_size + (kp - pi * p.page_size)) * W;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const long long row = __shfl_sync(0xffffffffu, at, j);
      __nv_bfloat16* dst = sK + (size_t)(st * LD_KEYS + warp * 8 + j) * WS;
      for (int c = lane * 8; c < W; c += 256) {
        if (row >= 0)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + c)),
                       "l"(p.pool + row + c));
        else
          *(uint4*)(dst + c) = make_uint4(0, 0, 0, 0);
      }
    }
    asm volatile("cp.async.commit_group;");
  };
  if (lo < hi) fetch(lo, 0);
  for (int i = threadIdx.x; i < 2 * LD_KEYS; i += LD_THREADS)       // columns past the rows
    for (int c = W; c < W32; ++c) sK[(size_t)i * WS + c] = __float2bfloat16_rn(0.f);
  for (int i = threadIdx.x; i < p.rot_dims / 2; i += LD_THREADS)
    pair_angle(pos, p.freq[i], &s_cs[i].x, &s_cs[i].y);
  __syncthreads();
  for (int hh = warp; hh < LD_HEADS; hh += 4) {
    const int head = h0 + hh;
    const bool live = head < H;
    const float* a = p.qa + ((size_t)t * H + head) * R;
    const float* b = p.qr + (size_t)t * p.qr_stride + (size_t)head * p.qr_hstride + p.qr_off;
#pragma unroll 4
    for (int d = 2 * lane; d < W32; d += 64) {
      float2 v = make_float2(0.f, 0.f);
      if (live && d < R) {
        v = *(const float2*)(a + d);
      } else if (live && d < W) {
        const int e = d - R;                              // R is even: a pair of the turned part
        const float x = b[e], y = e + 1 < P ? b[e + 1] : 0.f;
        if (e < p.rot_dims) {
          const float2 cs = s_cs[e >> 1];
          v = make_float2(x * cs.x - y * cs.y, y * cs.x + x * cs.y);
        } else {
          v = make_float2(x, y);
        }
      }
#pragma unroll
      for (int term = 0; term < LD_Q_TERMS; ++term) {
        const __nv_bfloat162 q2 = __floats2bfloat162_rn(v.x, v.y);
        *(__nv_bfloat162*)(sQ + (term * LD_HEADS + hh) * WS + d) = q2;
        v.x -= __bfloat162float(q2.x);                    // what this term leaves (exact)
        v.y -= __bfloat162float(q2.y);
      }
    }
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};     // rows g and g + 8
  float acc[NTW][4];
#pragma unroll
  for (int i = 0; i < NTW; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[i][c] = 0.f;
  const int nt_all = R >> 3;
  const __nv_bfloat16* qp = sQ + (lane & 15) * WS + (lane >> 4) * 8;
  for (int tile = lo; tile < hi; ++tile) {
    const int st = (tile - lo) & 1;
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                  // the tile is here (and the queries), the one before is used
    if (tile + 1 < hi) fetch(tile + 1, st ^ 1);
    const __nv_bfloat16* k = sK + (size_t)st * LD_KEYS * WS;
    const __nv_bfloat16* kp = k + (warp * 8 + (lane & 7)) * WS + (lane >> 3) * 8;
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
    for (int kk = 0; kk < W32; kk += 32) {
      uint32_t a0[4], a1[4], b[4];
      ldmatrix_x4(b, kp + kk);
#pragma unroll
      for (int term = LD_Q_TERMS - 1; term >= 0; --term) {            // the small terms first
        ldmatrix_x4(a0, qp + term * LD_HEADS * WS + kk);
        ldmatrix_x4(a1, qp + term * LD_HEADS * WS + kk + 16);
        mma_bf16(s, a0, b);
        mma_bf16(s2, a1, b + 2);
      }
    }
    const int key = tile * LD_KEYS + warp * 8 + 2 * tq;
#pragma unroll
    for (int c = 0; c < 4; ++c)
      s[c] = key + (c & 1) < n_keys ? (s[c] + s2[c]) * p.scale : -INFINITY;
    float mx[2] = {fmaxf(s[0], s[1]), fmaxf(s[2], s[3])};
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 1));
      mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 2));
      if (tq == 0) s_mx[warp][g + 8 * x] = mx[x];
    }
    __syncthreads();
    float corr[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int row = g + 8 * x;      // a tile has at least one visible key: the maximum is finite
      const float mn = fmaxf(m[x], fmaxf(fmaxf(s_mx[0][row], s_mx[1][row]),
                                         fmaxf(s_mx[2][row], s_mx[3][row])));
      corr[x] = expf(m[x] - mn);
      m[x] = mn;
      const float e0 = expf(s[2 * x] - mn), e1 = expf(s[2 * x + 1] - mn);
      l[x] = l[x] * corr[x] + (e0 + e1);
      const __nv_bfloat162 p0 = __floats2bfloat162_rn(e0, e1);
      *(__nv_bfloat162*)&s_p[0][row][warp * 8 + 2 * tq] = p0;
      *(__nv_bfloat162*)&s_p[1][row][warp * 8 + 2 * tq] =
          __floats2bfloat162_rn(e0 - __bfloat162float(p0.x), e1 - __bfloat162float(p0.y));
    }
    __syncthreads();
    uint32_t pa[LD_P_TERMS][2][4];
#pragma unroll
    for (int term = 0; term < LD_P_TERMS; ++term) {
      ldmatrix_x4(pa[term][0], &s_p[term][lane & 15][(lane >> 4) * 8]);
      ldmatrix_x4(pa[term][1], &s_p[term][lane & 15][16 + (lane >> 4) * 8]);
    }
    const uint32_t v_addr = smem_u32(k + lane * WS);
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      const int nt = warp + 4 * i;
      if (nt < nt_all) {
        acc[i][0] *= corr[0]; acc[i][1] *= corr[0];
        acc[i][2] *= corr[1]; acc[i][3] *= corr[1];
        uint32_t b[4];
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3])
                     : "r"(v_addr + (uint32_t)(nt * 16)));
#pragma unroll
        for (int term = LD_P_TERMS - 1; term >= 0; --term) {
          mma_bf16(acc[i], pa[term][0], b);
          mma_bf16(acc[i], pa[term][1], b + 2);
        }
      }
    }
  }
  // this block's share into shared memory
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
    if (tq == 0) s_l[warp][g + 8 * x] = l[x];
  }
  __syncthreads();                    // every warp is done with the tiles: sO may take their place
  if (warp == 0 && tq == 0)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int row = g + 8 * x;
      s_ml[row] = make_float2(m[x], (s_l[0][row] + s_l[1][row]) + (s_l[2][row] + s_l[3][row]));
    }
#pragma unroll
  for (int i = 0; i < NTW; ++i) {
    const int nt = warp + 4 * i;
    if (nt < nt_all) {
      *(float2*)(sO + g * R + nt * 8 + 2 * tq) = make_float2(acc[i][0], acc[i][1]);
      *(float2*)(sO + (g + 8) * R + nt * 8 + 2 * tq) = make_float2(acc[i][2], acc[i][3]);
    }
  }
  cluster_sync();
  {
    const int r = threadIdx.x >> 4, row = threadIdx.x & 15;
    if (r < share) s_all[r][row] = ld_cluster_f2(cluster_map(&s_ml[row], r));
  }
  __syncthreads();
  if (threadIdx.x < LD_HEADS) {
    const int row = threadIdx.x;
    const float sk = p.sink && h0 + row < H ? p.sink[h0 + row] : -INFINITY;
    float M = sk;
    for (int r = 0; r < share; ++r) M = fmaxf(M, s_all[r][row].x);
    float L = expf(sk - M);
    for (int r = 0; r < share; ++r) L += s_all[r][row].y * expf(s_all[r][row].x - M);
    for (int r = 0; r < share; ++r) s_w[r][row] = expf(s_all[r][row].x - M) / L;
  }
  __syncthreads();
  const int rows = min(LD_HEADS, H - h0), r4 = R >> 2;
  for (int i = rank * LD_THREADS + threadIdx.x; i < rows * r4; i += share * LD_THREADS) {
    const int row = i / r4, c = (i - row * r4) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r = 0; r < share; ++r) {
      const float w = s_w[r][row];
      const float4 o = ld_cluster_f4(cluster_map(sO + row * R + c, r));
      v.x = fmaf(w, o.x, v.x); v.y = fmaf(w, o.y, v.y);
      v.z = fmaf(w, o.z, v.z); v.w = fmaf(w, o.w, v.w);
    }
    *(float4*)(p.out + ((size_t)t * H + h0 + row) * R + c) = v;
  }
  cluster_sync();                     // nobody leaves while its share is still being read
}

template <int NTW>
static cudaError_t launch_latent_decode(const LatentDecodeParams& p, int n_tokens, int share,
                                        size_t smem, cudaStream_t st) {
  auto kern = latent_decode_mma_kernel<NTW>;
  if (smem > 32 * 1024) {       // with the static arrays a block may then pass 48 KB
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(n_tokens, (p.n_heads + LD_HEADS - 1) / LD_HEADS, share);
  cfg.blockDim = dim3(LD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = share;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = hs_pdl_enabled() ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

}  // namespace hs

// Works on the single-query tokens of `plan` (at most n_tokens).  Refuses (HS_ERR_UNSUPPORTED) rows
// that are no whole 16-byte pieces and latents of more than 512 numbers: the caller then uses the
// CUDA-core kernel.
HS_EXPORT int hs_latent_decode_mma(float* out, const float* qa, const float* qr, const void* pool,
                                   const int* table, const float* sink, const int* plan,
                                   int n_tokens, int n_heads, int R, int P, int qr_stride,
                                   int qr_hstride, int qr_off, float scale, int page_size,
                                   int num_pages, int max_pages, int* status, const float* freq,
                                   int rot_dims, int window, void* stream) {
  if (!out || !qa || !qr || !pool || !table || !plan || !status || window < 0)
    return HS_ERR_ARGUMENT;
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > P || (rot_dims && !freq)) return HS_ERR_ARGUMENT;
  if (R <= 0 || R % 8 || R > 512 || P < 0 || (R + P) % 8 || rot_dims > 512 || n_heads <= 0 ||
      page_size <= 0 || (((uintptr_t)pool | (uintptr_t)out | (uintptr_t)qa) & 15))
    return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  const int WS = ((R + P + 31) & ~31) + 8;
  const size_t smem = (size_t)(hs::LD_Q_TERMS * hs::LD_HEADS + 2 * hs::LD_KEYS) * WS * 2;
  if (smem > 200 * 1024) return HS_ERR_UNSUPPORTED;
  int share = hs::LD_MAX_SHARE;             // fixed by the window: no more blocks than tiles
  while (window > 0 && share > 1 && (share / 2) * hs::LD_KEYS >= window) share /= 2;
  hs::LatentDecodeParams p;
  p.out = out; p.qa = qa; p.qr = qr; p.pool = (const __nv_bfloat16*)pool; p.table = table;
  p.sink = sink; p.plan = plan; p.freq = freq; p.status = status; p.n_heads = n_heads; p.R = R;
  p.P = P; p.qr_stride = qr_stride; p.qr_hstride = qr_hstride; p.qr_off = qr_off;
  p.page_size = page_size; p.num_pages = num_pages; p.max_pages = max_pages;
  p.rot_dims = rot_dims; p.window = window; p.scale = scale;
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e = R <= 128   ? hs::launch_latent_decode<4>(p, n_tokens, share, smem, st)
                  : R <= 256 ? hs::launch_latent_decode<8>(p, n_tokens, share, smem, st)
                             : hs::launch_latent_decode<16>(p, n_tokens, share, smem, st);
  return e == cudaSuccess ? HS_OK : (int)e;
}
