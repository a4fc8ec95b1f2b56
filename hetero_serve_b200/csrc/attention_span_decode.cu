// The attention of attention_span.cu for the single-query tokens of a step, on the tensor cores
// (mma.sync m16n8k16, bfloat16 operands, float32 accumulators; bfloat16 cache).
//
// The query heads of one key/value head read the same rows, so up to 16 of them are the 16 rows of
// one product: a block works on one token and one such set of heads, 32 keys a tile in two cp.async
// stages.  A token's keys are shared out over a cluster of up to eight blocks; their shares (maximum,
// sum, weighted rows) stay in shared memory and are joined across the cluster, each block finishing a
// part of the output.  The split depends on the window alone, a row's result on its own request.
// The rows are bfloat16 numbers already; a query enters as the sum of three bfloat16 terms (a
// float32's whole mantissa) and a weight as the sum of two, so scores and weights keep what a float32
// product keeps.  Slope, cap, sink, gate and the visibility rule are those of attention_span.cu.
#include "mma_tiles.cuh"
#include "tcgen05.cuh"

namespace hs {

constexpr int SD_KEYS = 32, SD_HEADS = 16, SD_THREADS = 128, SD_MAX_SHARE = 8;
constexpr int SD_Q_TERMS = 3, SD_P_TERMS = 2;

struct SpanDecodeParams {
  __nv_bfloat16* out;        // [T, H * V]
  const float* q;            // [T, H * D]
  const __nv_bfloat16* pool;
  const int* table;
  const int* plan;
  const float* slopes;       // [H] or null
  const float* sinks;        // [H] or null
  const float* gate;         // [T, gate_stride] or null
  int* status;
  int H, G, D, V, page_size, num_pages, max_pages, window, keep_first, gate_stride, gate_offset;
  float scale, softcap, out_scale;
};

__device__ __forceinline__ float4 sd_cluster_f4(uint32_t a) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];"
               : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ float2 sd_cluster_f2(uint32_t a) {
  float2 v;
  asm volatile("ld.shared::cluster.v2.f32 {%0,%1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
  return v;
}

// NTW: output tiles of 8 columns a warp keeps at most (V <= 32 * NTW)
template <int NTW>
__global__ void __launch_bounds__(SD_THREADS)
span_decode_mma_kernel(const SpanDecodeParams p) {
  extern __shared__ __align__(16) uint8_t sd_smem[];
  __shared__ __align__(16) __nv_bfloat16 s_p[SD_P_TERMS][SD_HEADS][SD_KEYS + 8];
  __shared__ float s_mx[4][SD_HEADS], s_l[4][SD_HEADS];
  __shared__ __align__(8) float2 s_ml[SD_HEADS];          // this block's share: maximum, sum
  __shared__ float2 s_all[SD_MAX_SHARE][SD_HEADS];
  __shared__ float s_w[SD_MAX_SHARE][SD_HEADS];
  pdl_trigger();
  const int D = p.D, V = p.V, W = D + V, D32 = (D + 31) & ~31, WS = D32 + V + 8, QS = D32 + 8;
  const int per_kv = p.H / p.G, sets = (per_kv + SD_HEADS - 1) / SD_HEADS;
  const int kv = blockIdx.y / sets, set = blockIdx.y - kv * sets;
  const int h0 = kv * per_kv + set * SD_HEADS, n_rows = min(SD_HEADS, per_kv - set * SD_HEADS);
  __nv_bfloat16* sQ = (__nv_bfloat16*)sd_smem;            // [3 terms][16][QS]
  __nv_bfloat16* sK = sQ + SD_Q_TERMS * SD_HEADS * QS;    // [2][32][WS]: key, zeros up to D32, value
  float* sO = (float*)sK;                                 // [16][V], once the tiles are done
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  pdl_wait();
  if ((int)blockIdx.x >= p.plan[0]) return;               // the whole cluster
  const int t = p.plan[4 + 3 * blockIdx.x], req = p.plan[5 + 3 * blockIdx.x];
  const int pos = p.plan[6 + 3 * blockIdx.x];
  const int share = gridDim.z, rank = blockIdx.z;         // the cluster spans z
  const int first = p.window > 0 ? max(0, pos + 1 - p.window) : 0;
  const int kept = min(p.keep_first, first);              // first tokens that lie behind the window
  const int n_keys = kept + pos + 1 - first;
  const int n_tiles = (n_keys + SD_KEYS - 1) / SD_KEYS;
  const int per = (n_tiles + share - 1) / share;
  const int lo = rank * per, hi = min(n_tiles, lo + per);

  // a warp brings eight rows of a tile: the first eight lanes look their pages up
  auto fetch = [&](int tile, int st) {
    long long at = -1;
    const int kk = tile * SD_KEYS + warp * 8 + (lane & 7);
    if (kk < n_keys) {
      const int kp = kk < kept ? kk : first + kk - kept, pi = kp / p.page_size;
      const int page = pi < p.max_pages ? p.table[(size_t)req * p.max_pages + pi] : -1;
      if (page < 0 || page >= p.num_pages) atomicOr(p.status, HS_STATUS_BAD_PAGE);
      else at = (((long long)page * p.G + kv) * p.page_size + (kp - pi * p.page_size)) * W;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const long long row = __shfl_sync(0xffffffffu, at, j);
      __nv_bfloat16* dst = sK + (size_t)(st * SD_KEYS + warp * 8 + j) * WS;
      for (int c = lane * 8; c < W; c += 256) {
        __nv_bfloat16* d = dst + (c < D ? c : c - D + D32);
        if (row >= 0)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(d)),
                       "l"(p.pool + row + c));
        else
          *(uint4*)d = make_uint4(0, 0, 0, 0);
      }
    }
    asm volatile("cp.async.commit_group;");
  };
  if (lo < hi) fetch(lo, 0);
  if (D < D32)
    for (int i = threadIdx.x; i < 2 * SD_KEYS; i += SD_THREADS)
      for (int c = D; c < D32; ++c) sK[(size_t)i * WS + c] = __float2bfloat16_rn(0.f);
  for (int hh = warp; hh < SD_HEADS; hh += 4) {
    const float* a = p.q + ((size_t)t * p.H + h0 + hh) * D;
    for (int d = 2 * lane; d < D32; d += 64) {
      float2 v = make_float2(0.f, 0.f);
      if (hh < n_rows && d < D) v = *(const float2*)(a + d);
#pragma unroll
      for (int term = 0; term < SD_Q_TERMS; ++term) {
        const __nv_bfloat162 q2 = __floats2bfloat162_rn(v.x, v.y);
        *(__nv_bfloat162*)(sQ + (term * SD_HEADS + hh) * QS + d) = q2;
        v.x -= __bfloat162float(q2.x);                    // what this term leaves (exact)
        v.y -= __bfloat162float(q2.y);
      }
    }
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};     // rows g and g + 8
  float slope[2] = {0.f, 0.f};
  if (p.slopes) {
    if (g < n_rows) slope[0] = p.slopes[h0 + g];
    if (g + 8 < n_rows) slope[1] = p.slopes[h0 + g + 8];
  }
  float acc[NTW][4];
#pragma unroll
  for (int i = 0; i < NTW; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[i][c] = 0.f;
  const int nt_all = V >> 3;
  const __nv_bfloat16* qp = sQ + (lane & 15) * QS + (lane >> 4) * 8;
  for (int tile = lo; tile < hi; ++tile) {
    const int st = (tile - lo) & 1;
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                  // the tile is here (and the queries), the one before is used
    if (tile + 1 < hi) fetch(tile + 1, st ^ 1);
    const __nv_bfloat16* k = sK + (size_t)st * SD_KEYS * WS;
    const __nv_bfloat16* kp = k + (warp * 8 + (lane & 7)) * WS + (lane >> 3) * 8;
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
    for (int kk = 0; kk < D32; kk += 32) {
      uint32_t a0[4], a1[4], b[4];
      ldmatrix_x4(b, kp + kk);
#pragma unroll
      for (int term = SD_Q_TERMS - 1; term >= 0; --term) {            // the small terms first
        ldmatrix_x4(a0, qp + term * SD_HEADS * QS + kk);
        ldmatrix_x4(a1, qp + term * SD_HEADS * QS + kk + 16);
        mma_bf16(s, a0, b);
        mma_bf16(s2, a1, b + 2);
      }
    }
    const int key = tile * SD_KEYS + warp * 8 + 2 * tq;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int kk = key + (c & 1), j = kk < kept ? kk : first + kk - kept;
      float v = (s[c] + s2[c]) * p.scale - slope[c >> 1] * (float)(pos - j);
      if (p.softcap > 0.f) v = p.softcap * tanhf(v / p.softcap);
      s[c] = kk < n_keys ? v : -INFINITY;
    }
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
    uint32_t pa[SD_P_TERMS][2][4];
#pragma unroll
    for (int term = 0; term < SD_P_TERMS; ++term) {
      ldmatrix_x4(pa[term][0], &s_p[term][lane & 15][(lane >> 4) * 8]);
      ldmatrix_x4(pa[term][1], &s_p[term][lane & 15][16 + (lane >> 4) * 8]);
    }
    const uint32_t v_addr = smem_u32(k + lane * WS + D32);
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
        for (int term = SD_P_TERMS - 1; term >= 0; --term) {
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
      *(float2*)(sO + g * V + nt * 8 + 2 * tq) = make_float2(acc[i][0], acc[i][1]);
      *(float2*)(sO + (g + 8) * V + nt * 8 + 2 * tq) = make_float2(acc[i][2], acc[i][3]);
    }
  }
  cluster_sync();
  {
    const int r = threadIdx.x >> 4, row = threadIdx.x & 15;
    if (r < share) s_all[r][row] = sd_cluster_f2(cluster_map(&s_ml[row], r));
  }
  __syncthreads();
  if ((int)threadIdx.x < n_rows) {
    const int row = threadIdx.x;
    const float sk = p.sinks ? p.sinks[h0 + row] : -INFINITY;
    float M = sk;
    for (int r = 0; r < share; ++r) M = fmaxf(M, s_all[r][row].x);
    float L = expf(sk - M);
    for (int r = 0; r < share; ++r) L += s_all[r][row].y * expf(s_all[r][row].x - M);
    for (int r = 0; r < share; ++r) s_w[r][row] = expf(s_all[r][row].x - M) / L;
  }
  __syncthreads();
  const int v4 = V >> 2;
  for (int i = rank * SD_THREADS + threadIdx.x; i < n_rows * v4; i += share * SD_THREADS) {
    const int row = i / v4, c = (i - row * v4) * 4;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    for (int r = 0; r < share; ++r) {
      const float w = s_w[r][row];
      const float4 o = sd_cluster_f4(cluster_map(sO + row * V + c, r));
      v[0] = fmaf(w, o.x, v[0]); v[1] = fmaf(w, o.y, v[1]);
      v[2] = fmaf(w, o.z, v[2]); v[3] = fmaf(w, o.w, v[3]);
    }
    const size_t col = (size_t)(h0 + row) * V + c;
    if (p.gate) {
      const float* gr = p.gate + (size_t)t * p.gate_stride + p.gate_offset + col;
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] *= 1.0f / (1.0f + expf(-gr[j]));
    }
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0] * p.out_scale, v[1] * p.out_scale);
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[2] * p.out_scale, v[3] * p.out_scale);
    *(uint2*)(p.out + (size_t)t * p.H * V + col) = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
  }
  cluster_sync();                     // nobody leaves while its share is still being read
}

template <int NTW>
static cudaError_t launch_span_decode(const SpanDecodeParams& p, int n_tokens, int share, size_t smem,
                                      cudaStream_t st) {
  auto kern = span_decode_mma_kernel<NTW>;
  if (smem > 32 * 1024) {       // with the static arrays a block may then pass 48 KB
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  const int per_kv = p.H / p.G;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(n_tokens, p.G * ((per_kv + SD_HEADS - 1) / SD_HEADS), share);
  cfg.blockDim = dim3(SD_THREADS);
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
// that are no whole 16-byte pieces: the caller then uses the CUDA-core kernel.
HS_EXPORT int hs_span_decode_mma(void* out, const float* q, const void* pool, const int* table,
                                 int max_pages, int num_pages, const int* plan, int n_tokens,
                                 const float* slopes, const float* gate, int gate_stride,
                                 int gate_offset, float out_scale, int H, int G, int D, int V,
                                 int window, int keep_first, float scale, int page_size,
                                 float softcap, const float* sinks, int* status, void* stream) {
  using namespace hs;
  if (!out || !q || !pool || !table || !plan || !status) return HS_ERR_ARGUMENT;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || D % 8 || V <= 0 || V % 8 || V > 256 || window < 0 ||
      keep_first < 0 || page_size <= 0 || num_pages <= 0 || max_pages <= 0 ||
      (gate && (gate_offset < 0 || gate_offset + H * V > gate_stride)) ||
      (((uintptr_t)pool | (uintptr_t)out | (uintptr_t)q) & 15))
    return HS_ERR_UNSUPPORTED;
  if (n_tokens <= 0) return HS_OK;
  const int D32 = (D + 31) & ~31;
  size_t smem = (size_t)2 * (SD_Q_TERMS * SD_HEADS * (D32 + 8) + 2 * SD_KEYS * (D32 + V + 8));
  if (smem > 180 * 1024 || (long long)G * ((H / G + SD_HEADS - 1) / SD_HEADS) > 65535) return HS_ERR_UNSUPPORTED;
  int share = SD_MAX_SHARE;                 // fixed by the window: no more blocks than tiles
  while (window > 0 && share > 1 && (share / 2) * SD_KEYS >= window + keep_first) share /= 2;
  SpanDecodeParams p;
  p.out = (__nv_bfloat16*)out; p.q = q; p.pool = (const __nv_bfloat16*)pool; p.table = table;
  p.plan = plan; p.slopes = slopes; p.sinks = sinks; p.gate = gate; p.status = status;
  p.H = H; p.G = G; p.D = D; p.V = V; p.page_size = page_size; p.num_pages = num_pages;
  p.max_pages = max_pages; p.window = window; p.keep_first = keep_first;
  p.gate_stride = gate_stride; p.gate_offset = gate_offset; p.scale = scale; p.softcap = softcap;
  p.out_scale = out_scale;
  cudaStream_t st = (cudaStream_t)stream;
  const cudaError_t e = V <= 64    ? launch_span_decode<2>(p, n_tokens, share, smem, st)
                        : V <= 128 ? launch_span_decode<4>(p, n_tokens, share, smem, st)
                                   : launch_span_decode<8>(p, n_tokens, share, smem, st);
  return e == cudaSuccess ? HS_OK : (int)e;
}
