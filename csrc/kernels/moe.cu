// Mixture-of-experts plumbing for sm_100a: routers, the sync-free dispatch plan, row gather and the weighted combine.
//
// Reference: Mixtral top-2 on raw logits + softmax over the two (src/layers/mlp_mixtral.h:223-281); Qwen3 full
// softmax -> top-k -> renormalise (src/layers/moe_qwen3.h:283-315); DeepSeek noaux_tc — sigmoid, group score =
// sum of the top-2 biased scores of the group, keep topk_group groups, top-k experts by biased score, weights =
// unbiased scores / (sum + 1e-20) * routed_scaling_factor (src/layers/moe_deepseek.h:226-283,402-536); gather /
// scatter-add of rows (moe_deepseek.h:380-398, mlp_mixtral.h:204-219).
//
// The reference gathers on the host per expert.  Here nothing leaves the device: a plan kernel counts the rows of
// every local expert, lays the (token, slot) pairs out sorted by expert, and writes the tile table that the grouped
// tcgen05 GEMM (gemm_sm100.cu, xft_gemm_bf16_grouped) walks; the combine is a gather over each token's k slots in
// slot order, so results do not depend on where the rows landed.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

// ------------------------------------------------------------------------------------------ routers
// One warp per token.  kind: 0 mixtral, 1 softmax->topk(->renorm), 2 deepseek (sigmoid or softmax scores).
struct RouteParams {
  const float* logits; int ld; int T, E, k, kind;
  const float* bias; int n_group, topk_group; float scaling; int norm_topk; int sigmoid;
  int* idx; float* w;
};

__global__ void __launch_bounds__(128) route_kernel(const RouteParams p) {
  extern __shared__ float sm[];                 // per warp: score[E], sel[E], gscore[32]
  grid_dep_launch();
  grid_dep_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + warp;
  if (t >= p.T) return;
  const int E = p.E;
  float* score = sm + warp * (2 * E + 32);
  float* sel = score + E;
  float* gs = sel + E;
  const float* x = p.logits + (size_t)t * p.ld;
  // scores
  if (p.kind == 0) {
    for (int e = lane; e < E; e += 32) { score[e] = x[e]; sel[e] = x[e]; }
  } else {
    const bool softmax = p.kind == 1 || !p.sigmoid;
    float mx = -INFINITY;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, x[e]);
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
      const float v = softmax ? __expf(x[e] - mx) : 1.f / (1.f + __expf(-x[e]));
      score[e] = v;
      sum += v;
    }
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    for (int e = lane; e < E; e += 32) {
      if (softmax) score[e] /= sum;
      sel[e] = score[e] + ((p.kind == 2 && p.bias) ? p.bias[e] : 0.f);
    }
  }
  __syncwarp();
  if (p.kind == 2 && p.n_group > 1) {
    const int gsz = E / p.n_group;
    if (lane < p.n_group) {                     // group score = sum of its two best biased scores
      float a = -INFINITY, b = -INFINITY;
      for (int i = 0; i < gsz; ++i) {
        const float v = sel[lane * gsz + i];
        if (v > a) { b = a; a = v; } else if (v > b) b = v;
      }
      gs[lane] = gsz > 1 ? a + b : a;
    }
    __syncwarp();
    if (lane == 0) {                            // keep the topk_group best groups (first wins ties)
      unsigned keep = 0;
      for (int j = 0; j < p.topk_group; ++j) {
        int bi = -1; float bv = -INFINITY;
        for (int g = 0; g < p.n_group; ++g)
          if (!(keep >> g & 1) && (bi < 0 || gs[g] > bv)) { bv = gs[g]; bi = g; }
        keep |= 1u << bi;
      }
      gs[31] = __uint_as_float(keep);
    }
    __syncwarp();
    const unsigned keep = __float_as_uint(gs[31]);
    for (int e = lane; e < E; e += 32)
      if (!(keep >> (e / gsz) & 1)) sel[e] = -INFINITY;
    __syncwarp();
  }
  // top-k by repeated arg-max (lowest index wins ties)
  float wsum = 0.f;
  float myw = 0.f; int myi = 0;
  for (int j = 0; j < p.k; ++j) {
    float bv = -INFINITY; int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = sel[e];
      if (v > bv || (v == bv && e < bi)) { bv = v; bi = e; }
    }
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    if (bi == 0x7fffffff) bi = 0;
    const float sc = score[bi];
    wsum += sc;
    if (lane == j) { myw = sc; myi = bi; }
    __syncwarp();
    if (lane == 0) sel[bi] = -INFINITY;
    __syncwarp();
  }
  if (lane < p.k) {
    float w = myw;
    if (p.kind == 0) {
      // softmax over the selected logits only
      float mx = -INFINITY;
      for (int j = 0; j < p.k; ++j) mx = fmaxf(mx, __shfl_sync((1u << p.k) - 1, myw, j));
      float den = 0.f;
      for (int j = 0; j < p.k; ++j) den += __expf(__shfl_sync((1u << p.k) - 1, myw, j) - mx);
      w = __expf(myw - mx) / den;
    } else if (p.kind == 1) {
      if (p.norm_topk) w = myw / wsum;
    } else {
      if (p.norm_topk) w = myw / (wsum + 1e-20f);
      w *= p.scaling;
    }
    p.idx[(size_t)t * p.k + lane] = myi;
    p.w[(size_t)t * p.k + lane] = w;
  }
}

// ------------------------------------------------------------------------------------------ dispatch plan
// One block.  Pairs (t, s) whose expert lies in [e0, e1) are placed, grouped by expert, in rows
// [0, total).  Outputs: pos[T*k] (row of the pair or -1), src_tok[row], row_w[row], tile table
// {local expert, first row, rows, 0} for token tiles of `bn` rows, meta = {num_tiles, total rows}.
struct PlanParams {
  const int* idx; const float* w; int T, k, e0, e1, bn;
  int* pos; int* src_tok; float* row_w; int4* tiles; int* meta; int max_tiles; int max_rows;
};

// Counters are per warp (and expert), so that pairs only collide with those of their own 32 lanes.
__global__ void __launch_bounds__(1024) moe_plan_kernel(const PlanParams p) {
  extern __shared__ int cur[];                  // [32 warps][E]: counts, then the warp's next row of each expert
  __shared__ int cnt[256], off[257], toff[257];
  grid_dep_launch();
  grid_dep_wait();
  const int E = p.e1 - p.e0, n = p.T * p.k;
  int* mine = cur + (threadIdx.x >> 5) * E;
  for (int i = threadIdx.x; i < 32 * E; i += blockDim.x) cur[i] = 0;
  __syncthreads();
  // eight pairs per thread and round: their loads are in flight together
  for (int i0 = threadIdx.x; i0 < n; i0 += 8 * blockDim.x) {
    int e[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) { const int i = i0 + j * blockDim.x; e[j] = i < n ? p.idx[i] - p.e0 : -1; }
#pragma unroll
    for (int j = 0; j < 8; ++j) if (e[j] >= 0 && e[j] < E) atomicAdd(&mine[e[j]], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {      // counts of the warps -> where each one's rows start
    int o = 0;
    for (int w = 0; w < 32; ++w) { const int c = cur[w * E + e]; cur[w * E + e] = o; o += c; }
    cnt[e] = o;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int o = 0, to = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = o; toff[e] = to;
      o += cnt[e];
      to += (cnt[e] + p.bn - 1) / p.bn;
    }
    off[E] = o; toff[E] = to;
    p.meta[0] = to > p.max_tiles ? p.max_tiles : to;
    p.meta[1] = o;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int nt = toff[e + 1] - toff[e];
    for (int j = 0; j < nt; ++j) {
      const int ti = toff[e] + j;
      if (ti < p.max_tiles) p.tiles[ti] = make_int4(e, off[e] + j * p.bn, min(p.bn, cnt[e] - j * p.bn), 0);
    }
  }
  for (int i0 = threadIdx.x; i0 < n; i0 += 8 * blockDim.x) {
    int e[8], r[8];
    float w[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = i0 + j * blockDim.x;
      e[j] = i < n ? p.idx[i] - p.e0 : -1;
      w[j] = i < n ? p.w[i] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) r[j] = e[j] >= 0 && e[j] < E ? off[e[j]] + atomicAdd(&mine[e[j]], 1) : -1;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = i0 + j * blockDim.x;
      if (i >= n) break;
      if (r[j] >= p.max_rows) r[j] = -1;
      if (r[j] >= 0) { p.src_tok[r[j]] = i / p.k; p.row_w[r[j]] = w[j]; }
      p.pos[i] = r[j];
    }
  }
}

// Xs[row] = X[src_tok[row]] for row < total (one CTA per row slot; idle past the total)
__global__ void __launch_bounds__(128) moe_gather_kernel(const bf16* __restrict__ x, int ldx, const int* __restrict__ src_tok,
                                                         const int* __restrict__ meta, bf16* __restrict__ xs, int H) {
  grid_dep_launch();
  grid_dep_wait();
  const int r = blockIdx.x;
  if (r >= meta[1]) return;
  const uint4* s = reinterpret_cast<const uint4*>(x + (size_t)src_tok[r] * ldx);
  uint4* d = reinterpret_cast<uint4*>(xs + (size_t)r * H);
  for (int i = threadIdx.x; i < H / 8; i += 128) d[i] = s[i];
}

__device__ __forceinline__ void moe_load(const float* p, float (&v)[1]) { v[0] = p[0]; }
__device__ __forceinline__ void moe_load(const bf16* p, float (&v)[1]) { v[0] = __bfloat162float(p[0]); }
__device__ __forceinline__ void moe_load(const float* p, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void moe_load(const bf16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}

// y[t] = sum_s w[t,s] ys[pos[t,s]] + add1[t] + add2[t]   (fp32 sum, bf16 or fp32 out).  w null: the rows of ys carry their
// weight already.  VEC: four columns per thread (H and ld2 multiples of 4).  A row's positions are read first, so that all
// its loads are in flight together.
template <typename YT, bool VEC>
__global__ void __launch_bounds__(256) moe_combine_kernel(const YT* __restrict__ ys, const int* __restrict__ pos,
                                                          const float* __restrict__ w, int k, const float* __restrict__ add1,
                                                          const bf16* __restrict__ add2, int ld2, bf16* __restrict__ y,
                                                          float* __restrict__ y32, int H) {
  constexpr int V = VEC ? 4 : 1;
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x;
  const int i = (blockIdx.y * 256 + threadIdx.x) * V;
  if (i >= H) return;
  float a[V], v[V];
#pragma unroll
  for (int c = 0; c < V; ++c) a[c] = 0.f;
  for (int s0 = 0; s0 < k; s0 += 8) {
    int r[8];
    float f[8], x[8][V];
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      r[s] = s0 + s < k ? pos[t * k + s0 + s] : -1;
      f[s] = w && s0 + s < k ? w[t * k + s0 + s] : 1.f;
    }
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (r[s] >= 0) moe_load(ys + (size_t)r[s] * H + i, x[s]);
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (r[s] >= 0)
#pragma unroll
        for (int c = 0; c < V; ++c) a[c] += f[s] * x[s][c];
  }
  if (add1) {
    moe_load(add1 + (size_t)t * H + i, v);
#pragma unroll
    for (int c = 0; c < V; ++c) a[c] += v[c];
  }
  if (add2) {
    moe_load(add2 + (size_t)t * ld2 + i, v);
#pragma unroll
    for (int c = 0; c < V; ++c) a[c] += v[c];
  }
  if (y32) {
    if (VEC) *reinterpret_cast<float4*>(y32 + (size_t)t * H + i) = make_float4(a[0], a[V > 1 ? 1 : 0], a[V > 2 ? 2 : 0], a[V > 3 ? 3 : 0]);
    else y32[(size_t)t * H + i] = a[0];
  } else {
#pragma unroll
    for (int c = 0; c < V; ++c) y[(size_t)t * H + i + c] = __float2bfloat16(a[c]);
  }
}

}  // namespace xft

using namespace xft;

extern "C" int xft_moe_route(const float* logits, int ld, int T, int E, int k, int kind, const float* bias, int n_group,
                             int topk_group, float scaling, int norm_topk, int sigmoid, int* idx, float* w, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E > 4096 || k > 32 || n_group > 31) return -1;
  RouteParams p{logits, ld, T, E, k, kind, bias, n_group, topk_group, scaling, norm_topk, sigmoid, idx, w};
  const size_t smem = 4 * (2 * E + 32) * sizeof(float);
  cudaError_t e = launch_pdl(route_kernel, dim3((T + 3) / 4), dim3(128), smem, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

extern "C" int xft_moe_plan(const int* idx, const float* w, int T, int k, int e0, int e1, int bn, int* pos, int* src_tok,
                            float* row_w, void* tiles, int* meta, int max_tiles, int max_rows, cudaStream_t st) {
  if (e1 - e0 > 256 || e1 <= e0) return -1;
  PlanParams p{idx, w, T, k, e0, e1, bn, pos, src_tok, row_w, reinterpret_cast<int4*>(tiles), meta, max_tiles, max_rows};
  cudaError_t e = launch_pdl(moe_plan_kernel, dim3(1), dim3(1024), (size_t)32 * (e1 - e0) * sizeof(int), st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

extern "C" int xft_moe_gather(const void* x, int ldx, const int* src_tok, const int* meta, void* xs, int max_rows, int H,
                              cudaStream_t st) {
  if (max_rows <= 0) return 0;
  if (H % 8) return -1;
  cudaError_t e = launch_pdl(moe_gather_kernel, dim3(max_rows), dim3(128), 0, st, (const bf16*)x, ldx, src_tok, meta, (bf16*)xs, H);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

template <typename YT>
static int launch_combine(const YT* ys, const int* pos, const float* w, int k, const float* add1, const bf16* add2, int ld2, void* y,
                          float* y32, int T, int H, cudaStream_t st) {
  const bool vec = H % 4 == 0 && (!add2 || ld2 % 4 == 0) &&
                   ((reinterpret_cast<uintptr_t>(ys) | reinterpret_cast<uintptr_t>(add1) | reinterpret_cast<uintptr_t>(add2) |
                     reinterpret_cast<uintptr_t>(y32)) & 15) == 0;
  const int per = vec ? 1024 : 256;
  const dim3 grid(T, (H + per - 1) / per);
  cudaError_t e = vec ? launch_pdl(moe_combine_kernel<YT, true>, grid, dim3(256), 0, st, ys, pos, w, k, add1, add2, ld2, (bf16*)y, y32, H)
                      : launch_pdl(moe_combine_kernel<YT, false>, grid, dim3(256), 0, st, ys, pos, w, k, add1, add2, ld2, (bf16*)y, y32, H);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

extern "C" int xft_moe_combine(const float* ys, const int* pos, int k, const float* add1, const void* add2, int ld2, void* y,
                               float* y32, int T, int H, cudaStream_t st) {
  if (T <= 0) return 0;
  return launch_combine<float>(ys, pos, nullptr, k, add1, (const bf16*)add2, ld2, y, y32, T, H, st);
}

// Prompt sizes: bf16 rows, weighted here with w [T, k].
extern "C" int xft_moe_combine_bf16(const void* ys, const int* pos, const float* w, int k, const float* add1, const void* add2,
                                    int ld2, void* y, float* y32, int T, int H, cudaStream_t st) {
  if (T <= 0) return 0;
  return launch_combine<bf16>((const bf16*)ys, pos, w, k, add1, (const bf16*)add2, ld2, y, y32, T, H, st);
}
