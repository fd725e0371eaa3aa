// Plain kernels for any size: the 32-bit path of the layered decoder (fp32 weights, activations and cache), and what a
// bf16 model needs when its heads are larger than the tensor-core kernels take.
//
//   xft_gemm_f32        Y[T, N] = act(X[T, K] W[N, K]^T + bias) * times in fp32 (no reduced-precision mode); also one product per head,
//                       and products of rows grouped by expert
//   xft_gated_act_f32   act(gate) * up
//   xft_sigmoid_gate    x * sigmoid(gate)
//   xft_rope_cache      split q | k | v rows, rotate q and k, append k and v to the paged cache; key and value heads may
//                       have different sizes
//   xft_attention_plain one warp per (query, head): sliding window with kept first keys, capped scores, sinks
//
// This file is compiled without fast-math: tanhf, expf and the divisions are the accurate ones.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16(v); }

// ------------------------------------------------------------------------------------------ GEMM
struct GemmF32 {
  const float* X; int ldx; const float* W; int ldw; float* Y; int ldo; int T, N, K, act;
  long long sx, sw, sy;                        // blockIdx.z steps through a batch with these strides
  // grouped form: blockIdx.y is a tile {group, first row, rows, -} of 64 rows; X row r comes from src[r] when given
  const int4* tiles; const int* num_tiles; const int* src; const float* row_w; int group_w_rows;
  const float* bias; const float* times; int ldt;             // [N] and [T, N], or null
  float param;                                 // of the activation
};

__device__ __forceinline__ float act_f32(float x, int act, float param = 1.f) {
  if (act == 1) return fmaxf(x, 0.f);
  if (act == 2) return x / (1.f + expf(-x));
  if (act == 3) return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
  if (act == 4) { const float r = fmaxf(x, 0.f); return r * r; }
  if (act == 5) return 0.5f * x * (1.f + erff(x * 0.70710678118654752f));
  if (act == 7) return tanhf(x);
  if (act == 8) return param * tanhf(x / param);
  return x;
}

// 64 x 64 tile of Y per CTA, 256 threads with 4 x 4 values each, 16 columns of the reduction per step.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32 p) {
  __shared__ float xs[16][68], ws[16][68];
  const float* W = p.W + blockIdx.z * p.sw;
  int t0 = blockIdx.y * 64, rows = min(64, p.T - t0);
  if (p.tiles) {
    if ((int)blockIdx.y >= *p.num_tiles) return;
    const int4 e = p.tiles[blockIdx.y];
    t0 = e.y;
    rows = e.z;
    W += (size_t)e.x * p.group_w_rows * p.ldw;
  }
  const int n0 = blockIdx.x * 64, tid = threadIdx.x;
  const int lr = tid >> 2, lk = (tid & 3) * 4;             // this thread loads row lr, columns lk .. lk + 3
  const int tx = tid & 15, ty = tid >> 4;
  const float* xrow = p.X + blockIdx.z * p.sx + (size_t)(lr < rows ? (p.src ? p.src[t0 + lr] : t0 + lr) : 0) * p.ldx;
  const float* wrow = W + (size_t)(n0 + lr < p.N ? n0 + lr : 0) * p.ldw;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      xs[lk + j][lr] = (lr < rows && k < p.K) ? xrow[k] : 0.f;
      ws[lk + j][lr] = (n0 + lr < p.N && k < p.K) ? wrow[k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) { a[j] = xs[k][ty * 4 + j]; b[j] = ws[k][tx * 4 + j]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  float* Y = p.Y + blockIdx.z * p.sy;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = ty * 4 + i, n = n0 + tx * 4 + j;
      if (r < rows && n < p.N) {
        float v = act_f32(acc[i][j] + (p.bias ? p.bias[n] : 0.f), p.act, p.param);
        if (p.times) v *= p.times[(size_t)(t0 + r) * p.ldt + n];
        if (p.row_w) v *= p.row_w[t0 + r];
        Y[(size_t)(t0 + r) * p.ldo + n] = v;
      }
    }
}

__global__ void gated_act_f32_kernel(const float* __restrict__ gu, int ld, float* __restrict__ out, int T, int I, int act, float limit) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)T * I) return;
  const int t = (int)(i / I), c = (int)(i % I);
  const float g = gu[(size_t)t * ld + c], u = gu[(size_t)t * ld + I + c];
  if (act == 6) {                                        // gate bounded above, the other on both sides
    const float c = fminf(g, limit);
    out[i] = c / (1.f + expf(-1.702f * c)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
  } else out[i] = act_f32(g, act) * u;
}

// out[t, c] = x[t, c] * sigmoid(gate[t, c / per])
template <typename T>
__global__ void sigmoid_gate_kernel(const T* __restrict__ x, int ldx, const T* __restrict__ gate, int ldg, T* __restrict__ out,
                                    int ldo, int n_tok, int n, int per) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)n_tok * n) return;
  const int t = (int)(i / n), c = (int)(i % n);
  const float g = to_f32<T>(gate[(size_t)t * ldg + c / per]);
  out[(size_t)t * ldo + c] = from_f32<T>(to_f32<T>(x[(size_t)t * ldx + c]) / (1.f + expf(-g)));
}

// ------------------------------------------------------------------------------------------ rotary + cache append
// One warp per (token, head); rows are hq query heads of kd, hkv key heads of kd, hkv value heads of vd.
template <typename T>
__global__ void __launch_bounds__(128) rope_cache_kernel(const T* __restrict__ qkv, int ldq, int n_tok, int hq, int hkv, int kd,
                                                         int vd, const int* __restrict__ positions,
                                                         const float* __restrict__ table, int rot, int style, int max_pos,
                                                         T* __restrict__ q_out, T* __restrict__ kc, T* __restrict__ vc, int bs,
                                                         long long nslots, const int* __restrict__ slots, int* status) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nheads = hq + 2 * hkv;
  const long long gw = (long long)blockIdx.x * 4 + warp;
  if (gw >= (long long)n_tok * nheads) return;
  const int t = (int)(gw / nheads), h = (int)(gw % nheads);
  const bool is_v = h >= hq + hkv;
  const T* src = qkv + (size_t)t * ldq + (is_v ? (hq + hkv) * kd + (h - hq - hkv) * vd : h * kd);
  const int D = is_v ? vd : kd;
  T* dst;
  if (h < hq) {
    dst = q_out + ((size_t)t * hq + h) * kd;
  } else {
    const long long slot = slots[t];
    if (slot < 0 || slot >= nslots) { if (lane == 0 && status) atomicCAS(status, 0, XFT_ERR_BOUNDS); return; }
    const int kh = is_v ? h - hq - hkv : h - hq;
    dst = (is_v ? vc : kc) + ((size_t)((slot / bs) * hkv + kh) * bs + slot % bs) * D;
  }
  int pos = positions[t];
  if (table && (pos < 0 || pos >= max_pos)) { if (lane == 0 && status) atomicCAS(status, 0, XFT_ERR_BOUNDS); pos = 0; }
  const int half = rot >> 1;
  for (int d = lane; d < D; d += 32) {
    float x = to_f32<T>(src[d]);
    if (!is_v && table && d < rot) {
      const float* cs = table + (size_t)pos * rot;
      const int i = style == 0 ? (d < half ? d : d - half) : d >> 1;
      const bool second = style == 0 ? d >= half : (d & 1) != 0;
      const int partner = style == 0 ? (second ? d - half : d + half) : d ^ 1;
      const float y = to_f32<T>(src[partner]);
      x = x * cs[i] + (second ? y : -y) * cs[half + i];
    }
    dst[d] = from_f32<T>(x);
  }
}

// ------------------------------------------------------------------------------------------ attention
// One warp per (query token, head).  A lane owns one of 32 keys while scores are computed and every 32nd output feature
// while values are added up.
template <typename T>
__global__ void __launch_bounds__(128) attention_plain_kernel(const T* __restrict__ q, T* __restrict__ out,
                                                              const T* __restrict__ kc, const T* __restrict__ vc,
                                                              const int* __restrict__ block_table, int bt_stride,
                                                              const int* __restrict__ cu_q, const int* __restrict__ kv_lens,
                                                              int B, int n_tok, int hq, int hkv, int group, int q_off, int kd,
                                                              int vd, int vld, int bs, int num_blocks, float scale, float softcap,
                                                              int window, int keep, const float* __restrict__ sinks,
                                                              int* status) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* qs = sm + warp * (kd + vd + 64);
  float* acc = qs + kd;
  float* ps = acc + vd;                                   // 32 weights
  int* rs = reinterpret_cast<int*>(ps + 32);              // 32 cache rows
  const long long gw = (long long)blockIdx.x * 4 + warp;
  if (gw >= (long long)n_tok * hq) return;
  const int t = (int)(gw / hq), h = (int)(gw % hq);
  int lo_b = 0, hi_b = B - 1;                             // the sequence that owns token t
  while (lo_b < hi_b) {
    const int mid = (lo_b + hi_b + 1) >> 1;
    if (cu_q[mid] <= t) lo_b = mid; else hi_b = mid - 1;
  }
  const int b = lo_b, kv_len = kv_lens[b];
  const int qpos = kv_len - (cu_q[b + 1] - cu_q[b]) + (t - cu_q[b]);
  const int kvh = min((h + q_off) / group, hkv - 1);
  for (int d = lane; d < kd; d += 32) qs[d] = to_f32<T>(q[((size_t)t * hq + h) * kd + d]);
  for (int d = lane; d < vd; d += 32) acc[d] = 0.f;
  __syncwarp();
  // visible keys: [0, nk) and [lo, qpos]
  const int lo = max(0, qpos - window + 1);
  const int nk = min(keep, lo);
  const int total = nk + qpos + 1 - lo;
  const int* bt = block_table + (size_t)b * bt_stride;
  float m = -INFINITY, l = 0.f;
  if (sinks) { m = sinks[h]; l = 1.f; }
  for (int n0 = 0; n0 < total; n0 += 32) {
    const int n = n0 + lane;
    float s = -INFINITY;
    int row = 0;
    if (n < total) {
      const int key = n < nk ? n : n - nk + lo;
      int blk = bt[key / bs];
      if (blk < 0 || blk >= num_blocks) { if (status) atomicCAS(status, 0, XFT_ERR_BOUNDS); blk = 0; }
      row = (blk * hkv + kvh) * bs + key % bs;
      const T* kp = kc + (size_t)row * kd;
      float dot = 0.f;
      for (int d = 0; d < kd; ++d) dot = fmaf(qs[d], to_f32<T>(kp[d]), dot);
      s = dot * scale;
      if (softcap > 0.f) s = softcap * tanhf(s / softcap);
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx);
    const float c = m == -INFINITY ? 0.f : expf(m - mn);
    const float pr = n < total ? expf(s - mn) : 0.f;
    float sum = pr;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    m = mn;
    l = l * c + sum;
    ps[lane] = pr;
    rs[lane] = row;
    __syncwarp();
    const int cnt = min(32, total - n0);
    for (int d = lane; d < vd; d += 32) {
      float a = acc[d] * c;
      for (int i = 0; i < cnt; ++i) a = fmaf(ps[i], to_f32<T>(vc[(size_t)rs[i] * vld + d]), a);
      acc[d] = a;
    }
    __syncwarp();
  }
  for (int d = lane; d < vd; d += 32) out[((size_t)t * hq + h) * vd + d] = from_f32<T>(l > 0.f ? acc[d] / l : 0.f);
}

}  // namespace xft

using namespace xft;

// act: 0 none, 1 relu, 2 silu, 3 gelu (tanh), 4 relu squared, 5 gelu (erf), 7 tanh, 8 param * tanh(. / param)
extern "C" int xft_gemm_f32(const float* X, int ldx, const float* W, int ldw, float* Y, int ldo, int T, int N, int K, int act,
                            const float* bias, const float* times, int ldt, float param, cudaStream_t st) {
  if (T <= 0 || N <= 0) return 0;
  if (K <= 0 || ldx < K || ldw < K || ldo < N || (times && ldt < N)) return -1;
  const int ty = (T + 63) / 64;
  if (ty > 65535) return -2;
  GemmF32 p{X, ldx, W, ldw, Y, ldo, T, N, K, act};
  p.bias = bias; p.times = times; p.ldt = ldt; p.param = param;
  gemm_f32_kernel<<<dim3((N + 63) / 64, ty), 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}

// One product per head: Y[:, h * ys + n] = sum_k X[:, h * xs + k] W[h * N + n, k]; W [heads * N, K].
extern "C" int xft_gemm_f32_heads(const float* X, int ldx, int xs, const float* W, float* Y, int ldo, int ys, int heads, int T,
                                  int N, int K, cudaStream_t st) {
  if (T <= 0 || N <= 0 || heads <= 0) return 0;
  if (K <= 0 || ldx < (heads - 1) * xs + K || ldo < (heads - 1) * ys + N || heads > 65535) return -1;
  const int ty = (T + 63) / 64;
  if (ty > 65535) return -2;
  GemmF32 p{X, ldx, W, K, Y, ldo, T, N, K, 0, xs, (long long)N * K, ys};
  gemm_f32_kernel<<<dim3((N + 63) / 64, ty, heads), 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}

// Products of rows sorted by group (experts): tiles of 64 rows from xft_moe_plan; src: row r is X[src[r]] (null: X[r]);
// row_w: factor of a row's result (null: none).  W [groups * group_w_rows, K].
extern "C" int xft_gemm_f32_grouped(const float* X, int ldx, const float* W, int ldw, float* Y, int ldo, int N, int K,
                                    int group_w_rows, const void* tiles, const int* num_tiles, int max_tiles, const int* src,
                                    const float* row_w, int act, cudaStream_t st) {
  if (max_tiles <= 0 || N <= 0) return 0;
  if (K <= 0 || ldx < K || ldw < K || ldo < N || max_tiles > 65535) return -1;
  GemmF32 p{X, ldx, W, ldw, Y, ldo, 0, N, K, act, 0, 0, 0, (const int4*)tiles, num_tiles, src, row_w, group_w_rows};
  gemm_f32_kernel<<<dim3((N + 63) / 64, max_tiles), 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}

// per: columns that share a gate value
extern "C" int xft_sigmoid_gate(const void* x, int ldx, const void* gate, int ldg, void* out, int ldo, int T, int n, int per, int f32,
                                cudaStream_t st) {
  const size_t m = (size_t)T * n;
  if (!m) return 0;
  if (per < 1 || ldx < n || ldg < (n + per - 1) / per || ldo < n) return -1;
  const unsigned grid = (unsigned)((m + 255) / 256);
  if (f32) sigmoid_gate_kernel<float><<<grid, 256, 0, st>>>((const float*)x, ldx, (const float*)gate, ldg, (float*)out, ldo, T, n, per);
  else sigmoid_gate_kernel<bf16><<<grid, 256, 0, st>>>((const bf16*)x, ldx, (const bf16*)gate, ldg, (bf16*)out, ldo, T, n, per);
  return (int)cudaGetLastError();
}

// act 6: see ops.linear_gated ("clamped")
extern "C" int xft_gated_act_f32(const float* gu, int ld, float* out, int T, int I, int act, float limit, cudaStream_t st) {
  const size_t n = (size_t)T * I;
  if (!n) return 0;
  if (ld < 2 * I) return -1;
  gated_act_f32_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(gu, ld, out, T, I, act, limit);
  return (int)cudaGetLastError();
}

// f32: 1 = fp32 rows and cache, 0 = bf16.  hkv = 0: query heads only (a layer that reads another layer's cache).
extern "C" int xft_rope_cache(const void* qkv, int ldq, int T, int hq, int hkv, int kd, int vd, const int* positions,
                              const float* table, int rot, int style, int max_pos, void* q_out, void* kc, void* vc, int bs,
                              long long nslots, const int* slots, int f32, int* status, cudaStream_t st) {
  if (T <= 0) return 0;
  if (hq <= 0 || hkv < 0 || kd <= 0 || vd <= 0 || bs <= 0 || rot < 0 || rot > kd || (rot & 1) ||
      ldq < (hq + hkv) * kd + hkv * vd || (rot > 0 && !table)) return -1;
  if (rot == 0) table = nullptr;
  const long long warps = (long long)T * (hq + 2 * hkv);
  const unsigned grid = (unsigned)((warps + 3) / 4);
  if (f32)
    rope_cache_kernel<float><<<grid, 128, 0, st>>>((const float*)qkv, ldq, T, hq, hkv, kd, vd, positions, table, rot, style,
                                                   max_pos, (float*)q_out, (float*)kc, (float*)vc, bs, nslots, slots, status);
  else
    rope_cache_kernel<bf16><<<grid, 128, 0, st>>>((const bf16*)qkv, ldq, T, hq, hkv, kd, vd, positions, table, rot, style,
                                                  max_pos, (bf16*)q_out, (bf16*)kc, (bf16*)vc, bs, nslots, slots, status);
  return (int)cudaGetLastError();
}

// q [T, hq, kd], caches [num_blocks, hkv, bs, kd] and [num_blocks, hkv, bs, vld], out [T, hq, vd], all fp32 (f32 = 1) or
// bf16; values are the first vd of vld columns (latent attention: vc = kc, vld = kd).  window 0: every earlier key; softcap 0: none; sinks null: none.
extern "C" int xft_attention_plain(const void* q, void* out, const void* kc, const void* vc, const int* block_table,
                                   int bt_stride, const int* cu_q, const int* kv_lens, int B, int T, int hq, int hkv, int group,
                                   int q_off, int kd, int vd, int vld, int bs, int num_blocks, float scale, float softcap,
                                   int window, int keep, const float* sinks, int f32, int* status, cudaStream_t st) {
  if (B <= 0 || T <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || group <= 0 || kd <= 0 || vd <= 0 || vld < vd || bs <= 0 || softcap < 0.f || window < 0 || keep < 0) return -1;
  if ((long long)num_blocks * hkv * bs >= (1ll << 31)) return -2;
  const size_t smem = (size_t)4 * (kd + vd + 64) * sizeof(float);
  if (smem > 200 * 1024) return -3;
  const int win = window > 0 ? (window < (1 << 30) ? window : 1 << 30) : 1 << 30;
  const int kp = window > 0 ? keep : 0;
  const unsigned grid = (unsigned)(((long long)T * hq + 3) / 4);
  if (f32) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(attention_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    attention_plain_kernel<float><<<grid, 128, smem, st>>>((const float*)q, (float*)out, (const float*)kc, (const float*)vc,
                                                           block_table, bt_stride, cu_q, kv_lens, B, T, hq, hkv, group, q_off,
                                                           kd, vd, vld, bs, num_blocks, scale, softcap, win, kp, sinks, status);
  } else {
    if (smem > 48 * 1024) cudaFuncSetAttribute(attention_plain_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    attention_plain_kernel<bf16><<<grid, 128, smem, st>>>((const bf16*)q, (bf16*)out, (const bf16*)kc, (const bf16*)vc,
                                                          block_table, bt_stride, cu_q, kv_lens, B, T, hq, hkv, group, q_off,
                                                          kd, vd, vld, bs, num_blocks, scale, softcap, win, kp, sinks, status);
  }
  return (int)cudaGetLastError();
}
