// Attention whose heads' weights are mixed, for any size in fp32 or bf16, and the step in front of it:
//
//   xft_talking_prep    RMS norms over all of a row's q and over all of its k; appends k to the key cache and k as it was in front
//                       of the norm to the value cache
//   xft_talking_plain   scores q . k scale - r1 ln(1 + r2 (i - j)), a softmax per head over the keys within the window, head h's
//                       weights sum_g talk[h, g] weight_g applied to the values of its own key/value head, output gate
//
// The weights of all heads of a (query, key) pair meet in the mix, so a CTA takes a query token with all of its heads, and the
// softmax is done with before a weight is mixed: the keys are visited twice.  The tensor-core forms are in talking_mma.cu.
// This file is compiled without fast-math.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float tk_f32(T v);
template <> __device__ __forceinline__ float tk_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float tk_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T tk_from(float v);
template <> __device__ __forceinline__ float tk_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 tk_from<bf16>(float v) { return __float2bfloat16(v); }

// ------------------------------------------------------------------------------------------ norms + append
struct TalkingPrepParams {
  const void* x; int ldx; int k_at;
  int hq, hkv, dim, padded;
  const float* q_norm; const float* k_norm; float eps;
  void* q_out; void* kc; void* vc; int bs; long long nslots; const int* slots;
  int* status;
};

// one CTA per (token, q or k)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) talking_prep_kernel(const TalkingPrepParams p) {
  struct alignas(VEC * sizeof(T)) V { T e[VEC]; };
  __shared__ float sh[8];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const bool is_k = blockIdx.y != 0;
  const int heads = is_k ? p.hkv : p.hq, n = heads * p.dim;
  const T* row = reinterpret_cast<const T*>(p.x) + (size_t)t * p.ldx + (is_k ? p.k_at : 0);
  const float* gain = is_k ? p.k_norm : p.q_norm;
  float ss = 0.f;
  for (int i = tid * VEC; i < n; i += 256 * VEC) {
    const V v = *reinterpret_cast<const V*>(row + i);
#pragma unroll
    for (int k = 0; k < VEC; ++k) { const float f = tk_f32<T>(v.e[k]); ss = fmaf(f, f, ss); }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) sh[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += sh[i];
  const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
  long long slot = 0;
  if (is_k) {
    slot = p.slots[t];
    if (slot < 0 || slot >= p.nslots) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); return; }
  }
  const int per = p.padded / VEC;                          // pieces of a head; those behind dim are zeros
  for (int i = tid; i < heads * per; i += 256) {
    const int h = i / per, c = (i - h * per) * VEC;
    V v, y;
    if (c < p.dim) v = *reinterpret_cast<const V*>(row + h * p.dim + c);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      if (c >= p.dim) v.e[k] = tk_from<T>(0.f);
      y.e[k] = c < p.dim ? tk_from<T>(tk_f32<T>(v.e[k]) * inv * gain[h * p.dim + c + k]) : tk_from<T>(0.f);
    }
    if (is_k) {
      const size_t at = ((size_t)((slot / p.bs) * p.hkv + h) * p.bs + slot % p.bs) * p.padded + c;
      *reinterpret_cast<V*>(reinterpret_cast<T*>(p.kc) + at) = y;
      *reinterpret_cast<V*>(reinterpret_cast<T*>(p.vc) + at) = v;
    } else {
      *reinterpret_cast<V*>(reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.hq + h) * p.padded + c) = y;
    }
  }
}

// ------------------------------------------------------------------------------------------ plain attention
struct TalkingPlainParams {
  const void* q; const void* gate; int ldg; void* out; int ldo;
  const void* kc; const void* vc; const int* block_table; int bt_stride;
  const int* cu_q; const int* kv_lens;
  int B, hq, hkv, D, bs, num_blocks, window;
  float scale, mult;
  const float* r1; const float* r2; const float* talk;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(256) talking_plain_kernel(const TalkingPlainParams p) {
  extern __shared__ float tp_sm[];
  const int H = p.hq, D = p.D, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* qs = tp_sm;                                       // [H][D]
  float* acc = qs + H * D;                                 // [H][D]
  float* ps = acc + H * D;                                 // [H][32] weights, and mixed
  float* ws = ps + H * 32;
  float* sm = ws + H * 32;                                 // [H] maxima and sums
  float* sl = sm + H;
  int* rs = reinterpret_cast<int*>(sl + H);                // [32] cache rows of head 0
  const int t = blockIdx.x;
  int b = 0;
  {
    int hi = p.B - 1;
    while (b < hi) { const int mid = (b + hi + 1) >> 1; if (p.cu_q[mid] <= t) b = mid; else hi = mid - 1; }
  }
  const int qpos = p.kv_lens[b] - (p.cu_q[b + 1] - p.cu_q[b]) + (t - p.cu_q[b]);
  const int lo = max(0, qpos - p.window + 1), total = qpos + 1 - lo, group = H / p.hkv;
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * H * D;
  for (int i = tid; i < H * D; i += 256) { qs[i] = tk_f32<T>(q[i]); acc[i] = 0.f; }
  for (int i = tid; i < H; i += 256) { sm[i] = -INFINITY; sl[i] = 0.f; }
  const int* bt = p.block_table + (size_t)b * p.bt_stride;
  const T* kc = reinterpret_cast<const T*>(p.kc);
  const T* vc = reinterpret_cast<const T*>(p.vc);
  for (int pass = 0; pass < 2; ++pass) {
    for (int n0 = 0; n0 < total; n0 += 32) {
      const int cnt = min(32, total - n0);
      __syncthreads();
      if (tid < 32) {
        const int key = lo + n0 + min(tid, cnt - 1);
        int blk = bt[key / p.bs];
        if (blk < 0 || blk >= p.num_blocks) { if (p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); blk = 0; }
        rs[tid] = blk * p.hkv * p.bs + key % p.bs;
      }
      __syncthreads();
      for (int h = warp; h < H; h += 8) {
        const T* kp = kc + (size_t)(rs[lane] + h / group * p.bs) * D;
        float dot = 0.f;
        for (int d = 0; d < D; ++d) dot = fmaf(qs[h * D + d], tk_f32<T>(kp[d]), dot);
        const float far = (float)(qpos - (lo + n0 + lane));
        const float s = lane < cnt ? dot * p.scale - p.r1[h] * log1pf(p.r2[h] * far) : -INFINITY;
        if (pass == 0) {
          float mx = s;
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
          const float m = sm[h], mn = fmaxf(m, mx);
          float e = lane < cnt ? expf(s - mn) : 0.f;
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) e += __shfl_xor_sync(0xffffffffu, e, o);
          __syncwarp();
          if (lane == 0) { sl[h] = sl[h] * (m == -INFINITY ? 0.f : expf(m - mn)) + e; sm[h] = mn; }
          __syncwarp();
        } else {
          ps[h * 32 + lane] = lane < cnt ? expf(s - sm[h]) / sl[h] : 0.f;
        }
      }
      if (pass == 0) continue;
      __syncthreads();
      for (int i = tid; i < H * 32; i += 256) {
        const int h = i >> 5;
        float w = 0.f;
        for (int g = 0; g < H; ++g) w = fmaf(p.talk[h * H + g], ps[g * 32 + (i & 31)], w);
        ws[i] = w;
      }
      __syncthreads();
      for (int i = tid; i < H * D; i += 256) {
        const int h = i / D, d = i - h * D;
        float a = acc[i];
        for (int k = 0; k < cnt; ++k) a = fmaf(ws[h * 32 + k], tk_f32<T>(vc[(size_t)(rs[k] + h / group * p.bs) * D + d]), a);
        acc[i] = a;
      }
    }
  }
  const T* gate = reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ldg;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
  for (int i = tid; i < H * D; i += 256) out[i] = tk_from<T>(acc[i] / (1.f + expf(-tk_f32<T>(gate[i]))) * p.mult);
}

}  // namespace xft

using namespace xft;

// x rows [q: hq x dim | (from k_at) k: hkv x dim], q_out [T, hq, padded], caches [blocks, hkv, bs, padded], all fp32 (f32 = 1) or bf16.
extern "C" int xft_talking_prep(const void* x, int ldx, int T, int k_at, int hq, int hkv, int dim, int padded, const float* q_norm,
                                const float* k_norm, float eps, void* q_out, void* kc, void* vc, int bs, long long nslots, const int* slots,
                                int f32, int* status, cudaStream_t st) {
  if (T <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || dim <= 0 || padded < dim || k_at < hq * dim || ldx < k_at + hkv * dim || bs <= 0) return -1;
  TalkingPrepParams p{x, ldx, k_at, hq, hkv, dim, padded, q_norm, k_norm, eps, q_out, kc, vc, bs, nslots, slots, status};
  const bool vec = ((dim | padded | ldx | k_at) & 7) == 0 && (((uintptr_t)x | (uintptr_t)q_out | (uintptr_t)kc | (uintptr_t)vc) & 15) == 0;
  const dim3 grid(T, 2);
  cudaError_t e;
  if (f32) e = vec ? launch_pdl(talking_prep_kernel<float, 4>, grid, dim3(256), 0, st, p) : launch_pdl(talking_prep_kernel<float, 1>, grid, dim3(256), 0, st, p);
  else e = vec ? launch_pdl(talking_prep_kernel<bf16, 8>, grid, dim3(256), 0, st, p) : launch_pdl(talking_prep_kernel<bf16, 1>, grid, dim3(256), 0, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// q [T, hq, D], gate and out [T, ld] (head h at columns h * D), caches [num_blocks, hkv, bs, D], all fp32 (f32 = 1) or bf16; r1, r2 [hq],
// talk [hq, hq] fp32.  window 0: every earlier key.  Results are multiplied with sigmoid(gate) and mult.
extern "C" int xft_talking_plain(const void* q, const void* gate, int ldg, void* out, int ldo, const void* kc, const void* vc,
                                 const int* block_table, int bt_stride, const int* cu_q, const int* kv_lens, int B, int T, int hq, int hkv,
                                 int D, int bs, int num_blocks, float scale, const float* r1, const float* r2, const float* talk, int window,
                                 float mult, int f32, int* status, cudaStream_t st) {
  if (B <= 0 || T <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || hq % hkv || D <= 0 || bs <= 0 || window < 0 || ldg < hq * D || ldo < hq * D) return -1;
  if ((long long)num_blocks * hkv * bs >= (1ll << 31)) return -2;
  const size_t smem = ((size_t)2 * hq * D + 66 * hq + 32) * sizeof(float);
  if (smem > 200 * 1024) return -3;
  TalkingPlainParams p{q, gate, ldg, out, ldo, kc, vc, block_table, bt_stride, cu_q, kv_lens, B, hq, hkv, D, bs, num_blocks,
                       window > 0 ? min(window, 1 << 30) : 1 << 30, scale, mult, r1, r2, talk, status};
  if (f32) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(talking_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    talking_plain_kernel<float><<<T, 256, smem, st>>>(p);
  } else {
    if (smem > 48 * 1024) cudaFuncSetAttribute(talking_plain_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    talking_plain_kernel<bf16><<<T, 256, smem, st>>>(p);
  }
  return (int)cudaGetLastError();
}
