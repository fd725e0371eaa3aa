// What happens to the heads of attention whose values are its keys, between the projection and the paged cache, in one
// launch: a causal convolution over time on every channel of q and k, then on the heads an RMS norm and the rotation of
// their first dimensions.  The keys as they leave the convolution are the values.
//
//   u  rows [T, (hq + hkv) * dim] of the projection (bias included), u_t = 0 before a sequence's first token
//   y_t = sum_j w[j] u_(t - taps + 1 + j)           per channel
//   q, k = rotate(y / sqrt(mean(y^2) + eps) * gain)  per head;   v = y of the key heads
//
// The last taps - 1 rows of u that a sequence has seen are its state; a portion starts from them and leaves its own.  A
// state slot is never cleared: rows in front of a sequence's first token are taken as zero by position.
//
// One warp per head and run of consecutive tokens: weights, gains and the convolution's window stay in registers, a lane
// owns two or four neighbouring channels.  Heads are stored `padded` wide (zeros behind dim), as the attention kernels
// take them.  In a decode step the warp that reads a state also moves it on; otherwise a second, small kernel does, after
// all portions have read theirs.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

struct HeadPrepParams {
  const void* x; int ldx; int T, B, hq, hkv, dim, padded, taps;
  const float* conv;                       // [taps, (hq + hkv) * dim] or null (taps 1)
  const float* q_norm; const float* k_norm;          // [dim] or null
  float eps;
  const int* positions; const float* table; int rot, max_pos;      // table [max_pos, rot]: cosines | sines
  const int* cu_q; const int* kv_lens;
  void* state; const int* state_slots; int num_states;             // [slots, taps - 1, (hq + hkv) * dim]
  void* q_out; void* kc; void* vc; int bs; long long nslots; const int* slots;
  int run, decode;                         // tokens per warp; decode: one token per sequence, states move on here
  int* status;
};

template <typename T> __device__ __forceinline__ float hp_f32(T v);
template <> __device__ __forceinline__ float hp_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float hp_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T hp_from(float v);
template <> __device__ __forceinline__ float hp_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 hp_from<bf16>(float v) { return __float2bfloat16(v); }

template <int VEC>
__device__ __forceinline__ void hp_pack(float (&e)[VEC], const float (&v)[VEC]) {
#pragma unroll
  for (int k = 0; k < VEC; ++k) e[k] = v[k];
}
template <int VEC>
__device__ __forceinline__ void hp_pack(bf16 (&e)[VEC], const float (&v)[VEC]) {
#pragma unroll
  for (int k = 0; k < VEC; k += 2) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[k], v[k + 1]);
    e[k] = b.x;
    e[k + 1] = b.y;
  }
}

// VEC neighbouring channels of a row, `left` of which exist; whole: they are aligned and exist all or not at all
template <int VEC, typename T>
__device__ __forceinline__ void hp_load(const T* p, int left, bool whole, float (&v)[VEC]) {
  if (whole) {
    struct alignas(VEC * sizeof(T)) V { T e[VEC]; };
    V r;
    if (left > 0) r = *reinterpret_cast<const V*>(p);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = left > 0 ? hp_f32<T>(r.e[k]) : 0.f;
  } else {
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = k < left ? hp_f32<T>(p[k]) : 0.f;
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void hp_store(T* p, const float (&v)[VEC], int left, bool whole) {
  if (whole) {
    struct alignas(VEC * sizeof(T)) V { T e[VEC]; };
    V r;
    hp_pack<VEC>(r.e, v);
    if (left > 0) *reinterpret_cast<V*>(p) = r;
  } else {
#pragma unroll
    for (int k = 0; k < VEC; ++k) if (k < left) p[k] = hp_from<T>(v[k]);
  }
}

__device__ __forceinline__ int hp_sequence(const int* cu_q, int B, int t) {       // the sequence that owns token t
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// A lane owns VEC neighbouring channels of every 32 VEC, NV times (padded <= 32 VEC NV); TAPS >= taps.  VEC 4: dim, row
// strides and half the rotated dimensions are multiples of 4.
template <typename T, int VEC, int NV, int TAPS>
__global__ void __launch_bounds__(128, (TAPS + 3) * NV * VEC <= 28 ? 6 : 1) head_prep_kernel(const HeadPrepParams p) {
  extern __shared__ __align__(16) float hp_sm[];
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = p.hq + p.hkv, C = heads * p.dim;
  const long long gw = (long long)blockIdx.x * 4 + warp;
  const int t0 = (int)(gw / heads) * p.run, h = (int)(gw % heads);
  if (t0 >= p.T) { grid_dep_wait(); return; }
  const int t1 = min(t0 + p.run, p.T);
  const bool is_k = h >= p.hq;
  const bool whole = VEC == 4 || (p.dim & 1) == 0, out_whole = VEC == 4 || (p.padded & 1) == 0;
  float* row = hp_sm + warp * ((p.dim + 3) & ~3);
  const int skip = TAPS - p.taps;                        // leading taps that do not exist
  float w[TAPS][NV][VEC], gain[NV][VEC];
  const float* norm = is_k ? p.k_norm : p.q_norm;
  auto chan = [&](int i) { return VEC * lane + 32 * VEC * i; };
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = chan(i), left = p.dim - c;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      if (j >= skip && p.conv) {
        hp_load<VEC>(p.conv + (size_t)(j - skip) * C + h * p.dim + c, left, whole, w[j][i]);
      } else {
#pragma unroll
        for (int k = 0; k < VEC; ++k) w[j][i][k] = j < skip ? 0.f : 1.f;
      }
    }
    if (norm) hp_load<VEC>(norm + c, left, whole, gain[i]);
  }
  grid_dep_wait();
  const T* x = reinterpret_cast<const T*>(p.x) + h * p.dim;
  T* state = reinterpret_cast<T*>(p.state);
  int b = hp_sequence(p.cu_q, p.B, t0);
  float u[TAPS][NV][VEC], next[NV][VEC];                 // the window, newest last; the row behind it
#pragma unroll
  for (int i = 0; i < NV; ++i) hp_load<VEC>(x + (size_t)t0 * p.ldx + chan(i), p.dim - chan(i), whole, next[i]);
  int start = p.cu_q[b], end = p.cu_q[b + 1];
  int next_pos = p.rot > 0 ? p.positions[t0] : 0, next_slot = is_k ? p.slots[t0] : 0;
  const float inv_dim = 1.f / (float)p.dim;
  const int half = p.rot >> 1;
  bool fresh = true;
  for (int t = t0; t < t1; ++t) {
    while (b + 1 < p.B && t >= end) { ++b; start = end; end = p.cu_q[b + 1]; fresh = true; }
    const int li = t - start;
    // rotation: the angles' cosines and sines are on their way while the convolution runs
    float cosv[NV][VEC], sinv[NV][VEC];
    const int slot = next_slot;
    if (p.rot > 0) {
      int pos = next_pos;
      if (pos < 0 || pos >= p.max_pos) { if (lane == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); pos = 0; }
      const float* cs = p.table + (size_t)pos * p.rot;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = chan(i);
        if (c >= p.rot) continue;                        // rot is a multiple of VEC
        if (VEC == 4) {                                  // all of them in the same half
          const int f = c >= half ? c - half : c;
          hp_load<VEC>(cs + f, VEC, true, cosv[i]);
          hp_load<VEC>(cs + half + f, VEC, true, sinv[i]);
        } else {
#pragma unroll
          for (int k = 0; k < VEC; ++k) {
            const int f = c + k >= half ? c + k - half : c + k;
            cosv[i][k] = cs[f];
            sinv[i][k] = cs[half + f];
          }
        }
      }
    }
    if (t + 1 < t1) {
      if (p.rot > 0) next_pos = p.positions[t + 1];
      if (is_k) next_slot = p.slots[t + 1];
    }
    T* st = nullptr;
    if (p.taps > 1 && (fresh || p.decode)) {
      int s = p.state_slots[b];
      if (s < 0 || s >= p.num_states) { if (lane == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); s = 0; }
      st = state + (size_t)s * (p.taps - 1) * C + h * p.dim;
    }
    if (fresh) {
      const int past = p.kv_lens[b] - (end - start);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int idx = li - (TAPS - 1) + j;             // place in this portion; negative: before it
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = chan(i), left = p.dim - c;
          if (j >= skip && idx >= 0) hp_load<VEC>(x + (size_t)(start + idx) * p.ldx + c, left, whole, u[j][i]);
          else if (j >= skip && past + idx >= 0) hp_load<VEC>(st + (size_t)(p.taps - 1 + idx) * C + c, left, whole, u[j][i]);
          else {
#pragma unroll
            for (int k = 0; k < VEC; ++k) u[j][i][k] = 0.f;
          }
        }
      }
      fresh = false;
    }
    float y[NV][VEC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        u[TAPS - 1][i][k] = next[i][k];
        float a = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a = fmaf(w[j][i][k], u[j][i][k], a);
        y[i][k] = a;
        ss = fmaf(a, a, ss);
      }
      if (t + 1 < t1) hp_load<VEC>(x + (size_t)(t + 1) * p.ldx + chan(i), p.dim - chan(i), whole, next[i]);
    }
    if (p.decode && p.taps > 1) {                        // rows 1 .. taps - 1 of the window are the new state
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
        if (j > skip)
#pragma unroll
          for (int i = 0; i < NV; ++i) hp_store<VEC>(st + (size_t)(j - 1 - skip) * C + chan(i), u[j][i], p.dim - chan(i), whole);
    }
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int k = 0; k < VEC; ++k) u[j][i][k] = u[j + 1][i][k];
    T* dst;
    if (is_k) {
      if (slot < 0 || slot >= p.nslots) { if (lane == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); continue; }
      const int blk = slot / p.bs;
      const size_t at = ((size_t)(blk * p.hkv + (h - p.hq)) * p.bs + (slot - blk * p.bs)) * p.padded;
      dst = reinterpret_cast<T*>(p.kc) + at;
      T* v = reinterpret_cast<T*>(p.vc) + at;
#pragma unroll
      for (int i = 0; i < NV; ++i) hp_store<VEC>(v + chan(i), y[i], p.padded - chan(i), out_whole);
    } else {
      dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.hq + h) * p.padded;
    }
    if (norm) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = rsqrtf(ss * inv_dim + p.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[i][k] *= inv * gain[i][k];
    }
    if (p.rot > 0) {
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NV; ++i) hp_store<VEC>(row + chan(i), y[i], p.dim - chan(i), VEC == 4);
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = chan(i);
        if (c >= p.rot) continue;
        float other[VEC];
        if (VEC == 4) {
          hp_load<VEC>(row + (c >= half ? c - half : c + half), VEC, true, other);
        } else {
#pragma unroll
          for (int k = 0; k < VEC; ++k) other[k] = row[c + k >= half ? c + k - half : c + k + half];
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[i][k] = y[i][k] * cosv[i][k] + (c + k >= half ? other[k] : -other[k]) * sinv[i][k];
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) hp_store<VEC>(dst + chan(i), y[i], p.padded - chan(i), out_whole);
  }
}

// States of portions: row r of the new state is the row of u at distance taps - 1 - r from the portion's end.  A thread owns a
// channel and goes upwards, so the old rows it still needs lie above the ones it has written.
template <typename T>
__global__ void __launch_bounds__(256) conv_state_kernel(const T* __restrict__ x, int ldx, int C, int taps, const int* __restrict__ cu_q,
                                                         const int* __restrict__ kv_lens, T* state, const int* __restrict__ state_slots,
                                                         int num_states, int* status) {
  grid_dep_launch();
  grid_dep_wait();
  const int b = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C) return;
  const int start = cu_q[b], n = cu_q[b + 1] - start, past = kv_lens[b] - n;
  if (n <= 0) return;
  const int slot = state_slots[b];
  if (slot < 0 || slot >= num_states) { if (status) atomicCAS(status, 0, XFT_ERR_BOUNDS); return; }
  T* st = state + (size_t)slot * (taps - 1) * C + c;
  for (int r = 0; r < taps - 1; ++r) {
    const int idx = n - (taps - 1) + r;
    T v = hp_from<T>(0.f);
    if (idx >= 0) v = x[(size_t)(start + idx) * ldx + c];
    else if (past + idx >= 0) v = st[(size_t)(taps - 1 + idx) * C];
    st[(size_t)r * C] = v;
  }
}

}  // namespace xft

using namespace xft;

template <typename T, int VEC, int NV, int TAPS>
static cudaError_t launch_head_prep(const HeadPrepParams& p, cudaStream_t st) {
  const long long warps = (long long)((p.T + p.run - 1) / p.run) * (p.hq + p.hkv);
  return launch_pdl(head_prep_kernel<T, VEC, NV, TAPS>, dim3((unsigned)((warps + 3) / 4)), dim3(128),
                    (size_t)4 * ((p.dim + 3) / 4 * 4) * sizeof(float), st, p);
}
template <typename T, int VEC, int NV>
static cudaError_t pick_taps(const HeadPrepParams& p, cudaStream_t st) {
  if (p.taps <= 1) return launch_head_prep<T, VEC, NV, 1>(p, st);
  if (p.taps <= 2) return launch_head_prep<T, VEC, NV, 2>(p, st);
  if (p.taps <= 4) return launch_head_prep<T, VEC, NV, 4>(p, st);
  return launch_head_prep<T, VEC, NV, 8>(p, st);
}
template <typename T>
static cudaError_t pick_width(const HeadPrepParams& p, cudaStream_t st) {
  if (p.dim % 4 == 0 && p.padded % 4 == 0 && p.ldx % 4 == 0 && p.rot % 8 == 0) {
    if (p.padded <= 128) return pick_taps<T, 4, 1>(p, st);
    if (p.padded <= 256) return pick_taps<T, 4, 2>(p, st);
    return pick_taps<T, 4, 4>(p, st);
  }
  if (p.padded <= 64) return pick_taps<T, 2, 1>(p, st);
  if (p.padded <= 128) return pick_taps<T, 2, 2>(p, st);
  if (p.padded <= 256) return pick_taps<T, 2, 4>(p, st);
  return pick_taps<T, 2, 8>(p, st);
}

// The convolution's state [slots, taps - 1, C] behind a call's portions, from its input rows x [T, ldx] and the old state.
extern "C" int xft_conv_state(const void* x, int ldx, int C, int taps, const int* cu_q, const int* kv_lens, int B, void* state,
                              const int* state_slots, int num_states, int f32, int* status, cudaStream_t st) {
  const dim3 grid((C + 255) / 256, B);
  cudaError_t e = f32 ? launch_pdl(conv_state_kernel<float>, grid, dim3(256), 0, st, (const float*)x, ldx, C, taps, cu_q, kv_lens,
                                   (float*)state, state_slots, num_states, status)
                      : launch_pdl(conv_state_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)x, ldx, C, taps, cu_q, kv_lens,
                                   (bf16*)state, state_slots, num_states, status);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// x rows, q_out, caches and state all fp32 (f32 = 1) or bf16.  caches [blocks, hkv, bs, padded].  dim <= padded <= 512, up to 8
// taps; even dim wants even row strides.  decode: every sequence has one token in this call.
extern "C" int xft_head_prep(const void* x, int ldx, int T, int B, int hq, int hkv, int dim, int padded, int taps, const float* conv,
                             const float* q_norm, const float* k_norm, float eps, const int* positions, const float* table, int rot,
                             int max_pos, const int* cu_q, const int* kv_lens, void* state, const int* state_slots, int num_states,
                             void* q_out, void* kc, void* vc, int bs, long long nslots, const int* slots, int decode, int f32,
                             int* status, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  const int C = (hq + hkv) * dim;
  if (hq <= 0 || hkv <= 0 || dim <= 0 || padded < dim || padded > 512 || taps < 1 || taps > 8 || ldx < C || bs <= 0) return -1;
  if (rot < 0 || rot > dim || (rot & 1) || (rot > 0 && !table) || (taps > 1 && (!conv || !state || !state_slots || num_states <= 0))) return -2;
  if ((dim & 1) == 0 && (ldx & 1)) return -3;
  if (B > 65535) return -4;
  const int run = decode || T < 2048 ? 1 : T < 8192 ? 8 : 16;
  HeadPrepParams p{x, ldx, T, B, hq, hkv, dim, padded, taps, conv, q_norm, k_norm, eps, positions, table, rot, max_pos, cu_q, kv_lens,
                   state, state_slots, num_states, q_out, kc, vc, bs, nslots, slots, run, decode, status};
  cudaError_t e = f32 ? pick_width<float>(p, st) : pick_width<bf16>(p, st);
  if (e != cudaSuccess) return (int)e;
  if (taps > 1 && !decode) return xft_conv_state(x, ldx, C, taps, cu_q, kv_lens, B, state, state_slots, num_states, f32, status, st);
  return (int)cudaGetLastError();
}
