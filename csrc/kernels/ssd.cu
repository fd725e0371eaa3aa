// State-space layers (Mamba-2) and the input mixes of time mixing: what stands around the recurrences of gla.cu, and the
// recurrence of state-space layers over portions.
//
//   xft_channel_conv   silu(causal convolution + bias) of a run of channels, the last inputs kept as a state
//   xft_ssd_chunk      portions of the recurrence, 64 tokens at a time on the tensor cores
//   xft_gated_norm     y * silu(z), normalised in equal parts by their root mean square, times a gain
//   xft_token_shift    mixes of every row with the row of the token before it
//
// The recurrence per head, with dt_t = softplus(raw_t + bias) and a_t = -rate dt_t:
//
//   S_t = exp(a_t) S_(t-1) + dt_t B_t x_t^T        state x vdim, fp32
//   y_t = S_t^T C_t + D x_t
//
// In chunks, with L_t the running sum of a within the chunk (fp32):
//
//   y   = exp(L_t) C S + (tril(C B^T) * exp(L_t - L_s) dt_s) x + D x
//   S  <- exp(L_end) S + B^T (dt_s exp(L_end - L_s) x)
//
// All exponents are at most zero, whatever the decays.  The state stays in registers as the accumulator of its product; the
// products take bf16 operands.  Single tokens, short portions and fp32 run the step kernel of gla.cu (xft_ssd_step).
// This file is compiled without fast-math.
#include "mma_sync.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float ss_f32(T v);
template <> __device__ __forceinline__ float ss_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float ss_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T ss_from(float v);
template <> __device__ __forceinline__ float ss_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 ss_from<bf16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ int ss_sequence(const int* cu_q, int B, int t) {       // the sequence that owns token t
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}
__device__ __forceinline__ int ss_slot(const int* slots, int b, int num, int* status) {
  const int s = slots[b];
  if (s >= 0 && s < num) return s;
  if (status) atomicCAS(status, 0, XFT_ERR_BOUNDS);
  return 0;
}

// x * sigmoid(x): accurate in fp32, with the approximate instructions for bf16 results
template <typename T> __device__ __forceinline__ float ss_silu(float x);
template <> __device__ __forceinline__ float ss_silu<float>(float x) { return x / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float ss_silu<bf16>(float x) { return x * gl_rcp(1.f + gl_ex2(-x * 1.4426950408889634f)); }

// ------------------------------------------------------------------------------------------ convolution over time
struct ChannelConvParams {
  const void* x; int ldx; int T, B, C, taps;               // x points at the first channel
  const float* w; const float* bias;                       // [taps, C], [C]
  const int* cu_q; const int* kv_lens;
  void* state; const int* state_slots; int num_states;     // [slots, taps - 1, C]
  void* out; int ldo;
  int run, decode;                                         // tokens per thread; decode: one token per sequence, states move on here
  int* status;
};

// A thread owns VEC neighbouring channels and a run of tokens; the convolution's window stays in registers.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) channel_conv_kernel(const ChannelConvParams p) {
  struct alignas(VEC * sizeof(T)) V { T e[VEC]; };
  grid_dep_launch();
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, t0 = blockIdx.y * p.run, t1 = min(t0 + p.run, p.T);
  if (c >= p.C) { grid_dep_wait(); return; }               // C is a multiple of VEC
  const int skip = TAPS - p.taps;
  float w[TAPS][VEC], bias[VEC];
  auto row_of = [](const float* from, float (&v)[VEC]) {
    constexpr int N = VEC % 4 ? 1 : 4;
    struct alignas(4 * N) F { float e[N]; };
#pragma unroll
    for (int k = 0; k < VEC; k += N) {
      const F r = *reinterpret_cast<const F*>(from + k);
#pragma unroll
      for (int i = 0; i < N; ++i) v[k + i] = r.e[i];
    }
  };
  row_of(p.bias + c, bias);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    if (j >= skip) row_of(p.w + (size_t)(j - skip) * p.C + c, w[j]);
    else {
#pragma unroll
      for (int k = 0; k < VEC; ++k) w[j][k] = 0.f;
    }
  }
  grid_dep_wait();
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  auto load = [&](const T* from, float (&v)[VEC]) {
    const V r = *reinterpret_cast<const V*>(from);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = ss_f32<T>(r.e[k]);
  };
  int b = ss_sequence(p.cu_q, p.B, t0), start = p.cu_q[b], end = p.cu_q[b + 1];
  bool fresh = true;
  float u[TAPS][VEC];
  constexpr int AHEAD = 2;                                 // rows on their way while one is summed up
  V ahead[AHEAD];
#pragma unroll
  for (int s = 0; s < AHEAD; ++s)
    if (t0 + s < t1) ahead[s] = *reinterpret_cast<const V*>(x + (size_t)(t0 + s) * p.ldx);
  auto step = [&](int t, V& row) {
    while (b + 1 < p.B && t >= end) { ++b; start = end; end = p.cu_q[b + 1]; fresh = true; }
    const int li = t - start;
    T* st = nullptr;
    if (p.taps > 1 && (fresh || p.decode))
      st = reinterpret_cast<T*>(p.state) + (size_t)ss_slot(p.state_slots, b, p.num_states, p.status) * (p.taps - 1) * p.C + c;
    if (fresh) {
      const int past = p.kv_lens[b] - (end - start);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int idx = li - (TAPS - 1) + j;               // place in this portion; negative: before it
        if (j >= skip && idx >= 0) load(x + (size_t)(start + idx) * p.ldx, u[j]);
        else if (j >= skip && past + idx >= 0) load(st + (size_t)(p.taps - 1 + idx) * p.C, u[j]);
        else {
#pragma unroll
          for (int k = 0; k < VEC; ++k) u[j][k] = 0.f;
        }
      }
      fresh = false;
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) u[TAPS - 1][k] = ss_f32<T>(row.e[k]);
    if (t + AHEAD < t1) row = *reinterpret_cast<const V*>(x + (size_t)(t + AHEAD) * p.ldx);
    V y;
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      float a = bias[k];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) a = fmaf(w[j][k], u[j][k], a);
      y.e[k] = ss_from<T>(ss_silu<T>(a));
    }
    *reinterpret_cast<V*>(reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + c) = y;
    if (p.decode && p.taps > 1) {                          // rows 1 .. taps - 1 of the window are the new state
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
        if (j > skip) {
          V r;
#pragma unroll
          for (int k = 0; k < VEC; ++k) r.e[k] = ss_from<T>(u[j][k]);
          *reinterpret_cast<V*>(st + (size_t)(j - 1 - skip) * p.C) = r;
        }
    }
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int k = 0; k < VEC; ++k) u[j][k] = u[j + 1][k];
  };
  for (int t = t0; t < t1; t += AHEAD)
#pragma unroll
    for (int s = 0; s < AHEAD; ++s)
      if (t + s < t1) step(t + s, ahead[s]);
}

// ------------------------------------------------------------------------------------------ gate and grouped norm
// One CTA per (token, part); a thread has 8 neighbouring values up to twice.
__global__ void __launch_bounds__(1024) gated_norm_vec_kernel(const bf16* __restrict__ y, int ldy, const bf16* __restrict__ z, int ldz,
                                                             const float* __restrict__ gain, bf16* __restrict__ out, int ldo, int n, float eps) {
  __shared__ float sh[32];
  const int t = blockIdx.y, c0 = blockIdx.x * n, nt = blockDim.x;
  grid_dep_launch();
  grid_dep_wait();
  const bf16* yr = y + (size_t)t * ldy + c0;
  const bf16* zr = z + (size_t)t * ldz + c0;
  uint4 a[2], b[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = (threadIdx.x + k * nt) * 8;
    a[k] = b[k] = make_uint4(0, 0, 0, 0);
    if (i < n) { a[k] = *reinterpret_cast<const uint4*>(yr + i); b[k] = *reinterpret_cast<const uint4*>(zr + i); }
  }
  float v[16], ss = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 p = gl_unpack(reinterpret_cast<const uint32_t*>(&a[k])[j]), q = gl_unpack(reinterpret_cast<const uint32_t*>(&b[k])[j]);
      v[k * 8 + 2 * j] = p.x * ss_silu<bf16>(q.x);
      v[k * 8 + 2 * j + 1] = p.y * ss_silu<bf16>(q.y);
      ss = fmaf(v[k * 8 + 2 * j], v[k * 8 + 2 * j], fmaf(v[k * 8 + 2 * j + 1], v[k * 8 + 2 * j + 1], ss));
    }
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < (nt >> 5); ++i) ss += sh[i];
  const float inv = rsqrtf(ss / (float)n + eps);
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = (threadIdx.x + k * nt) * 8;
    if (i >= n) continue;
    const float4 g0 = *reinterpret_cast<const float4*>(gain + c0 + i), g1 = *reinterpret_cast<const float4*>(gain + c0 + i + 4);
    const float* w = v + k * 8;
    uint4 r;
    r.x = gl_pack(w[0] * inv * g0.x, w[1] * inv * g0.y);
    r.y = gl_pack(w[2] * inv * g0.z, w[3] * inv * g0.w);
    r.z = gl_pack(w[4] * inv * g1.x, w[5] * inv * g1.y);
    r.w = gl_pack(w[6] * inv * g1.z, w[7] * inv * g1.w);
    *reinterpret_cast<uint4*>(out + (size_t)t * ldo + c0 + i) = r;
  }
}

// Any size: a thread keeps up to 16 values; wider parts are read again.
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const T* __restrict__ y, int ldy, const T* __restrict__ z, int ldz,
                                                         const float* __restrict__ gain, T* __restrict__ out, int ldo, int n, float eps) {
  __shared__ float sh[8];
  grid_dep_launch();
  grid_dep_wait();
  const int t = blockIdx.y, c0 = blockIdx.x * n, nt = blockDim.x;
  const T* yr = y + (size_t)t * ldy + c0;
  const T* zr = z + (size_t)t * ldz + c0;
  auto value = [&](int i) { return ss_f32<T>(yr[i]) * ss_silu<T>(ss_f32<T>(zr[i])); };
  float v[16], ss = 0.f;
#pragma unroll
  for (int k = 0; k < 16; ++k) {
    const int i = threadIdx.x + k * nt;
    v[k] = i < n ? value(i) : 0.f;
    ss = fmaf(v[k], v[k], ss);
  }
  for (int i = threadIdx.x + 16 * nt; i < n; i += nt) { const float a = value(i); ss = fmaf(a, a, ss); }
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < (nt >> 5); ++i) ss += sh[i];
  const float inv = 1.f / sqrtf(ss / (float)n + eps);
  T* o = out + (size_t)t * ldo + c0;
#pragma unroll
  for (int k = 0; k < 16; ++k) {
    const int i = threadIdx.x + k * nt;
    if (i < n) o[i] = ss_from<T>(v[k] * inv * gain[c0 + i]);
  }
  for (int i = threadIdx.x + 16 * nt; i < n; i += nt) o[i] = ss_from<T>(value(i) * inv * gain[c0 + i]);
}

// ------------------------------------------------------------------------------------------ token shift
// Mix k of a row: x + (previous row - x) mu[k].  The CTA of a sequence's first token reads the row that the sequence left behind
// and replaces it by its last one.
template <typename T>
__global__ void __launch_bounds__(128) token_shift_kernel(const float* __restrict__ x, int ldx, int n_mix, int W, const float* __restrict__ mu,
                                                          const int* __restrict__ cu_q, const int* __restrict__ kv_lens, int B,
                                                          float* state, const int* __restrict__ state_slots, int num_states,
                                                          T* __restrict__ out, int* status) {
  grid_dep_launch();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4, t = blockIdx.y;
  grid_dep_wait();
  if (c >= W) return;                                      // W is a multiple of 4
  const int b = ss_sequence(cu_q, B, t), start = cu_q[b], end = cu_q[b + 1];
  const float4 v = *reinterpret_cast<const float4*>(x + (size_t)t * ldx + c);
  float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
  if (t > start) q = *reinterpret_cast<const float4*>(x + (size_t)(t - 1) * ldx + c);
  else {
    float4* st = reinterpret_cast<float4*>(state + (size_t)ss_slot(state_slots, b, num_states, status) * W + c);
    if (kv_lens[b] > end - start) q = *st;
    *st = *reinterpret_cast<const float4*>(x + (size_t)(end - 1) * ldx + c);
  }
  const float4 d = make_float4(q.x - v.x, q.y - v.y, q.z - v.z, q.w - v.w);
  for (int k = 0; k < n_mix; ++k) {
    const float4 m = *reinterpret_cast<const float4*>(mu + (size_t)k * W + c);
    struct alignas(4 * sizeof(T)) V { T e[4]; } r;
    r.e[0] = ss_from<T>(fmaf(d.x, m.x, v.x)); r.e[1] = ss_from<T>(fmaf(d.y, m.y, v.y));
    r.e[2] = ss_from<T>(fmaf(d.z, m.z, v.z)); r.e[3] = ss_from<T>(fmaf(d.w, m.w, v.w));
    *reinterpret_cast<V*>(out + ((size_t)t * n_mix + k) * W + c) = r;
  }
}

// ------------------------------------------------------------------------------------------ chunks of 64 tokens
struct SsdChunkParams {
  const bf16* u; int ldu; int b_at, c_at;                  // rows [x: heads x vdim | B | C: groups x state]
  const bf16* dt; int ld_dt;
  const float* dt_bias; const float* rate; const float* skip;
  int heads, per_group, state_n, vdim;
  float* state; const int* state_slots; int num_states;
  const int* cu_q; const int* kv_lens;
  bf16* y;                                                 // [T, heads * vdim]
  int min_q;
  int segs, carry;                                         // segments per portion; carry: the launch that runs the states alone
  float* seg_state;                                        // [B, heads, segs, state, vdim]: the initial state, then what segment j - 1 leaves
  float* seg_decay;                                        // [B, heads, segs]: sum of log2 of the decays of segment j - 1
  int* status;
};

constexpr int kSsdChunk = 64, kSsdThreads = 256;           // threads per head
template <int NP, int VS, int HPC>
struct SsdCfg {
  static constexpr int NS = NP + 8, XS = VS + 8, AS = kSsdChunk + 8;
  static constexpr int STAGE = kSsdChunk * (2 * NS + HPC * XS);            // C, B, x of every head of a chunk
  static constexpr int STAGES = NP <= 128 ? 2 : 1;
  static constexpr int HEAD = kSsdChunk * XS + NP * XS + kSsdChunk * AS;   // of a head: x with its factor, the state, scores
  static constexpr size_t SMEM = ((size_t)STAGES * STAGE + HPC * HEAD) * 2 + HPC * 2 * kSsdChunk * 4;
  static_assert(SMEM <= 227 * 1024, "shared memory");
};

// A CTA takes HPC heads that share B and C, with eight warps each.
template <int NP, int VS, int HPC>
__global__ void __launch_bounds__(kSsdThreads * HPC, 1) ssd_chunk_kernel(const SsdChunkParams p) {
  using Cfg = SsdCfg<NP, VS, HPC>;
  constexpr int NT = kSsdThreads * HPC, NS = Cfg::NS, XS = Cfg::XS, AS = Cfg::AS;
  constexpr int MT = NP / 16, SPLIT = MT < 8 ? 8 / MT : 1, MPW = MT < 8 ? 1 : MT / 8;    // the state: row tiles, column parts, tiles per warp
  constexpr int NSW = VS / 8 / SPLIT;                      // its 8-column tiles per warp
  constexpr int NO = VS / 16;                              // 8-column tiles of half the output columns
  static_assert(NSW % 2 == 0 && NO % 2 == 0, "warp tiles");
  extern __shared__ __align__(16) uint8_t sc_raw[];
  const int tid = threadIdx.x, lane = tid & 31, hw = tid / kSsdThreads, ht = tid % kSsdThreads, warp = ht >> 5;
  bf16* stage0 = reinterpret_cast<bf16*>(sc_raw);
  bf16* sX2 = stage0 + Cfg::STAGES * Cfg::STAGE + hw * Cfg::HEAD;          // x with its factor of the state's update
  bf16* sS = sX2 + kSsdChunk * XS;                         // the state as an operand [NP][XS]
  bf16* sA = sS + NP * XS;                                 // scores [64][AS]
  float* sL = reinterpret_cast<float*>(stage0 + Cfg::STAGES * Cfg::STAGE + HPC * Cfg::HEAD) + hw * 2 * kSsdChunk;   // running sums, base 2
  float* sDt = sL + kSsdChunk;
  const int h = blockIdx.y * HPC + hw, b = blockIdx.z, seg = blockIdx.x % p.segs, v0 = blockIdx.x / p.segs * VS;
  grid_dep_launch();
  const int start = p.cu_q[b], n = p.cu_q[b + 1] - start;
  const int chunks = (n + kSsdChunk - 1) / kSsdChunk, per_seg = (chunks + p.segs - 1) / p.segs;
  const int ch0 = seg * per_seg, ch1 = min(ch0 + per_seg, chunks);         // this CTA's chunks
  if (n < p.min_q || n <= 0 || ch0 >= chunks || (p.carry && ch1 == chunks)) { grid_dep_wait(); return; }
  const bool alone = per_seg >= chunks;                    // one segment has all of the portion
  const int past = p.kv_lens[b] - n;
  const int N = p.state_n, vw = min(VS, p.vdim - v0);
  const bool whole8 = (N & 7) == 0 && (p.vdim & 7) == 0 && (p.ldu & 7) == 0 && (p.b_at & 7) == 0 && (p.c_at & 7) == 0;
  float* st = p.state + ((size_t)ss_slot(p.state_slots, b, p.num_states, p.status) * p.heads + h) * N * p.vdim;
  for (int i = tid; i < Cfg::STAGES * Cfg::STAGE / 8; i += NT) reinterpret_cast<uint4*>(stage0)[i] = make_uint4(0, 0, 0, 0);
  // the state: MPW tiles of 16 rows, NSW x 8 columns; element e of tile (m, j): row sd + 128 m + 8 (e >> 1), column sc + 8 j + (e & 1)
  const int sd = (warp % (MT < 8 ? MT : 8)) * 16 + (lane >> 2), sn0 = MT < 8 ? warp / MT * NSW * 8 : 0, sc = sn0 + 2 * (lane & 3);
  float S[MPW][NSW][4];
  auto each_state = [&](auto f) {
#pragma unroll
    for (int m = 0; m < MPW; ++m)
#pragma unroll
      for (int j = 0; j < NSW; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = sd + m * 128 + (e >> 1) * 8, c = sc + j * 8 + (e & 1);
          f(S[m][j][e], (size_t)d * p.vdim + v0 + c, d < N && c < vw);
        }
  };
  each_state([&](float& v, size_t at, bool in) { v = past > 0 && seg == 0 && (alone || p.carry) && in ? st[at] : 0.f; });
  const float rate2 = p.rate[h] * 1.4426950408889634f, skip = p.skip[h], dtb = p.dt_bias[h];
  grid_dep_wait();
  float* seg_s = p.seg_state + ((size_t)b * p.heads + h) * p.segs * N * p.vdim;
  float* seg_d = p.seg_decay + ((size_t)b * p.heads + h) * p.segs;
  float carried = 0.f;                                     // carry: sum of the logarithms over the segment
  if (p.carry && seg == 0) {                               // the pool is written while later segments still start: keep a copy
    each_state([&](float& v, size_t at, bool in) { if (in) seg_s[at] = v; });
  } else if (!alone && !p.carry) {
    for (int k = seg == 0 ? 0 : 1; k <= seg; ++k) {
      const float f = k > 1 ? gl_ex2(seg_d[k]) : 1.f;
      const float* from = seg_s + (size_t)k * N * p.vdim;
      each_state([&](float& v, size_t at, bool in) { v = fmaf(v, f, in ? from[at] : 0.f); });
    }
  }
  __syncthreads();
  const bf16* u = p.u + (size_t)start * p.ldu;
  const int kg = h / p.per_group;                          // the same for all heads of the CTA
  auto load = [&](int ch) {
    bf16* sC = stage0 + (Cfg::STAGES > 1 ? (ch & 1) * Cfg::STAGE : 0);
    bf16* sB = sC + kSsdChunk * NS;
    bf16* sX = sB + kSsdChunk * NS + hw * kSsdChunk * XS;
    const int t0 = ch * kSsdChunk, rows = min(kSsdChunk, n - t0);
    auto part = [&](bf16* dst, int ld, int at, int width, int id, int nt) {
      if (whole8) {
        const int per = width >> 3, dr = nt / per, dc = nt % per;
        int r = id / per, c = id % per;
        while (r < kSsdChunk) {
          const bf16* src = u + (size_t)(t0 + min(r, rows - 1)) * p.ldu + at + c * 8;
          const int bytes = r < rows ? 16 : 0;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * ld + c * 8)), "l"(src), "r"(bytes) : "memory");
          r += dr;
          c += dc;
          if (c >= per) { c -= per; ++r; }
        }
      } else {
        for (int i = id; i < kSsdChunk * width; i += nt) {
          const int r = i / width, c = i - r * width;
          dst[r * ld + c] = r < rows ? u[(size_t)(t0 + r) * p.ldu + at + c] : __float2bfloat16(0.f);
        }
      }
    };
    if (!p.carry) part(sC, NS, p.c_at + kg * N, N, tid, NT);
    part(sB, NS, p.b_at + kg * N, N, tid, NT);
    part(sX, XS, h * p.vdim + v0, vw, ht, kSsdThreads);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto raw_dt = [&](int ch) {                              // of token ht of a chunk
    const int t = ch * kSsdChunk + ht;
    return ht < kSsdChunk && t < n ? __bfloat162float(p.dt[(size_t)(start + t) * p.ld_dt + h]) + dtb : -INFINITY;
  };
  const int fa_r = (lane & 7) + ((lane >> 3) & 1) * 8, fa_c = (lane >> 4) * 8;
  const int fb_r = (lane & 7) + ((lane >> 4) & 1) * 8, fb_c = ((lane >> 3) & 1) * 8;
  const int mt = warp & 3, half = warp >> 2, r0 = mt * 16 + (lane >> 2), cc = 2 * (lane & 3);
  load(ch0);
  float z = raw_dt(ch0);
  for (int ch = ch0; ch < ch1; ++ch) {
    bf16* sC = stage0 + (Cfg::STAGES > 1 ? (ch & 1) * Cfg::STAGE : 0);
    bf16* sB = sC + kSsdChunk * NS;
    bf16* sX = sB + kSsdChunk * NS + hw * kSsdChunk * XS;
    const int rows = min(kSsdChunk, n - ch * kSsdChunk);
    // step sizes and running sums: two warps per head, a token per lane
    if (warp < 2) {
      const float dt = z == -INFINITY ? 0.f : fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      float L = -rate2 * dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, L, o);
        if (lane >= o) L += v;
      }
      sL[ht] = L;
      sDt[ht] = dt;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // also: everyone is done with the chunk before
    if (Cfg::STAGES > 1 && ch + 1 < ch1) load(ch + 1);
    z = ch + 1 < ch1 ? raw_dt(ch + 1) : -INFINITY;
    const float half_sum = sL[31], end_sum = half_sum + sL[63];
    carried += end_sum;
    auto sum_at = [&](int t) { return sL[t] + (t >= 32 ? half_sum : 0.f); };
    // x with its factor; the state as an operand; the scores
    {
      const int c = ht % (VS / 2), dr = kSsdThreads / (VS / 2);
#pragma unroll 4
      for (int r = ht / (VS / 2); r < kSsdChunk; r += dr) {
        const float f = sDt[r] * gl_ex2(end_sum - sum_at(r));
        const float2 x = gl_unpack(*reinterpret_cast<const uint32_t*>(sX + r * XS + 2 * c));
        *reinterpret_cast<uint32_t*>(sX2 + r * XS + 2 * c) = gl_pack(x.x * f, x.y * f);
      }
    }
    const float l0 = sum_at(r0), l1 = sum_at(r0 + 8);
    if (!p.carry) {
#pragma unroll
      for (int m = 0; m < MPW; ++m)
#pragma unroll
        for (int j = 0; j < NSW; ++j) {
          *reinterpret_cast<uint32_t*>(sS + (sd + m * 128) * XS + sc + j * 8) = gl_pack(S[m][j][0], S[m][j][1]);
          *reinterpret_cast<uint32_t*>(sS + (sd + m * 128 + 8) * XS + sc + j * 8) = gl_pack(S[m][j][2], S[m][j][3]);
        }
      // the ten tiles of 16 x 16 scores on and below the diagonal
      for (int i = warp; i < 10; i += 8) {
        const int qt = i < 1 ? 0 : i < 3 ? 1 : i < 6 ? 2 : 3, kt = i - qt * (qt + 1) / 2;
        float A[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) A[j][0] = A[j][1] = A[j][2] = A[j][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < NP / 16; ++ks) {
          uint32_t a[4], w[4];
          gl_ldsm(a, sC + (qt * 16 + fa_r) * NS + ks * 16 + fa_c);
          gl_ldsm(w, sB + (kt * 16 + fb_r) * NS + ks * 16 + fb_c);
          gl_mma(A[0], a, w[0], w[1]);
          gl_mma(A[1], a, w[2], w[3]);
        }
        const int tq = qt * 16 + (lane >> 2);
        const float lq0 = sum_at(tq), lq1 = sum_at(tq + 8);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int s = kt * 16 + j * 8 + cc;
          const float ls0 = sum_at(s), ls1 = sum_at(s + 1), d0 = sDt[s], d1 = sDt[s + 1];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = tq + e * 8;
            const float lt = e ? lq1 : lq0;
            const float a0 = s <= t ? A[j][2 * e] * gl_ex2(lt - ls0) * d0 : 0.f, a1 = s + 1 <= t ? A[j][2 * e + 1] * gl_ex2(lt - ls1) * d1 : 0.f;
            *reinterpret_cast<uint32_t*>(sA + t * AS + s) = gl_pack(a0, a1);
          }
        }
      }
    }
    __syncthreads();
    // y = exp(L) C S + A x + D x: rows of this warp, half the columns
    if (!p.carry) {
      float O[NO][4];
#pragma unroll
      for (int j = 0; j < NO; ++j) O[j][0] = O[j][1] = O[j][2] = O[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < NP / 16; ++ks) {
        uint32_t a[4];
        gl_ldsm(a, sC + (mt * 16 + fa_r) * NS + ks * 16 + fa_c);
#pragma unroll
        for (int j = 0; j < NO; j += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, sS + (ks * 16 + fa_r) * XS + half * (VS / 2) + j * 8 + fa_c);
          gl_mma(O[j], a, w[0], w[1]);
          gl_mma(O[j + 1], a, w[2], w[3]);
        }
      }
      const float e0 = gl_ex2(l0), e1 = gl_ex2(l1);
#pragma unroll
      for (int j = 0; j < NO; ++j) { O[j][0] *= e0; O[j][1] *= e0; O[j][2] *= e1; O[j][3] *= e1; }
      for (int ks = 0; ks <= mt; ++ks) {                   // causal: 16 keys at a time
        uint32_t a[4];
        gl_ldsm(a, sA + (mt * 16 + fa_r) * AS + ks * 16 + fa_c);
#pragma unroll
        for (int j = 0; j < NO; j += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, sX + (ks * 16 + fa_r) * XS + half * (VS / 2) + j * 8 + fa_c);
          gl_mma(O[j], a, w[0], w[1]);
          gl_mma(O[j + 1], a, w[2], w[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = r0 + e * 8;
        if (r >= rows) continue;
        bf16* yr = p.y + (size_t)(start + ch * kSsdChunk + r) * p.heads * p.vdim + h * p.vdim + v0;
#pragma unroll
        for (int j = 0; j < NO; ++j) {
          const int c = half * (VS / 2) + j * 8 + cc;
          if (c >= vw) continue;
          const float2 x = gl_unpack(*reinterpret_cast<const uint32_t*>(sX + r * XS + c));
          const float2 v = make_float2(fmaf(skip, x.x, O[j][2 * e]), fmaf(skip, x.y, O[j][2 * e + 1]));
          if ((p.vdim & 1) == 0) *reinterpret_cast<uint32_t*>(yr + c) = gl_pack(v.x, v.y);
          else { yr[c] = __float2bfloat16(v.x); if (c + 1 < vw) yr[c + 1] = __float2bfloat16(v.y); }
        }
      }
    }
    // S = exp(L_end) S + B^T x2
    const float keep = gl_ex2(end_sum);
#pragma unroll
    for (int m = 0; m < MPW; ++m) {
#pragma unroll
      for (int j = 0; j < NSW; ++j) { S[m][j][0] *= keep; S[m][j][1] *= keep; S[m][j][2] *= keep; S[m][j][3] *= keep; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t a[4];
        gl_ldsm_t(a, sB + (ks * 16 + fb_r) * NS + (sd - (lane >> 2)) + m * 128 + fb_c);
#pragma unroll
        for (int j = 0; j < NSW; j += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, sX2 + (ks * 16 + fa_r) * XS + sn0 + j * 8 + fa_c);
          gl_mma(S[m][j], a, w[0], w[1]);
          gl_mma(S[m][j + 1], a, w[2], w[3]);
        }
      }
    }
    __syncthreads();                                       // the sums, and with one stage the tiles, are written again
    if (Cfg::STAGES == 1 && ch + 1 < ch1) load(ch + 1);
  }
  if (p.carry) {
    st = seg_s + (size_t)(seg + 1) * N * p.vdim;
    if (v0 == 0 && ht == 0) seg_d[seg + 1] = carried;
  } else if (ch1 < chunks) return;                         // the last segment leaves the state
  each_state([&](float& v, size_t at, bool in) { if (in) st[at] = v; });
}

}  // namespace xft

using namespace xft;

// States of portions (head_prep.cu).
extern "C" int xft_conv_state(const void* x, int ldx, int C, int taps, const int* cu_q, const int* kv_lens, int B, void* state,
                              const int* state_slots, int num_states, int f32, int* status, cudaStream_t st);

template <typename T, int VEC>
static cudaError_t launch_conv(const ChannelConvParams& p, cudaStream_t st) {
  const dim3 grid((p.C / VEC + 127) / 128, (p.T + p.run - 1) / p.run);
  if (p.taps <= 2) return launch_pdl(channel_conv_kernel<T, VEC, 2>, grid, dim3(128), 0, st, p);
  if (p.taps <= 4) return launch_pdl(channel_conv_kernel<T, VEC, 4>, grid, dim3(128), 0, st, p);
  return launch_pdl(channel_conv_kernel<T, VEC, 8>, grid, dim3(128), 0, st, p);
}

// x [T, ldx] (its first channel) and out [T, ldo], both fp32 (f32 = 1) or bf16, as is the state [slots, taps - 1, C]; up to 8 taps.
// decode: every sequence has one token in this call.
extern "C" int xft_channel_conv(const void* x, int ldx, int T, int B, int C, int taps, const float* w, const float* bias, const int* cu_q,
                                const int* kv_lens, void* state, const int* state_slots, int num_states, void* out, int ldo, int decode,
                                int f32, int* status, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (C <= 0 || taps < 1 || taps > 8 || ldx < C || ldo < C || (taps > 1 && (!state || !state_slots || num_states <= 0))) return -1;
  const int run = decode || T < 1024 ? 1 : T < 8192 ? 8 : 16;
  if ((T + run - 1) / run > 65535) return -2;
  ChannelConvParams p{x, ldx, T, B, C, taps, w, bias, cu_q, kv_lens, state, state_slots, num_states, out, ldo, run, decode, status};
  const bool vec = ((C | ldx | ldo) & 7) == 0 && (((uintptr_t)x | (uintptr_t)out | (uintptr_t)state | (uintptr_t)w | (uintptr_t)bias) & 15) == 0;
  cudaError_t e;
  if (f32) e = vec ? launch_conv<float, 4>(p, st) : launch_conv<float, 1>(p, st);
  else e = vec ? launch_conv<bf16, 8>(p, st) : launch_conv<bf16, 1>(p, st);
  if (e != cudaSuccess) return (int)e;
  if (taps > 1 && !decode) return xft_conv_state(x, ldx, C, taps, cu_q, kv_lens, B, state, state_slots, num_states, f32, status, st);
  return (int)cudaGetLastError();
}

// y, z and out [T, ld], all fp32 (f32 = 1) or bf16, `parts` parts of n columns each, gain fp32 [parts * n].
extern "C" int xft_gated_norm(const void* y, int ldy, const void* z, int ldz, const float* gain, void* out, int ldo, int T, int parts, int n,
                              float eps, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (parts <= 0 || n <= 0 || ldy < parts * n || ldz < parts * n || ldo < parts * n) return -1;
  const bool vec = !f32 && n <= 16384 && ((n | ldy | ldz | ldo) & 7) == 0 && (((uintptr_t)y | (uintptr_t)z | (uintptr_t)out | (uintptr_t)gain) & 15) == 0;
  const int nt = vec ? (n <= 512 ? 32 : n <= 1024 ? 64 : n <= 2048 ? 128 : n <= 4096 ? 256 : n <= 8192 ? 512 : 1024) : n <= 512 ? 64 : n <= 2048 ? 128 : 256;
  for (int t0 = 0; t0 < T; t0 += 65535) {                  // the grid's second dimension
    const dim3 grid(parts, T - t0 < 65535 ? T - t0 : 65535);
    const size_t ay = (size_t)t0 * ldy, az = (size_t)t0 * ldz, ao = (size_t)t0 * ldo;
    cudaError_t e;
    if (f32) e = launch_pdl(gated_norm_kernel<float>, grid, dim3(nt), 0, st, (const float*)y + ay, ldy, (const float*)z + az, ldz, gain,
                            (float*)out + ao, ldo, n, eps);
    else e = launch_pdl(vec ? gated_norm_vec_kernel : gated_norm_kernel<bf16>, grid, dim3(nt), 0, st, (const bf16*)y + ay, ldy,
                        (const bf16*)z + az, ldz, gain, (bf16*)out + ao, ldo, n, eps);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)cudaGetLastError();
}

// x fp32 [T, ldx], W a multiple of 4 columns, mu [n_mix, W], state fp32 [slots, W], out [T, n_mix * W] fp32 or bf16.
extern "C" int xft_token_shift(const float* x, int ldx, int T, int n_mix, int W, const float* mu, const int* cu_q, const int* kv_lens, int B,
                               float* state, const int* state_slots, int num_states, void* out, int f32, int* status, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (n_mix <= 0 || W <= 0 || (W & 3) || ldx < W || (ldx & 3) || num_states <= 0 || T > 65535) return -1;
  if (((uintptr_t)x | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)out) & 15) return -2;
  const dim3 grid((W / 4 + 127) / 128, T);
  cudaError_t e = f32 ? launch_pdl(token_shift_kernel<float>, grid, dim3(128), 0, st, x, ldx, n_mix, W, mu, cu_q, kv_lens, B, state,
                                   state_slots, num_states, (float*)out, status)
                      : launch_pdl(token_shift_kernel<bf16>, grid, dim3(128), 0, st, x, ldx, n_mix, W, mu, cu_q, kv_lens, B, state,
                                   state_slots, num_states, (bf16*)out, status);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

template <int NP, int VS, int HPC>
static int launch_ssd_heads(const SsdChunkParams& p, int B, cudaStream_t st) {
  using Cfg = SsdCfg<NP, VS, HPC>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(ssd_chunk_kernel<NP, VS, HPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM) != cudaSuccess)
      return 3000 + (int)cudaGetLastError();
    attr_set = true;
  }
  const dim3 grid((p.vdim + VS - 1) / VS * p.segs, p.heads / HPC, B), block(kSsdThreads * HPC);
  cudaError_t e = cudaSuccess;
  if (p.segs > 1) {
    SsdChunkParams q = p;
    q.carry = 1;
    e = launch_pdl(ssd_chunk_kernel<NP, VS, HPC>, grid, block, Cfg::SMEM, st, q);
  }
  if (e == cudaSuccess) e = launch_pdl(ssd_chunk_kernel<NP, VS, HPC>, grid, block, Cfg::SMEM, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
template <int NP, int VS>
static int launch_ssd_chunk(const SsdChunkParams& p, int B, cudaStream_t st) {
  if (p.per_group % 2 == 0) return launch_ssd_heads<NP, VS, 2>(p, B, st);
  return launch_ssd_heads<NP, VS, 1>(p, B, st);
}

// CTAs that a sequence occupies in the chunk kernel, 0: it has no instance for states of so many rows.
extern "C" int xft_ssd_chunk_ctas(int heads, int per_group, int state_n, int vdim) {
  if (state_n <= 0 || state_n > 256 || heads <= 0 || per_group <= 0 || vdim <= 0) return 0;
  const int cols = state_n > 128 || vdim <= 64 ? 64 : 128;
  const bool two = per_group % 2 == 0 && !(cols == 128) && state_n <= 128;
  return heads / (two ? 2 : 1) * ((vdim + cols - 1) / cols);
}

// bf16 portions of at least min_q tokens (others are left alone): u rows [x | B | C] behind the convolution, dt raw step sizes, y
// [T, heads * vdim] bf16.  segs > 1: portions are cut into so many segments (two launches), with scratch seg_state fp32 [B, heads, segs,
// state, vdim] and seg_decay fp32 [B, heads, segs].
extern "C" int xft_ssd_chunk(const void* u, int ldu, int b_at, int c_at, const void* dt, int ld_dt, const float* dt_bias, const float* rate,
                             const float* skip, int heads, int per_group, int state_n, int vdim, float* state, const int* state_slots,
                             int num_states, const int* cu_q, const int* kv_lens, int B, void* y, int min_q, int segs, float* seg_state,
                             float* seg_decay, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (!xft_ssd_chunk_ctas(heads, per_group, state_n, vdim) || heads % per_group || num_states <= 0) return -1;
  if (heads > 65535 || B > 65535 || ((uintptr_t)u & 15) || segs < 1 || (segs > 1 && (!seg_state || !seg_decay))) return -2;
  SsdChunkParams p{(const bf16*)u, ldu, b_at, c_at, (const bf16*)dt, ld_dt, dt_bias, rate, skip, heads, per_group, state_n, vdim, state,
                   state_slots, num_states, cu_q, kv_lens, (bf16*)y, min_q, segs, 0, seg_state, seg_decay, status};
  if (state_n <= 64) return vdim <= 64 ? launch_ssd_chunk<64, 64>(p, B, st) : launch_ssd_heads<64, 128, 1>(p, B, st);
  if (state_n <= 128) return vdim <= 64 ? launch_ssd_chunk<128, 64>(p, B, st) : launch_ssd_heads<128, 128, 1>(p, B, st);
  return launch_ssd_heads<256, 64, 1>(p, B, st);
}
