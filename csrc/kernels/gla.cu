// Gated linear attention: a recurrent layer whose state per head is a dim x vdim matrix that decays per key channel.
//
//   alpha_t = sigmoid(W_a2 a1_t + bias)^(1 / tau)         [dim]
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T                fp32
//   o_t = S_t^T (q_t / sqrt(dim))                          [vdim]
//   out = o / sqrt(mean(o^2) + eps) * gain * silu(g_t)
//
// and two relatives of it in the same kernels:
//
//   time mixing    alpha_t = exp(-exp(W_a2 a1_t + bias)), o_t = (S_(t-1) + diag(u) k_t v_t^T)^T (q_t scale): the state is read
//                  before it moves on, and the current token counts with a bonus u per channel
//   state space    (step kernel) one decay exp(-rate dt) per head and token, k scaled by dt = softplus(raw + bias), q and k shared by
//                  groups of heads; what leaves is o + D v, its gate and norm follow in a kernel of their own
//
// Rows of x are packed [q | k | v | g | a1] (queries, keys, values and gate of all heads, the decay's first product).  A
// sequence's state lives in its slot of a pool [slots, heads, dim, vdim]; its first token starts from zero whatever the slot
// holds.  Two kernels share a batch, by the length of a sequence's portion:
//
// gla_step_kernel (decode, short portions, and everything in fp32): token after token.  The state of a (sequence, head)
// stays in registers, spread over one CTA or, by columns, over a cluster of up to 8 that exchange the norm's sum of squares
// through distributed shared memory.  A decode step is bound by reading and writing the state once; the state is fetched
// before the kernel in front has finished.
//
// gla_chunk_kernel (bf16 portions): 64 tokens at a time on the tensor cores.  With b_t the running sum of log(alpha) within
// the chunk (fp32), its last value b_C and mid = b_C / 2 per channel,
//
//   q^_t = q_t exp(b_t - mid),  k^_t = k_t exp(mid - b_t)
//   O   = q^ (exp(mid) S) + tril(q^ k^^T) V
//   S  <- exp(mid) (exp(mid) S + k^^T V)
//
// which is exact algebra; the exponents stay within +-30 as long as no channel decays by more than e^-60 in a chunk.  A
// chunk with a faster channel goes in four pieces of 16 tokens, and a piece with such a channel forms its 16 x 16 scores
// from differences b_t - b_s <= 0, which cannot overflow.  S stays in registers as the accumulator of its product.
// Few sequences: a portion is cut into segments that run side by side.  A first launch carries the state alone through
// every segment but the last, from zero; in the second each segment starts from the decayed sum of the ones before it.
//
// This file is compiled without fast-math; the chunk kernel asks for the fast exponential and logarithm by name.
#include "mma_sync.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

struct GlaParams {
  const void* x; int ldx; int k_at, v_at, g_at, a_at;
  int heads, dim, vdim, rank, rank_ld;     // rank_ld: row stride of a2
  const void* a2; const float* bias;       // [heads * dim, rank_ld], [heads * dim]
  float inv_tau, scale, eps;
  const float* gain;                       // [vdim]
  float* state; const int* state_slots; int num_states;
  const int* cu_q; const int* kv_lens; int B;
  void* out; int ldo;                      // [T, heads * vdim]
  float* raw;                              // chunk kernel with split columns: o before its norm, fp32 [T, heads * vdim]
  int min_q, max_q;                        // only sequences with min_q <= tokens in this call < max_q
  int segs, carry;                         // segments per portion; carry: the launch that runs the states alone
  float* seg_state;                        // [B, heads, segs, dim, vdim]: the initial state, then what segment j - 1 leaves
  float* seg_decay;                        // [B, heads, segs, dim]: sum of log2(alpha) over segment j - 1
  int* status;
  const float* bonus;                      // [heads, dim] (time mixing)
  int gain_ld; float mult;                 // gain of head h at h * gain_ld; a factor of the result
  // state space: q columns start at q_at, heads_per_group heads share q and k, raw step sizes [T, ld_dt], fp32 vectors [heads]
  int q_at, heads_per_group;
  const void* dt; int ld_dt; const float* dt_bias; const float* rate; const float* skip;
};
enum GlaMode { kGla = 0, kTimeMix = 1, kStateSpace = 2 };

template <typename T> __device__ __forceinline__ float gl_f32(T v);
template <> __device__ __forceinline__ float gl_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float gl_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T gl_from(float v);
template <> __device__ __forceinline__ float gl_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 gl_from<bf16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ int gl_slot(const GlaParams& p, int b) {
  int s = p.state_slots[b];
  if (s < 0 || s >= p.num_states) { if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); s = 0; }
  return s;
}

// ------------------------------------------------------------------------------------------ token by token
constexpr int kStepThreads = 256;

// LC lanes share a row of the state (4 columns each), RPT rows per thread
template <typename T, int LC, int RPT, int MODE>
__global__ void __launch_bounds__(kStepThreads) gla_step_kernel(const GlaParams p) {
  constexpr int CW = LC * 4, GROUPS = kStepThreads / LC, NW = kStepThreads / 32;
  extern __shared__ float gs_sm[];
  float* sq = gs_sm;                       // [dim] each
  float* sk = sq + p.dim;
  float* sa = sk + p.dim;
  float* sb = sa + p.dim;                  // time mixing: the bonus' scores
  float* sr = sb + (MODE == kTimeMix ? p.dim : 0);        // [rank_ld]
  __shared__ float red[NW][CW];
  __shared__ float ssq[2][NW];
  __shared__ float peer_ss[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, b = blockIdx.z, slice = blockIdx.x, nslices = gridDim.x;
  grid_dep_launch();
  const int start = p.cu_q[b], n = p.cu_q[b + 1] - start;
  if (n < p.min_q || n >= p.max_q) { grid_dep_wait(); return; }
  const int past = p.kv_lens[b] - n;
  const int lc = tid % LC, grp = tid / LC;
  const int c0 = slice * CW + lc * 4;                     // this thread's columns c0 .. c0 + 3
  const bool vec = (p.vdim & 3) == 0;
  float* st = p.state + ((size_t)gl_slot(p, b) * p.heads + h) * p.dim * p.vdim;
  float S[RPT][4];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int d = r * GROUPS + grp;
    S[r][0] = S[r][1] = S[r][2] = S[r][3] = 0.f;
    if (past > 0 && d < p.dim) {
      const float* row = st + (size_t)d * p.vdim + c0;
      if (vec && c0 < p.vdim) {
        const float4 v = *reinterpret_cast<const float4*>(row);
        S[r][0] = v.x; S[r][1] = v.y; S[r][2] = v.z; S[r][3] = v.w;
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c0 + j < p.vdim) S[r][j] = row[j];
      }
    }
  }
  grid_dep_wait();
  const T* a2 = reinterpret_cast<const T*>(p.a2) + (size_t)h * p.dim * p.rank_ld;
  const int kh = MODE == kStateSpace ? h / p.heads_per_group : h;                      // the head of q and k
  for (int i = 0; i < n; ++i) {
    const T* row = reinterpret_cast<const T*>(p.x) + (size_t)(start + i) * p.ldx;
    if (MODE != kStateSpace)
    for (int r = tid; r < p.rank_ld; r += kStepThreads) sr[r] = r < p.rank ? gl_f32<T>(row[p.a_at + r]) : 0.f;
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = c0 + j < p.vdim ? gl_f32<T>(row[p.v_at + h * p.vdim + c0 + j]) : 0.f;
    float keep = 0.f, dt = 1.f;
    if (MODE == kStateSpace) {
      const float z = gl_f32<T>(reinterpret_cast<const T*>(p.dt)[(size_t)(start + i) * p.ld_dt + h]) + p.dt_bias[h];
      dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      keep = expf(-p.rate[h] * dt);
    }
    __syncthreads();
    for (int d = tid; d < p.dim; d += kStepThreads) {
      if (MODE == kStateSpace) {
        sq[d] = gl_f32<T>(row[p.q_at + kh * p.dim + d]);
        sk[d] = gl_f32<T>(row[p.k_at + kh * p.dim + d]) * dt;
        continue;
      }
      float z = p.bias[h * p.dim + d];
      const T* wr = a2 + (size_t)d * p.rank_ld;
      for (int r = 0; r < p.rank_ld; r += 8) {            // rows of a2 are multiples of 8 values, zeros behind the rank
        struct alignas(16) V8 { T e[8]; };
        const V8 w = *reinterpret_cast<const V8*>(wr + r);
#pragma unroll
        for (int e = 0; e < 8; ++e) z = fmaf(gl_f32<T>(w.e[e]), sr[r + e], z);
      }
      // log(sigmoid(z)) / tau, or -exp(z)
      const float la = MODE == kTimeMix ? -expf(z) : (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau;
      sa[d] = expf(la);
      sq[d] = gl_f32<T>(row[h * p.dim + d]) * p.scale;
      sk[d] = gl_f32<T>(row[p.k_at + h * p.dim + d]);
      if (MODE == kTimeMix) sb[d] = sq[d] * sk[d] * p.bonus[h * p.dim + d];
    }
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int d = r * GROUPS + grp;
      if (d < p.dim) {
        const float al = MODE == kStateSpace ? keep : sa[d], kk = sk[d], qq = sq[d];
        const float bb = MODE == kTimeMix ? sb[d] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (MODE == kTimeMix) o[j] = fmaf(qq, S[r][j], fmaf(bb, v[j], o[j]));
          S[r][j] = fmaf(al, S[r][j], kk * v[j]);
          if (MODE != kTimeMix) o[j] = fmaf(qq, S[r][j], o[j]);
        }
      }
    }
#pragma unroll
    for (int m = LC; m < 32; m <<= 1)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], m);
    if (lane < LC) {
#pragma unroll
      for (int j = 0; j < 4; ++j) red[warp][lc * 4 + j] = o[j];
    }
    __syncthreads();
    float y = 0.f;
    const int col = slice * CW + tid;
    const bool mine = tid < CW && col < p.vdim;
    if (tid < CW) {
#pragma unroll
      for (int w = 0; w < NW; ++w) y += red[w][tid];
    }
    if (MODE == kStateSpace) {
      if (mine)
        reinterpret_cast<T*>(p.out)[(size_t)(start + i) * p.heads * p.vdim + h * p.vdim + col] =
            gl_from<T>(fmaf(p.skip[h], gl_f32<T>(row[p.v_at + h * p.vdim + col]), y));
      continue;
    }
    float ss = mine ? y * y : 0.f;
#pragma unroll
    for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if (lane == 0) ssq[i & 1][warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) ss += ssq[i & 1][w];
    if (nslices > 1) {                                    // the other columns of the head are with the cluster's other CTAs
      if (tid == 0) peer_ss[i & 1] = ss;
      cluster_arrive();
      cluster_wait();
      ss = 0.f;
      for (int c = 0; c < nslices; ++c) ss += ld_dsmem(dsmem_addr(smem_u32(&peer_ss[i & 1]), c));
    }
    if (mine) {
      const float g = gl_f32<T>(row[p.g_at + h * p.vdim + col]);
      const float r = y / sqrtf(ss / (float)p.vdim + p.eps) * p.gain[h * p.gain_ld + col] * (g / (1.f + expf(-g))) * p.mult;
      reinterpret_cast<T*>(p.out)[(size_t)(start + i) * p.ldo + h * p.vdim + col] = gl_from<T>(r);
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int d = r * GROUPS + grp;
    if (d < p.dim) {
      float* row = st + (size_t)d * p.vdim + c0;
      if (vec && c0 < p.vdim) *reinterpret_cast<float4*>(row) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
      else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c0 + j < p.vdim) row[j] = S[r][j];
      }
    }
  }
  if (MODE != kStateSpace && nslices > 1) { cluster_arrive(); cluster_wait(); }  // nobody leaves while its shared memory may be read
}

// ------------------------------------------------------------------------------------------ chunks of 64 tokens
constexpr int kChunk = 64, kPiece = 16;
constexpr float kMaxDecay = 60.f;

// x * sigmoid(x); e^-x past the largest float makes it 0
__device__ __forceinline__ float gl_silu(float x) { return x * gl_rcp(1.f + gl_ex2(-x * kLog2e)); }

// DP: padded dim, VS: columns of the state per CTA, RP: padded rank.  16 warps: products of rows take 16 rows (of four) and a
// quarter of the columns per warp, the state is divided by 16 rows and, when they are fewer than 16 x 16, by columns.
constexpr int kChunkThreads = 512;
template <int DP, int VS, int RP>
struct ChunkCfg {
  static constexpr int QS = DP + 8, VSS = VS + 8, RS = RP + 8, AS = kChunk + 8;     // row strides (16 bytes of padding)
  static constexpr int BS = DP + 8;
  static constexpr int STAGE = kChunk * (2 * QS + VSS + RS);                         // q, k, v, a1 of a chunk, in values
  static constexpr int STAGES = DP <= 128 ? 2 : 1;
  // the running sums are done with when the state is written as an operand: one place for both
  static constexpr size_t SHARED = (size_t)kChunk * BS * 4 > (size_t)DP * VSS * 2 ? (size_t)kChunk * BS * 4 : (size_t)DP * VSS * 2;
  static constexpr size_t B16 = (size_t)STAGES * STAGE + kChunk * AS + DP * RS;
  static constexpr size_t F32 = 8 * DP + 4 * 2 * DP + 2 * DP + 5 * kChunk + VS;
  static constexpr size_t SMEM = B16 * 2 + SHARED + F32 * 4;
  static_assert(SMEM <= 227 * 1024, "shared memory");
};

template <int DP, int VS, int RP, bool BONUS>
__global__ void __launch_bounds__(kChunkThreads, 1) gla_chunk_kernel(const GlaParams p) {
  using Cfg = ChunkCfg<DP, VS, RP>;
  constexpr int NT = kChunkThreads;
  constexpr int QS = Cfg::QS, VSS = Cfg::VSS, RS = Cfg::RS, AS = Cfg::AS, BS = Cfg::BS;
  constexpr int MW = DP / 16, NGRP = 16 / MW, NPW = VS / 8 / NGRP;     // state: m-tiles, column groups, n-tiles per warp
  constexpr int NO = VS / 32, NZ = DP / 32;                            // n-tiles of a quarter of the columns
  static_assert(MW <= 16 && NPW >= 2 && NPW % 2 == 0 && NO % 2 == 0 && NZ % 2 == 0, "warp tiles");
  extern __shared__ __align__(16) uint8_t gc_raw[];
  bf16* stage0 = reinterpret_cast<bf16*>(gc_raw);
  bf16* sA = stage0 + Cfg::STAGES * Cfg::STAGE;           // scores [64][AS]
  bf16* sW = sA + kChunk * AS;                            // a2 of this head [DP][RS]
  float* sB = reinterpret_cast<float*>(sW + DP * RS);     // running sums of log2(alpha) [64][BS], restarting every 8 rows
  bf16* sS = reinterpret_cast<bf16*>(sB);                 // then the state as an operand [DP][VSS]
  float* sT = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(sB) + Cfg::SHARED);     // totals of the sums [8][DP]
  float* sPre = sT + 8 * DP;                              // [4][DP] factors of the state's rows, per piece: in front of the operand
  float* sMid = sPre + 4 * DP;                            // [4][DP] and behind it
  float* sBias = sMid + 4 * DP;
  float* sSS = sBias + DP;                                // [4][64] sums of squares of the output rows
  float* sGain = sSS + 4 * kChunk;
  float* sU = sGain + VS;                                 // the bonus [DP], and the scores it gives the rows [64]
  float* sDiag = sU + DP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, b = blockIdx.z, seg = blockIdx.x % p.segs, v0 = blockIdx.x / p.segs * VS;
  grid_dep_launch();
  const int start = p.cu_q[b], n = p.cu_q[b + 1] - start;
  const int chunks = (n + kChunk - 1) / kChunk, per_seg = (chunks + p.segs - 1) / p.segs;
  const int ch0 = seg * per_seg, ch1 = min(ch0 + per_seg, chunks);      // this CTA's chunks
  if (n < p.min_q || n >= p.max_q || ch0 >= chunks || (p.carry && ch1 == chunks)) { grid_dep_wait(); return; }
  const int past = p.kv_lens[b] - n;
  const bool alone = per_seg >= chunks;                   // one segment has all of the portion
  const int vw = min(VS, p.vdim - v0);
  const bool even = (p.vdim & 1) == 0;
  const bool whole8 = (p.dim & 7) == 0 && (p.vdim & 7) == 0 && (p.rank & 7) == 0;
  float* st = p.state + ((size_t)gl_slot(p, b) * p.heads + h) * p.dim * p.vdim;
  const bf16* a2 = reinterpret_cast<const bf16*>(p.a2) + (size_t)h * p.dim * p.rank_ld;

  // weights, and zeros where nothing is ever loaded
  for (int i = tid; i < Cfg::STAGES * Cfg::STAGE / 8; i += NT) reinterpret_cast<uint4*>(stage0)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < DP * RP; i += NT) {
    const int d = i / RP, r = i % RP;
    sW[d * RS + r] = d < p.dim && r < p.rank ? a2[(size_t)d * p.rank_ld + r] : __float2bfloat16(0.f);
  }
  for (int d = tid; d < DP; d += NT) {
    sBias[d] = d < p.dim ? p.bias[h * p.dim + d] : 0.f;
    if (BONUS) sU[d] = d < p.dim ? p.bonus[h * p.dim + d] * p.scale : 0.f;
  }
  for (int c = tid; c < VS; c += NT) sGain[c] = c < vw ? p.gain[h * p.gain_ld + v0 + c] * p.mult : 0.f;
  // the state: warp tile of 16 rows and NPW x 8 columns
  const int sd = (warp % MW) * 16 + (lane >> 2), sn0 = warp / MW * NPW * 8, sc = sn0 + 2 * (lane & 3);
  float post0 = 1.f, post1 = 1.f;                         // factors of the two rows still to come
  float S[NPW][4];                                        // element e: row sd + 8 (e >> 1), column sc + 8 j + (e & 1)
  auto each_state = [&](auto f) {
#pragma unroll
    for (int j = 0; j < NPW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = sd + (e >> 1) * 8, c = sc + j * 8 + (e & 1);
        f(S[j][e], (size_t)d * p.vdim + v0 + c, d < p.dim && c < vw, e >> 1);
      }
  };
  each_state([&](float& v, size_t at, bool in, int) { v = past > 0 && seg == 0 && (alone || p.carry) && in ? st[at] : 0.f; });
  grid_dep_wait();
  float* seg_s = p.seg_state + ((size_t)b * p.heads + h) * p.segs * p.dim * p.vdim;
  float* seg_d = p.seg_decay + ((size_t)b * p.heads + h) * p.segs * p.dim;
  float carried = 0.f;                                    // carry: sum of log2(alpha) of channel tid over the segment
  if (p.carry && seg == 0) {                              // the pool is written while later segments still start: keep a copy
    each_state([&](float& v, size_t at, bool in, int) { if (in) seg_s[at] = v; });
  } else if (!alone && !p.carry) {
    for (int k = seg == 0 ? 0 : 1; k <= seg; ++k) {
      float f[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) f[e] = k > 1 && sd + e * 8 < p.dim ? gl_ex2(seg_d[(size_t)k * p.dim + sd + e * 8]) : 1.f;
      const float* from = seg_s + (size_t)k * p.dim * p.vdim;
      each_state([&](float& v, size_t at, bool in, int e) { v = fmaf(v, f[e], in ? from[at] : 0.f); });
    }
  }
  __syncthreads();

  const bf16* x = reinterpret_cast<const bf16*>(p.x) + (size_t)start * p.ldx;
  auto load = [&](int chunk) {
    bf16* sq = stage0 + (Cfg::STAGES > 1 ? (chunk & 1) * Cfg::STAGE : 0);
    bf16* sk = sq + kChunk * QS;
    bf16* sv = sk + kChunk * QS;
    bf16* sr = sv + kChunk * VSS;
    const int t0 = chunk * kChunk, rows = min(kChunk, n - t0);
    // rows behind the portion's end become zero
    auto part = [&](bf16* dst, int ld, int at, int width) {
      if (whole8) {
        const int per = width >> 3, dr = NT / per, dc = NT % per;
        int r = tid / per, c = tid % per;
        while (r < kChunk) {
          const bf16* src = x + (size_t)(t0 + min(r, rows - 1)) * p.ldx + at + c * 8;
          const int bytes = r < rows ? 16 : 0;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * ld + c * 8)), "l"(src), "r"(bytes) : "memory");
          r += dr;
          c += dc;
          if (c >= per) { c -= per; ++r; }
        }
      } else {
        for (int i = tid; i < kChunk * width; i += NT) {
          const int r = i / width, c = i % width;
          dst[r * ld + c] = r < rows ? x[(size_t)(t0 + r) * p.ldx + at + c] : __float2bfloat16(0.f);
        }
      }
    };
    if (!p.carry) part(sq, QS, h * p.dim, p.dim);
    part(sk, QS, p.k_at + h * p.dim, p.dim);
    part(sv, VSS, p.v_at + h * p.vdim + v0, vw);
    part(sr, RS, p.a_at, p.rank);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // fragment addresses: A (rows x k) and B (columns x k) row-major, B (k x columns) through a transposing load
  const int fa_r = (lane & 7) + ((lane >> 3) & 1) * 8, fa_c = (lane >> 4) * 8;
  const int fb_r = (lane & 7) + ((lane >> 4) & 1) * 8, fb_c = ((lane >> 3) & 1) * 8;
  const int mt = warp & 3, quarter = warp >> 2;           // this warp's 16 rows of the chunk, and its part of the columns
  const int r0 = mt * 16 + (lane >> 2), cc = 2 * (lane & 3);
  const float tau2 = p.inv_tau * kLog2e, scale2 = log2f(p.scale);

  load(ch0);
  for (int ch = ch0; ch < ch1; ++ch) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (Cfg::STAGES > 1 && ch + 1 < ch1) load(ch + 1);
    bf16* sq = stage0 + (Cfg::STAGES > 1 ? (ch & 1) * Cfg::STAGE : 0);
    bf16* sk = sq + kChunk * QS;
    bf16* sv = sk + kChunk * QS;
    bf16* sr = sv + kChunk * VSS;
    const int rows = min(kChunk, n - ch * kChunk);

    // log2(alpha) of every row and channel
    {
      float z[NZ][4];
#pragma unroll
      for (int j = 0; j < NZ; ++j) z[j][0] = z[j][1] = z[j][2] = z[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < RP / 16; ++ks) {
        uint32_t a[4];
        gl_ldsm(a, sr + (mt * 16 + fa_r) * RS + ks * 16 + fa_c);
#pragma unroll
        for (int j = 0; j < NZ; j += 2) {
          uint32_t w[4];
          gl_ldsm(w, sW + (quarter * (DP / 4) + j * 8 + fb_r) * RS + ks * 16 + fb_c);
          gl_mma(z[j], a, w[0], w[1]);
          gl_mma(z[j + 1], a, w[2], w[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < NZ; ++j) {
        const int d = quarter * (DP / 4) + j * 8 + cc;
        const float2 bias = *reinterpret_cast<const float2*>(sBias + d);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = r0 + e * 8;
          float l[2];
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            const float zz = z[j][2 * e + k] + (k ? bias.y : bias.x);
            // (a decay of 2^-200 is none that fp32 could tell from zero)
            const float la = BONUS ? fmaxf(-kLog2e * gl_ex2(zz * kLog2e), -200.f)
                                   : fminf(zz, 0.f) * tau2 - gl_lg2(1.f + gl_ex2(-fabsf(zz) * kLog2e)) * p.inv_tau;
            l[k] = r < rows && d + k < p.dim ? la : 0.f;
          }
          *reinterpret_cast<float2*>(sB + r * BS + d) = make_float2(l[0], l[1]);
        }
      }
    }
    __syncthreads();
    // running sums within every 8 rows, and their totals
    for (int it = tid; it < 4 * DP; it += NT) {
      const int pr = it % (DP / 2), g = it / (DP / 2);
      float2* col = reinterpret_cast<float2*>(sB + g * 8 * BS + 2 * pr);
      float2 c = make_float2(0.f, 0.f), v[8];
#pragma unroll
      for (int r = 0; r < 8; ++r) v[r] = col[r * (BS / 2)];
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        c.x += v[r].x; c.y += v[r].y;
        col[r * (BS / 2)] = c;
      }
      *reinterpret_cast<float2*>(sT + g * DP + 2 * pr) = c;
    }
    __syncthreads();
    if (BONUS && !p.carry) {                               // the rows' scores with themselves, from q and k as they came
#pragma unroll
      for (int r = warp * 4; r < warp * 4 + 4; ++r) {
        float a = 0.f;
        for (int d = 2 * lane; d < DP; d += 64) {
          const float2 q = gl_unpack(*reinterpret_cast<const uint32_t*>(sq + r * QS + d)), k = gl_unpack(*reinterpret_cast<const uint32_t*>(sk + r * QS + d));
          a += q.x * k.x * sU[d] + q.y * k.y * sU[d + 1];
        }
#pragma unroll
        for (int m = 16; m > 0; m >>= 1) a += __shfl_xor_sync(0xffffffffu, a, m);
        if (lane == 0) sDiag[r] = a;
      }
    }
    bool ok = true;
    for (int d = tid; d < DP; d += NT) {
      float t = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) t += sT[g * DP + d];
      carried += t;
      ok = t >= -kMaxDecay * kLog2e;
    }
    const bool one = __syncthreads_and(ok);               // the whole chunk in one piece
    const int pieces = one ? 1 : (rows + kPiece - 1) / kPiece;
    float O[NO][4];
#pragma unroll
    for (int j = 0; j < NO; ++j) O[j][0] = O[j][1] = O[j][2] = O[j][3] = 0.f;
    uint32_t gate[NO][2];                                  // of this warp's output values
    // which pieces (groups of 16 rows) have a channel too fast for factors
    uint32_t harsh = 0;
    if (!one) {
      uint32_t mine = 0;
      for (int d = tid; d < DP; d += NT)
#pragma unroll
        for (int g = 0; g < 4; ++g) mine |= (sT[2 * g * DP + d] + sT[(2 * g + 1) * DP + d] < -kMaxDecay * kLog2e ? 1u : 0u) << g;
#pragma unroll
      for (int g = 0; g < 4; ++g) harsh |= (__syncthreads_or(mine >> g & 1) ? 1u : 0u) << g;
      if (harsh && !p.carry) {
        // their scores from differences of running sums: 256 pairs of rows each, a warp at a time
        for (int i = warp; i < 4 * kPiece * kPiece; i += NT / 32) {
          const int g = i / (kPiece * kPiece), t = g * kPiece + i / kPiece % kPiece, s = g * kPiece + i % kPiece;
          if (!(harsh >> g & 1)) continue;
          float a = 0.f;
          if (BONUS ? s < t : s <= t)
            for (int d = lane; d < p.dim; d += 32) {
              const float between = (t & 8) && !(s & 8) ? sT[2 * g * DP + d] : 0.f;       // the sums restart between s and t
              const float bt = !BONUS ? sB[t * BS + d] : t & 7 ? sB[(t - 1) * BS + d] : 0.f;
              a += __bfloat162float(sq[t * QS + d]) * __bfloat162float(sk[s * QS + d]) * gl_ex2(bt - sB[s * BS + d] + between);
            }
#pragma unroll
          for (int m = 16; m > 0; m >>= 1) a += __shfl_xor_sync(0xffffffffu, a, m);
          if (lane == 0) sA[t * AS + s] = __float2bfloat16(BONUS && s == t ? sDiag[t] : a * p.scale);
        }
        __syncthreads();
      }
    }
    // q^ and k^ in place; the factors of the state's rows
    for (int it = tid; it < 4 * DP; it += NT) {
      const int pr = it % (DP / 2), g = it / (DP / 2);
      const int lo = one ? 0 : g & ~1, hi = one ? 8 : lo + 2;        // the piece's groups of 8 rows
      float2 base = make_float2(0.f, 0.f), tot = make_float2(0.f, 0.f);
      for (int j = lo; j < hi; ++j) {
        const float2 v = *reinterpret_cast<const float2*>(sT + j * DP + 2 * pr);
        if (j < g) { base.x += v.x; base.y += v.y; }
        tot.x += v.x; tot.y += v.y;
      }
      // q^ = q exp2(b - qr), k^ = k exp2(kr - b)
      const bool gentle = !(harsh >> (g >> 1) & 1);
      const float2 qr = gentle ? make_float2(0.5f * tot.x, 0.5f * tot.y) : make_float2(0.f, 0.f);
      const float2 kr = gentle ? qr : tot;
      if (g == lo) {
        const float2 e = make_float2(gl_ex2(qr.x), gl_ex2(qr.y));
        *reinterpret_cast<float2*>(sMid + (lo >> 1) * DP + 2 * pr) = gentle ? make_float2(1.f, 1.f) : make_float2(gl_ex2(tot.x), gl_ex2(tot.y));
        *reinterpret_cast<float2*>(sPre + (lo >> 1) * DP + 2 * pr) = e;
      }
      const float2 qo = make_float2(base.x - qr.x + scale2, base.y - qr.y + scale2), ko = make_float2(kr.x - base.x, kr.y - base.y);
      float2 before = make_float2(0.f, 0.f);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const int t = g * 8 + r;
        const float2 bb = *reinterpret_cast<const float2*>(sB + t * BS + 2 * pr);
        const float2 bq = BONUS ? before : bb;             // the state is read before this token's decay
        before = bb;
        uint32_t* qp = reinterpret_cast<uint32_t*>(sq + t * QS + 2 * pr);
        uint32_t* kp = reinterpret_cast<uint32_t*>(sk + t * QS + 2 * pr);
        const float2 k = gl_unpack(*kp);
        if (!p.carry) {
          const float2 q = gl_unpack(*qp);
          *qp = gl_pack(q.x * gl_ex2(bq.x + qo.x), q.y * gl_ex2(bq.y + qo.y));
        }
        *kp = gl_pack(k.x * gl_ex2(ko.x - bb.x), k.y * gl_ex2(ko.y - bb.y));
      }
    }
    __syncthreads();
    for (int pc = 0; pc < pieces; ++pc) {
      const int g_lo = one ? 0 : pc, g_hi = one ? 4 : pc + 1;       // groups of 16 rows in this piece
      const bool gentle = !(harsh >> pc & 1);
      // the state as an operand, and the scores
      {
        // the factor behind the last update and the one in front of the operand; the same one follows this update
        const float e0 = sPre[pc * DP + sd], e1 = sPre[pc * DP + sd + 8], f0 = post0 * e0, f1 = post1 * e1;
        post0 = e0;
        post1 = e1;
#pragma unroll
        for (int j = 0; j < NPW; ++j) {
          S[j][0] *= f0; S[j][1] *= f0; S[j][2] *= f1; S[j][3] *= f1;
          if (!p.carry) {
            *reinterpret_cast<uint32_t*>(sS + sd * VSS + sc + j * 8) = gl_pack(S[j][0], S[j][1]);
            *reinterpret_cast<uint32_t*>(sS + (sd + 8) * VSS + sc + j * 8) = gl_pack(S[j][2], S[j][3]);
          }
        }
        if (!gentle) {
          const float m0 = sMid[pc * DP + sd], m1 = sMid[pc * DP + sd + 8];
#pragma unroll
          for (int j = 0; j < NPW; ++j) { S[j][0] *= m0; S[j][1] *= m0; S[j][2] *= m1; S[j][3] *= m1; }
        }
      }
      const bool my_rows = mt >= g_lo && mt < g_hi && !p.carry;
      const int kt = one ? quarter : mt;                   // the 16 keys of this warp's scores
      if (gentle && my_rows && kt <= mt && (one || quarter == 0)) {
        float A[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) A[j][0] = A[j][1] = A[j][2] = A[j][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
          uint32_t a[4], w[4];
          gl_ldsm(a, sq + (mt * 16 + fa_r) * QS + ks * 16 + fa_c);
          gl_ldsm(w, sk + (kt * 16 + fb_r) * QS + ks * 16 + fb_c);
          gl_mma(A[0], a, w[0], w[1]);
          gl_mma(A[1], a, w[2], w[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int t = r0 + (e >> 1) * 8, s = kt * 16 + j * 8 + cc;
            float a0 = s <= t ? A[j][e] : 0.f, a1 = s + 1 <= t ? A[j][e + 1] : 0.f;
            if (BONUS && s == t) a0 = sDiag[t];
            if (BONUS && s + 1 == t) a1 = sDiag[t];
            *reinterpret_cast<uint32_t*>(sA + t * AS + s) = gl_pack(a0, a1);
          }
      }
      if (pc == 0 && even && !p.raw && !p.carry) {         // fetched here, used behind the products
#pragma unroll
        for (int j = 0; j < NO; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int c = quarter * (VS / 4) + j * 8 + cc, r = r0 + e * 8;
            gate[j][e] = r < rows && c < p.vdim ? __ldg(reinterpret_cast<const uint32_t*>(
                x + (size_t)(ch * kChunk + r) * p.ldx + p.g_at + h * p.vdim + c)) : 0u;
          }
      }
      __syncthreads();
      // O = q^ S + A V, rows of this warp, a quarter of the columns
      if (my_rows) {
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
          uint32_t a[4];
          gl_ldsm(a, sq + (mt * 16 + fa_r) * QS + ks * 16 + fa_c);
#pragma unroll
          for (int j = 0; j < NO; j += 2) {
            uint32_t w[4];
            gl_ldsm_t(w, sS + (ks * 16 + fa_r) * VSS + quarter * (VS / 4) + j * 8 + fa_c);
            gl_mma(O[j], a, w[0], w[1]);
            gl_mma(O[j + 1], a, w[2], w[3]);
          }
        }
        for (int ks = g_lo; ks <= mt; ++ks) {              // causal: 16 keys at a time
          uint32_t a[4];
          gl_ldsm(a, sA + (mt * 16 + fa_r) * AS + ks * 16 + fa_c);
#pragma unroll
          for (int j = 0; j < NO; j += 2) {
            uint32_t w[4];
            gl_ldsm_t(w, sv + (ks * 16 + fa_r) * VSS + quarter * (VS / 4) + j * 8 + fa_c);
            gl_mma(O[j], a, w[0], w[1]);
            gl_mma(O[j + 1], a, w[2], w[3]);
          }
        }
      }
      // S += k^^T V
      for (int ks = g_lo; ks < g_hi; ++ks) {
        uint32_t a[4];
        gl_ldsm_t(a, sk + (ks * 16 + fb_r) * QS + (warp % MW) * 16 + fb_c);
#pragma unroll
        for (int j = 0; j < NPW; j += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, sv + (ks * 16 + fa_r) * VSS + sn0 + j * 8 + fa_c);
          gl_mma(S[j], a, w[0], w[1]);
          gl_mma(S[j + 1], a, w[2], w[3]);
        }
      }
      if (pc + 1 < pieces) __syncthreads();               // the next piece writes sS, sA and the factors again
    }
    // norm and gate (or the bare output, when other CTAs have the head's other columns)
    if (p.carry) {
    } else if (p.raw) {
#pragma unroll
      for (int j = 0; j < NO; ++j) {
        const int c = quarter * (VS / 4) + j * 8 + cc;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = r0 + (e >> 1) * 8;
          if (r < rows && c + (e & 1) < vw)
            p.raw[(size_t)(start + ch * kChunk + r) * p.heads * p.vdim + h * p.vdim + v0 + c + (e & 1)] = O[j][e];
        }
      }
    } else {
      float ss[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < NO; ++j) {
        ss[0] += O[j][0] * O[j][0] + O[j][1] * O[j][1];
        ss[1] += O[j][2] * O[j][2] + O[j][3] * O[j][3];
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 1);
        ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 2);
        if ((lane & 3) == 0) sSS[quarter * kChunk + r0 + e * 8] = ss[e];
      }
      named_bar_sync(1 + mt, 128);                         // the four warps that have these rows
      const float inv_n = 1.f / (float)p.vdim;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = r0 + e * 8;
        const float inv = rsqrtf((sSS[r] + sSS[kChunk + r] + sSS[2 * kChunk + r] + sSS[3 * kChunk + r]) * inv_n + p.eps);
        const size_t trow = (size_t)(ch * kChunk + r);
        bf16* orow = reinterpret_cast<bf16*>(p.out) + (start + trow) * p.ldo + h * p.vdim;
        const bf16* grow = x + trow * p.ldx + p.g_at + h * p.vdim;
#pragma unroll
        for (int j = 0; j < NO; ++j) {
          const int c = quarter * (VS / 4) + j * 8 + cc;
          if (r >= rows || c >= p.vdim) continue;
          const float2 w = *reinterpret_cast<const float2*>(sGain + c);
          if (even) {
            const float2 g = gl_unpack(gate[j][e]);
            *reinterpret_cast<uint32_t*>(orow + c) = gl_pack(O[j][2 * e] * inv * w.x * gl_silu(g.x), O[j][2 * e + 1] * inv * w.y * gl_silu(g.y));
          } else {
            orow[c] = __float2bfloat16(O[j][2 * e] * inv * w.x * gl_silu(__bfloat162float(grow[c])));
            if (c + 1 < p.vdim) orow[c + 1] = __float2bfloat16(O[j][2 * e + 1] * inv * w.y * gl_silu(__bfloat162float(grow[c + 1])));
          }
        }
      }
    }
    if (Cfg::STAGES == 1) {
      __syncthreads();                                     // everything of this chunk has been read
      if (ch + 1 < ch1) load(ch + 1);
    }
  }
  __syncthreads();
  if (p.carry) {
    st = seg_s + (size_t)(seg + 1) * p.dim * p.vdim;
    if (v0 == 0 && tid < p.dim) seg_d[(size_t)(seg + 1) * p.dim + tid] = carried;
  } else if (ch1 < chunks) return;                         // the last segment leaves the state
  each_state([&](float& v, size_t at, bool in, int e) { if (in) st[at] = v * (e ? post1 : post0); });
}

// Norm and gate of rows whose columns came from several CTAs: one warp per (token, head) of the sequences in question.
__global__ void __launch_bounds__(128) gla_norm_kernel(const GlaParams p, int n_tok) {
  grid_dep_launch();
  grid_dep_wait();
  const int lane = threadIdx.x & 31;
  const long long gw = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (gw >= (long long)n_tok * p.heads) return;
  const int t = (int)(gw / p.heads), h = (int)(gw % p.heads);
  int lo = 0, hi = p.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int n = p.cu_q[lo + 1] - p.cu_q[lo];
  if (n < p.min_q || n >= p.max_q) return;
  const float* o = p.raw + (size_t)t * p.heads * p.vdim + h * p.vdim;
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) ss += o[c] * o[c];
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float inv = rsqrtf(ss / (float)p.vdim + p.eps);
  const bf16* gp = reinterpret_cast<const bf16*>(p.x) + (size_t)t * p.ldx + p.g_at + h * p.vdim;
  bf16* op = reinterpret_cast<bf16*>(p.out) + (size_t)t * p.ldo + h * p.vdim;
  for (int c = lane; c < p.vdim; c += 32) {
    const float g = __bfloat162float(gp[c]);
    op[c] = __float2bfloat16(o[c] * inv * p.gain[h * p.gain_ld + c] * p.mult * __fdividef(g, 1.f + __expf(-g)));
  }
}

}  // namespace xft

using namespace xft;

template <typename T, int LC, int RPT, int MODE>
static int launch_step(const GlaParams& p, cudaStream_t st) {
  const int slices = (p.vdim + LC * 4 - 1) / (LC * 4);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, p.heads, p.B);
  cfg.blockDim = dim3(kStepThreads);
  cfg.dynamicSmemBytes = (size_t)((MODE == kTimeMix ? 4 : 3) * p.dim + p.rank_ld) * sizeof(float);
  cfg.stream = st;
  cudaLaunchAttribute at[2];
  int na = 0;
  if (slices > 1 && MODE != kStateSpace) {
    at[na].id = cudaLaunchAttributeClusterDimension;
    at[na].val.clusterDim.x = slices; at[na].val.clusterDim.y = 1; at[na].val.clusterDim.z = 1;
    ++na;
  }
  if (g_xft_pdl) {
    at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = at;
  cfg.numAttrs = na;
  cudaError_t e = cudaLaunchKernelEx(&cfg, gla_step_kernel<T, LC, RPT, MODE>, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
template <typename T, int LC, int MODE>
static int step_rows(const GlaParams& p, cudaStream_t st) {
  const int rows = (p.dim + kStepThreads / LC - 1) / (kStepThreads / LC);
  if (rows <= 2) return launch_step<T, LC, 2, MODE>(p, st);
  if (rows <= 4) return launch_step<T, LC, 4, MODE>(p, st);
  if (rows <= 8) return launch_step<T, LC, 8, MODE>(p, st);
  if (rows <= 16) return launch_step<T, LC, 16, MODE>(p, st);
  if (rows <= 32) return launch_step<T, LC, 32, MODE>(p, st);
  return -5;
}
template <typename T, int MODE>
static int step_columns(const GlaParams& p, int columns, cudaStream_t st) {
  if (columns == 32) return step_rows<T, 8, MODE>(p, st);
  if (columns == 64) return step_rows<T, 16, MODE>(p, st);
  if (columns == 128) return step_rows<T, 32, MODE>(p, st);
  return -6;
}

template <int DP, int VS, int RP, bool BONUS>
static int launch_chunk_mode(const GlaParams& p, cudaStream_t st) {
  using Cfg = ChunkCfg<DP, VS, RP>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(gla_chunk_kernel<DP, VS, RP, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM) != cudaSuccess)
      return 3000 + (int)cudaGetLastError();
    attr_set = true;
  }
  const dim3 grid((p.vdim + VS - 1) / VS * p.segs, p.heads, p.B);
  cudaError_t e = cudaSuccess;
  if (p.segs > 1) {
    GlaParams q = p;
    q.carry = 1;
    e = launch_pdl(gla_chunk_kernel<DP, VS, RP, BONUS>, grid, dim3(kChunkThreads), Cfg::SMEM, st, q);
  }
  if (e == cudaSuccess) e = launch_pdl(gla_chunk_kernel<DP, VS, RP, BONUS>, grid, dim3(kChunkThreads), Cfg::SMEM, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
template <int DP, int VS, int RP>
static int launch_chunk(const GlaParams& p, cudaStream_t st) {
  return p.bonus ? launch_chunk_mode<DP, VS, RP, true>(p, st) : launch_chunk_mode<DP, VS, RP, false>(p, st);
}
template <int DP, int VS>
static int chunk_rank(const GlaParams& p, cudaStream_t st) {
  if (p.rank <= 16) return launch_chunk<DP, VS, 16>(p, st);
  if (p.rank <= 64) return launch_chunk<DP, VS, 64>(p, st);
  return -7;
}

// Columns of the state per CTA of the chunk kernel for a key size, 0: it has no instance (the step kernel runs everything).
extern "C" int xft_gla_chunk_columns(int dim, int vdim, int rank) {
  if (dim > 256 || rank > (dim > 128 ? 16 : 64) || dim <= 0) return 0;
  return vdim <= 64 ? 64 : 128;
}

// x, a2 and out all fp32 (f32 = 1) or bf16; row strides and offsets as the file comment says, all multiples of 8 (a2's rows
// too).  Sequences with min_q <= tokens < max_q take part, the others are left alone.  columns: of the state per CTA, 32, 64
// or 128, at most 8 CTAs per head; rows per CTA: dim <= columns-dependent limit (1024, 512, 256).  bonus [heads, dim] (fp32): time
// mixing, null: gated linear attention.  gain [vdim] (gain_ld 0) or [heads, gain_ld].
extern "C" int xft_gla_step(const void* x, int ldx, int k_at, int v_at, int g_at, int a_at, int heads, int dim, int vdim, int rank,
                            int rank_ld, const void* a2, const float* bias, float tau, float scale, float eps, const float* bonus, int gain_ld, float mult, const float* gain,
                            float* state, const int* state_slots, int num_states, const int* cu_q, const int* kv_lens, int B,
                            void* out, int ldo, int min_q, int max_q, int columns, int f32, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || rank <= 0 || rank_ld < rank || (rank_ld & 7) || tau <= 0.f || num_states <= 0 ||
      columns <= 0) return -1;
  if (heads > 65535 || B > 65535 || (vdim + columns - 1) / columns > 8 || (size_t)(4 * dim + rank_ld) * 4 > 40000) return -2;
  if (((uintptr_t)a2 | (uintptr_t)state) & 15) return -3;
  GlaParams p{x, ldx, k_at, v_at, g_at, a_at, heads, dim, vdim, rank, rank_ld, a2, bias, 1.f / tau, scale, eps, gain, state, state_slots,
              num_states, cu_q, kv_lens, B, out, ldo, nullptr, min_q, max_q, 1, 0, nullptr, nullptr, status};
  p.bonus = bonus; p.gain_ld = gain_ld; p.mult = mult;
  if (bonus) return f32 ? step_columns<float, kTimeMix>(p, columns, st) : step_columns<bf16, kTimeMix>(p, columns, st);
  return f32 ? step_columns<float, kGla>(p, columns, st) : step_columns<bf16, kGla>(p, columns, st);
}

// The recurrence of a state-space layer, token by token: x rows hold q, k (groups x dim each) and v (heads x vdim) from columns q_at,
// k_at and v_at; dt [T, ld_dt] raw step sizes of the rows' type; dt_bias, rate, skip fp32 [heads]; out [T, heads * vdim]
// of the rows' type.
extern "C" int xft_ssd_step(const void* x, int ldx, int q_at, int k_at, int v_at, int heads, int heads_per_group, int dim, int vdim,
                            const void* dt, int ld_dt, const float* dt_bias, const float* rate, const float* skip, float* state,
                            const int* state_slots, int num_states, const int* cu_q, const int* kv_lens, int B, void* out, int min_q,
                            int max_q, int columns, int f32, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || heads_per_group <= 0 || heads % heads_per_group || num_states <= 0 || columns <= 0) return -1;
  if (heads > 65535 || B > 65535 || (size_t)3 * dim * 4 > 40000 || ((uintptr_t)state & 15)) return -2;
  GlaParams p{};
  p.x = x; p.ldx = ldx; p.q_at = q_at; p.k_at = k_at; p.v_at = v_at; p.heads = heads; p.heads_per_group = heads_per_group;
  p.dim = dim; p.vdim = vdim; p.dt = dt; p.ld_dt = ld_dt; p.dt_bias = dt_bias; p.rate = rate; p.skip = skip;
  p.state = state; p.state_slots = state_slots; p.num_states = num_states; p.cu_q = cu_q; p.kv_lens = kv_lens; p.B = B;
  p.out = out; p.min_q = min_q; p.max_q = max_q; p.segs = 1; p.status = status;
  return f32 ? step_columns<float, kStateSpace>(p, columns, st) : step_columns<bf16, kStateSpace>(p, columns, st);
}

// bf16 portions.  raw: fp32 [T, heads * vdim], needed when a head has more columns than xft_gla_chunk_columns says.
// segs > 1: portions are cut into so many segments (two launches), with scratch seg_state fp32 [B, heads, segs, dim, vdim] and
// seg_decay fp32 [B, heads, segs, dim].
extern "C" int xft_gla_chunk(const void* x, int ldx, int k_at, int v_at, int g_at, int a_at, int heads, int dim, int vdim, int rank,
                             int rank_ld, const void* a2, const float* bias, float tau, float scale, float eps, const float* bonus, int gain_ld, float mult, const float* gain,
                             float* state, const int* state_slots, int num_states, const int* cu_q, const int* kv_lens, int B, int T,
                             void* out, int ldo, float* raw, int min_q, int max_q, int segs, float* seg_state, float* seg_decay,
                             int* status, cudaStream_t st) {
  if (B <= 0 || T <= 0) return 0;
  if (segs < 1 || (segs > 1 && (!seg_state || !seg_decay))) return -4;
  const int cols = xft_gla_chunk_columns(dim, vdim, rank);
  if (!cols || heads <= 0 || vdim <= 0 || rank <= 0 || rank_ld < rank || tau <= 0.f || num_states <= 0) return -1;
  if (heads > 65535 || B > 65535 || (vdim > cols && !raw)) return -2;
  if ((ldx & 7) || (k_at & 7) || (v_at & 7) || (g_at & 7) || (a_at & 7) || ((uintptr_t)x & 15)) return -3;
  GlaParams p{x, ldx, k_at, v_at, g_at, a_at, heads, dim, vdim, rank, rank_ld, a2, bias, 1.f / tau, scale, eps, gain, state, state_slots,
              num_states, cu_q, kv_lens, B, out, ldo, vdim > cols ? raw : nullptr, min_q, max_q, segs, 0, seg_state, seg_decay, status};
  p.bonus = bonus; p.gain_ld = gain_ld; p.mult = mult;
  int r;
  if (dim > 128) r = cols == 64 ? launch_chunk<256, 64, 16>(p, st) : launch_chunk<256, 128, 16>(p, st);
  else if (dim > 64) r = cols == 64 ? chunk_rank<128, 64>(p, st) : chunk_rank<128, 128>(p, st);
  else r = cols == 64 ? chunk_rank<64, 64>(p, st) : chunk_rank<64, 128>(p, st);
  if (r || !p.raw) return r;
  const long long warps = (long long)T * heads;
  cudaError_t e = launch_pdl(gla_norm_kernel, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, st, p, T);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
