// Prompt attention over keys and values that lie next to each other in memory, on the 5th-generation tensor cores: the
// expanded form of latent attention.  The latents of the positions a prompt portion can see are multiplied with the
// per-head matrices once (a plain GEMM), and this kernel attends to the result.
//
// A key has two parts: `nc1` chunks of 64 dimensions of its own head (columns of the expanded matrix) and `nc2` chunks that
// all heads share (the rotated part, columns of the gathered cache rows).  Values are `nv` chunks of 64.
//
// One CTA takes 256 query rows of one head as two tiles of 128, each with four softmax warps of its own, so that one tile's
// softmax runs while the tensor core works for the other:
//
//   S_i = Q_i K^T   tcgen05.mma, 128 x 128, both operands K-major in shared memory, D in TMEM
//   P_i = softmax   one query row (= one TMEM lane) per thread: the row of S is read into registers once; P goes back as
//                   bf16 over the first half of S's columns
//   O_i += P_i V    tcgen05.mma with A = P from TMEM, B = V MN-major, D in TMEM for the whole loop.  When a row's maximum
//                   has grown by more than 2^8 since O was last scaled, its warp rescales O in place; a smaller growth
//                   stays in P (at most 2^8), and the row sum uses the same maximum, so the quotient is the same
//
// Tensor-core instructions of a CTA run in the order of issue: S_i of the next key tile is issued after O_i += P_i V, so it
// may overwrite P_i, and when its barrier completes O_i is complete too.
//
// Key tiles start at the first key that the CTA's first row sees (sliding window), not at a multiple of anything.
//
// Warp roles (384 threads): warp 0 = TMA producer, warp 1 = TMEM owner + MMA issuer, warps 2 and 3 idle (they complete the
// warpgroup that hands registers over), warps 4-7 and 8-11 = softmax and output of the two tiles.  Every wait is bounded and
// reports through the status word.
#include "ptx.cuh"

namespace xft {

int make_tensor_map(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                    uint32_t esize);

struct FlatAttnParams {
  __nv_bfloat16* out; int ldo;               // row t, head h: columns h * 64 nv ...
  const __nv_bfloat16* gate; int ldg;        // same layout, or null
  int head_gate;                             // the gate has one column per head instead
  const float* sinks;                        // [heads] a score without a key per head (of all launches), or null
  const int* q_start; const int* q_len;      // [B] first row and number of rows of a sequence's queries
  const int* kv_len;                         // [B] keys visible after this call's append
  const int* span_lo; const int* span_row;   // [B] first key that lies in the flat arrays, and its row there
  int q_head;                                // columns of one query head in Q
  int head0;                                 // first head of this launch (the flat arrays hold its heads from column 0)
  int nc1, nc2, nv, k_stages, v_stages;
  int v_col0;                                // first value column of the expanded matrix
  int r_col0;                                // first column of the shared key part in the gathered rows
  float scale_log2;                          // softmax scale * log2(e), > 0
  int window;                                // keys within `window` positions are visible (2^30: all)
  int* status;
};

constexpr int kFlChunk = 128 * 128;          // bytes of 128 rows x 64 dimensions

__global__ void __launch_bounds__(384, 1) attn_flat_tc_kernel(const __grid_constant__ CUtensorMap tmQ,
                                                              const __grid_constant__ CUtensorMap tmK,
                                                              const __grid_constant__ CUtensorMap tmR, const FlatAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nq = p.nc1 + p.nc2;
  uint8_t* sQ = smem;                                                  // [2 tiles][nq chunks]
  uint8_t* sK = sQ + 2 * nq * kFlChunk;                                // [k_stages][nq chunks]
  uint8_t* sV = sK + p.k_stages * nq * kFlChunk;                       // [v_stages][nv chunks]
  __shared__ uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_full[2], o_full[2];
  __shared__ uint32_t tmem_base_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, hl = blockIdx.y;
  const int q0 = p.q_start[b], q_len = p.q_len[b], kv_len = p.kv_len[b];
  const int n_qt = (q_len + 255) / 256;
  if ((int)blockIdx.x >= n_qt) return;
  const int row0 = (n_qt - 1 - (int)blockIdx.x) * 256;                 // the rows with the most keys first
  const int tiles_q = q_len - row0 > 128 ? 2 : 1;
  const int past = kv_len - q_len;
  const int last = min(row0 + 256, q_len) - 1;
  const int k_begin = max(p.span_lo[b], past + row0 - p.window + 1);   // first key any row of this CTA sees
  const int n_tiles = (past + last + 1 - k_begin + 127) / 128;
  const int flat0 = p.span_row[b] - p.span_lo[b] + k_begin;            // its row in the flat arrays

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1); mbar_init(&o_full[s], 1);
      mbar_init(&p_full[s], 4);                                        // one arrival per softmax warp
    }
    fence_barrier_init();
    fence_proxy_async();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmR);
  }
  if (warp == 1) {
    tmem_alloc(&tmem_base_s, 512);                                     // S_0, S_1, O_0, O_1
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem = tmem_base_s;
  grid_dep_launch();
  grid_dep_wait();

  // registers: 384 x 168 at launch, 128 x 72 + 256 x 216 from here on
  if (warp < 4) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 72;");
    if (warp == 0) {
      // ------------------------------------------------------------------ TMA producer
      if (lane == 0) {
        mbar_expect_tx(&q_full, tiles_q * nq * kFlChunk);
        for (int i = 0; i < tiles_q; ++i)
          for (int c = 0; c < nq; ++c)
            tma_load_2d(sQ + (i * nq + c) * kFlChunk, &tmQ, &q_full, (p.head0 + hl) * p.q_head + c * 64, q0 + row0 + i * 128,
                        kEvictNormal);
        auto load_k = [&](int j) -> bool {
          const int s = j % p.k_stages;
          if (!mbar_wait(&k_empty[s], ((j / p.k_stages) & 1) ^ 1, p.status, XFT_ERR_WAIT_EMPTY)) return false;
          mbar_expect_tx(&k_full[s], nq * kFlChunk);
          uint8_t* k = sK + s * nq * kFlChunk;
          for (int c = 0; c < nq; ++c) {
            if (c < p.nc1) tma_load_2d(k + c * kFlChunk, &tmK, &k_full[s], (hl * p.nc1 + c) * 64, flat0 + j * 128, kEvictNormal);
            else tma_load_2d(k + c * kFlChunk, &tmR, &k_full[s], p.r_col0 + (c - p.nc1) * 64, flat0 + j * 128, kEvictNormal);
          }
          return true;
        };
        bool ok = load_k(0);
        for (int j = 0; j < n_tiles && ok; ++j) {
          if (j + 1 < n_tiles && !load_k(j + 1)) break;
          const int s = j % p.v_stages;
          ok = mbar_wait(&v_empty[s], ((j / p.v_stages) & 1) ^ 1, p.status, XFT_ERR_WAIT_EMPTY);
          if (!ok) break;
          mbar_expect_tx(&v_full[s], p.nv * kFlChunk);
          for (int c = 0; c < p.nv; ++c)
            tma_load_2d(sV + (s * p.nv + c) * kFlChunk, &tmK, &v_full[s], p.v_col0 + (hl * p.nv + c) * 64, flat0 + j * 128,
                        kEvictNormal);
        }
      }
    } else if (warp == 1) {
      // ------------------------------------------------------------------ MMA issuer
      if (lane == 0) {
        constexpr uint32_t IDESC_S = umma_idesc(128, 128, 1, 1, 1);
        const uint32_t idesc_o = umma_idesc(128, 64, 1, 1, 1) + (p.nv > 1 ? (8u << 17) : 0u) | (1u << 16);   // N = 64 nv, B MN-major
        auto issue_s = [&](int i, int j) {
          const uint32_t qa = smem_u32(sQ + i * nq * kFlChunk), ka = smem_u32(sK + (j % p.k_stages) * nq * kFlChunk);
          for (int c = 0; c < nq; ++c)
  #pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              umma_bf16(tmem + i * 128, umma_desc_k128(qa + c * kFlChunk + kk * 32), umma_desc_k128(ka + c * kFlChunk + kk * 32),
                        IDESC_S, c > 0 || kk > 0);
          if (i + 1 == tiles_q) tcgen05_commit(&k_empty[j % p.k_stages]);
          tcgen05_commit(&s_full[i]);
        };
        auto wait_k = [&](int j) {
          const bool ok = mbar_wait(&k_full[j % p.k_stages], (j / p.k_stages) & 1, p.status, XFT_ERR_WAIT_FULL);
          tcgen05_fence_after();
          return ok;
        };
        bool ok = mbar_wait(&q_full, 0, p.status, XFT_ERR_WAIT_FULL) && wait_k(0);
        for (int i = 0; i < tiles_q && ok; ++i) issue_s(i, 0);
        for (int j = 0; j < n_tiles && ok; ++j) {
          for (int i = 0; i < tiles_q && ok; ++i) {
            ok = mbar_wait(&p_full[i], j & 1, p.status, XFT_ERR_WAIT_TMEM);
            if (ok && i == 0) ok = mbar_wait(&v_full[j % p.v_stages], (j / p.v_stages) & 1, p.status, XFT_ERR_WAIT_FULL);
            if (!ok) break;
            tcgen05_fence_after();
            const uint32_t va = smem_u32(sV + (j % p.v_stages) * p.nv * kFlChunk);
  #pragma unroll
            for (int kk = 0; kk < 8; ++kk)                               // 16 keys = 8 columns of P, 16 rows of V
              umma_bf16_ta(tmem + 256 + i * 128, tmem + i * 128 + kk * 8, umma_desc_mn128(va + kk * 2048, kFlChunk), idesc_o,
                           j > 0 || kk > 0);
            if (i + 1 == tiles_q) tcgen05_commit(&v_empty[j % p.v_stages]);
            if (j + 1 == n_tiles) {
              tcgen05_commit(&o_full[i]);
            } else {
              if (i == 0) ok = wait_k(j + 1);
              if (ok) issue_s(i, j + 1);
            }
          }
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + output: one query row per thread
    asm volatile("setmaxnreg.inc.sync.aligned.u32 216;");
    const int i = (warp - 4) >> 2, qd = warp & 3;
    if (i < tiles_q) {
      const int qrow = row0 + i * 128 + qd * 32 + lane;
      const int qpos = past + min(qrow, q_len - 1);                    // rows past the end attend like the last one
      const uint32_t lane_addr = tmem + (uint32_t(qd * 32) << 16);
      const uint32_t sa = lane_addr + i * 128, oa = lane_addr + 256 + i * 128;
      float m = -INFINITY, l = 0.f;
      if (p.sinks) { m = p.sinks[p.head0 + hl] * 1.4426950408889634f; l = 1.f; }
      bool ok = true;
      for (int j = 0; j < n_tiles; ++j) {
        if (!mbar_wait(&s_full[i], j & 1, p.status, XFT_ERR_WAIT_TMEM)) { ok = false; break; }
        tcgen05_fence_after();
        uint32_t v[4][32];
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_ld32(sa + c * 32, v[c]);
        tmem_ld_wait();
        const int k0 = k_begin + j * 128;
        const int hi = min(qpos + 1, kv_len) - k0, lo = qpos - p.window + 1 - k0;      // keys lo .. hi - 1 of the tile are visible
        if (!__all_sync(0xffffffffu, hi >= 128 && lo <= 0)) {
#pragma unroll
          for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int e = 0; e < 32; ++e)
              if (c * 32 + e >= hi || c * 32 + e < lo) v[c][e] = 0xff800000u;          // -inf
        }
        float mx4[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          mx4[c] = __uint_as_float(v[c][0]);
#pragma unroll
          for (int e = 1; e < 32; ++e) mx4[c] = fmaxf(mx4[c], __uint_as_float(v[c][e]));
        }
        const float mt = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
        float f = 1.f;
        if (mt > m + 8.f || m == -INFINITY) {                          // m = -inf: nothing seen yet, O and l are zero (or unset)
          if (m != -INFINITY) { f = exp2f(m - mt); l *= f; }
          m = mt;
        }
        if (j > 0 && __any_sync(0xffffffffu, f != 1.f)) {
          for (int c = 0; c < p.nv * 64; c += 32) {
            uint32_t o[32];
            tmem_ld32(oa + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
            tmem_st32(oa + c, o);
          }
        }
        const float mu = m == -INFINITY ? 0.f : m;
        float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          uint32_t w[32];
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const float a = exp2f(fmaf(__uint_as_float(v[g * 2 + (e >> 4)][(2 * e) & 31]), p.scale_log2, -mu));
            const float c = exp2f(fmaf(__uint_as_float(v[g * 2 + (e >> 4)][(2 * e + 1) & 31]), p.scale_log2, -mu));
            sum4[(e & 1) * 2] += a;
            sum4[(e & 1) * 2 + 1] += c;
            const __nv_bfloat162 pb = __floats2bfloat162_rn(a, c);
            w[e] = *reinterpret_cast<const uint32_t*>(&pb);
          }
          tmem_st32(sa + g * 32, w);
        }
        l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
        tmem_st_wait();
        tcgen05_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[i]);
      }
      ok = ok && mbar_wait(&o_full[i], 0, p.status, XFT_ERR_WAIT_TMEM);
      tcgen05_fence_after();
      if (__all_sync(0xffffffffu, ok)) {
        const float inv = l > 0.f ? 1.f / l : 0.f;
        const size_t col = (size_t)(p.head0 + hl) * p.nv * 64;
        __nv_bfloat16* dst = p.out + (size_t)(q0 + qrow) * p.ldo + col;
        const __nv_bfloat16* gt = p.gate ? p.gate + (size_t)(q0 + qrow) * p.ldg + (p.head_gate ? p.head0 + hl : col) : nullptr;
        const float hg = gt && p.head_gate && qrow < q_len ? __fdividef(inv, 1.f + __expf(-__bfloat162float(*gt))) : inv;
        for (int c = 0; c < p.nv * 64; c += 32) {
          uint32_t o[32];
          tmem_ld32(oa + c, o);
          tmem_ld_wait();
          if (qrow < q_len) {
#pragma unroll
            for (int g = 0; g < 4; ++g) {
              float x[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) x[e] = __uint_as_float(o[g * 8 + e]) * hg;
              if (gt && !p.head_gate) {
                const uint4 u = *reinterpret_cast<const uint4*>(gt + c + g * 8);
                const __nv_bfloat162* hb = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  const float2 y = __bfloat1622float2(hb[e]);
                  x[2 * e] = __fdividef(x[2 * e], 1.f + __expf(-y.x));
                  x[2 * e + 1] = __fdividef(x[2 * e + 1], 1.f + __expf(-y.y));
                }
              }
              uint32_t w[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const __nv_bfloat162 ob = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
                w[e] = *reinterpret_cast<const uint32_t*>(&ob);
              }
              *reinterpret_cast<uint4*>(dst + c + g * 8) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        }
      }
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace xft

using namespace xft;

// Causal attention of prompt rows over flat keys (see the file comment).  Q [T, ldq] (head h at columns h * q_head: nc1 + nc2
// chunks of 64); kv [rows, ldkv]: per head of this launch nc1 * 64 key columns, then, from v_col0 on, nv * 64 value columns;
// shared [rows, lds]: the shared key part at columns r_col0 ...; out [T, ldo] and gate [T, ldg] (or null): head h at columns
// h * nv * 64 (head_gate: column h of the gate).  sinks [all heads] or null.  Heads head0 .. head0 + heads - 1.  Per sequence of B: q_start, q_len, kv_len, span_lo, span_row.
// Returns 0, -1 for sizes it does not have, or a CUDA / tensor-map error.
extern "C" int xft_attn_flat_tc(const void* q, int ldq, int q_cols, int q_head, const void* kv, int ldkv, int v_col0,
                                const void* shared, int lds, int r_col0, int rows, void* out, int ldo, const void* gate, int ldg, int head_gate,
                                const int* q_start, const int* q_len, const int* kv_len, const int* span_lo, const int* span_row,
                                int B, int T, int max_q, int head0, int heads, int nc1, int nc2, int nv, float scale, const float* sinks, int window,
                                int* status, cudaStream_t st) {
  if (B <= 0 || T <= 0 || max_q <= 0 || heads <= 0) return 0;
  const int nq = nc1 + nc2;
  if (nc1 < 1 || nc2 < 1 || nq > 4 || nv < 1 || nv > 2 || scale <= 0.f || window < 0 || rows <= 0) return -1;
  if ((q_head & 7) || (v_col0 & 7) || (r_col0 & 7) || (ldo & 7) || (ldg & 7) || v_col0 + heads * nv * 64 > ldkv ||
      heads * nc1 * 64 > v_col0 || r_col0 + nc2 * 64 > lds || (head0 + heads - 1) * q_head + nq * 64 > q_cols || q_cols > ldq ||
      (head0 + heads) * nv * 64 > ldo)
    return -2;
  if (((uintptr_t)out | (head_gate ? 0 : (uintptr_t)gate)) & 15) return -3;
  FlatAttnParams p{};
  p.head_gate = head_gate; p.sinks = sinks;
  p.out = (__nv_bfloat16*)out; p.ldo = ldo; p.gate = (const __nv_bfloat16*)gate; p.ldg = ldg;
  p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len; p.span_lo = span_lo; p.span_row = span_row;
  p.q_head = q_head; p.head0 = head0; p.nc1 = nc1; p.nc2 = nc2; p.nv = nv; p.v_col0 = v_col0; p.r_col0 = r_col0;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = window > 0 ? min(window, 1 << 30) : 1 << 30;
  p.status = status;
  // 227 KB: two query tiles, then as many key and value stages (at most two each) as fit
  const int room = 14 - 2 * nq;                                        // chunks of 16 KB besides Q
  p.k_stages = 2 * nq + nv <= room ? 2 : 1;
  p.v_stages = p.k_stages * nq + 2 * nv <= room ? 2 : 1;
  if (p.k_stages * nq + p.v_stages * nv > room) return -1;
  const size_t smem = (size_t)(2 * nq + p.k_stages * nq + p.v_stages * nv) * kFlChunk + 1024;
  CUtensorMap tmQ, tmK, tmR;
  if (make_tensor_map(&tmQ, q, (uint64_t)T, (uint64_t)q_cols, (uint64_t)ldq, 128, 2)) return -4;
  if (make_tensor_map(&tmK, kv, (uint64_t)rows, (uint64_t)ldkv, (uint64_t)ldkv, 128, 2)) return -4;
  if (make_tensor_map(&tmR, shared, (uint64_t)rows, (uint64_t)lds, (uint64_t)lds, 128, 2)) return -4;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(attn_flat_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 14 * kFlChunk + 1024) != cudaSuccess)
      return 3000 + (int)cudaGetLastError();
    attr_set = true;
  }
  dim3 grid((max_q + 255) / 256, heads, B);
  cudaError_t e = launch_pdl(attn_flat_tc_kernel, grid, dim3(384), smem, st, tmQ, tmK, tmR, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
