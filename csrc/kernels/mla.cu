// Latent attention over the paged latent cache, absorbed form, for sm_100a: DeepSeek's multi-head latent attention and the
// latent layers of layered designs.
//
// Reference: crossAttnByHead_DS (src/kernels/attention_kernels.h:1132-1206) — per (head, batch):
// S = (Q_nope·W_uk)·C_kv^T + Q_rope·K_rope^T, O = (softmax(S)·C_kv)·W_uv — and selfAttention_MLA (:569-766) for
// prefill.  The cache holds one row per token: c_kv[LAT] ‖ k_rope[64] (src/layers/attn_deepseek.h:129-376).
//
// Here the two absorb products are per-head tcgen05 GEMMs (gemm_sm100.cu); this kernel does the middle: every head reads the
// SAME latent rows (multi-query attention with a LAT + 64 wide key and a LAT wide value), so a CTA takes 16 heads of one
// query token as its 16 MMA rows and streams the sequence's latent tiles once.
//
// One lane of the ninth warp feeds a ring of 32-key half tiles with TMA, 64 columns per box; the other eight warps work on
// 64-key tiles (a cache block, or a part of one).
// Warps 0-7: warp w computes the partial scores of keys 16 (w / 2) .. + 15 over one half of the dimensions, with that half
// of Q in its registers for the whole kernel; the partial scores meet in shared memory, where warp w does the online softmax
// of rows 2w and 2w + 1 and leaves their weights as bf16; then warp w adds P C for its eighth of the value columns.  Long
// contexts are split over the CTAs of a cluster, which merge through distributed shared memory, each a part of the columns;
// when that leaves SMs idle, over several clusters, whose parts meet in global scratch (the CTA that arrives last on a part
// of the columns finishes it; nobody waits).
//
// A sliding window restricts the tiles to those that hold a visible key.  A sink starts a head's online softmax in the first part.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

int make_tensor_map(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                    uint32_t esize);

constexpr int ROPE = 64, MKT = 64;               // rotated columns, keys per tile
constexpr int kMlaSx = 72;                       // row pitch of the score exchange: 16-row float2 reads without conflicts

struct MlaParams {
  const bf16* q_abs; long long qa_sh, qa_st;     // [head][token][LAT] strides in elements
  const bf16* q_rope; long long qr_sh, qr_st;    // [.][.][64]
  bf16* out; long long o_sh, o_st;               // [head][token][LAT]
  const int* block_table; int bt_stride;
  const int* cu_q; const int* kv_lens;
  int B, T, hl, bs, num_blocks;
  float scale;
  const float* sinks;                            // [hl] a score without a key per head, or null
  int window;                                    // keys within `window` positions are visible (2^30: all)
  int nsplit, groups;                            // cluster size; clusters per (token, 16 heads)
  float* part_o; float* part_ml; int* counters;  // groups > 1: [unit][group][16][LAT], [unit][group][rank][16][2], [unit][rank]
  int* status;
};

__device__ __forceinline__ void mla_cp16(void* s, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(s)), "l"(g) : "memory");
}
__device__ __forceinline__ void mla_ldsm(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mla_ldsm_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mla_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t mla_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// 16-byte chunk `chunk` of row `row`: boxes of 64 columns (128 bytes, swizzled by row & 7), ROWS rows each
template <int ROWS>
__device__ __forceinline__ bf16* mla_ptr(bf16* base, int row, int chunk) {
  return base + (chunk >> 3) * (ROWS * 64) + row * 64 + (((chunk & 7) ^ (row & 7)) << 3);
}

template <int LAT>
struct MlaCfg {
  static constexpr int DK = LAT + ROPE;
  static constexpr int STAGE_BYTES = MKT / 2 * DK * 2;                 // half a tile
  static constexpr int SX_BYTES = 2 * 16 * kMlaSx * 4 + 16 * MKT * 2;  // scores [half of the dimensions][row][key], weights
  static constexpr int FIXED = 16 * DK * 2 + SX_BYTES + 1024;
  static constexpr int STAGES = (225 * 1024 - FIXED) / STAGE_BYTES < 12 ? (225 * 1024 - FIXED) / STAGE_BYTES : 12;
  static constexpr int SMEM = FIXED + STAGES * STAGE_BYTES;
};

// grid (tokens * head_chunks, nsplit * groups), clusters of (1, nsplit); 384 threads
template <int LAT>
__global__ void __launch_bounds__(384, 1) mla_attn_kernel(const __grid_constant__ CUtensorMap tmC, const MlaParams p) {
  using Cfg = MlaCfg<LAT>;
  constexpr int DK = Cfg::DK, STAGES = Cfg::STAGES, KS = DK / 32;      // KS: 16-wide steps of half the dimensions
  constexpr int NT = LAT / 64 > 2 ? LAT / 64 : 2;                      // 8-column output tiles per warp
  constexpr int PITCH = LAT + 4;                                       // merge buffer row
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  bf16* ring = reinterpret_cast<bf16*>(base);                          // [STAGES][DK / 64][32][64]
  bf16* qs = reinterpret_cast<bf16*>(base + STAGES * Cfg::STAGE_BYTES);
  float* sx = reinterpret_cast<float*>(qs + 16 * DK);
  bf16* ps = reinterpret_cast<bf16*>(sx + 2 * 16 * kMlaSx);
  __shared__ uint64_t full_bar[STAGES], empty_bar[STAGES];
  __shared__ float s_ml[16][2], s_fac[16][8], s_corr[16], s_top[16][2];
  __shared__ int s_last;
  static_assert(16 * PITCH * 4 <= STAGES * Cfg::STAGE_BYTES, "the merge buffer lies over the ring");
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < STAGES; ++i) { mbar_init(&full_bar[i], 1); mbar_init(&empty_bar[i], 8); }
    fence_barrier_init();
    tma_prefetch_desc(&tmC);
  }
  __syncthreads();
  grid_dep_launch();
  // Until grid_dep_wait() only step inputs are read (lengths, block table) and cache rows of EARLIER calls.
  const int chunks = (p.hl + 15) / 16;
  const int t = blockIdx.x / chunks, h0 = (blockIdx.x % chunks) * 16, split = blockIdx.y;
  int b;
  {                                                                    // sequence of token t
    int lo = 0, hi = p.B - 1;
    while (lo < hi) { int mid = (lo + hi + 1) >> 1; if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1; }
    b = lo;
  }
  const int q0 = p.cu_q[b], past = p.kv_lens[b] - (p.cu_q[b + 1] - q0);
  const int n_keys = past + t - q0 + 1;                                // causal: keys 0 .. n_keys - 1
  const int nq = min(16, p.hl - h0);
  const int key_lo = max(0, n_keys - p.window);                        // and not before the window
  const int t_first = key_lo / MKT, t_all = (n_keys + MKT - 1) / MKT;
  const int parts = p.nsplit * p.groups;
  const int per = (t_all - t_first + parts - 1) / parts;
  const int t_begin = t_first + split * per, t_end = min(t_all, t_begin + per);
  const int nloc = max(0, t_end - t_begin);

  // registers: 384 x 168 at launch, 128 x 40 + 256 x 232 from here on (warps 9-11 only complete their warpgroup)
  if (warp >= 8) {
    // ------------------------------------------------------------------ TMA producer
    asm volatile("setmaxnreg.dec.sync.aligned.u32 40;");
    if (warp == 8 && lane == 0) {
      const int* bt = p.block_table + (size_t)b * p.bt_stride;
      auto issue = [&](int n) {
        const int s = n % STAGES, key = t_begin * MKT + n * (MKT / 2);
        int blk = bt[key / p.bs];
        if (blk < 0 || blk >= p.num_blocks) { if (p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); blk = 0; }
        mbar_expect_tx(&full_bar[s], Cfg::STAGE_BYTES);
        for (int c = 0; c < DK / 64; ++c)
          tma_load_2d(reinterpret_cast<uint8_t*>(ring) + s * Cfg::STAGE_BYTES + c * (MKT * 64), &tmC, &full_bar[s], c * 64,
                      blk * p.bs + key % p.bs, kEvictNormal);
      };
      // half tiles without a row of this call
      const int halves = 2 * nloc, pre = min(min(STAGES, halves), max(0, past / (MKT / 2) - 2 * t_begin));
      for (int n = 0; n < pre; ++n) issue(n);
      grid_dep_wait();
      for (int n = pre; n < halves; ++n) {
        if (!mbar_wait(&empty_bar[n % STAGES], ((n / STAGES) & 1) ^ 1, p.status, XFT_ERR_WAIT_EMPTY)) break;
        issue(n);
      }
    }
  }
  float* mo = reinterpret_cast<float*>(base);                          // merge buffer [16][PITCH], over the ring
  if (warp < 8) {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 232;");
    grid_dep_wait();
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    if (p.sinks && split == 0) {                                       // it counts once: in the first part
#pragma unroll
      for (int r = 0; r < 2; ++r)
        if (2 * warp + r < nq) { m[r] = p.sinks[h0 + 2 * warp + r]; l[r] = lane == 0 ? 1.f : 0.f; }
    }
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    const int r0 = lane >> 2, r1 = r0 + 8, qc = 2 * (lane & 3);
    const bool has_cols = warp * NT * 8 < LAT;
    // Q: row r = head h0 + r : [q_abs(LAT) | q_rope(64)]
    for (int i = tid; i < 16 * (DK / 8); i += 256) {
      const int r = i / (DK / 8), c = i % (DK / 8);
      bf16* dst = mla_ptr<16>(qs, r, c);
      if (r < nq) {
        mla_cp16(dst, c < LAT / 8 ? p.q_abs + (h0 + r) * p.qa_sh + (long long)t * p.qa_st + c * 8
                                  : p.q_rope + (h0 + r) * p.qr_sh + (long long)t * p.qr_st + (c - LAT / 8) * 8);
      } else {
        *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    named_bar_sync(1, 256);
    const int kg = warp >> 1, dh = warp & 1;
    uint32_t qa[KS][4];
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
      mla_ldsm(qa[ks], mla_ptr<16>(qs, (lane & 7) + ((lane >> 3) & 1) * 8, (dh * KS + ks) * 2 + (lane >> 4)));
    for (int n = 0; n < nloc; ++n) {
      const int sa = (2 * n) % STAGES, sb = (2 * n + 1) % STAGES;
      bf16* ka = ring + (size_t)sa * (Cfg::STAGE_BYTES / 2);
      bf16* kb = ring + (size_t)sb * (Cfg::STAGE_BYTES / 2);
      bool ok = mbar_wait(&full_bar[sa], ((2 * n) / STAGES) & 1, p.status, XFT_ERR_WAIT_FULL);
      ok = mbar_wait(&full_bar[sb], ((2 * n + 1) / STAGES) & 1, p.status, XFT_ERR_WAIT_FULL) && ok;
      bf16* kq = kg < 2 ? ka : kb;                                     // the half with this warp's keys
      {
        float s[4][4];                                                 // two 8-key tiles, even and odd steps
#pragma unroll
        for (int i = 0; i < 4; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          uint32_t bb[4];
          mla_ldsm(bb, mla_ptr<MKT / 2>(kq, (kg & 1) * 16 + (lane & 7) + ((lane >> 4) & 1) * 8, (dh * KS + ks) * 2 + ((lane >> 3) & 1)));
          mla_mma(s[(ks & 1) * 2], qa[ks], bb[0], bb[1]);
          mla_mma(s[(ks & 1) * 2 + 1], qa[ks], bb[2], bb[3]);
        }
        float* sd = sx + dh * (16 * kMlaSx) + kg * 16 + qc;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          *reinterpret_cast<float2*>(sd + r0 * kMlaSx + j * 8) = make_float2(s[j][0] + s[j + 2][0], s[j][1] + s[j + 2][1]);
          *reinterpret_cast<float2*>(sd + r1 * kMlaSx + j * 8) = make_float2(s[j][2] + s[j + 2][2], s[j][3] + s[j + 2][3]);
        }
      }
      if (named_bar_or(1, 256, !ok)) break;                            // scores complete (or all warps give up together)
      // ---- online softmax of this warp's two rows: two keys per lane ----
      const int k0 = (t_begin + n) * MKT, key = k0 + 2 * lane;
      const bool see0 = key < n_keys && key >= key_lo, see1 = key + 1 < n_keys && key + 1 >= key_lo;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int row = 2 * warp + r;
        const float* a = sx + row * kMlaSx + 2 * lane;
        const float2 x = *reinterpret_cast<const float2*>(a), y = *reinterpret_cast<const float2*>(a + 16 * kMlaSx);
        const float v0 = see0 ? (x.x + y.x) * p.scale : -INFINITY, v1 = see1 ? (x.y + y.y) * p.scale : -INFINITY;
        float mx = fmaxf(v0, v1);
#pragma unroll
        for (int i = 16; i > 0; i >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, i));
        const float mn = fmaxf(m[r], mx);                              // finite: every visited tile holds a visible key
        const float c = __expf(m[r] - mn), p0 = __expf(v0 - mn), p1 = __expf(v1 - mn);
        m[r] = mn;
        l[r] = l[r] * c + p0 + p1;                                     // per-lane partial sums
        if (lane == 0) s_corr[row] = c;
        *reinterpret_cast<uint32_t*>(mla_ptr<16>(ps, row, lane >> 2) + 2 * (lane & 3)) = mla_pack(p0, p1);
      }
      named_bar_sync(1, 256);
      if (has_cols) {
        const float c0 = s_corr[r0], c1 = s_corr[r1];
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
          for (int i = 0; i < NT; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
        }
        // ---- O[:, this warp's columns] += P · C ----
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          uint32_t a[4];
          mla_ldsm(a, mla_ptr<16>(ps, (lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4)));
#pragma unroll
          for (int j = 0; j < NT; j += 2) {
            uint32_t bb[4];
            mla_ldsm_t(bb, mla_ptr<MKT / 2>(ks < 2 ? ka : kb, (ks & 1) * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, warp * NT + j + (lane >> 4)));
            mla_mma(o[j], a, bb[0], bb[1]);
            mla_mma(o[j + 1], a, bb[2], bb[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) { mbar_arrive(&empty_bar[sa]); mbar_arrive(&empty_bar[sb]); }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
      for (int i = 16; i > 0; i >>= 1) l[r] += __shfl_xor_sync(0xffffffffu, l[r], i);
      if (lane == 0) { s_ml[2 * warp + r][0] = m[r]; s_ml[2 * warp + r][1] = l[r]; }
    }
    named_bar_sync(1, 256);                                            // every issued tile was consumed: the ring is idle
    if (has_cols) {
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int d = (warp * NT + j) * 8 + qc;
        *reinterpret_cast<float2*>(mo + r0 * PITCH + d) = make_float2(o[j][0], o[j][1]);
        *reinterpret_cast<float2*>(mo + r1 * PITCH + d) = make_float2(o[j][2], o[j][3]);
      }
    }
  }
  // ---- merge: each CTA of the cluster finishes LAT / nsplit columns ----
  __syncwarp();
  const int ns = p.nsplit;
  if (ns > 1) { cluster_arrive(); cluster_wait(); } else __syncthreads();
  if (tid < 16) {                                                      // factor of every CTA's part of row `tid`
    float mm[8], ll[8], top = -INFINITY, sum = 0.f;
    const uint32_t a = smem_u32(&s_ml[tid][0]);
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      if (s < ns) {
        const uint32_t ra = ns > 1 ? dsmem_addr(a, s) : a;
        mm[s] = ns > 1 ? ld_dsmem(ra) : s_ml[tid][0];
        ll[s] = ns > 1 ? ld_dsmem(ra + 4) : s_ml[tid][1];
        top = fmaxf(top, mm[s]);
      }
    }
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < ns) { mm[s] = mm[s] == -INFINITY ? 0.f : __expf(mm[s] - top); sum += mm[s] * ll[s]; }
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < ns) s_fac[tid][s] = p.groups > 1 ? mm[s] : sum > 0.f ? mm[s] / sum : 0.f;
    if (p.groups > 1) { s_top[tid][0] = top; s_top[tid][1] = sum; }
  }
  __syncthreads();
  const int rank = split % ns, group = split / ns;
  const int cols = LAT / ns, c0 = rank * cols;
  float* po = p.groups > 1 ? p.part_o + ((size_t)blockIdx.x * p.groups + group) * 16 * LAT : nullptr;
  for (int i = tid; i < nq * (cols / 2); i += 384) {
    const int r = i / (cols / 2), d = c0 + 2 * (i % (cols / 2));
    const uint32_t a = smem_u32(mo + r * PITCH + d);
    float x = 0.f, y = 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      if (s < ns) {
        const uint32_t ra = ns > 1 ? dsmem_addr(a, s) : a;
        const float f = s_fac[r][s];
        x += f * (ns > 1 ? ld_dsmem(ra) : mo[r * PITCH + d]);
        y += f * (ns > 1 ? ld_dsmem(ra + 4) : mo[r * PITCH + d + 1]);
      }
    }
    if (po) *reinterpret_cast<float2*>(po + r * LAT + d) = make_float2(x, y);
    else *reinterpret_cast<uint32_t*>(p.out + (h0 + r) * p.o_sh + (long long)t * p.o_st + d) = mla_pack(x, y);
  }
  if (po) {
    // this rank's columns of every group: the last CTA to arrive adds them up
    auto ml_of = [&](int g) { return p.part_ml + (((size_t)blockIdx.x * p.groups + g) * ns + rank) * 32; };
    if (tid < 32) ml_of(group)[tid] = s_top[tid >> 1][tid & 1];
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      int* c = p.counters + (size_t)blockIdx.x * ns + rank;
      s_last = atomicAdd(c, 1) == p.groups - 1;
      if (s_last) *c = 0;
    }
    __syncthreads();
    if (s_last) {
      __threadfence();
      for (int i = tid; i < nq * (cols / 2); i += 384) {
        const int r = i / (cols / 2), d = c0 + 2 * (i % (cols / 2));
        float top = -INFINITY, sum = 0.f, x = 0.f, y = 0.f;
        for (int g = 0; g < p.groups; ++g) top = fmaxf(top, __ldcg(ml_of(g) + 2 * r));
        for (int g = 0; g < p.groups; ++g) {
          const float mg = __ldcg(ml_of(g) + 2 * r), f = mg == -INFINITY ? 0.f : __expf(mg - top);
          const float2 v = __ldcg(reinterpret_cast<const float2*>(p.part_o + (((size_t)blockIdx.x * p.groups + g) * 16 + r) * LAT + d));
          sum += f * __ldcg(ml_of(g) + 2 * r + 1);
          x += f * v.x;
          y += f * v.y;
        }
        const float inv = sum > 0.f ? 1.f / sum : 0.f;
        *reinterpret_cast<uint32_t*>(p.out + (h0 + r) * p.o_sh + (long long)t * p.o_st + d) = mla_pack(x * inv, y * inv);
      }
    }
  }
  if (ns > 1) { cluster_arrive(); cluster_wait(); }                    // a peer may still read this CTA's part
}

}  // namespace xft

using namespace xft;

template <int LAT>
static int launch_mla(const MlaParams& p, const void* cache, cudaStream_t st) {
  using Cfg = MlaCfg<LAT>;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(mla_attn_kernel<LAT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) != cudaSuccess) return -5;
    attr = true;
  }
  CUtensorMap tm;
  if (make_tensor_map(&tm, cache, (uint64_t)p.num_blocks * p.bs, Cfg::DK, Cfg::DK, MKT / 2, 2)) return -4;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.T * ((p.hl + 15) / 16), p.nsplit * p.groups);
  cfg.blockDim = dim3(384);
  cfg.dynamicSmemBytes = Cfg::SMEM;
  cfg.stream = st;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = 1; at[0].val.clusterDim.y = p.nsplit; at[0].val.clusterDim.z = 1;
  at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = at;
  cfg.numAttrs = g_xft_pdl ? 2 : 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, mla_attn_kernel<LAT>, tm, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// Sizes of the latent (64, 128, 256 or 512, with 64 rotated key dimensions next to it) and a sliding window: position i
// sees the keys j <= i with i - j < window (0: all).  sinks [hl] or null.  nsplit: CTAs per (token, 16 heads) and
// cluster, rounded down to 1, 2, 4 or 8; groups: clusters per (token, 16 heads).  With groups > 1 and u = T * ceil(hl / 16):
// part_o of u * groups * 16 * lat floats, part_ml of u * groups * nsplit * 32, counters of u * nsplit zeros (left as zeros).
extern "C" int xft_mla_attention_ext(const void* q_abs, long long qa_sh, long long qa_st, const void* q_rope, long long qr_sh,
                                     long long qr_st, void* out, long long o_sh, long long o_st, const void* cache,
                                     const int* block_table, int bt_stride, const int* cu_q, const int* kv_lens, int B, int T,
                                     int hl, int lat, int bs, int num_blocks, float scale, const float* sinks, int window,
                                     int nsplit, int groups, float* part_o, float* part_ml, int* counters, int* status,
                                     cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (bs <= 0 || bs % MKT) return -2;
  if (window < 0 || hl <= 0) return -1;
  MlaParams p{(const bf16*)q_abs, qa_sh, qa_st, (const bf16*)q_rope, qr_sh, qr_st, (bf16*)out, o_sh, o_st, block_table,
              bt_stride, cu_q, kv_lens, B, T, hl, bs, num_blocks, scale, sinks, window > 0 ? min(window, 1 << 30) : 1 << 30,
              nsplit >= 8 ? 8 : nsplit >= 4 ? 4 : nsplit >= 2 ? 2 : 1, groups < 1 ? 1 : groups, part_o, part_ml, counters, status};
  if (p.groups > 1 && (!part_o || !part_ml || !counters)) return -3;
  switch (lat) {
    case 64: return launch_mla<64>(p, cache, st);
    case 128: return launch_mla<128>(p, cache, st);
    case 256: return launch_mla<256>(p, cache, st);
    case 512: return launch_mla<512>(p, cache, st);
  }
  return -1;
}

// The scratch arguments are not used any more: slices merge through distributed shared memory.
extern "C" int xft_mla_attention(const void* q_abs, long long qa_sh, long long qa_st, const void* q_rope, long long qr_sh,
                                 long long qr_st, void* out, long long o_sh, long long o_st, const void* cache,
                                 const int* block_table, int bt_stride, const int* cu_q, const int* kv_lens, int B, int T,
                                 int hl, int bs, int num_blocks, float scale, int nsplit, float* /*part_o*/,
                                 float* /*part_ml*/, int* /*counters*/, int* status, cudaStream_t st) {
  return xft_mla_attention_ext(q_abs, qa_sh, qa_st, q_rope, qr_sh, qr_st, out, o_sh, o_st, cache, block_table, bt_stride, cu_q,
                               kv_lens, B, T, hl, 512, bs, num_blocks, scale, nullptr, 0, nsplit, 1, nullptr, nullptr, nullptr, status, st);
}
