// Attention whose heads' weights are mixed, on the tensor cores (bf16, heads of 64 or 128; see talking.cu for what it computes).
//
// Prompt portions, talking_prefill_kernel: a CTA takes a tile of queries with all of their heads, since the weights of all heads
// of a (query, key) pair meet in the mix.  A warp owns a unit of 16 rows: 16 queries of one head, or (more than 16 heads) 8
// queries of two heads that share keys.  The keys are visited twice.  The first pass carries a running maximum and sum per row.
// The second forms the scores again, and from them the finished weights; they go to shared memory as two bf16 halves, are
// multiplied with the mixing matrix there (a product over the heads, both halves with fp32 sums: nothing of their 16 bits of
// mantissa is lost before the mix), and come back as the operand of the product with the values.
//
// Decode steps: talking_scores_kernel writes the scores of a key range of one key/value head with its maxima and sums,
// talking_values_kernel merges those of all ranges, mixes in fp32 and adds up the values of its range; the CTA that arrives last
// on a head adds up the ranges and applies the gate.
#include "mma_sync.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;
constexpr float kTalkLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------ prompt portions
struct TalkPrefillParams {
  const bf16* q; const bf16* gate; int ldg; bf16* out; int ldo;
  const bf16* kc; const bf16* vc; const int* block_table; int bt_stride;
  const int* cu_q; const int* kv_lens;
  int hq, hkv, group, bs, num_blocks, window;
  int units, blocks;                         // units of 16 rows, blocks of queries (units = blocks * hq / heads per unit)
  float scale2, mult;                        // softmax scale * log2(e)
  const float* r1; const float* r2; const float* talk;
  int* status;
};

constexpr int kTalkThreads = 512;

template <int D, int HB, int KT>
__global__ void __launch_bounds__(kTalkThreads, 1) talking_prefill_kernel(const TalkPrefillParams p) {
  constexpr int QPB = 16 / HB, HP = HB == 1 ? 16 : 32;                 // queries of a block; heads, padded
  constexpr int KS = D + 8, QP = KT + 8, PITCH = QPB * QP + 8;         // row strides: keys and values, weights of a query, of a head
  constexpr int KH = D > 64 || KT < 32 ? 16 : 32;                                // keys whose scores are in registers at a time
  constexpr int MT = HP / 16, MP = HP + 8;
  extern __shared__ __align__(16) uint8_t tk_raw[];
  bf16* sK = reinterpret_cast<bf16*>(tk_raw);                          // [hkv][KT][KS]
  bf16* sV = sK + (size_t)p.hkv * KT * KS;
  bf16* sM = sV + (size_t)p.hkv * KT * KS;                             // the mixing matrix [HP][MP]
  bf16* sP = sM + HP * MP;                                             // [2 halves][blocks][HP][PITCH]
  const int half_size = p.blocks * HP * PITCH;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.y;
  grid_dep_launch();
  const int q0 = p.cu_q[b], q_len = p.cu_q[b + 1] - q0, kv_len = p.kv_lens[b], QT = p.blocks * QPB;
  const int tiles_q = (q_len + QT - 1) / QT;
  if ((int)blockIdx.x >= tiles_q) { grid_dep_wait(); return; }
  const int row0 = (tiles_q - 1 - (int)blockIdx.x) * QT, past = kv_len - q_len;
  const int last = min(row0 + QT, q_len) - 1;
  const int k_lo = max(0, past + row0 - p.window + 1) / KT * KT;       // a tile lies in one page
  const int n_tiles = (past + last + 1 - k_lo + KT - 1) / KT;
  // this warp's unit
  const int per_block = p.hq / HB, qb = warp / per_block, h0 = (warp % per_block) * HB;
  const bool active = warp < p.units;
  const int kvh = active ? h0 / p.group : 0;
  const int r = lane >> 2, cc = 2 * (lane & 3);
  int qi[2], qpos[2], head[2];
  float r1[2], r2[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {                                        // rows r and r + 8
    qi[e] = row0 + (active ? qb : 0) * QPB + (HB == 1 ? r + 8 * e : r);
    head[e] = active ? h0 + (HB == 1 ? 0 : e) : 0;
    qpos[e] = past + min(qi[e], q_len - 1);                            // rows past the end attend like the last one
    r1[e] = p.r1[head[e]];
    r2[e] = p.r2[head[e]];
  }
  // the mixing matrix as an operand
  for (int i = tid; i < HP * HP; i += kTalkThreads) {
    const int h = i / HP, g = i % HP;
    sM[h * MP + g] = __float2bfloat16(h < p.hq && g < p.hq ? p.talk[h * p.hq + g] : 0.f);
  }
  for (int i = tid; i < half_size / 4; i += kTalkThreads) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);   // both halves
  grid_dep_wait();
  uint32_t qa[D / 16][4];
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = e & 1;
      qa[ks][e] = active && qi[i] < q_len ? *reinterpret_cast<const uint32_t*>(
          p.q + ((size_t)(q0 + qi[i]) * p.hq + head[i]) * D + ks * 16 + cc + (e >> 1) * 8) : 0u;
    }
  const int* bt = p.block_table + (size_t)b * p.bt_stride;
  auto load = [&](bf16* dst, const bf16* cache, int tile) {
    const int key = k_lo + tile * KT;
    int blk = bt[key / p.bs];
    if (blk < 0 || blk >= p.num_blocks) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); blk = 0; }
    const bf16* src = cache + ((size_t)blk * p.hkv * p.bs + key % p.bs) * D;
    for (int i = tid; i < p.hkv * KT * (D / 8); i += kTalkThreads) {
      const int row = i / (D / 8), c = i % (D / 8), g = row / KT, k = row % KT;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + (size_t)row * KS + c * 8)),
                   "l"(src + ((size_t)g * p.bs + k) * D + c * 8) : "memory");
    }
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
  const int fa_r = (lane & 7) + ((lane >> 3) & 1) * 8, fa_c = (lane >> 4) * 8;
  const int fb_r = (lane & 7) + ((lane >> 4) & 1) * 8, fb_c = ((lane >> 3) & 1) * 8;
  // scores (base 2) of this warp's rows and KH keys from `k` on of the tile in `s`; -inf where a key is not visible
  float S[KH / 8][4];
  auto scores = [&](const bf16* s, int tile, int k) {
#pragma unroll
    for (int j = 0; j < KH / 8; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
    const bf16* base = s + ((size_t)kvh * KT + k) * KS;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
#pragma unroll
      for (int j = 0; j < KH / 8; j += 2) {
        uint32_t w[4];
        gl_ldsm(w, base + (j * 8 + fb_r) * KS + ks * 16 + fb_c);
        gl_mma(S[j], qa[ks], w[0], w[1]);
        gl_mma(S[j + 1], qa[ks], w[2], w[3]);
      }
    const int key0 = k_lo + tile * KT + k + cc;
#pragma unroll
    for (int j = 0; j < KH / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int far = qpos[e >> 1] - (key0 + j * 8 + (e & 1));
        const float v = fmaf(S[j][e], p.scale2, -r1[e >> 1] * gl_lg2(fmaf(r2[e >> 1], (float)max(far, 0), 1.f)));
        S[j][e] = far >= 0 && far < p.window ? v : -INFINITY;
      }
  };
  // ---- first pass: maxima and sums; both tile buffers hold keys
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  load(sK, p.kc, 0);
  commit();
  for (int j = 0; j < n_tiles; ++j) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (j + 1 < n_tiles) load(j & 1 ? sK : sV, p.kc, j + 1);
    commit();
    if (!active) continue;
#pragma unroll 1
    for (int k = 0; k < KT; k += KH) {
      scores(j & 1 ? sV : sK, j, k);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float mx = m[e];
#pragma unroll
        for (int i = 0; i < KH / 8; ++i) mx = fmaxf(mx, fmaxf(S[i][2 * e], S[i][2 * e + 1]));
        const float ref = mx == -INFINITY ? 0.f : mx;                  // nothing seen yet: every term is zero
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < KH / 8; ++i) sum += gl_ex2(S[i][2 * e] - ref) + gl_ex2(S[i][2 * e + 1] - ref);
        l[e] = fmaf(l[e], gl_ex2(m[e] - ref), sum);                    // this lane's columns alone
        m[e] = mx;
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {                                        // the four lanes of a row; m becomes log2 of the row's sum
    float mx = m[e];
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    float s = m[e] == -INFINITY ? 0.f : l[e] * gl_ex2(m[e] - mx);
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    m[e] = mx;
    l[e] = s > 0.f ? __fdividef(1.f, s) : 0.f;
  }
  // ---- second pass
  float O[D / 8][4];
#pragma unroll
  for (int j = 0; j < D / 8; ++j) O[j][0] = O[j][1] = O[j][2] = O[j][3] = 0.f;
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  load(sK, p.kc, 0);
  commit();
  bf16* pw = sP + (size_t)(active ? qb : 0) * HP * PITCH;              // this unit's block
  for (int j = 0; j < n_tiles; ++j) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                                   // keys are here, everyone is done with the values
    load(sV, p.vc, j);
    commit();
    if (active) {
#pragma unroll 1
      for (int k = 0; k < KT; k += KH) {
        scores(sK, j, k);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          bf16* dst = pw + (size_t)head[e] * PITCH + (HB == 1 ? r + 8 * e : r) * QP + k + cc;
#pragma unroll
          for (int i = 0; i < KH / 8; ++i) {
            const float a = gl_ex2(S[i][2 * e] - m[e]) * l[e], c = gl_ex2(S[i][2 * e + 1] - m[e]) * l[e];
            const uint32_t hi = gl_pack(a, c);
            const float2 f = gl_unpack(hi);
            *reinterpret_cast<uint32_t*>(dst + i * 8) = hi;
            *reinterpret_cast<uint32_t*>(dst + half_size + i * 8) = gl_pack(a - f.x, c - f.y);
          }
        }
      }
    }
    __syncthreads();                                                   // weights are here, everyone is done with the keys
    if (j + 1 < n_tiles) load(sK, p.kc, j + 1);
    commit();
    // the mix, in place: 16 keys of a query at a time
    for (int c = warp; c < p.blocks * QPB * (KT / 16); c += kTalkThreads / 32) {
      const int qq = c / (KT / 16), k = c % (KT / 16) * 16;
      bf16* at = sP + (size_t)(qq / QPB) * HP * PITCH + qq % QPB * QP + k;
      float w[MT][2][4];
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int i = 0; i < 2; ++i) w[a][i][0] = w[a][i][1] = w[a][i][2] = w[a][i][3] = 0.f;
#pragma unroll
      for (int g = 0; g < MT; ++g)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t x[4];
          gl_ldsm_t(x, at + (size_t)part * half_size + (g * 16 + fa_r) * PITCH + fa_c);
#pragma unroll
          for (int a = 0; a < MT; ++a) {
            uint32_t mix[4];
            gl_ldsm(mix, sM + (a * 16 + fa_r) * MP + g * 16 + fa_c);
            gl_mma(w[a][0], mix, x[0], x[1]);
            gl_mma(w[a][1], mix, x[2], x[3]);
          }
        }
      __syncwarp();
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          *reinterpret_cast<uint32_t*>(at + (a * 16 + r) * PITCH + i * 8 + cc) = gl_pack(w[a][i][0], w[a][i][1]);
          *reinterpret_cast<uint32_t*>(at + (a * 16 + r + 8) * PITCH + i * 8 + cc) = gl_pack(w[a][i][2], w[a][i][3]);
        }
    }
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();                                                   // mixed weights and values are here
    if (active) {
      const bf16* wrow = HB == 1 ? pw + (size_t)h0 * PITCH + fa_r * QP : pw + (size_t)(h0 + ((lane >> 3) & 1)) * PITCH + (lane & 7) * QP;
      const bf16* vb = sV + (size_t)kvh * KT * KS;
#pragma unroll
      for (int ks = 0; ks < KT / 16; ++ks) {
        uint32_t a[4];
        gl_ldsm(a, wrow + ks * 16 + fa_c);
#pragma unroll
        for (int i = 0; i < D / 8; i += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, vb + (ks * 16 + fa_r) * KS + i * 8 + fa_c);
          gl_mma(O[i], a, w[0], w[1]);
          gl_mma(O[i + 1], a, w[2], w[3]);
        }
      }
    }
  }
  if (!active) return;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    if (qi[e] >= q_len) continue;
    const size_t t = q0 + qi[e];
    const bf16* g = p.gate + t * p.ldg + head[e] * D + cc;
    bf16* o = p.out + t * p.ldo + head[e] * D + cc;
#pragma unroll
    for (int i = 0; i < D / 8; ++i) {
      const float2 x = gl_unpack(*reinterpret_cast<const uint32_t*>(g + i * 8));
      *reinterpret_cast<uint32_t*>(o + i * 8) = gl_pack(O[i][2 * e] * p.mult * gl_rcp(1.f + gl_ex2(-x.x * kTalkLog2e)),
                                                        O[i][2 * e + 1] * p.mult * gl_rcp(1.f + gl_ex2(-x.y * kTalkLog2e)));
    }
  }
}

// ------------------------------------------------------------------------------------------ decode steps
struct TalkDecodeParams {
  const bf16* q; const bf16* gate; int ldg; bf16* out; int ldo;
  const bf16* kc; const bf16* vc; const int* block_table; int bt_stride;
  const int* kv_lens;
  int B, hq, hkv, group, bs, num_blocks, window;
  int splits, span;                          // key ranges; positions per head of the score buffer (a multiple of 64)
  float scale2, mult;
  const float* r1; const float* r2; const float* talk;
  float* scores;                             // [B][hq][span], base 2, from the first visited page's first key on
  float* part_ml;                            // [B][hq][splits][2]
  float* part_o;                             // [B][hq][splits][D] (splits > 1)
  int* counters;                             // [B * hkv], zero between launches
  int* status;
};

// pages [first, stop) of a split; `base` is the first key of the first visited page
__device__ __forceinline__ void talk_pages(const TalkDecodeParams& p, int n_keys, int split, int& first, int& stop, int& base) {
  const int lo = max(0, n_keys - p.window), p0 = lo / 64, p1 = (n_keys + 63) / 64;
  const int per = (p1 - p0 + p.splits - 1) / p.splits;
  first = p0 + split * per;
  stop = min(p1, first + per);
  base = p0 * 64;
}
__device__ __forceinline__ const bf16* talk_page(const TalkDecodeParams& p, const bf16* cache, int b, int page, int kvh, int D) {
  int blk = p.block_table[(size_t)b * p.bt_stride + page * 64 / p.bs];
  if (blk < 0 || blk >= p.num_blocks) { if (p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); blk = 0; }
  return cache + (((size_t)blk * p.hkv + kvh) * p.bs + page * 64 % p.bs) * D;
}

// grid (splits, hkv * ceil(group / 16), B), 4 warps: 8 keys per warp and step, straight from the cache (the two operands share a
// permutation of the dimensions in which a lane's 16 bytes serve two products)
template <int D>
__global__ void __launch_bounds__(128) talking_scores_kernel(const TalkDecodeParams p) {
  __shared__ float red[4][16][2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, b = blockIdx.z;
  const int chunks = (p.group + 15) / 16, kvh = blockIdx.y / chunks, hc = blockIdx.y % chunks * 16;
  const int h0 = kvh * p.group + hc, rows = min(16, p.group - hc);
  grid_dep_launch();
  const int n_keys = p.kv_lens[b], qpos = n_keys - 1;
  int first, stop, base;
  talk_pages(p, n_keys, blockIdx.x, first, stop, base);
  const int r = lane >> 2, kq = lane & 3;
  float r1[2], r2[2], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int h = h0 + min(r + 8 * e, rows - 1);
    r1[e] = p.r1[h];
    r2[e] = p.r2[h];
  }
  grid_dep_wait();
  uint32_t qa[D / 32][2][4];
#pragma unroll
  for (int s = 0; s < D / 32; ++s) {
    uint4 v[2];
#pragma unroll
    for (int e = 0; e < 2; ++e)
      v[e] = r + 8 * e < rows ? *reinterpret_cast<const uint4*>(p.q + ((size_t)b * p.hq + h0 + r + 8 * e) * D + s * 32 + kq * 8) : make_uint4(0, 0, 0, 0);
    qa[s][0][0] = v[0].x; qa[s][0][1] = v[1].x; qa[s][0][2] = v[0].y; qa[s][0][3] = v[1].y;
    qa[s][1][0] = v[0].z; qa[s][1][1] = v[1].z; qa[s][1][2] = v[0].w; qa[s][1][3] = v[1].w;
  }
  for (int page = first; page < stop; ++page) {
    const bf16* k = talk_page(p, p.kc, b, page, kvh, D);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int k8 = (warp * 2 + i) * 8;
      float c[4] = {0.f, 0.f, 0.f, 0.f};
      uint4 v[D / 32];
#pragma unroll
      for (int s = 0; s < D / 32; ++s) v[s] = *reinterpret_cast<const uint4*>(k + (size_t)(k8 + r) * D + s * 32 + kq * 8);
#pragma unroll
      for (int s = 0; s < D / 32; ++s) {
        gl_mma(c, qa[s][0], v[s].x, v[s].y);
        gl_mma(c, qa[s][1], v[s].z, v[s].w);
      }
      const int key = page * 64 + k8 + 2 * kq;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float s[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int far = qpos - (key + x);
          const float val = fmaf(c[2 * e + x], p.scale2, -r1[e] * gl_lg2(fmaf(r2[e], (float)max(far, 0), 1.f)));
          s[x] = far >= 0 && far < p.window ? val : -INFINITY;
        }
        if (r + 8 * e < rows)
          *reinterpret_cast<float2*>(p.scores + ((size_t)b * p.hq + h0 + r + 8 * e) * p.span + key - base) = make_float2(s[0], s[1]);
        const float mx = fmaxf(m[e], fmaxf(s[0], s[1])), ref = mx == -INFINITY ? 0.f : mx;
        l[e] = l[e] * gl_ex2(m[e] - ref) + gl_ex2(s[0] - ref) + gl_ex2(s[1] - ref);
        m[e] = mx;
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float mx = m[e];
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    float s = m[e] == -INFINITY ? 0.f : l[e] * gl_ex2(m[e] - mx);
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    if (kq == 0) { red[warp][r + 8 * e][0] = mx; red[warp][r + 8 * e][1] = s; }
  }
  __syncthreads();
  if (tid < rows) {
    float mx = -INFINITY, s = 0.f;
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, red[w][tid][0]);
    for (int w = 0; w < 4; ++w) s += red[w][tid][0] == -INFINITY ? 0.f : red[w][tid][1] * gl_ex2(red[w][tid][0] - mx);
    float* o = p.part_ml + (((size_t)b * p.hq + h0 + tid) * p.splits + blockIdx.x) * 2;
    o[0] = mx;
    o[1] = s;
  }
}

// grid (splits, hkv, B), 128 threads: a thread owns four columns of the head and every (512 / D)-th key of a page
template <int D, int GR>
__global__ void __launch_bounds__(128) talking_values_kernel(const TalkDecodeParams p) {
  constexpr int CG = D / 4, KSUB = 128 / CG;
  extern __shared__ float tv_sm[];
  const int H = p.hq, tid = threadIdx.x, b = blockIdx.z, kvh = blockIdx.y, h0 = kvh * p.group;
  float* sp = tv_sm;                         // [H][64] weights
  float* sw = sp + H * 64;                   // [64][GR] mixed
  float* st = sw + 64 * GR;                  // [group][H] mixing matrix
  float* sm = st + p.group * H;              // [H] maxima and inverse sums
  float* si = sm + H;
  float* so = tv_sm;                         // [KSUB][GR][D] at the end
  __shared__ int s_last;
  grid_dep_launch();
  const int n_keys = p.kv_lens[b];
  int first, stop, base;
  talk_pages(p, n_keys, blockIdx.x, first, stop, base);
  for (int i = tid; i < p.group * H; i += 128) st[i] = p.talk[(size_t)h0 * H + i];
  grid_dep_wait();
  for (int h = tid; h < H; h += 128) {
    const float* ml = p.part_ml + ((size_t)b * H + h) * p.splits * 2;
    float mx = -INFINITY, s = 0.f;
    for (int i = 0; i < p.splits; ++i) mx = fmaxf(mx, __ldcg(ml + 2 * i));
    for (int i = 0; i < p.splits; ++i) { const float m = __ldcg(ml + 2 * i); s += m == -INFINITY ? 0.f : __ldcg(ml + 2 * i + 1) * gl_ex2(m - mx); }
    sm[h] = mx;
    si[h] = s > 0.f ? 1.f / s : 0.f;
  }
  float acc[GR][4];
#pragma unroll
  for (int g = 0; g < GR; ++g) acc[g][0] = acc[g][1] = acc[g][2] = acc[g][3] = 0.f;
  const int c4 = tid % CG * 4, ksub = tid / CG;
  for (int page = first; page < stop; ++page) {
    __syncthreads();
    for (int i = tid; i < H * 16; i += 128) {
      const int h = i >> 4, k = (i & 15) * 4;
      const float4 s = __ldcg(reinterpret_cast<const float4*>(p.scores + ((size_t)b * H + h) * p.span + page * 64 - base + k));
      const float m = sm[h], f = si[h];
      *reinterpret_cast<float4*>(sp + h * 64 + k) = make_float4(gl_ex2(s.x - m) * f, gl_ex2(s.y - m) * f, gl_ex2(s.z - m) * f, gl_ex2(s.w - m) * f);
    }
    __syncthreads();
    for (int i = tid; i < 64 * GR; i += 128) {
      const int g = i >> 6, k = i & 63;
      float w = 0.f;
      if (g < p.group)
        for (int x = 0; x < H; ++x) w = fmaf(st[g * H + x], sp[x * 64 + k], w);
      sw[k * GR + g] = w;
    }
    __syncthreads();
    const bf16* v = talk_page(p, p.vc, b, page, kvh, D) + c4;
#pragma unroll 4
    for (int k = ksub; k < 64; k += KSUB) {
      const uint2 u = *reinterpret_cast<const uint2*>(v + (size_t)k * D);
      const float2 a = gl_unpack(u.x), c = gl_unpack(u.y);
#pragma unroll
      for (int g = 0; g < GR; ++g) {
        const float w = sw[k * GR + g];
        acc[g][0] = fmaf(w, a.x, acc[g][0]); acc[g][1] = fmaf(w, a.y, acc[g][1]);
        acc[g][2] = fmaf(w, c.x, acc[g][2]); acc[g][3] = fmaf(w, c.y, acc[g][3]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int g = 0; g < GR; ++g) *reinterpret_cast<float4*>(so + ((size_t)ksub * GR + g) * D + c4) = make_float4(acc[g][0], acc[g][1], acc[g][2], acc[g][3]);
  __syncthreads();
  auto finish = [&](int g, int d, float x) {
    const float y = __bfloat162float(p.gate[(size_t)b * p.ldg + (h0 + g) * D + d]);
    p.out[(size_t)b * p.ldo + (h0 + g) * D + d] = __float2bfloat16(x * p.mult * gl_rcp(1.f + gl_ex2(-y * kTalkLog2e)));
  };
  for (int i = tid; i < p.group * D; i += 128) {
    const int g = i / D, d = i % D;
    float x = 0.f;
#pragma unroll
    for (int k = 0; k < KSUB; ++k) x += so[((size_t)k * GR + g) * D + d];
    if (p.splits == 1) finish(g, d, x);
    else p.part_o[(((size_t)b * H + h0 + g) * p.splits + blockIdx.x) * D + d] = x;
  }
  if (p.splits == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int* c = p.counters + b * p.hkv + kvh;
    s_last = atomicAdd(c, 1) == p.splits - 1;
    if (s_last) *c = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int i = tid; i < p.group * D; i += 128) {
    const int g = i / D, d = i % D;
    const float* o = p.part_o + ((size_t)b * H + h0 + g) * p.splits * D + d;
    float x = 0.f;
    for (int s = 0; s < p.splits; ++s) x += __ldcg(o + (size_t)s * D);
    finish(g, d, x);
  }
}

}  // namespace xft

using namespace xft;

template <int D, int HB, int KT>
static int launch_prefill(const TalkPrefillParams& p, int B, int max_q, cudaStream_t st) {
  constexpr int QPB = 16 / HB, HP = HB == 1 ? 16 : 32;
  const size_t smem = ((size_t)2 * p.hkv * KT * (D + 8) + HP * (HP + 8) + (size_t)2 * p.blocks * HP * (QPB * (KT + 8) + 8)) * 2;
  if (smem > 227 * 1024) return -6;
  static size_t allowed = 0;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(talking_prefill_kernel<D, HB, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return 3000 + (int)cudaGetLastError();
    allowed = smem;
  }
  const int qt = p.blocks * QPB;
  cudaError_t e = launch_pdl(talking_prefill_kernel<D, HB, KT>, dim3((max_q + qt - 1) / qt, B), dim3(kTalkThreads), smem, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
template <int D, int HB>
static int prefill_keys(const TalkPrefillParams& p, int keys, int B, int max_q, cudaStream_t st) {
  if (keys == 64) return launch_prefill<D, HB, 64>(p, B, max_q, st);
  if (keys == 32) return launch_prefill<D, HB, 32>(p, B, max_q, st);
  return launch_prefill<D, HB, 16>(p, B, max_q, st);
}

// Keys per tile of the prompt kernel for these sizes, 0: it has no instance.
extern "C" int xft_talking_prefill_keys(int hq, int hkv, int D) {
  if (hq <= 0 || hkv <= 0 || hq % hkv || hq > 32 || (D != 64 && D != 128)) return 0;
  const int hb = hq > 16 ? 2 : 1;
  if (hb == 2 && (hq / hkv) % 2) return 0;                 // two heads of a unit share their keys
  const int blocks = 16 * hb / hq > 0 ? 16 * hb / hq : 1, hp = hb == 1 ? 16 : 32, qpb = 16 / hb;
  for (int kt = 64; kt >= 16; kt /= 2)
    if (((size_t)2 * hkv * kt * (D + 8) + hp * (hp + 8) + (size_t)2 * blocks * hp * (qpb * (kt + 8) + 8)) * 2 <= 227 * 1024) return kt;
  return 0;
}

// bf16: q [T, hq, D], gate and out [T, ld] (head h at columns h * D), caches [num_blocks, hkv, bs, D] with bs a multiple of 64; r1, r2
// [hq], talk [hq, hq] fp32 (of bf16 values).  window 0: every earlier key.
extern "C" int xft_talking_prefill(const void* q, const void* gate, int ldg, void* out, int ldo, const void* kc, const void* vc,
                                   const int* block_table, int bt_stride, const int* cu_q, const int* kv_lens, int B, int max_q, int hq,
                                   int hkv, int D, int bs, int num_blocks, float scale, const float* r1, const float* r2, const float* talk,
                                   int window, float mult, int* status, cudaStream_t st) {
  if (B <= 0 || max_q <= 0) return 0;
  const int keys = xft_talking_prefill_keys(hq, hkv, D);
  if (!keys || bs <= 0 || bs % 64 || window < 0 || ldg < hq * D || ldo < hq * D || ((ldg | ldo) & 1) || B > 65535) return -1;
  if (((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc) & 15 || ((uintptr_t)gate | (uintptr_t)out) & 3) return -2;
  const int hb = hq > 16 ? 2 : 1, blocks = 16 * hb / hq > 0 ? 16 * hb / hq : 1;
  TalkPrefillParams p{(const bf16*)q, (const bf16*)gate, ldg, (bf16*)out, ldo, (const bf16*)kc, (const bf16*)vc, block_table, bt_stride, cu_q,
                      kv_lens, hq, hkv, hq / hkv, bs, num_blocks, window > 0 ? min(window, 1 << 30) : 1 << 30, blocks * hq / hb, blocks,
                      scale * kTalkLog2e, mult, r1, r2, talk, status};
  if (D == 64) return hb == 1 ? prefill_keys<64, 1>(p, keys, B, max_q, st) : prefill_keys<64, 2>(p, keys, B, max_q, st);
  return hb == 1 ? prefill_keys<128, 1>(p, keys, B, max_q, st) : prefill_keys<128, 2>(p, keys, B, max_q, st);
}

template <int D, int GR>
static cudaError_t launch_values(const TalkDecodeParams& p, cudaStream_t st) {
  const size_t work = (size_t)p.hq * 64 + 64 * GR + p.group * p.hq + 2 * p.hq, end = (size_t)512 / D * GR * D;
  const size_t smem = (work > end ? work : end) * sizeof(float);
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(talking_values_kernel<D, GR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  return launch_pdl(talking_values_kernel<D, GR>, dim3(p.splits, p.hkv, p.B), dim3(128), smem, st, p);
}
template <int D>
static int launch_decode(const TalkDecodeParams& p, cudaStream_t st) {
  cudaError_t e = launch_pdl(talking_scores_kernel<D>, dim3(p.splits, p.hkv * ((p.group + 15) / 16), p.B), dim3(128), 0, st, p);
  if (e != cudaSuccess) return (int)e;
  e = p.group <= 1 ? launch_values<D, 1>(p, st) : p.group <= 2 ? launch_values<D, 2>(p, st) : p.group <= 4 ? launch_values<D, 4>(p, st)
      : p.group <= 8 ? launch_values<D, 8>(p, st) : launch_values<D, 16>(p, st);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// One token per sequence: q [B, hq, D] and the rest as above, heads of 64, 128 or 256, up to 16 per key/value head and 128 in all.  Scratch:
// scores [B * hq * span] with span a multiple of 64, at least 64 * (pages that a window can touch); part_ml [B * hq * splits * 2], part_o
// [B * hq * splits * D], counters [B * hkv] zeros (left as zeros).
extern "C" int xft_talking_decode(const void* q, const void* gate, int ldg, void* out, int ldo, const void* kc, const void* vc,
                                  const int* block_table, int bt_stride, const int* kv_lens, int B, int hq, int hkv, int D, int bs,
                                  int num_blocks, float scale, const float* r1, const float* r2, const float* talk, int window, float mult,
                                  int splits, int span, float* scores, float* part_ml, float* part_o, int* counters, int* status,
                                  cudaStream_t st) {
  if (B <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || hq % hkv || hq / hkv > 16 || hq > 128 || bs <= 0 || bs % 64 || window < 0 || splits < 1 || (span & 63) || span <= 0)
    return -1;
  if (ldg < hq * D || ldo < hq * D || B > 65535 || hkv > 65535) return -2;
  if (((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)scores) & 15) return -3;
  TalkDecodeParams p{(const bf16*)q, (const bf16*)gate, ldg, (bf16*)out, ldo, (const bf16*)kc, (const bf16*)vc, block_table, bt_stride, kv_lens,
                     B, hq, hkv, hq / hkv, bs, num_blocks, window > 0 ? min(window, 1 << 30) : 1 << 30, splits, span, scale * kTalkLog2e, mult,
                     r1, r2, talk, scores, part_ml, part_o, counters, status};
  if (D == 64) return launch_decode<64>(p, st);
  if (D == 128) return launch_decode<128>(p, st);
  if (D == 256) return launch_decode<256>(p, st);
  return -4;
}
