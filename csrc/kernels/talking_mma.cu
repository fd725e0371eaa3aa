// Attention whose heads' weights are mixed, on the tensor cores (bf16, heads of 64 or 128; see talking.cu for what it computes).
//
// Prompt portions, talking_prefill_kernel: a CTA takes a tile of queries with all of their heads, since the weights of all heads
// of a (query, key) pair meet in the mix.  A warp owns a unit of 16 rows: 16 queries of one head, or (more than 16 heads) 8
// queries of two heads that share keys.  Where the heads of a group allow it a warp has two such units side by side, which halves the
// operands that it reads from shared memory.  The keys are visited twice.  The first pass carries a running maximum and sum per row.
// The second forms the scores again, and from them the finished weights; they go to shared memory as two bf16 halves, are
// multiplied with the mixing matrix there (a product over the heads, both halves with fp32 sums: nothing of their 16 bits of
// mantissa is lost before the mix), and come back as the operand of the product with the values.
//
// Decode steps: talking_scores_kernel writes the scores of a key range of one key/value head with its maxima and sums,
// talking_values_kernel merges those of all ranges, mixes in fp32 and adds up the values of its range.  The ranges of a head are a
// cluster, whose CTAs add up their results through distributed shared memory, each a part of the columns, and apply the gate.
#include "mma_sync.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;
int make_tensor_map_groups(CUtensorMap* out, const void* ptr, uint64_t groups, uint64_t rows, uint64_t cols, uint32_t box_groups,
                           uint32_t box_rows);
constexpr float kTalkLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------ prompt portions
struct TalkPrefillParams {
  const bf16* q; const bf16* gate; int ldg; bf16* out; int ldo;
  const int* block_table; int bt_stride;
  const int* cu_q; const int* kv_lens;
  int hq, hkv, group, num_blocks, window;
  int units, blocks;                         // units of 16 rows, blocks of queries (units = blocks * hq / heads per unit)
  int bs_shift;                              // log2 of the page size
  int stages;                                // tiles of keys in shared memory, 1 or 2
  float scale2, mult;                        // softmax scale * log2(e)
  const float* r1; const float* r2; const float* talk;
  int* status;
};

constexpr int kTalkUnits = 16;               // units of 16 rows per CTA at most
constexpr int kTalkPages = 64;
constexpr size_t kTalkSmem = 227 * 1024 - 512;          // beside the static part

// Shared memory: `stages` tiles of keys and one of values as TMA leaves them (per 64 columns and head KT rows of 128 bytes, swizzled
// by row & 7), the queries in the order of their fragments, the mixing matrix, weights (two buffers of the upper halves, which the mixed
// weights replace, and one of the lower), biases.
template <int D, int HB, int KT>
struct TalkCfg {
  static constexpr int QPB = 16 / HB, HP = HB == 1 ? 16 : 32;          // queries of a block; heads, padded
  static constexpr int QP = KT + 8, PITCH = QPB * QP + 8, MP = HP + 8;      // row strides: weights of a query, of a head, matrix
  static constexpr int TAB = KT + QPB;                                 // biases of a head: distances of a tile and a block
  static size_t bytes(int hkv, int blocks, int stages) {
    return 1024 + ((size_t)(stages + 1) * hkv * KT * D + HP * MP + (size_t)3 * blocks * HP * PITCH) * 2 +
           (size_t)kTalkUnits * (HB * TAB * 4 + D / 16 * 512);
  }
};

// U: units per warp.  With two their queries stay in registers, with one they are read from shared memory.
template <int D, int HB, int KT, int U>
__global__ void __launch_bounds__(kTalkUnits / U * 32, 1) talking_prefill_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const TalkPrefillParams p) {
  using Cfg = TalkCfg<D, HB, KT>;
  constexpr int QPB = Cfg::QPB, HP = Cfg::HP, QP = Cfg::QP, PITCH = Cfg::PITCH, MP = Cfg::MP, MT = HP / 16;
  constexpr int NW = kTalkUnits / U, NT = NW * 32;
  constexpr int KH = U == 1 ? KT : 16;                                 // keys whose scores are in registers at a time
  constexpr int BOX = KT * 128;                                        // bytes of a head's 64 columns
  extern __shared__ uint8_t tk_raw[];
  __shared__ uint64_t full[4];                                         // one per tile buffer
  __shared__ int pages[kTalkPages];                                    // the first entries of the block table that matter
  const int tile_size = p.hkv * KT * D, half_size = p.blocks * HP * PITCH, nbuf = p.stages + 1;
  // tile buffers; the offset is added to the array itself, so that the compiler sees every address to be one of shared memory
  bf16* sT = reinterpret_cast<bf16*>(tk_raw + ((1024 - (smem_u32(tk_raw) & 1023)) & 1023));
  uint4* qa = reinterpret_cast<uint4*>(sT + (size_t)nbuf * tile_size) + (threadIdx.x >> 5) * (U * D / 16 * 32) + (threadIdx.x & 31);   // this lane's
  bf16* sM = sT + (size_t)nbuf * tile_size + kTalkUnits * D * 16;               // the mixing matrix [HP][MP]
  bf16* sP = sM + HP * MP;                                             // [2 upper, 1 lower][blocks][HP][PITCH]
  bf16* sLow = sP + (size_t)2 * half_size;
  float* tab = reinterpret_cast<float*>(sLow + half_size) + (threadIdx.x >> 5) * U * HB * Cfg::TAB;      // this warp's
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
  // this warp's units, neighbouring heads of one group
  const int per_block = p.hq / HB, qb = warp * U / per_block, h0 = (warp * U % per_block) * HB;
  const bool active = warp * U < p.units;
  const int kvh = active ? h0 / p.group : 0;
  const int r = lane >> 2, cc = 2 * (lane & 3);
  auto query = [&](int e) { return row0 + (active ? qb : 0) * QPB + (HB == 1 ? r + 8 * e : r); };       // of rows r and r + 8
  auto head = [&](int u, int e) { return active ? h0 + (HB == 1 ? u : 2 * u + e) : 0; };
  // the mixing matrix as an operand
  for (int i = tid; i < HP * HP; i += NT) {
    const int h = i / HP, g = i % HP;
    sM[h * MP + g] = __float2bfloat16(h < p.hq && g < p.hq ? p.talk[h * p.hq + g] : 0.f);
  }
  for (int i = tid; i < 3 * half_size / 8; i += NT) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);
  if (tid == 0) {
    for (int i = 0; i < nbuf; ++i) mbar_init(&full[i], 1);
    fence_barrier_init();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  __syncthreads();
  grid_dep_wait();
  uint32_t qr[U == 1 ? 1 : U][U == 1 ? 1 : D / 16][4];
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e & 1;
        v[e] = active && query(i) < q_len ? *reinterpret_cast<const uint32_t*>(
            p.q + ((size_t)(q0 + query(i)) * p.hq + head(u, i)) * D + ks * 16 + cc + (e >> 1) * 8) : 0u;
        if (U > 1) qr[u % (U == 1 ? 1 : U)][ks % (U == 1 ? 1 : D / 16)][e] = v[e];
      }
      if (U == 1) qa[ks * 32] = make_uint4(v[0], v[1], v[2], v[3]);    // read back by the same lane
    }
  const int* bt = p.block_table + (size_t)b * p.bt_stride;
  // tile buffers are filled by one thread, behind a barrier that says everyone is done with what was there
  uint32_t phases = 0;
  const int page0 = k_lo >> p.bs_shift;
  for (int i = tid; i < kTalkPages && i <= ((k_lo + (n_tiles - 1) * KT) >> p.bs_shift) - page0; i += NT) pages[i] = bt[page0 + i];
  __syncthreads();
  auto load = [&](int buf, const CUtensorMap& map, int tile, int by) {
    if (tile >= n_tiles || tid != by * 32) return;
    const int key = k_lo + tile * KT, page = (key >> p.bs_shift) - page0;
    int blk = page < kTalkPages ? pages[page] : bt[page0 + page];
    if (blk < 0 || blk >= p.num_blocks) { if (p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); blk = 0; }
    mbar_expect_tx(&full[buf], tile_size * 2);
    uint8_t* dst = reinterpret_cast<uint8_t*>(sT + (size_t)buf * tile_size);
#pragma unroll
    for (int c = 0; c < D / 64; ++c)
      tma_load_3d(dst + c * p.hkv * BOX, &map, &full[buf], c * 64, key & ((1 << p.bs_shift) - 1), blk * p.hkv, kEvictNormal);
  };
  auto arrived = [&](int buf) {                                        // a wait that runs out is reported; what was there is read
    mbar_wait(&full[buf], phases >> buf & 1, p.status, XFT_ERR_WAIT_FULL);
    phases ^= 1u << buf;
  };
  const int fa_r = (lane & 7) + ((lane >> 3) & 1) * 8, fa_c = (lane >> 4) * 8;
  const int fb_r = (lane & 7) + ((lane >> 4) & 1) * 8;
  // a lane's 16-byte piece of the first 16 columns, swizzled: keys (two pieces along a row) and values (two along the columns)
  const int xk = (((lane >> 3) & 1) ^ (lane & 7)) * 16, xv = ((lane >> 4) ^ (lane & 7)) * 16;
  // The bias of a key depends on its distance alone: -r1 log2(1 + r2 distance), and -inf for one that is not visible.  Entry i of a
  // head's table belongs to the distance top - i, where `top` is that of the block's last query and the tile's first key.
  float ra[U * HB], rc[U * HB];
#pragma unroll
  for (int e = 0; e < U * HB; ++e) {
    ra[e] = active ? -p.r1[h0 + e] : 0.f;
    rc[e] = active ? p.r2[h0 + e] : 0.f;
  }
  const int top0 = past + row0 + ((active ? qb : 0) + 1) * QPB - 1 - k_lo;
  auto biases = [&](int tile) {
    if (!active || tile >= n_tiles) return;
    __syncwarp();
#pragma unroll
    for (int e = 0; e < U * HB; ++e)
#pragma unroll
      for (int i = 0; i < Cfg::TAB - 1; i += 32) {
        const int far = top0 - tile * KT - i - lane;
        const float v = ra[e] * gl_lg2(fmaf(rc[e], (float)far, 1.f));
        if (i + lane < Cfg::TAB - 1) tab[e * Cfg::TAB + i + lane] = far >= 0 && far < p.window ? v : -INFINITY;
      }
    __syncwarp();
  };
  const int chunk = p.hkv * BOX;                                       // bytes of 64 columns of all heads
  const float* my_tab = tab + QPB - 1 - r + cc;
  // scores (base 2) of this warp's rows and KH keys from `k` on of the tile in `s`
  float S[U][KH / 8][4];
  auto scores = [&](const bf16* s, int k) {
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int j = 0; j < KH / 8; ++j) S[u][j][0] = S[u][j][1] = S[u][j][2] = S[u][j][3] = 0.f;
    const uint8_t* base = reinterpret_cast<const uint8_t*>(s) + kvh * BOX + (k + fb_r) * 128;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t a[U][4];
      if (U == 1) {
        const uint4 q = qa[ks * 32];
        a[0][0] = q.x; a[0][1] = q.y; a[0][2] = q.z; a[0][3] = q.w;
      } else {
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
          for (int e = 0; e < 4; ++e) a[u][e] = qr[u % (U == 1 ? 1 : U)][ks % (U == 1 ? 1 : D / 16)][e];
      }
#pragma unroll
      for (int j = 0; j < KH / 8; j += 2) {
        uint32_t w[4];
        gl_ldsm(w, base + ks / 4 * chunk + j * 1024 + (xk ^ (ks % 4 * 32)));
#pragma unroll
        for (int u = 0; u < U; ++u) {
          gl_mma(S[u][j], a[u], w[0], w[1]);
          gl_mma(S[u][j + 1], a[u], w[2], w[3]);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int j = 0; j < KH / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int at = HB == 1 ? u * Cfg::TAB - (e >> 1) * 8 : (2 * u + (e >> 1)) * Cfg::TAB;
          S[u][j][e] = fmaf(S[u][j][e], p.scale2, my_tab[at + k + j * 8 + (e & 1)]);
        }
  };
  // ---- first pass: maxima and sums; all buffers take turns with keys
  float m[U][2], l[U][2];
#pragma unroll
  for (int u = 0; u < U; ++u) { m[u][0] = m[u][1] = -INFINITY; l[u][0] = l[u][1] = 0.f; }
  for (int j = 0; j + 1 < nbuf; ++j) load(j, tmK, j, j);
  biases(0);
  for (int j = 0, buf = 0, ahead = nbuf - 1; j < n_tiles; ++j, buf = buf + 1 == nbuf ? 0 : buf + 1, ahead = ahead + 1 == nbuf ? 0 : ahead + 1) {
    __syncthreads();
    load(ahead, tmK, j + nbuf - 1, j % NW);
    arrived(buf);
    if (!active) continue;
#pragma unroll
    for (int k = 0; k < KT; k += KH) {
      scores(sT + buf * tile_size, k);
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float mx = m[u][e];
#pragma unroll
          for (int i = 0; i < KH / 8; ++i) mx = fmaxf(mx, fmaxf(S[u][i][2 * e], S[u][i][2 * e + 1]));
          const float ref = mx == -INFINITY ? 0.f : mx;                // nothing seen yet: every term is zero
          float sum = 0.f;
#pragma unroll
          for (int i = 0; i < KH / 8; ++i) sum += gl_ex2(S[u][i][2 * e] - ref) + gl_ex2(S[u][i][2 * e + 1] - ref);
          l[u][e] = fmaf(l[u][e], gl_ex2(m[u][e] - ref), sum);         // this lane's columns alone
          m[u][e] = mx;
        }
    }
    biases(j + 1);
  }
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int e = 0; e < 2; ++e) {                                      // the four lanes of a row
      float mx = m[u][e];
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      float s = m[u][e] == -INFINITY ? 0.f : l[u][e] * gl_ex2(m[u][e] - mx);
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      m[u][e] = s > 0.f ? mx + gl_lg2(s) : INFINITY;                   // log2 of the row's sum
    }
  // ---- second pass: the scores of one tile beside the values of the one before
  float O[U][D / 8][4];
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int j = 0; j < D / 8; ++j) O[u][j][0] = O[u][j][1] = O[u][j][2] = O[u][j][3] = 0.f;
  const int block_at = (active ? qb : 0) * HP * PITCH;                 // this unit's block
  auto weights = [&](int j) {                                          // of tile j, in two halves
    bf16* dst = sP + (j & 1) * half_size + block_at;
    const bf16* keys = sT + (p.stages > 1 ? (j & 1) * tile_size : 0);
#pragma unroll
    for (int k = 0; k < KT; k += KH) {
      scores(keys, k);
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int at = head(u, e) * PITCH + (HB == 1 ? r + 8 * e : r) * QP + k + cc;
#pragma unroll
          for (int i = 0; i < KH / 8; ++i) {
            const float a = gl_ex2(S[u][i][2 * e] - m[u][e]), c = gl_ex2(S[u][i][2 * e + 1] - m[u][e]);
            const uint32_t hi = gl_pack(a, c);
            const float2 f = gl_unpack(hi);
            *reinterpret_cast<uint32_t*>(dst + at + i * 8) = hi;
            *reinterpret_cast<uint32_t*>(sLow + block_at + at + i * 8) = gl_pack(a - f.x, c - f.y);
          }
        }
    }
  };
  // the mix of tile j, in place: 16 keys of a query at a time, two such pieces side by side
  const int pieces = p.blocks * QPB * (KT / 16);
  auto mix = [&](int j) {
    bf16* upper = sP + (j & 1) * half_size;
    constexpr int N2 = MT == 1 ? 2 : 1;
    uint32_t t[MT][MT][4];
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
      for (int g = 0; g < MT; ++g) gl_ldsm(t[a][g], sM + (a * 16 + fa_r) * MP + g * 16 + fa_c);
    for (int c0 = warp; c0 < pieces; c0 += N2 * NW) {
      int at[N2];
      uint32_t x[N2][2][MT][4];
#pragma unroll
      for (int n = 0; n < N2; ++n) {
        const int c = min(c0 + n * NW, pieces - 1), qq = c / (KT / 16), k = c % (KT / 16) * 16;
        at[n] = qq / QPB * HP * PITCH + qq % QPB * QP + k;
#pragma unroll
        for (int g = 0; g < MT; ++g) {
          gl_ldsm_t(x[n][0][g], upper + at[n] + (g * 16 + fa_r) * PITCH + fa_c);
          gl_ldsm_t(x[n][1][g], sLow + at[n] + (g * 16 + fa_r) * PITCH + fa_c);
        }
      }
      float w[N2][MT][2][4];
#pragma unroll
      for (int n = 0; n < N2; ++n)
#pragma unroll
        for (int a = 0; a < MT; ++a) {
#pragma unroll
          for (int i = 0; i < 2; ++i) w[n][a][i][0] = w[n][a][i][1] = w[n][a][i][2] = w[n][a][i][3] = 0.f;
#pragma unroll
          for (int g = 0; g < MT; ++g)
#pragma unroll
            for (int part = 0; part < 2; ++part) {
              gl_mma(w[n][a][0], t[a][g], x[n][part][g][0], x[n][part][g][1]);
              gl_mma(w[n][a][1], t[a][g], x[n][part][g][2], x[n][part][g][3]);
            }
        }
      __syncwarp();
#pragma unroll
      for (int n = 0; n < N2; ++n)
        if (n == 0 || c0 + n * NW < pieces)
#pragma unroll
          for (int a = 0; a < MT; ++a)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              *reinterpret_cast<uint32_t*>(upper + at[n] + (a * 16 + r) * PITCH + i * 8 + cc) = gl_pack(w[n][a][i][0], w[n][a][i][1]);
              *reinterpret_cast<uint32_t*>(upper + at[n] + (a * 16 + r + 8) * PITCH + i * 8 + cc) = gl_pack(w[n][a][i][2], w[n][a][i][3]);
            }
    }
  };
  const bool two = p.stages > 1;
  auto key_buf = [&](int j) { return two ? j & 1 : 0; };
  const int value_buf = p.stages;
  auto load_keys = [&](int j) { load(key_buf(j), tmK, j, j % NW); };
  auto load_values = [&](int j) { load(value_buf, tmV, j, (j + NW / 2) % NW); };
  __syncthreads();                                                     // everyone is done with the first pass's tiles
  load_keys(0);
  if (two) load_keys(1);
  load_values(0);
  biases(0);
  arrived(key_buf(0));
  if (active) weights(0);
  __syncthreads();
  if (!two) load_keys(1);
  mix(0);
  biases(1);
  __syncthreads();
  for (int j = 0; j < n_tiles; ++j) {
    // here: mixed weights of tile j; its values and the keys of tile j + 1 are on their way
    if (two) load_keys(j + 2);
    if (j + 1 < n_tiles) {
      arrived(key_buf(j + 1));
      if (active) weights(j + 1);
    }
    arrived(value_buf);
    if (active) {
      const bf16* pw = sP + (j & 1) * half_size + block_at;
      const bf16* wrow = HB == 1 ? pw + h0 * PITCH + fa_r * QP : pw + (h0 + ((lane >> 3) & 1)) * PITCH + (lane & 7) * QP;
      const uint8_t* vb = reinterpret_cast<const uint8_t*>(sT + (size_t)value_buf * tile_size) + kvh * BOX + fa_r * 128;
#pragma unroll
      for (int ks = 0; ks < KT / 16; ++ks) {
        uint32_t a[U][4];
#pragma unroll
        for (int u = 0; u < U; ++u) gl_ldsm(a[u], wrow + u * HB * PITCH + ks * 16 + fa_c);
#pragma unroll
        for (int i = 0; i < D / 8; i += 2) {
          uint32_t w[4];
          gl_ldsm_t(w, vb + i / 8 * chunk + ks * 2048 + (xv ^ (i % 8 * 16)));
#pragma unroll
          for (int u = 0; u < U; ++u) {
            gl_mma(O[u][i], a[u], w[0], w[1]);
            gl_mma(O[u][i + 1], a[u], w[2], w[3]);
          }
        }
      }
    }
    __syncthreads();
    if (!two) load_keys(j + 2);
    load_values(j + 1);
    if (j + 1 < n_tiles) mix(j + 1);
    biases(j + 2);
    __syncthreads();
  }
  if (!active) return;
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      if (query(e) >= q_len) continue;
      const size_t t = q0 + query(e);
      const bf16* g = p.gate + t * p.ldg + head(u, e) * D + cc;
      bf16* o = p.out + t * p.ldo + head(u, e) * D + cc;
#pragma unroll
      for (int i = 0; i < D / 8; ++i) {
        const float2 x = gl_unpack(*reinterpret_cast<const uint32_t*>(g + i * 8));
        *reinterpret_cast<uint32_t*>(o + i * 8) = gl_pack(O[u][i][2 * e] * p.mult * gl_rcp(1.f + gl_ex2(-x.x * kTalkLog2e)),
                                                          O[u][i][2 * e + 1] * p.mult * gl_rcp(1.f + gl_ex2(-x.y * kTalkLog2e)));
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

// grid (splits, hkv, B), clusters of (splits), 256 threads: a thread owns four columns of the head and every (1024 / D)-th key of a page
constexpr int kTalkValues = 256;
template <int D, int GR>
__global__ void __launch_bounds__(kTalkValues) talking_values_kernel(const TalkDecodeParams p) {
  constexpr int CG = D / 4, KSUB = kTalkValues / CG, NT = kTalkValues;
  extern __shared__ __align__(16) float tv_sm[];
  const int H = p.hq, tid = threadIdx.x, lane = tid & 31, b = blockIdx.z, kvh = blockIdx.y, h0 = kvh * p.group, ns = p.splits;
  float* so = tv_sm;                         // [GR][D] this range's result, which the cluster reads
  float* sp = so + GR * D;                   // [H][64] weights
  float* sw = sp + H * 64;                   // [64][GR] mixed
  float* st = sw + 64 * GR;                  // [group][H] mixing matrix
  float* sm = st + p.group * H;              // [H] maxima and inverse sums
  float* si = sm + H;
  float* sr = sp;                            // [KSUB][GR][D] at the end
  grid_dep_launch();
  const int n_keys = p.kv_lens[b];
  int first, stop, base;
  talk_pages(p, n_keys, blockIdx.x, first, stop, base);
  for (int i = tid; i < p.group * H; i += NT) st[i] = p.talk[(size_t)h0 * H + i];
  const int c4 = tid % CG * 4, ksub = tid / CG;
  grid_dep_wait();
  for (int h = tid >> 5; h < H; h += NT / 32) {            // a warp per head, a range per lane
    const float2 ml = lane < ns ? __ldcg(reinterpret_cast<const float2*>(p.part_ml) + ((size_t)b * H + h) * ns + lane) : make_float2(-INFINITY, 0.f);
    float mx = ml.x;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float s = ml.x == -INFINITY ? 0.f : ml.y * gl_ex2(ml.x - mx);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) { sm[h] = mx; si[h] = s > 0.f ? 1.f / s : 0.f; }
  }
  float acc[GR][4];
#pragma unroll
  for (int g = 0; g < GR; ++g) acc[g][0] = acc[g][1] = acc[g][2] = acc[g][3] = 0.f;
  constexpr int KN = 64 / KSUB;              // keys of a page per thread
  for (int page = first; page < stop; ++page) {
    // values on their way while the weights are mixed
    const bf16* v = talk_page(p, p.vc, b, page, kvh, D) + c4;
    uint2 u[KN];
#pragma unroll
    for (int k = 0; k < KN; ++k) u[k] = *reinterpret_cast<const uint2*>(v + (size_t)(k * KSUB + ksub) * D);
    __syncthreads();
    for (int i = tid; i < H * 16; i += NT) {
      const int h = i >> 4, k = (i & 15) * 4;
      const float4 s = __ldcg(reinterpret_cast<const float4*>(p.scores + ((size_t)b * H + h) * p.span + page * 64 - base + k));
      const float m = sm[h], f = si[h];
      *reinterpret_cast<float4*>(sp + h * 64 + k) = make_float4(gl_ex2(s.x - m) * f, gl_ex2(s.y - m) * f, gl_ex2(s.z - m) * f, gl_ex2(s.w - m) * f);
    }
    __syncthreads();
    for (int i = tid; i < 64 * GR; i += NT) {
      const int g = i >> 6, k = i & 63;
      float w = 0.f;
      if (g < p.group)
#pragma unroll 8
        for (int x = 0; x < H; ++x) w = fmaf(st[g * H + x], sp[x * 64 + k], w);
      sw[k * GR + g] = w;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      const float2 a = gl_unpack(u[k].x), c = gl_unpack(u[k].y);
#pragma unroll
      for (int g = 0; g < GR; ++g) {
        const float w = sw[(k * KSUB + ksub) * GR + g];
        acc[g][0] = fmaf(w, a.x, acc[g][0]); acc[g][1] = fmaf(w, a.y, acc[g][1]);
        acc[g][2] = fmaf(w, c.x, acc[g][2]); acc[g][3] = fmaf(w, c.y, acc[g][3]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int g = 0; g < GR; ++g) *reinterpret_cast<float4*>(sr + ((size_t)ksub * GR + g) * D + c4) = make_float4(acc[g][0], acc[g][1], acc[g][2], acc[g][3]);
  __syncthreads();
  for (int i = tid; i < GR * D; i += NT) {
    float x = 0.f;
#pragma unroll
    for (int k = 0; k < KSUB; ++k) x += sr[(size_t)k * GR * D + i];
    so[i] = x;
  }
  if (ns > 1) { cluster_arrive(); cluster_wait(); } else __syncthreads();
  // this CTA's part of the columns
  const int n = p.group * D, per = (n + ns - 1) / ns, i0 = blockIdx.x * per, i1 = min(i0 + per, n);
  for (int i = i0 + tid; i < i1; i += NT) {
    float x = 0.f;
    if (ns > 1) {
      const uint32_t a = smem_u32(so + i);
#pragma unroll 8
      for (int c = 0; c < ns; ++c) x += ld_dsmem(dsmem_addr(a, c));
    } else x = so[i];
    const size_t col = (size_t)h0 * D + i;
    const float y = __bfloat162float(p.gate[(size_t)b * p.ldg + col]);
    p.out[(size_t)b * p.ldo + col] = __float2bfloat16(x * p.mult * gl_rcp(1.f + gl_ex2(-y * kTalkLog2e)));
  }
  if (ns > 1) { cluster_arrive(); cluster_wait(); }        // nobody leaves while its shared memory may be read
}

}  // namespace xft

using namespace xft;

template <int D, int HB, int KT, int U>
static int launch_units(const TalkPrefillParams& p, const void* kc, const void* vc, int bs, int B, int max_q, cudaStream_t st) {
  using Cfg = TalkCfg<D, HB, KT>;
  const size_t smem = Cfg::bytes(p.hkv, p.blocks, p.stages);
  if (smem > kTalkSmem) return -6;
  static size_t allowed = 0;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(talking_prefill_kernel<D, HB, KT, U>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return 3000 + (int)cudaGetLastError();
    allowed = smem;
  }
  const int qt = p.blocks * Cfg::QPB;
  CUtensorMap tmK, tmV;
  const uint64_t groups = (uint64_t)p.num_blocks * p.hkv;
  if (make_tensor_map_groups(&tmK, kc, groups, bs, D, p.hkv, KT) || make_tensor_map_groups(&tmV, vc, groups, bs, D, p.hkv, KT)) return -4;
  cudaError_t e = launch_pdl(talking_prefill_kernel<D, HB, KT, U>, dim3((max_q + qt - 1) / qt, B), dim3(kTalkUnits / U * 32), smem, st, tmK, tmV, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

template <int D, int HB, int KT>
static int launch_prefill(const TalkPrefillParams& p, const void* kc, const void* vc, int bs, int B, int max_q, cudaStream_t st) {
  if (p.group % (2 * HB) == 0) return launch_units<D, HB, KT, 2>(p, kc, vc, bs, B, max_q, st);
  return launch_units<D, HB, KT, 1>(p, kc, vc, bs, B, max_q, st);
}

// Keys per tile, stages and blocks of queries of the prompt kernel for these sizes; false: it has no instance.
template <int D, int HB>
static bool plan_prefill(int hq, int hkv, int& keys, int& stages, int& blocks) {
  const int most = 16 * HB / hq > 0 ? 16 * HB / hq : 1;
  for (int st = 2; st >= 1; --st)
    for (int kt = 32; kt >= 16; kt /= 2)
      for (int n = most; n >= (most + 1) / 2; --n) {
        const size_t b = kt == 32 ? TalkCfg<D, HB, 32>::bytes(hkv, n, st) : TalkCfg<D, HB, 16>::bytes(hkv, n, st);
        if (b <= kTalkSmem) { keys = kt; stages = st; blocks = n; return true; }
      }
  return false;
}
static bool plan_prefill(int hq, int hkv, int D, int& keys, int& stages, int& blocks) {
  if (hq <= 0 || hkv <= 0 || hq % hkv || hq > 32 || (D != 64 && D != 128)) return false;
  if (hq <= 16) return D == 64 ? plan_prefill<64, 1>(hq, hkv, keys, stages, blocks) : plan_prefill<128, 1>(hq, hkv, keys, stages, blocks);
  if (hq / hkv % 2) return false;                          // two heads of a unit share their keys
  return D == 64 ? plan_prefill<64, 2>(hq, hkv, keys, stages, blocks) : plan_prefill<128, 2>(hq, hkv, keys, stages, blocks);
}
extern "C" int xft_talking_prefill_keys(int hq, int hkv, int D) {
  int keys, stages, blocks;
  return plan_prefill(hq, hkv, D, keys, stages, blocks) ? keys : 0;
}

// bf16: q [T, hq, D], gate and out [T, ld] (head h at columns h * D), caches [num_blocks, hkv, bs, D] with bs a power of two, at least 64;
// r1, r2 [hq], talk [hq, hq] fp32 (of bf16 values).  window 0: every earlier key.
extern "C" int xft_talking_prefill(const void* q, const void* gate, int ldg, void* out, int ldo, const void* kc, const void* vc,
                                   const int* block_table, int bt_stride, const int* cu_q, const int* kv_lens, int B, int max_q, int hq,
                                   int hkv, int D, int bs, int num_blocks, float scale, const float* r1, const float* r2, const float* talk,
                                   int window, float mult, int* status, cudaStream_t st) {
  if (B <= 0 || max_q <= 0) return 0;
  int keys, stages, blocks;
  int shift = 6;
  while (shift < 20 && (1 << shift) < bs) ++shift;
  if (!plan_prefill(hq, hkv, D, keys, stages, blocks) || bs != 1 << shift || window < 0 || ldg < hq * D || ldo < hq * D || ((ldg | ldo) & 1) ||
      B > 65535 || (long long)num_blocks * hkv * bs >= (1ll << 31)) return -1;
  if (((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc) & 15 || ((uintptr_t)gate | (uintptr_t)out) & 3) return -2;
  const int hb = hq > 16 ? 2 : 1;
  TalkPrefillParams p{(const bf16*)q, (const bf16*)gate, ldg, (bf16*)out, ldo, block_table, bt_stride, cu_q,
                      kv_lens, hq, hkv, hq / hkv, num_blocks, window > 0 ? min(window, 1 << 30) : 1 << 30, blocks * hq / hb, blocks, shift, stages,
                      scale * kTalkLog2e, mult, r1, r2, talk, status};
  if (D == 64) {
    if (hb == 1) return keys == 32 ? launch_prefill<64, 1, 32>(p, kc, vc, bs, B, max_q, st) : launch_prefill<64, 1, 16>(p, kc, vc, bs, B, max_q, st);
    return keys == 32 ? launch_prefill<64, 2, 32>(p, kc, vc, bs, B, max_q, st) : launch_prefill<64, 2, 16>(p, kc, vc, bs, B, max_q, st);
  }
  if (hb == 1) return keys == 32 ? launch_prefill<128, 1, 32>(p, kc, vc, bs, B, max_q, st) : launch_prefill<128, 1, 16>(p, kc, vc, bs, B, max_q, st);
  return keys == 32 ? launch_prefill<128, 2, 32>(p, kc, vc, bs, B, max_q, st) : launch_prefill<128, 2, 16>(p, kc, vc, bs, B, max_q, st);
}

template <int D, int GR>
static cudaError_t launch_values(const TalkDecodeParams& p, cudaStream_t st) {
  const size_t work = (size_t)p.hq * 64 + 64 * GR + p.group * p.hq + 2 * p.hq, end = (size_t)kTalkValues * 4 * GR;
  const size_t smem = (GR * D + (work > end ? work : end)) * sizeof(float);
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(talking_values_kernel<D, GR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.splits, p.hkv, p.B);
  cfg.blockDim = dim3(kTalkValues);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[2];
  int na = 0;
  if (p.splits > 1) {
    at[na].id = cudaLaunchAttributeClusterDimension;
    at[na].val.clusterDim.x = p.splits; at[na].val.clusterDim.y = 1; at[na].val.clusterDim.z = 1;
    ++na;
  }
  if (g_xft_pdl) {
    at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = at;
  cfg.numAttrs = na;
  return cudaLaunchKernelEx(&cfg, talking_values_kernel<D, GR>, p);
}
template <int D>
static int launch_decode(const TalkDecodeParams& p, cudaStream_t st) {
  cudaError_t e = launch_pdl(talking_scores_kernel<D>, dim3(p.splits, p.hkv * ((p.group + 15) / 16), p.B), dim3(128), 0, st, p);
  if (e != cudaSuccess) return (int)e;
  e = p.group <= 1 ? launch_values<D, 1>(p, st) : p.group <= 2 ? launch_values<D, 2>(p, st) : p.group <= 4 ? launch_values<D, 4>(p, st)
      : p.group <= 8 ? launch_values<D, 8>(p, st) : launch_values<D, 16>(p, st);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// One token per sequence: q [B, hq, D] and the rest as above, heads of 64, 128 or 256, up to 16 per key/value head and 128 in all.  splits:
// key ranges, up to 8.  Scratch: scores [B * hq * span] with span a multiple of 64, at least 64 * (pages that a window can touch); part_ml
// [B * hq * splits * 2].
extern "C" int xft_talking_decode(const void* q, const void* gate, int ldg, void* out, int ldo, const void* kc, const void* vc,
                                  const int* block_table, int bt_stride, const int* kv_lens, int B, int hq, int hkv, int D, int bs,
                                  int num_blocks, float scale, const float* r1, const float* r2, const float* talk, int window, float mult,
                                  int splits, int span, float* scores, float* part_ml, int* status, cudaStream_t st) {
  if (B <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || hq % hkv || hq / hkv > 16 || hq > 128 || bs <= 0 || bs % 64 || window < 0 || splits < 1 || splits > 8 || (span & 63) || span <= 0)
    return -1;
  if (ldg < hq * D || ldo < hq * D || B > 65535 || hkv > 65535) return -2;
  if (((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)scores | (uintptr_t)part_ml) & 15) return -3;
  TalkDecodeParams p{(const bf16*)q, (const bf16*)gate, ldg, (bf16*)out, ldo, (const bf16*)kc, (const bf16*)vc, block_table, bt_stride, kv_lens,
                     B, hq, hkv, hq / hkv, bs, num_blocks, window > 0 ? min(window, 1 << 30) : 1 << 30, splits, span, scale * kTalkLog2e, mult,
                     r1, r2, talk, scores, part_ml, status};
  if (D == 64) return launch_decode<64>(p, st);
  if (D == 128) return launch_decode<128>(p, st);
  if (D == 256) return launch_decode<256>(p, st);
  return -4;
}
