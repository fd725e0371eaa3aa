// The residual stream kept in 32 bits, with everything that happens to it between two products in one launch:
//
//   x <- carry * x + mult * post(y) + add   y = output of the sublayer just finished; post = a norm with its own gain, or
//                                   nothing; add = a vector, the same for every row, or nothing
//   or x <- post(carry * x + mult * y + add), the norm of the sum being the stream
//   h <- next(x)                    input of the sublayer that follows, for the next product (bf16 or fp32); next = a norm,
//                                   or x as it is
//
// and, for the first layer, x <- table[id] * scale instead of the first line.  The norm is LayerNorm (mean and variance) or
// RMSNorm, with a gain and an optional bias.  Either half can be left out; `rows` restricts the work to some rows of
// the batch (the ones whose logits are wanted).  One CTA per row: the row stays in registers between the reductions,
// so x and y are read once and x and h written once.  Row buffers may be wider than H (`HP`, a multiple of 8, so that
// the products that follow see 16-byte rows); the columns from H on are written as zeros.
//
// The reference adds the residual inside its GEMMs and normalises in a kernel of its own (src/layers/decoder_block.h:122-134,
// src/kernels/layernorm_kernels.cpp:27-160), with a residual in the activation type.
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

struct ResidualNormParams {
  const int* ids; const bf16* table; int vocab; long long ldt;      // embedding form (ids != null)
  const float* x; int ldx;                                          // residual stream in (unless ids)
  float* x_out; int ldxo;                                           // residual stream out, or null
  const void* y; int ldy, y_f32;                                    // sublayer output, or null
  const float* post_w; const float* post_b;                         // gain / bias of its norm (post_w null: no norm)
  const float* next_w; const float* next_b;                         // gain / bias of the following norm
  void* h; int ldh, h_f32;                                          // normalised output, or null
  const int* rows;                                                  // row r of the outputs comes from rows[r], or null
  int n_in;                                                         // rows of x and y
  int H, HP, rms;
  float eps, embed_scale, mult;
  const float* add;                                                 // [H] or null
  int raw;                                                          // h is x itself
  float carry; int post_sum;                                        // factor of x; the norm `post` is that of the sum
  int* status;
};

template <int NT>
__device__ __forceinline__ float row_sum(float v, float* sh) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if (NT == 32) return v;
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) r += sh[i];
  return r;
}

// eight consecutive values of a row, columns past H read as zero
__device__ __forceinline__ void load8(const float* p, int left, float (&v)[8]) {
  if (left >= 8) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = j < left ? p[j] : 0.f;
  }
}
__device__ __forceinline__ void load8(const bf16* p, int left, float (&v)[8]) {
  if (left >= 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(b[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = j < left ? __bfloat162float(p[j]) : 0.f;
  }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8]) {
  uint4 u;
  __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int j = 0; j < 4; ++j) b[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
  *reinterpret_cast<uint4*>(p) = u;
}

// in-place norm of the CTA's row; columns from H on become zero
template <int NT, int CH, bool PRE>
__device__ __forceinline__ void norm_row(float (&v)[CH][8], const ResidualNormParams& p, const float* w, const float* b,
                                         const float (&pre)[PRE ? CH : 1][8], float* sh) {
  float mean = 0.f;
  if (!p.rms) {
    float s = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[c][j];
    mean = row_sum<NT>(s, sh) / (float)p.H;
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int left = p.H - (threadIdx.x + c * NT) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      v[c][j] = j < left ? v[c][j] - mean : 0.f;
      ss += v[c][j] * v[c][j];
    }
  }
  const float inv = rsqrtf(row_sum<NT>(ss, sh + NT / 32) / (float)p.H + p.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (threadIdx.x + c * NT) * 8;
    if (i < p.H) {
      float g[8];
      if (!PRE) load8(w + i, p.H - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[c][j] *= inv * (PRE ? pre[PRE ? c : 0][j] : g[j]);
      if (b) {
        load8(b + i, p.H - i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[c][j] += g[j];
      }
    }
  }
}

// PRE: the gains, which are weights, are read before the kernel in front has finished (few rows: latency counts)
template <int NT, int CH, bool PRE>
__global__ void __launch_bounds__(NT) residual_norm_kernel(const ResidualNormParams p) {
  __shared__ float sh[4][NT / 32 > 0 ? NT / 32 : 1];
  grid_dep_launch();
  float g1[PRE ? CH : 1][8], g2[PRE ? CH : 1][8];
  if (PRE) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = (threadIdx.x + c * NT) * 8, left = p.H - i;
      if (p.post_w) load8(p.post_w + (left > 0 ? i : 0), left, g1[PRE ? c : 0]);
      if (p.next_w) load8(p.next_w + (left > 0 ? i : 0), left, g2[PRE ? c : 0]);
    }
  }
  grid_dep_wait();
  const int r = blockIdx.x;
  int src = r;
  if (p.rows) {
    src = p.rows[r];
    if (src < 0 || src >= p.n_in) { if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); src = 0; }
  }
  float x[CH][8], y[CH][8];
  int id = 0;
  if (p.ids) {
    id = p.ids[src];
    if (id < 0 || id >= p.vocab) { if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); id = 0; }
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (threadIdx.x + c * NT) * 8;
    const int left = p.H - i;                              // <= 0: nothing of the row here
    if (p.ids) {
      load8(p.table + (size_t)id * p.ldt + (left > 0 ? i : 0), left, x[c]);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] *= p.embed_scale;
    } else load8(p.x + (size_t)src * p.ldx + (left > 0 ? i : 0), left, x[c]);
    if (p.y) {
      if (p.y_f32) load8(reinterpret_cast<const float*>(p.y) + (size_t)src * p.ldy + (left > 0 ? i : 0), left, y[c]);
      else load8(reinterpret_cast<const bf16*>(p.y) + (size_t)src * p.ldy + (left > 0 ? i : 0), left, y[c]);
    }
  }
  if (p.carry != 1.f) {
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] *= p.carry;
  }
  if (p.y) {
    if (p.post_w && !p.post_sum) norm_row<NT, CH, PRE>(y, p, p.post_w, p.post_b, g1, sh[0]);
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] += p.mult * y[c][j];
  }
  if (p.add) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = (threadIdx.x + c * NT) * 8, left = p.H - i;
      load8(p.add + (left > 0 ? i : 0), left, y[c]);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] += y[c][j];
    }
  }
  if (p.post_sum) norm_row<NT, CH, PRE>(x, p, p.post_w, p.post_b, g1, sh[0]);
  if (p.x_out) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = (threadIdx.x + c * NT) * 8;
      if (i < p.HP) store8(p.x_out + (size_t)r * p.ldxo + i, x[c]);
    }
  }
  if (p.h) {
    if (!p.raw) norm_row<NT, CH, PRE>(x, p, p.next_w, p.next_b, g2, sh[2]);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int i = (threadIdx.x + c * NT) * 8;
      if (i < p.HP) {
        if (p.h_f32) store8(reinterpret_cast<float*>(p.h) + (size_t)r * p.ldh + i, x[c]);
        else store8(reinterpret_cast<bf16*>(p.h) + (size_t)r * p.ldh + i, x[c]);
      }
    }
  }
}

}  // namespace xft

using namespace xft;

// One launch over n_out rows (see the file comment).  H <= 32768; HP = H rounded up to 8, at most every row stride; row
// strides multiples of 8, pointers 16-byte aligned (gains, biases and the added vector too).  kind: 0 LayerNorm, 1 RMSNorm.
extern "C" int xft_residual_norm(const int* ids, const void* table, int vocab, long long ldt, const float* x, int ldx,
                                 float* x_out, int ldxo, const void* y, int ldy, int y_f32, const float* post_w,
                                 const float* post_b, const float* next_w, const float* next_b, void* h, int ldh, int h_f32,
                                 const int* rows, int n_in, int n_out, int H, int kind, float eps, float embed_scale,
                                 float mult, const float* add, int raw, float carry, int post_sum, int* status, cudaStream_t st) {
  if (n_out <= 0) return 0;
  const int HP = (H + 7) / 8 * 8;
  if (H <= 0 || H > 32768 || (!ids && !x) || (h && !next_w && !raw) || (post_sum && !post_w) || (!rows && n_out > n_in)) return -1;
  if ((ids && ((ldt & 7) || ldt < HP)) || (!ids && ((ldx & 7) || ldx < HP))) return -2;
  if ((x_out && ((ldxo & 7) || ldxo < HP)) || (y && ((ldy & 7) || ldy < HP)) || (h && ((ldh & 7) || ldh < HP))) return -2;
  if (((uintptr_t)table | (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)post_w | (uintptr_t)post_b |
       (uintptr_t)next_w | (uintptr_t)next_b | (uintptr_t)h | (uintptr_t)add) & 15) return -3;
  if (rows && x_out == x && x_out) return -4;              // gathered rows cannot be written back in place
  ResidualNormParams p{ids, (const bf16*)table, vocab, ldt, x, ldx, x_out, ldxo, y, ldy, y_f32, post_w, post_b, next_w,
                       next_b, h, ldh, h_f32, rows, n_in, H, HP, kind, eps, embed_scale, mult, add, raw, carry, post_sum, status};
  cudaError_t e;
#define XFT_RN(NT, CH, PRE) e = launch_pdl(residual_norm_kernel<NT, CH, PRE>, dim3(n_out), dim3(NT), 0, st, p)
  const bool few = n_out <= 296;                           // decode: a wide CTA per row, everything in one round of loads
  if (HP <= 256) XFT_RN(32, 1, true);
  else if (few && HP <= 1024) XFT_RN(128, 1, true);
  else if (few && HP <= 2048) XFT_RN(256, 1, true);
  else if (few && HP <= 4096) XFT_RN(512, 1, true);
  else if (few && HP <= 8192) XFT_RN(1024, 1, true);
  else if (HP <= 1024) XFT_RN(128, 1, false);
  else if (HP <= 2048) XFT_RN(128, 2, false);
  else if (HP <= 4096) XFT_RN(256, 2, false);
  else if (HP <= 8192) XFT_RN(512, 2, false);
  else if (HP <= 16384) XFT_RN(512, 4, false);
  else XFT_RN(1024, 4, false);
#undef XFT_RN
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
