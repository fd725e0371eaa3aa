// Latent attention: what sits between a layer's packed projection and its attention, in one launch.
//
// A packed row is [q: heads x (dim + rot) | latent: rank | shared rotated key: rot | gate ...].  The kernel rotates the
// rotated part of every query head in place (pairs 2i, 2i + 1; the first `rot_dims` of its `rot` columns, the rest pass),
// and, for a layer with a cache of its own, writes [RMS norm of the latent * gain | rotated key part] to the token's cache
// row.  Columns of `rank` beyond `rank_real` are padding: zeros that do not count in the mean.
//
//   xft_latent_prep     bf16 or fp32 rows
//   xft_latent_gather   the cache rows of a span of positions per sequence, next to each other (bf16)
#include "ptx.cuh"

namespace xft {

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float lat_f32(T v);
template <> __device__ __forceinline__ float lat_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float lat_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T lat_from(float v);
template <> __device__ __forceinline__ float lat_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 lat_from<bf16>(float v) { return __float2bfloat16(v); }

struct LatentPrepParams {
  void* x; int ldx;
  int heads, dim, rot, rot_dims, rank, rank_real, own_kv;
  const int* positions; const float* table; int max_pos;
  const float* norm_w; float eps;
  void* cache; long long nslots; const int* slots;
  int* status;
};

// one CTA per token
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float sh[8];
  const int tid = threadIdx.x, t = blockIdx.x;
  grid_dep_launch();
  grid_dep_wait();
  T* row = reinterpret_cast<T*>(p.x) + (size_t)t * p.ldx;
  int pos = p.positions[t];
  if (p.table && (pos < 0 || pos >= p.max_pos)) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); pos = 0; }
  const int half = p.table ? p.rot_dims >> 1 : 0;
  const float* cs = p.table ? p.table + (size_t)pos * p.rot_dims : nullptr;
  const int hd = p.dim + p.rot;
  for (int i = tid; i < p.heads * half; i += 256) {
    const int h = i / half, j = i - h * half;
    T* q = row + (size_t)h * hd + p.dim + 2 * j;
    const float u = lat_f32<T>(q[0]), v = lat_f32<T>(q[1]), c = cs[j], s = cs[half + j];
    q[0] = lat_from<T>(u * c - v * s);
    q[1] = lat_from<T>(v * c + u * s);
  }
  if (!p.own_kv) return;
  const T* c_in = row + (size_t)p.heads * hd;
  float ss = 0.f;
  for (int i = tid; i < p.rank; i += 256) { const float v = lat_f32<T>(c_in[i]); ss += v * v; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) sh[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += sh[i];
  const float inv = 1.f / sqrtf(ss / (float)p.rank_real + p.eps);
  const long long slot = p.slots[t];
  if (slot < 0 || slot >= p.nslots) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); return; }
  T* dst = reinterpret_cast<T*>(p.cache) + (size_t)slot * (p.rank + p.rot);
  for (int i = tid; i < p.rank; i += 256) dst[i] = lat_from<T>(lat_f32<T>(c_in[i]) * inv * p.norm_w[i]);
  const T* k_in = c_in + p.rank;
  T* kd = dst + p.rank;
  for (int i = tid; i < p.rot; i += 256) {
    if (i < 2 * half) {
      if (i & 1) continue;
      const int j = i >> 1;
      const float u = lat_f32<T>(k_in[i]), v = lat_f32<T>(k_in[i + 1]), c = cs[j], s = cs[half + j];
      kd[i] = lat_from<T>(u * c - v * s);
      kd[i + 1] = lat_from<T>(v * c + u * s);
    } else {
      kd[i] = k_in[i];
    }
  }
}

// The same for bf16 rows whose parts are multiples of 8: 16 bytes (four pairs) per thread and step.  gridDim.y CTAs share a
// token when there are few of them; the last one then takes the cache row.
__device__ __forceinline__ uint4 rotate8(const uint4 u, const float* cs, int half, int j) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
  const float4 c = *reinterpret_cast<const float4*>(cs + j), s = *reinterpret_cast<const float4*>(cs + half + j);
  const float cc[4] = {c.x, c.y, c.z, c.w}, sn[4] = {s.x, s.y, s.z, s.w};
  uint4 r;
  __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 x = __bfloat1622float2(h[i]);
    o[i] = __floats2bfloat162_rn(x.x * cc[i] - x.y * sn[i], x.y * cc[i] + x.x * sn[i]);
  }
  return r;
}

__global__ void __launch_bounds__(256) latent_prep_vec_kernel(const LatentPrepParams p) {
  __shared__ float sh[8];
  const int tid = threadIdx.x, t = blockIdx.x;
  grid_dep_launch();
  grid_dep_wait();
  bf16* row = reinterpret_cast<bf16*>(p.x) + (size_t)t * p.ldx;
  int pos = p.positions[t];
  if (p.table && (pos < 0 || pos >= p.max_pos)) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); pos = 0; }
  const int half = p.table ? p.rot_dims >> 1 : 0;
  const float* cs = p.table ? p.table + (size_t)pos * p.rot_dims : nullptr;
  const int hd = p.dim + p.rot, per = half >> 2;                       // 16-byte pieces of a head's rotated dimensions
  const int q_ctas = gridDim.y > 1 && p.own_kv ? gridDim.y - 1 : gridDim.y;
  if ((int)blockIdx.y < q_ctas) {
#pragma unroll 4
    for (int i = blockIdx.y * 256 + tid; i < p.heads * per; i += q_ctas * 256) {
      const int h = i / per, j = i - h * per;
      uint4* q = reinterpret_cast<uint4*>(row + (size_t)h * hd + p.dim + 8 * j);
      *q = rotate8(*q, cs, half, 4 * j);
    }
  }
  if (!p.own_kv || blockIdx.y + 1 != gridDim.y) return;
  const long long slot = p.slots[t];
  const bf16* c_in = row + (size_t)p.heads * hd;
  uint4 u[2];                                                          // the first 4096 values stay in registers
  float ss = 0.f;
  for (int i = tid, n = 0; i < p.rank / 8; i += 256, ++n) {
    const uint4 v = reinterpret_cast<const uint4*>(c_in)[i];
    if (n == 0) u[0] = v;
    if (n == 1) u[1] = v;
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 x = __bfloat1622float2(h[e]); ss += x.x * x.x + x.y * x.y; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) sh[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += sh[i];
  const float inv = 1.f / sqrtf(ss / (float)p.rank_real + p.eps);
  if (slot < 0 || slot >= p.nslots) { if (tid == 0 && p.status) atomicCAS(p.status, 0, XFT_ERR_BOUNDS); return; }
  uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.cache) + (size_t)slot * (p.rank + p.rot));
  for (int i = tid, n = 0; i < p.rank / 8; i += 256, ++n) {
    const uint4 v = n == 0 ? u[0] : n == 1 ? u[1] : reinterpret_cast<const uint4*>(c_in)[i];
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
    const float4 a = reinterpret_cast<const float4*>(p.norm_w)[2 * i], b = reinterpret_cast<const float4*>(p.norm_w)[2 * i + 1];
    const float g[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    uint4 r;
    __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 x = __bfloat1622float2(h[e]);
      o[e] = __floats2bfloat162_rn(x.x * inv * g[2 * e], x.y * inv * g[2 * e + 1]);
    }
    dst[i] = r;
  }
  // the shared key part, by the threads that have the least to do above
  for (int i = 255 - tid; i < p.rot / 8; i += 256) {
    const uint4 v = reinterpret_cast<const uint4*>(c_in + p.rank)[i];
    dst[p.rank / 8 + i] = i < per ? rotate8(v, cs, half, 4 * i) : v;
  }
}

// One warp per row: row r of the output is position span_lo[b] + (r - span_row[b]) of the sequence b whose rows hold r.
// span_row [B] is increasing and starts at 0; lanes copy 16-byte pieces.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* __restrict__ cache, int width16, int bs, int num_blocks,
                                                            const int* __restrict__ block_table, int bt_stride,
                                                            const int* __restrict__ seq, const int* __restrict__ span_lo,
                                                            const int* __restrict__ span_row, int B, int rows,
                                                            uint4* __restrict__ out, int* status) {
  grid_dep_launch();
  grid_dep_wait();
  const int r = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  int lo = 0, hi = B - 1;
  while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (span_row[mid] <= r) lo = mid; else hi = mid - 1; }
  const int key = span_lo[lo] + r - span_row[lo];
  int blk = block_table[(size_t)seq[lo] * bt_stride + key / bs];
  if (blk < 0 || blk >= num_blocks) { if (lane == 0 && status) atomicCAS(status, 0, XFT_ERR_BOUNDS); blk = 0; }
  const uint4* src = cache + ((size_t)blk * bs + key % bs) * width16;
  for (int i = lane; i < width16; i += 32) out[(size_t)r * width16 + i] = src[i];
}

}  // namespace xft

using namespace xft;

// cache [num_blocks, bs, width] bf16, width a multiple of 8; out [rows, width].  seq [B]: a span's row of the block table.
extern "C" int xft_latent_gather(const void* cache, int width, int bs, int num_blocks, const int* block_table, int bt_stride,
                                 const int* seq, const int* span_lo, const int* span_row, int B, int rows, void* out, int* status,
                                 cudaStream_t st) {
  if (B <= 0 || rows <= 0) return 0;
  if (width <= 0 || (width & 7) || bs <= 0) return -1;
  cudaError_t e = launch_pdl(latent_gather_kernel, dim3((rows + 3) / 4), dim3(128), 0, st, (const uint4*)cache, width / 8, bs,
                             num_blocks, block_table, bt_stride, seq, span_lo, span_row, B, rows, (uint4*)out, status);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// x [T, ldx] packed rows; table [max_pos, rot_dims] = cos | sin, or null (no rotation); cache [nslots, rank + rot].
// f32: 1 = fp32 rows and cache, 0 = bf16.
extern "C" int xft_latent_prep(void* x, int ldx, int T, int heads, int dim, int rot, int rot_dims, int rank, int rank_real,
                               int own_kv, const int* positions, const float* table, int max_pos, const float* norm_w, float eps,
                               void* cache, long long nslots, const int* slots, int f32, int* status, cudaStream_t st) {
  if (T <= 0) return 0;
  if (heads <= 0 || dim < 0 || rot < 0 || rot_dims < 0 || (rot_dims & 1) || rot_dims > rot || rank_real <= 0 || rank_real > rank)
    return -1;
  if (ldx < heads * (dim + rot) + (own_kv ? rank + rot : 0) || (own_kv && (!norm_w || !cache || !slots))) return -2;
  LatentPrepParams p{x, ldx, heads, dim, rot, rot_dims, rank, rank_real, own_kv, positions, rot_dims > 0 ? table : nullptr, max_pos,
                     norm_w, eps, cache, nslots, slots, status};
  const bool vec = !f32 && !((ldx | dim | rot | rank) & 7) && !(p.table && (rot_dims & 7)) &&
                   !(((uintptr_t)x | (uintptr_t)cache | (uintptr_t)norm_w | (uintptr_t)table) & 15);
  if (vec) {
    const int pieces = p.table ? heads * (rot_dims / 8) : 0;
    const int parts = T > 128 ? 1 : max(1, min(16, (pieces + 255) / 256)) + (own_kv ? 1 : 0);
    cudaError_t e = launch_pdl(latent_prep_vec_kernel, dim3(T, parts), dim3(256), 0, st, p);
    return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
  }
  cudaError_t e = f32 ? launch_pdl(latent_prep_kernel<float>, dim3(T), dim3(256), 0, st, p)
                      : launch_pdl(latent_prep_kernel<bf16>, dim3(T), dim3(256), 0, st, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
