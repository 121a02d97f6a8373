// Row ops of decoders that mix recurrent and attention layers over a 32-bit residual stream. Activations and parameters are
// bf16 or fp32 (template parameter T); rows are padded to multiples of 8 columns, pads are kept zero.
//
//   embed_normed   x = norm(table[id] * scale + position[p]), the fp32 stream's first rows
//   token_shift    m_t = h_t + (h_(t-1) - h_t) * mu per column; the row before a sequence's first new one comes from a ring of
//                  two rows in the sequence's state slot (position p in row p mod 2; zero before the sequence)
//   gated_norm     root-mean-square norm of equal parts of a row, with a silu gate in front or a sigmoid gate behind, and a factor
//   panel_append   columns of a projection to the paged cache
//   softcap        cap * tanh(z / cap)
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>

namespace ksana {

// in the activations' precision
template <typename T> __device__ __forceinline__ float sigmoid_as(float x) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-x)) : 1.f / (1.f + expf(-x));
}

// Sum over the CTA, in every thread. `red`: 32 floats of shared memory
__device__ __forceinline__ float cta_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int nw = blockDim.x >> 5;
  if (nw == 1) return v;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = (threadIdx.x & 31) < nw ? red[threadIdx.x & 31] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ------------------------------------------------------------------------------------------------ embedding
template <typename T, int VPT>
__global__ void embed_normed_kernel(const int* __restrict__ ids, const int* __restrict__ positions, const T* __restrict__ table,
                                    const T* __restrict__ pos_table, const T* __restrict__ w, float* __restrict__ x, int H, int real,
                                    int vocab, int max_pos, float scale, float eps, int* err) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x, nvec = H >> 3;
  int id = ids[t], pos = positions[t];
  if (id < 0 || id >= vocab) { if (threadIdx.x == 0) guard_report(err, kGuardGatherRow, id); id = 0; }
  if (pos < 0 || pos >= max_pos) { if (threadIdx.x == 0) guard_report(err, kGuardPosition, pos); pos = 0; }
  float f[VPT][8], s = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      float g[8];
      load8(table + static_cast<size_t>(id) * H + i * 8, f[j]);
      load8(pos_table + static_cast<size_t>(pos) * H + i * 8, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        f[j][e] = fmaf(f[j][e], scale, g[e]);
        s = fmaf(f[j][e], f[j][e], s);
      }
    }
  }
  const float rstd = 1.f / sqrtf(cta_sum(s, red) / static_cast<float>(real) + eps);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      float g[8];
      load8(w + i * 8, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[j][e] *= rstd * g[e];
      store8(x + static_cast<size_t>(t) * H + i * 8, f[j]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ token shift
constexpr int kShiftRows = 8;
// grid (channel tiles, row tiles, sequences); 8 columns per thread, the row before in registers. The CTA of a sequence's first
// rows also stores its last row to the ring (after it has read the ring).
template <typename T>
__global__ void token_shift_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ mu, T* __restrict__ out, long long ldo,
                                   T* ring, long long slot_stride, const int* __restrict__ cu_q, const int* __restrict__ kv_lens,
                                   const int* __restrict__ slots, int num_slots, int W, int* err) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, c = (blockIdx.x * blockDim.x + threadIdx.x) * 8, row0 = blockIdx.y * kShiftRows;
  const int q0 = cu_q[s], n = cu_q[s + 1] - q0, past = kv_lens[s] - n;
  if (row0 >= n || c >= W) return;
  int slot = slots[s];
  if (slot >= num_slots) { if (threadIdx.x == 0) guard_report(err, kGuardSlot, slot); slot = -1; }
  T* mine = ring + static_cast<long long>(slot < 0 ? 0 : slot) * slot_stride + c;
  const T* src = h + static_cast<long long>(q0) * ldh + c;
  float m[8], prev[8] = {};
  load8(mu + c, m);
  if (row0 > 0) load8(src + (row0 - 1) * ldh, prev);
  else if (past > 0 && slot >= 0) load8(mine + static_cast<size_t>((past - 1) & 1) * W, prev);
  const int end = min(row0 + kShiftRows, n);
  float f[8];
  for (int t = row0; t < end; ++t) {
    float o[8];
    load8(src + t * ldh, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) { o[e] = fmaf(prev[e] - f[e], m[e], f[e]); prev[e] = f[e]; }
    store8(out + static_cast<long long>(q0 + t) * ldo + c, o);
  }
  if (row0 == 0 && slot >= 0 && past >= 0) {
    if (end < n) load8(src + (n - 1) * ldh, f);
    store8(mine + static_cast<size_t>((past + n - 1) & 1) * W, f);
  }
}

// ------------------------------------------------------------------------------------------------ gated part norm
template <typename T>
struct GatedNormParams {
  const T* y; long long ldy;
  const T* z; long long ldz;                 // silu(z) multiplies y before the norm (null: none)
  const T* g; long long ldg;                 // sigmoid(g) multiplies the normed row (null: none)
  const T* w;                                // [cols]
  T* out; long long ldo;
  int cols;                                  // padded: heads of `pad` columns, of which `real` count
  int pad, real, parts;                      // parts of (cols / pad) * real / parts real columns each
  float eps, factor;
};

// One CTA per row, VPT vectors of 8 per thread. Squares are summed per unit (a vector, or a single column where parts or heads
// are not multiples of 8) in dynamic shared memory, then one warp per part.
template <typename T, int VPT>
__global__ void gated_norm_kernel(const GatedNormParams<T> p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sums[];
  const int m = blockIdx.x, nvec = p.cols >> 3, total = p.cols / p.pad * p.real, size = total / p.parts;
  const bool whole = p.real == p.pad && size % 8 == 0;
  const int units = whole ? nvec : total, per = whole ? size >> 3 : size;
  float* rstd = sums + units;
  float v[VPT][8];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      load8(p.y + static_cast<long long>(m) * p.ldy + i * 8, v[j]);
      if (p.z) {
        float f[8];
        load8(p.z + static_cast<long long>(m) * p.ldz + i * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[j][e] *= f[e] * sigmoid_as<T>(f[e]);
      }
      if (whole) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(v[j][e], v[j][e], s);
        sums[i] = s;
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int c = i * 8 + e, k = c % p.pad;
          if (k < p.real) sums[c / p.pad * p.real + k] = v[j][e] * v[j][e];
        }
      }
    }
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  for (int q = threadIdx.x >> 5; q < p.parts; q += warps) {
    float s = 0.f;
    for (int k = lane; k < per; k += 32) s += sums[q * per + k];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) rstd[q] = 1.f / sqrtf(s / static_cast<float>(size) + p.eps) * p.factor;
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      float w[8];
      load8(p.w + i * 8, w);
      if (whole) {
        const float r = rstd[i / per];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[j][e] *= r * w[e];
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int c = i * 8 + e, k = c % p.pad;
          v[j][e] = k < p.real ? v[j][e] * w[e] * rstd[(c / p.pad * p.real + k) / size] : 0.f;
        }
      }
      if (p.g) {
        float f[8];
        load8(p.g + static_cast<long long>(m) * p.ldg + i * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[j][e] *= sigmoid_as<T>(f[e]);
      }
      store8(p.out + static_cast<long long>(m) * p.ldo + i * 8, v[j]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ append, soft cap
// Panel of a block: [heads][block_tokens][D]. slot < 0: a padding row.
template <typename T>
__global__ void panel_append_kernel(const T* __restrict__ k, long long ldk, const int* __restrict__ slots, T* __restrict__ cache,
                                    long long block_stride, int block_tokens, int num_blocks, int heads, int D, int T_, int* err) {
  pdl_trigger();
  pdl_wait();
  const int nv = heads * (D >> 3);
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < static_cast<long long>(T_) * nv;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int t = static_cast<int>(i / nv), c = static_cast<int>(i % nv) * 8, slot = slots[t];
    if (slot < 0) continue;
    const int blk = slot / block_tokens;
    if (blk >= num_blocks) { guard_report(err, kGuardSlot, slot); continue; }
    float f[8];
    load8(k + static_cast<long long>(t) * ldk + c, f);
    store8(cache + static_cast<long long>(blk) * block_stride +
               (static_cast<long long>(c / D) * block_tokens + slot % block_tokens) * D + c % D, f);
  }
}

__global__ void softcap_kernel(float* __restrict__ z, long long ld, int M, int N, float cap) {
  pdl_trigger();
  pdl_wait();
  for (int m = blockIdx.y; m < M; m += gridDim.y)
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < N; i += gridDim.x * blockDim.x) {
      float* at = z + m * ld + i;
      *at = cap * tanhf(*at / cap);
    }
}

template <typename T>
static int run_embed(const int* ids, const int* positions, const void* table, const void* pos_table, const void* w, float* x, int T_, int H,
                     int real, int vocab, int max_pos, float scale, float eps, int* err, cudaStream_t st) {
  const int nvec = H / 8;
  auto go = [&](auto* kernel, int vpt) {
    const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
    return launch_pdl(kernel, dim3(T_), dim3(threads), 0, st, ids, positions, static_cast<const T*>(table), static_cast<const T*>(pos_table),
                      static_cast<const T*>(w), x, H, real, vocab, max_pos, scale, eps, err) == cudaSuccess ? 0 : -4;
  };
  if (nvec <= 256) return go(embed_normed_kernel<T, 1>, 1);
  if (nvec <= 1024) return go(embed_normed_kernel<T, 2>, 2);
  return nvec <= 4096 ? go(embed_normed_kernel<T, 4>, 4) : -10;
}

template <typename T>
static int run_gated_norm(const GatedNormParams<T>& p, int M, cudaStream_t st) {
  const int nvec = p.cols / 8, total = p.cols / p.pad * p.real, size = total / p.parts;
  const size_t smem = ((p.real == p.pad && size % 8 == 0 ? nvec : total) + p.parts) * sizeof(float);
  if (smem > 46 * 1024) return -10;
  auto go = [&](auto* kernel, int vpt) {
    const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
    return launch_pdl(kernel, dim3(M), dim3(threads), smem, st, p) == cudaSuccess ? 0 : -4;
  };
  if (nvec <= 256) return go(gated_norm_kernel<T, 1>, 1);
  if (nvec <= 1024) return go(gated_norm_kernel<T, 2>, 2);
  return nvec <= 4096 ? go(gated_norm_kernel<T, 4>, 4) : -10;
}

}  // namespace ksana

using namespace ksana;

extern "C" int ksana_embed_normed(const int* ids, const int* positions, const void* table, const void* pos_table, const void* w, float* x,
                                  int T_, int H, int real, int vocab, int max_pos, float scale, float eps, int f32, int* err,
                                  cudaStream_t st) {
  if (T_ <= 0) return 0;
  if (H <= 0 || H % 8 || real <= 0 || real > H) return -10;
  return f32 ? run_embed<float>(ids, positions, table, pos_table, w, x, T_, H, real, vocab, max_pos, scale, eps, err, st)
             : run_embed<bf16>(ids, positions, table, pos_table, w, x, T_, H, real, vocab, max_pos, scale, eps, err, st);
}

// ring: [slots] of [2][W], slot_stride elements apart; every sequence of the step in one launch
extern "C" int ksana_token_shift(const void* h, long long ldh, const void* mu, void* out, long long ldo, void* ring, long long slot_stride,
                                 const int* cu_q, const int* kv_lens, const int* slots, int num_slots, int B, int max_q, int W, int f32,
                                 int* err, cudaStream_t st) {
  if (B <= 0 || max_q <= 0) return 0;
  if (W <= 0 || W % 8 || ldh % 8 || ldo % 8 || slot_stride % (f32 ? 4 : 8) || B > 65535 || !aligned16(h) || !aligned16(out) ||
      !aligned16(ring))
    return -10;
  const int vec = W / 8, threads = vec < 256 ? (vec + 31) / 32 * 32 : 256;
  const dim3 grid((vec + threads - 1) / threads, (max_q + kShiftRows - 1) / kShiftRows, B);
  const cudaError_t e = f32 ? launch_pdl(token_shift_kernel<float>, grid, dim3(threads), 0, st, static_cast<const float*>(h), ldh,
                                         static_cast<const float*>(mu), static_cast<float*>(out), ldo, static_cast<float*>(ring),
                                         slot_stride, cu_q, kv_lens, slots, num_slots, W, err)
                            : launch_pdl(token_shift_kernel<bf16>, grid, dim3(threads), 0, st, static_cast<const bf16*>(h), ldh,
                                         static_cast<const bf16*>(mu), static_cast<bf16*>(out), ldo, static_cast<bf16*>(ring), slot_stride,
                                         cu_q, kv_lens, slots, num_slots, W, err);
  return e == cudaSuccess ? 0 : -4;
}

extern "C" int ksana_gated_norm(const void* y, long long ldy, const void* z, long long ldz, const void* g, long long ldg, const void* w,
                                void* out, long long ldo, int M, int cols, int pad, int real, int parts, float eps, float factor, int f32,
                                cudaStream_t st) {
  if (M <= 0) return 0;
  if (cols <= 0 || cols % 8 || pad <= 0 || pad % 8 || cols % pad || real <= 0 || real > pad || parts <= 0 || (cols / pad * real) % parts ||
      ldy % 8 || ldz % 8 || ldg % 8 || ldo % 8 || !aligned16(y) || !aligned16(z) || !aligned16(g) || !aligned16(out))
    return -10;
  auto run = [&](auto tag) {
    typedef decltype(tag) T;
    const GatedNormParams<T> p{static_cast<const T*>(y), ldy, static_cast<const T*>(z), ldz, static_cast<const T*>(g), ldg,
                               static_cast<const T*>(w), static_cast<T*>(out), ldo, cols, pad, real, parts, eps, factor};
    return run_gated_norm<T>(p, M, st);
  };
  return f32 ? run(0.f) : run(bf16());
}

extern "C" int ksana_panel_append(const void* k, long long ldk, const int* slots, void* cache, long long block_stride, int block_tokens,
                                  int num_blocks, int heads, int D, int T_, int f32, int* err, cudaStream_t st) {
  if (T_ <= 0) return 0;
  if (heads <= 0 || D <= 0 || D % 8 || ldk % 8 || block_stride % 8 || block_tokens <= 0 || !aligned16(k) || !aligned16(cache)) return -10;
  const long long n = static_cast<long long>(T_) * heads * (D / 8);
  const dim3 grid(static_cast<unsigned>(n + 255 < 256LL * 4096 ? (n + 255) / 256 : 4096));
  const cudaError_t e = f32 ? launch_pdl(panel_append_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(k), ldk, slots,
                                         static_cast<float*>(cache), block_stride, block_tokens, num_blocks, heads, D, T_, err)
                            : launch_pdl(panel_append_kernel<bf16>, grid, dim3(256), 0, st, static_cast<const bf16*>(k), ldk, slots,
                                         static_cast<bf16*>(cache), block_stride, block_tokens, num_blocks, heads, D, T_, err);
  return e == cudaSuccess ? 0 : -4;
}

extern "C" int ksana_softcap(float* z, long long ld, int M, int N, float cap, cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (!(cap > 0.f)) return -10;
  const int gx = (N + 1023) / 1024;
  return launch_pdl(softcap_kernel, dim3(gx, M < 65535 ? M : 65535), dim3(256), 0, st, z, ld, M, N, cap) == cudaSuccess ? 0 : -4;
}
