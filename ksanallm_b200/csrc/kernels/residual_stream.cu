// Ops around a 32-bit residual stream, for decoders that keep the sum of their sublayers in fp32 and normalise before
// (and some after) every sublayer. Activations (GEMM operands and results) are bf16, or fp32 in the all-32-bit mode
// (template parameter T); parameters have the activations' type.
//
//   embed_pair        x = table[id] * scale (+ pair[hash(previous id, id)]), fp32, plus an optional copy in T
//   residual_norm     x += scale * norm(y) ; z = norm(x)  - one pass for "norm after the sublayer, layer scale, residual
//                     add, norm before the next sublayer"; every part is optional (a plain norm, a cast, a row gather)
//                     The addend may have a scalar factor, and the stream's norm may be taken per part of a row
//   glu_clamp         min(g, limit) * sigmoid(alpha * g) * (clamp(u, -limit, limit) + offset)
//   xielu             pos z^2 + lin z (z > 0), neg (exp(z) - 1 - z) + lin z (z <= 0)
//   qkv_rope_append   rotary embedding on the first rot dims of q and k, k and v into the paged cache; k and v may have
//                     different head sizes and live in separate panels
//   refit_rows_f32    rows of x overwritten with given embeddings
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>
#include <stdint.h>

namespace ksana {

// ------------------------------------------------------------------------------------------------ embedding
// One CTA per token. H is the padded row width (a multiple of 8; pad columns of the tables are zero). The pair row of
// (previous id a, id b) is (a * mul_prev + b * mul_cur) mod buckets, and row `buckets` for a sequence's first token
// (prev < 0). Ids outside the table are recorded in the error word and read as row 0.
template <typename T>
__global__ void embed_pair_kernel(const int* __restrict__ ids, const int* __restrict__ prev, const T* __restrict__ table,
                                  const T* __restrict__ pair, float* __restrict__ x, T* __restrict__ copy, int ldc, int H,
                                  int vocab, long long buckets, long long mul_prev, long long mul_cur, float scale, int* err) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) { if (threadIdx.x == 0) guard_report(err, kGuardGatherRow, id); id = 0; }
  const T* src = table + static_cast<size_t>(id) * H;
  const T* psrc = nullptr;
  if (pair) {
    long long a = prev[t];
    if (a >= vocab) { if (threadIdx.x == 0) guard_report(err, kGuardGatherRow, a); a = 0; }
    long long r = a < 0 ? buckets : (a * mul_prev + id * mul_cur) % buckets;
    if (r < 0) r += buckets;
    psrc = pair + static_cast<size_t>(r) * H;
  }
  for (int i = threadIdx.x * 8; i < H; i += blockDim.x * 8) {
    float f[8];
    load8(src + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= scale;
    if (psrc) {
      float g[8];
      load8(psrc + i, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += g[e];
    }
    store8(x + static_cast<size_t>(t) * H + i, f);
    if (copy) store8(copy + static_cast<size_t>(t) * ldc + i, f);
  }
}

// ------------------------------------------------------------------------------------------------ norms
// Running mean and sum of squared deviations of a set of values; two sets merge exactly (pairwise update), so a row's
// statistics need one pass over the registers and one block reduction instead of two.
struct Moments { float n, mean, m2; };
__device__ __forceinline__ Moments merge(const Moments& a, const Moments& b) {
  Moments r;
  r.n = a.n + b.n;
  if (r.n <= 0.f) return Moments{0.f, 0.f, 0.f};
  const float inv = 1.f / r.n, d = b.mean - a.mean;
  r.mean = (a.n * a.mean + b.n * b.mean) * inv;
  r.m2 = a.m2 + b.m2 + d * d * (a.n * b.n * inv);
  return r;
}
__device__ __forceinline__ Moments warp_moments(Moments v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const Moments w{__shfl_xor_sync(0xffffffffu, v.n, o), __shfl_xor_sync(0xffffffffu, v.mean, o),
                    __shfl_xor_sync(0xffffffffu, v.m2, o)};
    v = merge(v, w);
  }
  return v;
}
// `red`: 32 entries of shared memory, different for the two reductions of a row
__device__ __forceinline__ Moments block_moments(Moments v, Moments* red) {
  v = warp_moments(v);
  const int nw = blockDim.x >> 5;
  if (nw == 1) return v;
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  v = l < nw ? red[l] : Moments{0.f, 0.f, 0.f};
  return warp_moments(v);
}

template <typename T>
struct ResNormParams {
  const float* x; int ldx;              // residual stream in
  const int* rows; int in_rows;         // optional: output row m reads stream row rows[m]
  const T* y; int ldy;                  // sublayer result to add (null: none)
  const T* w1; const T* b1;             // norm of y (w1 null: y is added as it is)
  const T* ls;                          // per-column factor of the addend (null: 1)
  float* x_out;                         // updated stream (may alias x); null: not stored
  const T* w2; const T* b2;             // norm of the updated stream (w2 null: z is a plain copy)
  T* z; int ldz;                        // null: no second output
  int H;                                // real row width; buffers are padded to a multiple of 8, pads are kept zero
  float eps;
  int rms;                              // 1: root-mean-square norms (no mean, no bias needed)
  float alpha;                          // factor of the addend, all columns
  int groups;                           // > 1: the stream's norm takes its mean square per consecutive part of H / groups columns
  int* err;
};

// z = the row v scaled by the reciprocal root mean square of each of its `groups` parts of equal size, times w2. Squares are
// summed per unit (a vector of 8, or a single element where a part is not a multiple of 8) in dynamic shared memory, one
// warp per part. `part` holds H / unit sums, then one reciprocal per part.
template <typename T, int VPT>
__device__ __forceinline__ void grouped_norm(const ResNormParams<T>& p, int m, float (&v)[VPT][8], int nvec) {
  extern __shared__ float part[];
  const int size = p.H / p.groups, unit = size % 8 == 0 ? 8 : 1, per = size / unit;
  float* rstd = part + p.H / unit;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      if (unit == 8) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(v[j][e], v[j][e], s);
        part[i] = s;
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) if (i * 8 + e < p.H) part[i * 8 + e] = v[j][e] * v[j][e];
      }
    }
  }
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int g = threadIdx.x >> 5; g < p.groups; g += blockDim.x >> 5) {
    float s = 0.f;
    for (int k = lane; k < per; k += 32) s += part[g * per + k];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) rstd[g] = rsqrtf(s / static_cast<float>(size) + p.eps);
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      float wf[8], r0 = unit == 8 ? rstd[i / per] : 0.f;
      load8(p.w2 + i * 8, wf);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int c = i * 8 + e;
        if (unit != 8) r0 = c < p.H ? rstd[c / size] : 0.f;
        v[j][e] = c < p.H ? v[j][e] * r0 * wf[e] : 0.f;
      }
      store8(p.z + static_cast<size_t>(m) * p.ldz + i * 8, v[j]);
    }
  }
}

// One CTA per row, VPT vectors of 8 elements per thread.
template <typename T, int VPT>
__global__ void residual_norm_kernel(const ResNormParams<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ Moments red[2][32];
  const int m = blockIdx.x;
  int r = m;
  if (p.rows) {
    r = p.rows[m];
    if (r < 0 || r >= p.in_rows) { if (threadIdx.x == 0) guard_report(p.err, kGuardGatherRow, r); r = 0; }
  }
  const int nvec = (p.H + 7) >> 3;
  float v[VPT][8], y[VPT][8];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      load8(p.x + static_cast<size_t>(r) * p.ldx + i * 8, v[j]);
      if (p.y) load8(p.y + static_cast<size_t>(r) * p.ldy + i * 8, y[j]);
    }
  }
  // statistics of the valid elements of f: (n, mean, m2), or for RMS (n, 0, sum of squares)
  auto moments_of = [&](float (&f)[VPT][8], Moments* rd) {
    Moments t{0.f, 0.f, 0.f};
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) {
        const int k = min(8, p.H - i * 8);
        t.n += static_cast<float>(k);
#pragma unroll
        for (int e = 0; e < 8; ++e) s += e < k ? f[j][e] : 0.f;
      }
    }
    if (!p.rms && t.n > 0.f) t.mean = s / t.n;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) {
        const int k = min(8, p.H - i * 8);
#pragma unroll
        for (int e = 0; e < 8; ++e) { const float d = f[j][e] - t.mean; t.m2 += e < k ? d * d : 0.f; }
      }
    }
    return block_moments(t, rd);
  };
  auto affine = [&](float (&f)[8], int i, float mean, float rstd, const T* w, const T* b) {
    float wf[8];
    load8(w + i * 8, wf);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = (f[e] - mean) * rstd * wf[e];
    if (b) {
      float bf[8];
      load8(b + i * 8, bf);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += bf[e];
    }
  };
  if (p.y) {
    float mean = 0.f, rstd = 1.f;
    if (p.w1) {
      const Moments s = moments_of(y, red[0]);
      mean = s.mean;
      rstd = rsqrtf(s.m2 / static_cast<float>(p.H) + p.eps);
    }
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) {
        if (p.w1) affine(y[j], i, mean, rstd, p.w1, p.b1);
        if (p.ls) {
          float lf[8];
          load8(p.ls + i * 8, lf);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[j][e] *= lf[e];
        }
        const int k = min(8, p.H - i * 8);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[j][e] = e < k ? fmaf(p.alpha, y[j][e], v[j][e]) : 0.f;
      }
    }
  }
  if (p.x_out) {
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) store8(p.x_out + static_cast<size_t>(m) * p.ldx + i * 8, v[j]);
    }
  }
  if (!p.z) return;
  if (p.groups > 1) {                   // same for every thread of the launch
    grouped_norm<T, VPT>(p, m, v, nvec);
    return;
  }
  float mean = 0.f, rstd = 1.f;
  if (p.w2) {
    const Moments s = moments_of(v, red[1]);
    mean = s.mean;
    rstd = rsqrtf(s.m2 / static_cast<float>(p.H) + p.eps);
  }
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nvec) {
      if (p.w2) affine(v[j], i, mean, rstd, p.w2, p.b2);
      const int k = min(8, p.H - i * 8);
      if (k < 8) {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[j][e] = e < k ? v[j][e] : 0.f;
      }
      store8(p.z + static_cast<size_t>(m) * p.ldz + i * 8, v[j]);
    }
  }
}

template <typename T>
static int launch_residual_norm(const ResNormParams<T>& p, int M, cudaStream_t st) {
  const int nvec = (p.H + 7) >> 3;
  auto threads = [&](int vpt) { return ((nvec + vpt - 1) / vpt + 31) / 32 * 32; };
  size_t smem = 0;
  if (p.groups > 1) {
    const int size = p.H / p.groups;
    smem = (static_cast<size_t>(p.H) / (size % 8 == 0 ? 8 : 1) + p.groups) * sizeof(float);
    if (smem > 46 * 1024) return -10;
  }
  cudaError_t e;
  if (nvec <= 256) e = launch_pdl(residual_norm_kernel<T, 1>, dim3(M), dim3(threads(1)), smem, st, p);
  else if (nvec <= 1024) e = launch_pdl(residual_norm_kernel<T, 2>, dim3(M), dim3(threads(2)), smem, st, p);
  else if (nvec <= 4096) e = launch_pdl(residual_norm_kernel<T, 4>, dim3(M), dim3(threads(4)), smem, st, p);
  else return -10;
  return e == cudaSuccess ? 0 : -4;
}

// ------------------------------------------------------------------------------------------------ gated unit
template <typename T>
__global__ void glu_clamp_kernel(const T* __restrict__ in, T* __restrict__ out, int M, int I, int in_ld, float limit,
                                 float alpha, float offset) {
  pdl_trigger();
  pdl_wait();
  const int nvec = I >> 3;
  const long long total = static_cast<long long>(M) * nvec;
  for (long long idx = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; idx < total;
       idx += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int m = static_cast<int>(idx / nvec), i = static_cast<int>(idx - static_cast<long long>(m) * nvec);
    const T* row = in + static_cast<size_t>(m) * in_ld;
    float g[8], u[8];
    load8(row + i * 8, g);
    load8(row + I + i * 8, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float gv = fminf(g[e], limit), uv = fminf(fmaxf(u[e], -limit), limit);
      g[e] = gv / (1.f + __expf(-alpha * gv)) * (uv + offset);
    }
    store8(out + static_cast<size_t>(m) * I + i * 8, g);
  }
}

// ------------------------------------------------------------------------------------------------ elementwise units
// Piecewise unit of a plain feed-forward: pos z^2 + lin z above zero, neg (exp(z) - 1 - z) + lin z below. Near zero
// exp(z) - 1 - z is the Taylor series of the exponential from its quadratic term on (relative error below 1e-6 for
// |z| < 1/4); elsewhere the cancellation in the difference costs at most a few ulps.
__device__ __forceinline__ float xielu_f(float z, float pos, float neg, float lin) {
  const float zz = z * z;
  const float series = zz * (0.5f + z * (1.f / 6 + z * (1.f / 24 + z * (1.f / 120 + z * (1.f / 720)))));
  const float low = z > -0.25f ? series : __expf(z) - 1.f - z;
  return (z > 0.f ? pos * zz : neg * low) + lin * z;
}

// Rows of I elements, 8 per thread; grid.y walks the rows.
template <typename T>
__global__ void xielu_kernel(const T* __restrict__ in, int ldi, T* __restrict__ out, int ldo, int M, int I, float pos, float neg,
                             float lin) {
  pdl_trigger();
  pdl_wait();
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (i >= I) return;
  for (int m = blockIdx.y; m < M; m += gridDim.y) {
    float f[8];
    load8(in + static_cast<size_t>(m) * ldi + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = xielu_f(f[e], pos, neg, lin);
    store8(out + static_cast<size_t>(m) * ldo + i, f);
  }
}

// ------------------------------------------------------------------------------------------------ rotary + append
// One CTA per token. qkv row: [Hq*D | Hkv*D | Hkv*Dv]; cos_sin [max_pos][rot] = cos(rot/2) | sin(rot/2). K panel of a
// block: [Hkv][block_tokens][D] at kc + block * block_stride, V panel [Hkv][block_tokens][Dv] at vc + block * block_stride.
// q is rotated in place, k goes rotated to the cache only. slot < 0: no cache write (padding row). rot 0: no rotation.
// Items are 8-element vectors: whole-vector copies, and for the rotated part 8 pairs (j, j + rot/2) at a time when
// rot/2 is a multiple of 8, single pairs otherwise.
template <typename T>
__global__ void qkv_rope_append_kernel(T* __restrict__ qkv, const int* __restrict__ positions, const int* __restrict__ slots,
                                       const float* __restrict__ cos_sin, int max_pos, T* __restrict__ kc, T* __restrict__ vc,
                                       long long block_stride, int block_tokens, int num_blocks, int Hq, int Hkv, int D,
                                       int Dv, int rot, int* err) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  T* row = qkv + static_cast<size_t>(t) * ((Hq + Hkv) * D + Hkv * Dv);
  const int half = rot >> 1;
  int pos = rot ? positions[t] : 0;
  if (pos < 0 || (rot && pos >= max_pos)) { if (threadIdx.x == 0) guard_report(err, kGuardPosition, pos); pos = 0; }
  int slot = slots[t];
  if (slot >= 0 && slot / block_tokens >= num_blocks) { if (threadIdx.x == 0) guard_report(err, kGuardSlot, slot); slot = -1; }
  const int blk = slot < 0 ? 0 : slot / block_tokens, off = slot < 0 ? 0 : slot - blk * block_tokens;
  T* kdst = kc + static_cast<size_t>(blk) * block_stride + static_cast<size_t>(off) * D;
  T* vdst = vc + static_cast<size_t>(blk) * block_stride + static_cast<size_t>(off) * Dv;
  const size_t kh = static_cast<size_t>(block_tokens) * D, vh = static_cast<size_t>(block_tokens) * Dv;   // per-head panels
  const float* cs = cos_sin + static_cast<size_t>(pos) * rot;
  // one item list per token, so that all of a token's loads are in flight at once: rotated vectors of q and k, then
  // the rest of k, then v (the rest of q stays where it is)
  const bool vec = (half & 7) == 0;
  const int unit = vec ? 8 : 1;
  const int hv = half / unit, pv = (D - rot) / unit, dv8 = Dv >> 3;
  const int n_rot = (Hq + (slot >= 0 ? Hkv : 0)) * hv, n_rest = slot >= 0 ? Hkv * pv : 0, n_v = slot >= 0 ? Hkv * dv8 : 0;
  for (int i = threadIdx.x; i < n_rot + n_rest + n_v; i += blockDim.x) {
    if (i < n_rot) {
      const int h = i / hv, j = (i - h * hv) * unit;
      T* src = row + static_cast<size_t>(h) * D;
      T* dst = h >= Hq ? kdst + (h - Hq) * kh : src;
      if (vec) {
        float a[8], b[8], c[8], s[8], ra[8], rb[8];
        load8(src + j, a);
        load8(src + half + j, b);
        load8(cs + j, c);
        load8(cs + half + j, s);
#pragma unroll
        for (int e = 0; e < 8; ++e) { ra[e] = a[e] * c[e] - b[e] * s[e]; rb[e] = b[e] * c[e] + a[e] * s[e]; }
        store8(dst + j, ra);
        store8(dst + half + j, rb);
      } else {
        const float a = to_f(src[j]), b = to_f(src[half + j]), c = cs[j], s = cs[half + j];
        dst[j] = from_f<T>(a * c - b * s);
        dst[half + j] = from_f<T>(b * c + a * s);
      }
    } else if (i < n_rot + n_rest) {
      const int k = i - n_rot, h = k / pv, j = rot + (k - h * pv) * unit;
      const T* src = row + static_cast<size_t>(Hq + h) * D;
      if (vec) {
        float a[8];
        load8(src + j, a);
        store8(kdst + h * kh + j, a);
      } else {
        kdst[h * kh + j] = src[j];
      }
    } else {
      const int k = i - n_rot - n_rest, h = k / dv8, j = (k - h * dv8) * 8;
      float a[8];
      load8(row + static_cast<size_t>(Hq + Hkv) * D + h * Dv + j, a);
      store8(vdst + h * vh + j, a);
    }
  }
}

// x[pos[r], :] = emb[r, :] (fp32 rows of H real columns, stream rows ldx apart)
__global__ void refit_rows_f32_kernel(float* __restrict__ x, int ldx, const int* __restrict__ pos, const float* __restrict__ emb,
                                      int H, int rows, int* err) {
  const int r = pos[blockIdx.x];
  if (r < 0 || r >= rows) { if (threadIdx.x == 0) guard_report(err, kGuardGatherRow, r); return; }
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    x[static_cast<size_t>(r) * ldx + i] = emb[static_cast<size_t>(blockIdx.x) * H + i];
}

}  // namespace ksana

using namespace ksana;

// f32: activations and tables are fp32 instead of bf16 (all entry points below)
extern "C" int ksana_embed_pair(const int* ids, const int* prev, const void* table, const void* pair, float* x, void* copy,
                                int ldc, int T, int H, int vocab, long long buckets, long long mul_prev, long long mul_cur,
                                float scale, int f32, int* err, cudaStream_t st) {
  if (T <= 0) return 0;
  if (H % 8 || vocab <= 0 || (copy && ldc % 8) || (pair && (buckets <= 0 || !prev))) return -10;
  if (!aligned16(table) || !aligned16(pair) || !aligned16(x) || !aligned16(copy)) return -11;
  const int threads = H >= 2048 ? 256 : (H / 8 + 31) / 32 * 32;
  cudaError_t e;
  if (f32)
    e = launch_pdl(embed_pair_kernel<float>, dim3(T), dim3(threads), 0, st, ids, prev, (const float*)table, (const float*)pair, x,
                   (float*)copy, ldc, H, vocab, buckets, mul_prev, mul_cur, scale, err);
  else
    e = launch_pdl(embed_pair_kernel<bf16>, dim3(T), dim3(threads), 0, st, ids, prev, (const bf16*)table, (const bf16*)pair, x,
                   (bf16*)copy, ldc, H, vocab, buckets, mul_prev, mul_cur, scale, err);
  return e == cudaSuccess ? 0 : -4;
}

extern "C" int ksana_residual_norm(const float* x, int ldx, const int* rows, int in_rows, const void* y, int ldy,
                                   const void* w1, const void* b1, const void* ls, float* x_out, const void* w2,
                                   const void* b2, void* z, int ldz, int M, int H, float eps, int rms, int f32,
                                   float alpha, int groups, int* err, cudaStream_t st) {
  if (M <= 0) return 0;
  const int hp = (H + 7) / 8 * 8;
  if (H <= 0 || ldx % 8 || ldx < hp || (y && (ldy % 8 || ldy < hp)) || (z && (ldz % 8 || ldz < hp))) return -10;
  for (const void* q : {(const void*)x, y, w1, b1, ls, (const void*)x_out, w2, b2, (const void*)z})
    if (!aligned16(q)) return -11;
  if (rows && x_out == x) return -12;
  if (groups > 1 && (!rms || H % groups || w1 || b2 || !w2)) return -13;
  if (f32) {
    typedef float T;
    const ResNormParams<T> p{x, ldx, rows, in_rows, (const T*)y, ldy, (const T*)w1, (const T*)b1, (const T*)ls, x_out,
                             (const T*)w2, (const T*)b2, (T*)z, ldz, H, eps, rms, alpha, groups, err};
    return launch_residual_norm(p, M, st);
  }
  typedef bf16 T;
  const ResNormParams<T> p{x, ldx, rows, in_rows, (const T*)y, ldy, (const T*)w1, (const T*)b1, (const T*)ls, x_out,
                           (const T*)w2, (const T*)b2, (T*)z, ldz, H, eps, rms, alpha, groups, err};
  return launch_residual_norm(p, M, st);
}

// in [M, in_ld]: gate columns [0, I), up columns [I, 2I); out [M, I]. I a multiple of 8.
extern "C" int ksana_glu_clamp(const void* in, void* out, int M, int I, int in_ld, float limit, float alpha, float offset,
                               int f32, cudaStream_t st) {
  if (M <= 0) return 0;
  if (I % 8 || in_ld % 8 || in_ld < 2 * I || !aligned16(in) || !aligned16(out)) return -10;
  const long long total = static_cast<long long>(M) * (I >> 3);
  long long g = (total + 255) / 256;
  if (g > 148 * 8) g = 148 * 8;
  cudaError_t e;
  if (f32)
    e = launch_pdl(glu_clamp_kernel<float>, dim3((unsigned)g), dim3(256), 0, st, (const float*)in, (float*)out, M, I, in_ld, limit,
                   alpha, offset);
  else
    e = launch_pdl(glu_clamp_kernel<bf16>, dim3((unsigned)g), dim3(256), 0, st, (const bf16*)in, (bf16*)out, M, I, in_ld, limit,
                   alpha, offset);
  return e == cudaSuccess ? 0 : -4;
}

// in [M, I] -> out [M, I], I a multiple of 8
extern "C" int ksana_xielu(const void* in, int ldi, void* out, int ldo, int M, int I, float pos, float neg, float lin, int f32,
                           cudaStream_t st) {
  if (M <= 0) return 0;
  if (I <= 0 || I % 8 || ldi % 8 || ldi < I || ldo % 8 || ldo < I || !aligned16(in) || !aligned16(out)) return -10;
  const int vec = I / 8, threads = vec >= 256 ? 256 : (vec + 31) / 32 * 32, gx = (vec + threads - 1) / threads;
  const int most = 148 * 2048 / threads * 4;                 // about four waves of resident CTAs
  const int gy = min(M, max(1, min(65535, most / gx)));
  const dim3 grid(gx, gy), block(threads);
  const cudaError_t e =
      f32 ? launch_pdl(xielu_kernel<float>, grid, block, 0, st, (const float*)in, ldi, (float*)out, ldo, M, I, pos, neg, lin)
          : launch_pdl(xielu_kernel<bf16>, grid, block, 0, st, (const bf16*)in, ldi, (bf16*)out, ldo, M, I, pos, neg, lin);
  return e == cudaSuccess ? 0 : -4;
}

extern "C" int ksana_qkv_rope_append(void* qkv, const int* positions, const int* slots, const float* cos_sin, int max_pos,
                                     void* kc, void* vc, long long block_stride, int block_tokens, int num_blocks, int T,
                                     int Hq, int Hkv, int D, int Dv, int rot, int f32, int* err, cudaStream_t st) {
  if (T <= 0) return 0;
  if (D % 8 || Dv % 8 || rot < 0 || rot > D || (rot & 1) || block_tokens <= 0 || block_stride % 8 || (rot && !cos_sin)) return -10;
  if (!aligned16(qkv) || !aligned16(kc) || !aligned16(vc) || !aligned16(cos_sin)) return -11;
  const int items = (rot % 16 ? (Hq + Hkv) * (rot / 2) : (Hq + Hkv) * (rot / 16) + Hkv * ((D - rot) / 8)) + Hkv * (Dv / 8);
  const int threads = items >= 512 ? 512 : (items + 31) / 32 * 32;
  cudaError_t e;
  if (f32)
    e = launch_pdl(qkv_rope_append_kernel<float>, dim3(T), dim3(threads), 0, st, (float*)qkv, positions, slots, cos_sin, max_pos,
                   (float*)kc, (float*)vc, block_stride, block_tokens, num_blocks, Hq, Hkv, D, Dv, rot, err);
  else
    e = launch_pdl(qkv_rope_append_kernel<bf16>, dim3(T), dim3(threads), 0, st, (bf16*)qkv, positions, slots, cos_sin, max_pos,
                   (bf16*)kc, (bf16*)vc, block_stride, block_tokens, num_blocks, Hq, Hkv, D, Dv, rot, err);
  return e == cudaSuccess ? 0 : -4;
}

extern "C" int ksana_refit_rows_f32(float* x, int ldx, const int* pos, const float* emb, int R, int H, int rows, int* err,
                                    cudaStream_t st) {
  if (R <= 0) return 0;
  refit_rows_f32_kernel<<<R, 256, 0, st>>>(x, ldx, pos, emb, H, rows, err);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
