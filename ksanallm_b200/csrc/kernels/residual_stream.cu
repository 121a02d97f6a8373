// Ops around a 32-bit residual stream, for decoders that keep the sum of their sublayers in fp32 and normalise before
// (and some after) every sublayer. Activations (GEMM operands and results) are bf16, or fp32 in the all-32-bit mode
// (template parameter T); parameters have the activations' type.
//
//   embed_pair        x = table[id] * scale (+ pair[hash(previous id, id)]), fp32, plus an optional copy in T
//   residual_norm     x += scale * norm(y) ; z = norm(x)  - one pass for "norm after the sublayer, layer scale, residual
//                     add, norm before the next sublayer"; every part is optional (a plain norm, a cast, a row gather)
//                     The addend may have a scalar factor, and the stream's norm may be taken per part of a row. It may be
//                     the weighted sum of a token's expert outputs, gathered here; other stream rows (the embedding output,
//                     say) and a vector may be added as well
//   glu_clamp         min(g, limit) * sigmoid(alpha * g) * (clamp(u, -limit, limit) + offset)
//   xielu             pos z^2 + lin z (z > 0), neg (exp(z) - 1 - z) + lin z (z <= 0)
//   qkv_rope_append   rotary embedding on the first rot dims of q and k, k and v into the paged cache; k and v may have
//                     different head sizes and live in separate panels
//   qkv_norm_rope_append   the same with a norm over all of q and over all of k first, and rotated pairs (2i, 2i + 1)
//   latent_norms      the norms of a row's query latent (to a buffer) and key/value latent (to the paged cache)
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
// Sum of v over the CTA, in every thread. `red`: 32 floats of shared memory, other ones for every sum of a kernel
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int nw = blockDim.x >> 5;
  if (nw == 1) return v;
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  v = l < nw ? red[l] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
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
  const float* add; const T* vec;       // optional: stream rows (ldx apart) and a vector that are added too
  float z_scale;                        // factor of the normed row
  // addend = sum over k < top of w[row][k] * y[dst_row[row][k]] (+ w[row][top] * shared[row], or + shared[row] where a row has
  // no weight for it); rows of `ldw` weights. A negative dst_row is an expert that lives elsewhere
  const int* dst_row; const float* w; int ldw, top, cap;
  const T* shared; int lds;
  int* err;
};
constexpr int kMaxTop = 64;

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

// One CTA per row, VPT vectors of 8 elements per thread. EXPERTS: the addend is gathered from expert outputs.
template <typename T, int VPT, bool EXPERTS>
__global__ void residual_norm_kernel(const ResNormParams<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[4][32];
  __shared__ int src_row[EXPERTS ? kMaxTop : 1], src_n;
  __shared__ float src_w[EXPERTS ? kMaxTop : 1], shared_w;
  const int m = blockIdx.x;
  if (EXPERTS) {
    if (threadIdx.x < 32) {             // the rows that are here, in order, so that the loop over them has no branch
      int n = 0;
      for (int k0 = 0; k0 < p.top; k0 += 32) {
        const int k = k0 + threadIdx.x;
        int d = k < p.top ? p.dst_row[static_cast<size_t>(m) * p.top + k] : -1;
        if (d >= p.cap) { guard_report(p.err, kGuardDstRow, d); d = -1; }
        const unsigned here = __ballot_sync(0xffffffffu, d >= 0);
        if (d >= 0) {
          const int at = n + __popc(here & ((1u << threadIdx.x) - 1u));
          src_row[at] = d;
          src_w[at] = p.w[static_cast<size_t>(m) * p.ldw + k];
        }
        n += __popc(here);
      }
      if (threadIdx.x == 0) {
        src_n = n;
        if (p.shared) shared_w = p.ldw > p.top ? p.w[static_cast<size_t>(m) * p.ldw + p.top] : 1.f;
      }
    }
    __syncthreads();
  }
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
      if (EXPERTS) {
#pragma unroll
        for (int e = 0; e < 8; ++e) y[j][e] = 0.f;
        if (p.shared) {
          load8(p.shared + static_cast<size_t>(r) * p.lds + i * 8, y[j]);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[j][e] *= shared_w;
        }
        const int n = src_n;
#pragma unroll 4
        for (int k = 0; k < n; ++k) {
          float f[8];
          load8(p.y + static_cast<size_t>(src_row[k]) * p.ldy + i * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[j][e] = fmaf(src_w[k], f[e], y[j][e]);
        }
      } else if (p.y) {
        load8(p.y + static_cast<size_t>(r) * p.ldy + i * 8, y[j]);
      }
    }
  }
  // mean of the valid elements of f (RMS: 0) and reciprocal root of their mean squared distance from it; two sums, the
  // second over the distances, so nothing cancels
  auto statistics = [&](float (&f)[VPT][8], float (&rd)[4][32], int first, float& mean, float& rstd) {
    mean = 0.f;
    if (!p.rms) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < nvec) {
          const int k = min(8, p.H - i * 8);
#pragma unroll
          for (int e = 0; e < 8; ++e) s += e < k ? f[j][e] : 0.f;
        }
      }
      mean = block_sum(s, rd[first]) / static_cast<float>(p.H);
    }
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) {
        const int k = min(8, p.H - i * 8);
#pragma unroll
        for (int e = 0; e < 8; ++e) { const float d = f[j][e] - mean; s += e < k ? d * d : 0.f; }
      }
    }
    rstd = rsqrtf(block_sum(s, rd[first + 1]) / static_cast<float>(p.H) + p.eps);
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
    if (p.w1) statistics(y, red, 0, mean, rstd);
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
  if (p.add || p.vec) {                 // pad columns of both are zero
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < nvec) {
        float f[8];
        if (p.add) {
          load8(p.add + static_cast<size_t>(r) * p.ldx + i * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) v[j][e] += f[e];
        }
        if (p.vec) {
          load8(p.vec + i * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) v[j][e] += f[e];
        }
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
  if (p.w2) statistics(v, red, 2, mean, rstd);
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
#pragma unroll
      for (int e = 0; e < 8; ++e) v[j][e] *= p.z_scale;
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
  auto launch = [&](auto* plain, auto* experts, int vpt) {
    return launch_pdl(p.dst_row ? experts : plain, dim3(M), dim3(threads(vpt)), smem, st, p);
  };
  if (nvec <= 256) e = launch(residual_norm_kernel<T, 1, false>, residual_norm_kernel<T, 1, true>, 1);
  else if (nvec <= 1024) e = launch(residual_norm_kernel<T, 2, false>, residual_norm_kernel<T, 2, true>, 2);
  else if (nvec <= 4096) e = launch(residual_norm_kernel<T, 4, false>, residual_norm_kernel<T, 4, true>, 4);
  else return -10;
  return e == cudaSuccess ? 0 : -4;
}

// ------------------------------------------------------------------------------------------------ gated unit
template <typename T>
__global__ void glu_clamp_kernel(const T* __restrict__ in, T* __restrict__ out, int M, int I, int in_ld, float limit,
                                 float alpha, float offset, const int* __restrict__ tile_rows) {
  pdl_trigger();
  pdl_wait();
  const int nvec = I >> 3;
  const long long total = static_cast<long long>(M) * nvec;
  for (long long idx = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; idx < total;
       idx += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int m = static_cast<int>(idx / nvec), i = static_cast<int>(idx - static_cast<long long>(m) * nvec);
    if (tile_rows && (m & 127) >= tile_rows[m >> 7]) continue;       // of every 128 rows only so many hold anything
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

// q and k normed by the root mean square of all of q's (k's) columns at once, pairs (2i, 2i + 1) of the first `rot` dimensions
// of a head rotated, k and v into the paged cache (layout as above), q in place. One CTA per token, VPT vectors of q | k per
// thread in registers between the reduction and the rotation. Pad columns (head sizes that are not multiples of 8) are zero
// and have zero weights. sums: optional [T, 2] sums of squares of the whole q and k rows where this rank holds a part of them.
template <typename T>
struct NormRopeParams {
  T* qkv;
  const int* positions; const int* slots;
  const float* cos_sin; int max_pos;
  const T* qw; const T* kw; float eps;
  int nq, nk;                           // real columns of the whole q and k
  const float* sums;
  T* kc; T* vc; long long block_stride;
  int block_tokens, num_blocks, Hq, Hkv, D, Dv, rot;
  int* err;
};

template <typename T, int VPT>
__global__ void qkv_norm_rope_append_kernel(const NormRopeParams<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[2][32];
  const int t = blockIdx.x, D = p.D, Dv = p.Dv;
  T* row = p.qkv + static_cast<size_t>(t) * ((p.Hq + p.Hkv) * D + p.Hkv * Dv);
  int pos = p.rot ? p.positions[t] : 0;
  if (pos < 0 || (p.rot && pos >= p.max_pos)) { if (threadIdx.x == 0) guard_report(p.err, kGuardPosition, pos); pos = 0; }
  int slot = p.slots[t];
  if (slot >= 0 && slot / p.block_tokens >= p.num_blocks) { if (threadIdx.x == 0) guard_report(p.err, kGuardSlot, slot); slot = -1; }
  const int blk = slot < 0 ? 0 : slot / p.block_tokens, off = slot < 0 ? 0 : slot - blk * p.block_tokens;
  T* kdst = p.kc + static_cast<size_t>(blk) * p.block_stride + static_cast<size_t>(off) * D;
  T* vdst = p.vc + static_cast<size_t>(blk) * p.block_stride + static_cast<size_t>(off) * Dv;
  const size_t kh = static_cast<size_t>(p.block_tokens) * D, vh = static_cast<size_t>(p.block_tokens) * Dv;
  const int half = p.rot >> 1, d8 = D >> 3, dv8 = Dv >> 3;
  const int nqv = p.Hq * d8, nv = nqv + p.Hkv * d8;
  float f[VPT][8], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nv) {
      load8(row + static_cast<size_t>(i) * 8, f[j]);
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(f[j][e], f[j][e], s);
      if (i < nqv) sq += s; else sk += s;
    }
  }
  // v needs neither: its copies are in flight during the reduction
  if (slot >= 0) {
    for (int i = threadIdx.x; i < p.Hkv * dv8; i += blockDim.x) {
      const int h = i / dv8, j = (i - h * dv8) * 8;
      float a[8];
      load8(row + static_cast<size_t>(p.Hq + p.Hkv) * D + h * Dv + j, a);
      store8(vdst + h * vh + j, a);
    }
  }
  if (p.sums) {
    sq = p.sums[2 * t];
    sk = p.sums[2 * t + 1];
  } else {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
      sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) { sq += red[0][w]; sk += red[1][w]; }
  }
  const float rq = rsqrtf(sq / static_cast<float>(p.nq) + p.eps), rk = rsqrtf(sk / static_cast<float>(p.nk) + p.eps);
  const float* cs = p.cos_sin + static_cast<size_t>(pos) * p.rot;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nv && (i < nqv || slot >= 0)) {
      float w[8];
      load8(i < nqv ? p.qw + static_cast<size_t>(i) * 8 : p.kw + static_cast<size_t>(i - nqv) * 8, w);
      const float r = i < nqv ? rq : rk;
#pragma unroll
      for (int e = 0; e < 8; ++e) f[j][e] *= r * w[e];
      const int h = i / d8, c = (i - h * d8) * 8, pr = c >> 1;
      if (c < p.rot) {
        float co[4], si[4];
        if ((p.rot & 7) == 0) {         // the same for all; table rows and their halves start on 16-byte boundaries
          *reinterpret_cast<float4*>(co) = *reinterpret_cast<const float4*>(cs + pr);
          *reinterpret_cast<float4*>(si) = *reinterpret_cast<const float4*>(cs + half + pr);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const bool on = pr + e < half;
            co[e] = on ? cs[pr + e] : 1.f;
            si[e] = on ? cs[half + pr + e] : 0.f;
          }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float u = f[j][2 * e], v = f[j][2 * e + 1];
          f[j][2 * e] = u * co[e] - v * si[e];
          f[j][2 * e + 1] = v * co[e] + u * si[e];
        }
      }
      store8(i < nqv ? row + static_cast<size_t>(i) * 8 : kdst + (h - p.Hq) * kh + c, f[j]);
    }
  }
}

template <typename T>
static cudaError_t launch_norm_rope(const NormRopeParams<T>& p, int T_, cudaStream_t st) {
  const int nv = (p.Hq + p.Hkv) * (p.D >> 3);
  auto threads = [&](int vpt) { return dim3(((nv + vpt - 1) / vpt + 31) / 32 * 32); };
  if (nv <= 256) return launch_pdl(qkv_norm_rope_append_kernel<T, 1>, dim3(T_), threads(1), 0, st, p);
  if (nv <= 1024) return launch_pdl(qkv_norm_rope_append_kernel<T, 2>, dim3(T_), threads(2), 0, st, p);
  if (nv <= 4096) return launch_pdl(qkv_norm_rope_append_kernel<T, 4>, dim3(T_), threads(4), 0, st, p);
  return cudaErrorInvalidValue;
}

// Root-mean-square norms of two column ranges of a row: the query latent to q_out, the key/value latent to its place in the
// paged panel (slot < 0: a padding row, skipped). One warp per row and range. Sizes are rounded up to multiples of 8 in
// storage; pad columns and their weights are zero.
template <typename T>
struct LatentNormsParams {
  const T* q; const T* kv; long long ld;
  const T* qw; const T* kvw; float eps;
  T* q_out; int q_rank, kv_rank;
  const int* slots; T* cache; long long block_stride; int block_tokens; long long num_slots;
  int rows;
  int* err;
};
constexpr int kLnWarps = 4;

template <typename T>
__global__ void __launch_bounds__(32 * kLnWarps) latent_norms_kernel(const LatentNormsParams<T> p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, unit = blockIdx.x * kLnWarps + (threadIdx.x >> 5), t = unit >> 1;
  if (t >= p.rows) return;
  const bool is_q = (unit & 1) == 0;
  const int n = is_q ? p.q_rank : p.kv_rank, np = (n + 7) / 8 * 8;
  const T* src = (is_q ? p.q : p.kv) + static_cast<size_t>(t) * p.ld;
  const T* w = is_q ? p.qw : p.kvw;
  T* dst;
  if (is_q) {
    dst = p.q_out + static_cast<size_t>(t) * np;
  } else {
    const int slot = p.slots[t];
    if (slot < 0) return;
    if (slot >= p.num_slots) { if (lane == 0) guard_report(p.err, kGuardSlot, slot); return; }
    dst = p.cache + static_cast<size_t>(slot / p.block_tokens) * p.block_stride + static_cast<size_t>(slot % p.block_tokens) * np;
  }
  constexpr int kKeep = 6;              // vectors per lane that stay in registers between the two passes
  float keep[kKeep][8], ss = 0.f;
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int i = (lane + j * 32) * 8;
    if (i < np) {
      load8(src + i, keep[j]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(keep[j][e], keep[j][e], ss);
    }
  }
  for (int i = (lane + kKeep * 32) * 8; i < np; i += 32 * 8) {
    float f[8];
    load8(src + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(f[e], f[e], ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = rsqrtf(ss / static_cast<float>(n) + p.eps);
  auto put = [&](int i, float (&f)[8]) {
    float g[8];
    load8(w + i, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= r * g[e];
    store8(dst + i, f);
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int i = (lane + j * 32) * 8;
    if (i < np) put(i, keep[j]);
  }
  for (int i = (lane + kKeep * 32) * 8; i < np; i += 32 * 8) {
    float f[8];
    load8(src + i, f);
    put(i, f);
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

template <typename T>
static int residual_norm_entry(const float* x, int ldx, const int* rows, int in_rows, const void* y, int ldy, const void* w1,
                               const void* b1, const void* ls, float* x_out, const void* w2, const void* b2, void* z, int ldz,
                               int M, int H, float eps, int rms, float alpha, int groups, const float* add, const void* vec,
                               float z_scale, const int* dst_row, const float* w, int ldw, int top, int cap, const void* shared,
                               int lds, int* err, cudaStream_t st) {
  const ResNormParams<T> p{x, ldx, rows, in_rows, (const T*)y, ldy, (const T*)w1, (const T*)b1, (const T*)ls, x_out, (const T*)w2,
                           (const T*)b2, (T*)z, ldz, H, eps, rms, alpha, groups, add, (const T*)vec, z_scale, dst_row, w, ldw, top,
                           cap, (const T*)shared, lds, err};
  return launch_residual_norm(p, M, st);
}

// dst_row [M, top] / w [M, ldw] / shared: the addend is gathered from the expert outputs y [cap, ldy] (see ResNormParams)
extern "C" int ksana_residual_norm(const float* x, int ldx, const int* rows, int in_rows, const void* y, int ldy,
                                   const void* w1, const void* b1, const void* ls, float* x_out, const void* w2,
                                   const void* b2, void* z, int ldz, int M, int H, float eps, int rms, int f32,
                                   float alpha, int groups, const float* add, const void* vec, float z_scale, const int* dst_row,
                                   const float* w, int ldw, int top, int cap, const void* shared, int lds, int* err, cudaStream_t st) {
  if (M <= 0) return 0;
  const int hp = (H + 7) / 8 * 8;
  if (H <= 0 || ldx % 8 || ldx < hp || (y && (ldy % 8 || ldy < hp)) || (z && (ldz % 8 || ldz < hp))) return -10;
  for (const void* q : {(const void*)x, y, w1, b1, ls, (const void*)x_out, w2, b2, (const void*)z, (const void*)add, vec, shared})
    if (!aligned16(q)) return -11;
  if (rows && x_out == x) return -12;
  if (groups > 1 && (!rms || H % groups || w1 || b2 || !w2 || z_scale != 1.f)) return -13;
  if (dst_row && (!y || !w || rows || top <= 0 || top > kMaxTop || ldw < top || cap <= 0)) return -14;
  if (shared && (!dst_row || lds % 8 || lds < hp)) return -15;
  auto entry = f32 ? residual_norm_entry<float> : residual_norm_entry<bf16>;
  return entry(x, ldx, rows, in_rows, y, ldy, w1, b1, ls, x_out, w2, b2, z, ldz, M, H, eps, rms, alpha, groups, add, vec, z_scale,
               dst_row, w, ldw, top, cap, shared, lds, err, st);
}

// in [M, in_ld]: gate columns [0, I), up columns [I, 2I); out [M, I]. I a multiple of 8.
extern "C" int ksana_glu_clamp(const void* in, void* out, int M, int I, int in_ld, float limit, float alpha, float offset,
                               const int* tile_rows, int f32, cudaStream_t st) {
  if (M <= 0) return 0;
  if (I % 8 || in_ld % 8 || in_ld < 2 * I || !aligned16(in) || !aligned16(out)) return -10;
  const long long total = static_cast<long long>(M) * (I >> 3);
  long long g = (total + 255) / 256;
  if (g > 148 * 8) g = 148 * 8;
  cudaError_t e;
  if (f32)
    e = launch_pdl(glu_clamp_kernel<float>, dim3((unsigned)g), dim3(256), 0, st, (const float*)in, (float*)out, M, I, in_ld, limit,
                   alpha, offset, tile_rows);
  else
    e = launch_pdl(glu_clamp_kernel<bf16>, dim3((unsigned)g), dim3(256), 0, st, (const bf16*)in, (bf16*)out, M, I, in_ld, limit,
                   alpha, offset, tile_rows);
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

template <typename T>
static cudaError_t norm_rope_entry(void* qkv, const int* positions, const int* slots, const float* cos_sin, int max_pos,
                                   const void* qw, const void* kw, float eps, int nq, int nk, const float* sums, void* kc, void* vc,
                                   long long block_stride, int block_tokens, int num_blocks, int T_, int Hq, int Hkv, int D, int Dv,
                                   int rot, int* err, cudaStream_t st) {
  const NormRopeParams<T> p{(T*)qkv, positions, slots, cos_sin, max_pos, (const T*)qw, (const T*)kw, eps, nq, nk, sums, (T*)kc, (T*)vc,
                            block_stride, block_tokens, num_blocks, Hq, Hkv, D, Dv, rot, err};
  return launch_norm_rope(p, T_, st);
}

extern "C" int ksana_qkv_norm_rope_append(void* qkv, const int* positions, const int* slots, const float* cos_sin, int max_pos,
                                          const void* qw, const void* kw, float eps, int nq, int nk, const float* sums, void* kc,
                                          void* vc, long long block_stride, int block_tokens, int num_blocks, int T, int Hq, int Hkv,
                                          int D, int Dv, int rot, int f32, int* err, cudaStream_t st) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || Dv <= 0 || D % 8 || Dv % 8 || rot < 0 || rot > D || (rot & 1) || block_tokens <= 0 ||
      block_stride % 8 || (rot && !cos_sin) || !qw || !kw || nq <= 0 || nk <= 0 || (Hq + Hkv) * (D / 8) > 4096) return -10;
  if (!aligned16(qkv) || !aligned16(kc) || !aligned16(vc) || !aligned16(qw) || !aligned16(kw) || !aligned16(cos_sin)) return -11;
  auto entry = f32 ? norm_rope_entry<float> : norm_rope_entry<bf16>;
  return entry(qkv, positions, slots, cos_sin, max_pos, qw, kw, eps, nq, nk, sums, kc, vc, block_stride, block_tokens, num_blocks, T, Hq,
               Hkv, D, Dv, rot, err, st) == cudaSuccess ? 0 : -4;
}

template <typename T>
static cudaError_t latent_norms_entry(const void* q, const void* kv, long long ld, const void* qw, const void* kvw, float eps,
                                      void* q_out, int q_rank, int kv_rank, const int* slots, void* cache, long long block_stride,
                                      int block_tokens, long long num_slots, int T_, int* err, cudaStream_t st) {
  const LatentNormsParams<T> p{(const T*)q, (const T*)kv, ld, (const T*)qw, (const T*)kvw, eps, (T*)q_out, q_rank, kv_rank, slots,
                               (T*)cache, block_stride, block_tokens, num_slots, T_, err};
  return launch_pdl(latent_norms_kernel<T>, dim3((2 * T_ + kLnWarps - 1) / kLnWarps), dim3(32 * kLnWarps), 0, st, p);
}

// q, kv: column ranges of the same projection's rows, ld elements apart; q_out [T, q_rank rounded up to 8]
extern "C" int ksana_latent_norms(const void* q, const void* kv, long long ld, const void* qw, const void* kvw, float eps,
                                  void* q_out, int q_rank, int kv_rank, const int* slots, void* cache, long long block_stride,
                                  int block_tokens, long long num_slots, int T, int f32, int* err, cudaStream_t st) {
  if (T <= 0) return 0;
  if (q_rank <= 0 || kv_rank <= 0 || ld % 8 || block_stride % 8 || block_tokens <= 0) return -10;
  for (const void* a : {q, kv, qw, kvw, (const void*)q_out, (const void*)cache})
    if (!a || !aligned16(a)) return -11;
  auto entry = f32 ? latent_norms_entry<float> : latent_norms_entry<bf16>;
  return entry(q, kv, ld, qw, kvw, eps, q_out, q_rank, kv_rank, slots, cache, block_stride, block_tokens, num_slots, T, err, st) ==
                 cudaSuccess ? 0 : -4;
}

extern "C" int ksana_refit_rows_f32(float* x, int ldx, const int* pos, const float* emb, int R, int H, int rows, int* err,
                                    cudaStream_t st) {
  if (R <= 0) return 0;
  refit_rows_f32_kernel<<<R, 256, 0, st>>>(x, ldx, pos, emb, H, rows, err);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
