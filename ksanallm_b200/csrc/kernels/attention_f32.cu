// Paged attention in true 32-bit arithmetic: one CTA per (query row, head), new rows of any number of sequences in one
// launch. Serves models that run entirely in fp32, and (over bf16 storage) latent attention in sizes that the tensor-core
// kernel does not cover. Keys are walked in chunks of 128 (one key per thread for the scores, one output
// column per thread for the sum) with an online softmax. Sliding window with kept first tokens, grouped query heads,
// different key and value sizes (values may be the leading columns of the key rows), an optional per-head sink logit in the
// denominator and an optional gate per query row and head, or per output element (with a common factor). With a bias table
// [heads][distances] the weights are sigmoid(score + bias) instead, without normalisation.
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>

namespace ksana {

constexpr int kAfThreads = 128;
constexpr int kAfMaxD = 256;                 // head sizes of the ordinary form
constexpr int kAfMaxWide = 1024;             // ... and of the wide one (latent rows)

template <typename T>
struct AttnF32Params {
  const T* q; long long q_stride;
  T* out; long long out_stride;
  const T* kc; const T* vc;                  // K panel [Hkv][bt][D], V panel [Hkv][bt][ldv] of block 0 of the layer
  int ldv;                                   // elements between value rows (at least Dv)
  long long block_stride; int block_tokens, num_blocks;
  const int* block_table; int table_stride;
  const int* cu_q; const int* kv_lens;
  const float* sinks;
  const T* gate; long long gate_ld;          // optional [rows][gate_ld]: a head's output is multiplied by sigmoid(gate)
  int gate_wide; float out_factor;           // gate_wide: a gate per output element (columns like out's)
  const float* bias; int bias_len;           // sigmoid weights: [Hq][bias_len] by distance (the last entry holds beyond)
  int Hq, Hkv, D, Dv, window, keep;
  float scale;
  int* err;
};

__device__ __forceinline__ float block_reduce(float v, float* red, bool is_max) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float w = __shfl_xor_sync(0xffffffffu, v, o);
    v = is_max ? fmaxf(v, w) : v + w;
  }
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = red[0];
#pragma unroll
  for (int i = 1; i < kAfThreads / 32; ++i) v = is_max ? fmaxf(v, red[i]) : v + red[i];
  __syncthreads();
  return v;
}

template <typename T, int MAXD>
__global__ void __launch_bounds__(kAfThreads) attention_f32_kernel(const AttnF32Params<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float qs[MAXD];
  __shared__ float ps[kAfThreads];
  __shared__ long long voff[kAfThreads];
  __shared__ float red[kAfThreads / 32];
  const int s = blockIdx.z, head = blockIdx.y;
  const int q0 = p.cu_q[s], q_len = p.cu_q[s + 1] - q0;
  const int qi = blockIdx.x;
  if (qi >= q_len) return;
  const int pos = p.kv_lens[s] - q_len + qi;
  const int g = head / (p.Hq / p.Hkv);
  const int* table = p.block_table + static_cast<size_t>(s) * p.table_stride;
  const T* q = p.q + static_cast<size_t>(q0 + qi) * p.q_stride + static_cast<size_t>(head) * p.D;
  for (int d = threadIdx.x; d < p.D; d += kAfThreads) qs[d] = to_f(q[d]);
  // visible keys in order: the kept first tokens below the window, then the window
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int nkeep = min(p.keep, lo), nvis = nkeep + pos + 1 - lo;
  const float sink = p.sinks ? p.sinks[head] : -CUDART_INF_F;
  float m = sink, l = p.sinks ? 1.f : 0.f;
  float o[MAXD / kAfThreads] = {};
  __syncthreads();
  for (int c0 = 0; c0 < nvis; c0 += kAfThreads) {
    const int i = c0 + threadIdx.x;
    float sc = -CUDART_INF_F;
    long long vo = -1;
    if (i < nvis) {
      const int tok = i < nkeep ? i : lo + i - nkeep;
      const int blk = table[tok / p.block_tokens], off = tok % p.block_tokens;
      if (blk < 0 || blk >= p.num_blocks) {
        guard_report(p.err, kGuardBlockId, blk);
      } else {
        const T* k = p.kc + static_cast<long long>(blk) * p.block_stride + (static_cast<long long>(g) * p.block_tokens + off) * p.D;
        float acc = 0.f;
        for (int d = 0; d < p.D; d += 8) {
          float kv[8];
          load8(k + d, kv);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc = fmaf(kv[e], qs[d + e], acc);
        }
        sc = acc * p.scale;
        vo = static_cast<long long>(blk) * p.block_stride + (static_cast<long long>(g) * p.block_tokens + off) * p.ldv;
      }
    }
    if (p.bias) {                             // same for every thread of the launch
      const int tok = i < nkeep ? i : lo + i - nkeep;
      const float b = vo >= 0 ? p.bias[static_cast<size_t>(head) * p.bias_len + min(pos - tok, p.bias_len - 1)] : 0.f;
      ps[threadIdx.x] = vo >= 0 ? 1.f / (1.f + expf(-(sc + b))) : 0.f;
      voff[threadIdx.x] = vo;
      l = 1.f;
      __syncthreads();
      const int n = min(kAfThreads, nvis - c0);
#pragma unroll
      for (int c = 0; c < MAXD / kAfThreads; ++c) {
        const int d = threadIdx.x + c * kAfThreads;
        if (d < p.Dv)
          for (int k = 0; k < n; ++k) if (voff[k] >= 0) o[c] = fmaf(ps[k], to_f(p.vc[voff[k] + d]), o[c]);
      }
      __syncthreads();
      continue;
    }
    const float mx = fmaxf(m, block_reduce(sc, red, true));
    const float corr = (m == -CUDART_INF_F) ? 0.f : expf(m - mx);
    const float pr = (sc == -CUDART_INF_F) ? 0.f : expf(sc - mx);
    m = mx;
    ps[threadIdx.x] = pr;
    voff[threadIdx.x] = vo;
    l = l * corr + block_reduce(pr, red, false);       // its barriers also publish ps and voff
    const int n = min(kAfThreads, nvis - c0);
#pragma unroll
    for (int c = 0; c < MAXD / kAfThreads; ++c) {
      const int d = threadIdx.x + c * kAfThreads;
      if (d < p.Dv) {
        float acc = o[c] * corr;
        for (int k = 0; k < n; ++k) if (voff[k] >= 0) acc = fmaf(ps[k], to_f(p.vc[voff[k] + d]), acc);
        o[c] = acc;
      }
    }
    __syncthreads();
  }
  if (p.gate && p.gate_wide) {
#pragma unroll
    for (int c = 0; c < MAXD / kAfThreads; ++c) {
      const int d = threadIdx.x + c * kAfThreads;
      if (d < p.Dv) o[c] *= p.out_factor * sigmoid_f(to_f(p.gate[static_cast<size_t>(q0 + qi) * p.gate_ld + static_cast<size_t>(head) * p.Dv + d]));
    }
  } else if (p.gate) {
    const float f = sigmoid_f(to_f(p.gate[static_cast<size_t>(q0 + qi) * p.gate_ld + head]));
#pragma unroll
    for (int c = 0; c < MAXD / kAfThreads; ++c) o[c] *= f;
  }
#pragma unroll
  for (int c = 0; c < MAXD / kAfThreads; ++c) {
    const int d = threadIdx.x + c * kAfThreads;
    if (d < p.Dv) p.out[static_cast<size_t>(q0 + qi) * p.out_stride + static_cast<size_t>(head) * p.Dv + d] = from_f<T>(l > 0.f ? o[c] / l : 0.f);
  }
}

template <typename T>
static int launch_attention_f32(const void* q, long long q_stride, void* out, long long out_stride, const void* kc, const void* vc,
                                int ldv, long long block_stride, int block_tokens, int num_blocks, const int* block_table,
                                int table_stride, const int* cu_q, const int* kv_lens, const float* sinks, const void* gate,
                                long long gate_ld, int gate_wide, float out_factor, const float* bias, int bias_len, int B, int max_q_len,
                                int Hq, int Hkv, int D, int Dv, int window, int keep, float scale, int* err, cudaStream_t st) {
  AttnF32Params<T> p{};
  p.q = static_cast<const T*>(q); p.q_stride = q_stride; p.out = static_cast<T*>(out); p.out_stride = out_stride;
  p.kc = static_cast<const T*>(kc); p.vc = static_cast<const T*>(vc); p.ldv = ldv;
  p.block_stride = block_stride; p.block_tokens = block_tokens; p.num_blocks = num_blocks;
  p.block_table = block_table; p.table_stride = table_stride; p.cu_q = cu_q; p.kv_lens = kv_lens; p.sinks = sinks;
  p.gate = static_cast<const T*>(gate); p.gate_ld = gate_ld; p.gate_wide = gate_wide; p.out_factor = out_factor;
  p.bias = bias; p.bias_len = bias_len;
  p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.Dv = Dv; p.window = window; p.keep = window > 0 ? keep : 0; p.scale = scale; p.err = err;
  const dim3 grid(max_q_len, Hq, B), block(kAfThreads);
  const cudaError_t e = (D > kAfMaxD || Dv > kAfMaxD)
      ? launch_pdl(attention_f32_kernel<T, kAfMaxWide>, grid, block, 0, st, p)
      : launch_pdl(attention_f32_kernel<T, kAfMaxD>, grid, block, 0, st, p);
  return e == cudaSuccess ? 0 : -4;
}

}  // namespace ksana

using namespace ksana;

// window 0: full causal attention. bias: sigmoid weights. D and Dv multiples of 8, at most 1024. ldv: elements between value
// rows. f32: q, out and the panels are fp32 instead of bf16.
extern "C" int ksana_attention_f32(const void* q, long long q_stride, void* out, long long out_stride, const void* kc,
                                   const void* vc, int ldv, long long block_stride, int block_tokens, int num_blocks,
                                   const int* block_table, int table_stride, const int* cu_q, const int* kv_lens,
                                   const float* sinks, const void* gate, long long gate_ld, int gate_wide, float out_factor,
                                   const float* bias, int bias_len, int B, int max_q_len, int Hq, int Hkv, int D, int Dv, int window,
                                   int keep, float scale, int f32, int* err, cudaStream_t st) {
  if (B <= 0 || max_q_len <= 0) return 0;
  if (bias && bias_len <= 0) return -14;
  if (Hkv <= 0 || Hq % Hkv || D <= 0 || Dv <= 0 || D > kAfMaxWide || Dv > kAfMaxWide || D % 8 || Dv % 8 || ldv < Dv || Hq > 65535 ||
      B > 65535 || block_tokens <= 0 || block_stride % 8 || !aligned16(kc)) return -10;
  return f32 ? launch_attention_f32<float>(q, q_stride, out, out_stride, kc, vc, ldv, block_stride, block_tokens, num_blocks, block_table,
                                           table_stride, cu_q, kv_lens, sinks, gate, gate_ld, gate_wide, out_factor, bias, bias_len, B, max_q_len, Hq,
                                           Hkv, D, Dv, window, keep, scale, err, st)
             : launch_attention_f32<bf16>(q, q_stride, out, out_stride, kc, vc, ldv, block_stride, block_tokens, num_blocks, block_table,
                                          table_stride, cu_q, kv_lens, sinks, gate, gate_ld, gate_wide, out_factor, bias, bias_len, B, max_q_len, Hq,
                                          Hkv, D, Dv, window, keep, scale, err, st);
}
