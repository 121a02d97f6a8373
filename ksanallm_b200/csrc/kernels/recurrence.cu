// Gated linear recurrence over the new tokens of a step, for recurrent layers whose gates read the current token only:
//
//   gate_t = sigmoid(z_t),  cand_t = u_t + offset where u_t >= 0, sigmoid(u_t) elsewhere
//   S_t = (1 - gate_t) S_(t-1) + gate_t cand_t,   out_t = S_t silu(g_t)        element by element
//
// Everything between the projections and the output product is fp32. The state lives in the paged cache: a block's
// record holds one fp32 row per recurrent layer, the state after the last of the block's tokens that has been computed.
// A portion that starts at position p therefore reads the row of the block of position p - 1 (zero at p = 0), and every
// block that the portion fills keeps the state at its end, so that whole blocks can be shared, swapped and copied like
// the keys and values beside them.
//
//   gated_scan_kernel   sequences of any number of new tokens: one CTA per (sequence, channel tile), the time axis split
//                       over the threads, prefixes combined in registers, shuffles and one exchange per chunk
//   gated_step_kernel   sequences of one new token
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>

namespace ksana {

constexpr int kScanThreads = 256, kScanWarps = kScanThreads / 32;
constexpr int kScanPer = 4;                    // consecutive tokens per thread and chunk

template <typename T>
struct ScanParams {
  const T* z; const T* u; const T* g; long long ld;      // columns of one projection's rows, ld elements apart
  T* out; long long ldo;
  float* state; long long block_stride;                  // state row of block 0 of the layer; floats between blocks
  int block_tokens, num_blocks;
  const int* block_table; int table_stride;
  const int* cu_q; const int* kv_lens;                   // cu_q null: one row per sequence
  int W;                                                 // channels (a multiple of 8)
  float offset;
  int* err;
};

// decay and increment of one element
__device__ __forceinline__ void gate_pair(float z, float u, float offset, float& a, float& b) {
  const float gate = sigmoid_f(z);
  a = 1.f - gate;
  b = gate * (u >= 0.f ? u + offset : sigmoid_f(u));
}

// State row of the block that holds position `pos` of a sequence, or null for an id outside the cache.
template <typename T>
__device__ __forceinline__ float* state_row(const ScanParams<T>& p, const int* table, int pos) {
  const int blk = table[pos / p.block_tokens];
  if (blk < 0 || blk >= p.num_blocks) { guard_report(p.err, kGuardBlockId, blk); return nullptr; }
  return p.state + static_cast<long long>(blk) * p.block_stride;
}

// TPR threads cover the channels of one token (8 each); the others take later tokens of the chunk.
template <typename T, int TPR>
__global__ void __launch_bounds__(kScanThreads, 2) gated_scan_kernel(const ScanParams<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float tot[2][kScanWarps][2][TPR * 8];       // per warp: product of the decays, state from zero
  const int s = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cl = (threadIdx.x % TPR) * 8, c = blockIdx.x * TPR * 8 + cl;
  const bool live = c < p.W;
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.kv_lens[s] - n;
  if (n <= 0) return;
  if (past < 0) { if (threadIdx.x == 0) guard_report(p.err, kGuardQueryRow, q0 + n); return; }
  const int* table = p.block_table + static_cast<size_t>(s) * p.table_stride;
  float S0[8] = {};
  if (past > 0 && live) {
    const float* row = state_row(p, table, past - 1);
    if (row) load8(row + c, S0);
  }
  constexpr int kLanes = kScanThreads / TPR, kChunk = kLanes * kScanPer;
  const int tl = threadIdx.x / TPR;
  for (int t0 = 0, buf = 0; t0 < n; t0 += kChunk, buf ^= 1) {
    const int first = t0 + tl * kScanPer;
    float a[kScanPer][8], b[kScanPer][8], A[8], B[8];
#pragma unroll
    for (int l = 0; l < kScanPer; ++l) {
      if (live && first + l < n) {
        load8(p.z + (q0 + first + l) * p.ld + c, a[l]);
        load8(p.u + (q0 + first + l) * p.ld + c, b[l]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) { A[e] = 1.f; B[e] = 0.f; }
#pragma unroll
    for (int l = 0; l < kScanPer; ++l) {
      const bool on = live && first + l < n;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (on) gate_pair(a[l][e], b[l][e], p.offset, a[l][e], b[l][e]);
        else { a[l][e] = 1.f; b[l][e] = 0.f; }
        B[e] = fmaf(a[l][e], B[e], b[l][e]);
        A[e] *= a[l][e];
      }
    }
    // inclusive prefixes over the warp's token lanes, then the exclusive one of this thread
#pragma unroll
    for (int o = TPR; o < 32; o <<= 1) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float pa = __shfl_up_sync(0xffffffffu, A[e], o), pb = __shfl_up_sync(0xffffffffu, B[e], o);
        if (lane >= o) { B[e] = fmaf(A[e], pb, B[e]); A[e] *= pa; }
      }
    }
    if (lane >= 32 - TPR) {
      store8(&tot[buf][warp][0][cl], A);
      store8(&tot[buf][warp][1][cl], B);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float pa = __shfl_up_sync(0xffffffffu, A[e], TPR), pb = __shfl_up_sync(0xffffffffu, B[e], TPR);
      A[e] = lane >= TPR ? pa : 1.f;
      B[e] = lane >= TPR ? pb : 0.f;
    }
    __syncthreads();            // the other buffer is free again once every thread has passed the next chunk's barrier
    float S[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) S[e] = S0[e];
#pragma unroll
    for (int w = 0; w < kScanWarps; ++w) {
      float wa[8], wb[8];
      load8(&tot[buf][w][0][cl], wa);
      load8(&tot[buf][w][1][cl], wb);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        S0[e] = fmaf(wa[e], S0[e], wb[e]);
        if (w < warp) S[e] = S0[e];
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) S[e] = fmaf(A[e], S[e], B[e]);
#pragma unroll
    for (int l = 0; l < kScanPer; ++l) {
      const int t = first + l;
#pragma unroll
      for (int e = 0; e < 8; ++e) S[e] = fmaf(a[l][e], S[e], b[l][e]);
      if (live && t < n) {
        float o[8];
        load8(p.g + (q0 + t) * p.ld + c, o);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = S[e] * o[e] * sigmoid_f(o[e]);
        store8(p.out + (q0 + t) * p.ldo + c, o);
        if (t == n - 1 || (past + t + 1) % p.block_tokens == 0) {
          float* row = state_row(p, table, past + t);
          if (row) store8(row + c, S);
        }
      }
    }
  }
}

// One thread per 8 channels of a sequence's single new token. kv_len 0: a padding row, its output is zero.
template <typename T>
__global__ void gated_step_kernel(const ScanParams<T> p) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= p.W) return;
  const int pos = p.kv_lens[s] - 1;
  float o[8] = {};
  if (pos >= 0) {
    const int* table = p.block_table + static_cast<size_t>(s) * p.table_stride;
    float a[8], b[8], S[8] = {};
    load8(p.z + s * p.ld + c, a);
    load8(p.u + s * p.ld + c, b);
    load8(p.g + s * p.ld + c, o);
    if (pos > 0) {
      const float* row = state_row(p, table, pos - 1);
      if (row) load8(row + c, S);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      gate_pair(a[e], b[e], p.offset, a[e], b[e]);
      S[e] = fmaf(a[e], S[e], b[e]);
      o[e] = S[e] * o[e] * sigmoid_f(o[e]);
    }
    float* row = state_row(p, table, pos);
    if (row) store8(row + c, S);
  }
  store8(p.out + s * p.ldo + c, o);
}

template <typename T>
static int launch_gated(const void* z, const void* u, const void* g, long long ld, void* out, long long ldo, float* state,
                        long long block_stride, int block_tokens, int num_blocks, const int* block_table, int table_stride,
                        const int* cu_q, const int* kv_lens, int B, int W, float offset, int* err, cudaStream_t st) {
  ScanParams<T> p{};
  p.z = static_cast<const T*>(z); p.u = static_cast<const T*>(u); p.g = static_cast<const T*>(g); p.ld = ld;
  p.out = static_cast<T*>(out); p.ldo = ldo; p.state = state; p.block_stride = block_stride;
  p.block_tokens = block_tokens; p.num_blocks = num_blocks; p.block_table = block_table; p.table_stride = table_stride;
  p.cu_q = cu_q; p.kv_lens = kv_lens; p.W = W; p.offset = offset; p.err = err;
  cudaError_t e;
  if (!cu_q) {
    const int vec = W / 8, threads = vec >= 128 ? 128 : (vec + 31) / 32 * 32;
    e = launch_pdl(gated_step_kernel<T>, dim3((vec + threads - 1) / threads, B), dim3(threads), 0, st, p);
  } else if (static_cast<long long>(B) * ((W + 63) / 64) >= 2 * 148) {
    e = launch_pdl(gated_scan_kernel<T, 8>, dim3((W + 63) / 64, B), dim3(kScanThreads), 0, st, p);
  } else {
    e = launch_pdl(gated_scan_kernel<T, 4>, dim3((W + 31) / 32, B), dim3(kScanThreads), 0, st, p);
  }
  return e == cudaSuccess ? 0 : -4;
}

}  // namespace ksana

using namespace ksana;

// z, u, g: columns of the projections' rows (ld elements apart), bf16 or (f32) fp32; out [rows, ldo]. cu_q null: every
// sequence has one row. state: fp32 row of block 0 of the layer, block_stride floats between blocks.
extern "C" int ksana_gated_recurrence(const void* z, const void* u, const void* g, long long ld, void* out, long long ldo,
                                      float* state, long long block_stride, int block_tokens, int num_blocks,
                                      const int* block_table, int table_stride, const int* cu_q, const int* kv_lens, int B, int W,
                                      float offset, int f32, int* err, cudaStream_t st) {
  if (B <= 0) return 0;
  if (W <= 0 || W % 8 || ld % 8 || ldo % 8 || ldo < W || block_stride % 4 || block_tokens <= 0 || num_blocks <= 0 || B > 65535)
    return -10;
  for (const void* q : {z, u, g, (const void*)out, (const void*)state})
    if (!aligned16(q)) return -11;
  return f32 ? launch_gated<float>(z, u, g, ld, out, ldo, state, block_stride, block_tokens, num_blocks, block_table, table_stride,
                                   cu_q, kv_lens, B, W, offset, err, st)
             : launch_gated<bf16>(z, u, g, ld, out, ldo, state, block_stride, block_tokens, num_blocks, block_table, table_stride,
                                  cu_q, kv_lens, B, W, offset, err, st);
}
