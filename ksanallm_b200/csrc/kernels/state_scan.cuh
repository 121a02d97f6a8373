// What the kernels of matrix-state recurrences (state_scan.cu: CUDA cores, fp32; state_chunk.cu: tensor cores, bf16 operands)
// share: where a sequence's state and convolution inputs live, and the parameters of both recurrences.
#pragma once
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>

namespace ksana {

constexpr int kMaxTaps = 16;
constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// exp(-x), x >= 0, rounded to nearest near 1: a decay is applied once per token, a bias of its last bit would add up
__device__ __forceinline__ float decay_f(float x) { return 1.f + expm1f(-x); }
__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
// in the activations' precision
template <typename T> __device__ __forceinline__ float sigmoid_as(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
  else return sigmoid_exact(x);
}

struct StateRef {                            // where sequences keep their state
  const int* slots; int num_slots;           // per sequence; < 0: padding
  const int* kv_lens;
  int* err;
};
// The slot of sequence s, or -1 where it has none (padding, or an id outside the pool, which is recorded).
__device__ __forceinline__ int slot_of(const StateRef& r, int s) {
  const int slot = r.slots[s];
  if (slot >= r.num_slots) { if (threadIdx.x == 0) guard_report(r.err, kGuardSlot, slot); return -1; }
  return slot;
}

template <typename T>
struct ConvRef {                             // a short convolution's inputs, weights and ring
  const T* x; long long ld;                  // raw projection rows, first channel
  const T* w; const T* bias;                 // [taps][C] (the last tap is the current token's), [C] or null
  T* ring; long long slot_stride;            // ring of slot 0, elements between slots
  int taps, C;
};

// Channels [c0, c0 + n) of the last inputs of a sequence's new tokens go to the ring.
template <typename T>
__device__ __forceinline__ void ring_store(const ConvRef<T>& v, const T* rows, T* ring, int past, int n, int c0, int count, int tid, int threads) {
  const int vecs = count >> 3, keep = min(v.taps, n);
  for (int i = tid; i < vecs * keep; i += threads) {
    const int t = n - 1 - i / vecs, c = c0 + (i % vecs) * 8;
    float f[8];
    load8(rows + static_cast<long long>(t) * v.ld + c, f);
    store8(ring + static_cast<size_t>((past + t) % v.taps) * v.C + c, f);
  }
}

template <typename T>
struct SpaceParams {
  ConvRef<T> conv;                           // channels: x [H][P] | B [G][N] | C [G][N]
  const T* c; long long ldc;                 // convolved rows (scan)
  const T* dt; long long ld_dt;              // raw step sizes, [rows][H]
  const float* dt_bias; const float* A; const float* D;      // [H]
  T* y; long long ldy;                       // [rows][H * P]
  float* state; long long slot_stride;       // matrix state of slot 0 of the layer, floats between slots
  StateRef ref;
  const int* cu_q;
  int H, G, P, N;
};

// Channels of the ring that the CTA of (head, slab of columns [p0, p0 + np)) stores: its own x, and B and C of the head's group
// where it is the group's first.
template <typename T>
__device__ __forceinline__ void space_ring(const SpaceParams<T>& p, const T* rows, int slot, int past, int n, int h, int p0, int np, int tid,
                                           int threads) {
  T* ring = p.conv.ring + static_cast<long long>(slot) * p.conv.slot_stride;
  ring_store(p.conv, rows, ring, past, n, h * p.P + p0, np, tid, threads);
  const int per = p.H / p.G, g = h / per;
  if (h % per == 0 && p0 == 0) {
    ring_store(p.conv, rows, ring, past, n, p.H * p.P + g * p.N, p.N, tid, threads);
    ring_store(p.conv, rows, ring, past, n, p.H * p.P + (p.G + g) * p.N, p.N, tid, threads);
  }
}

template <typename T>
struct DeltaParams {
  ConvRef<T> conv;                           // channels: q [G][K] | k [G][K] | v [H][V]
  const T* c; long long ldc;                 // convolved rows (scan)
  const T* beta; long long ld_beta;          // raw, [rows][H]
  const T* decay; long long ld_decay;        // raw, [rows][H * K]
  const float* decay_bias; const float* A;   // [H * K], [H]
  T* o; long long ldo;                       // [rows][H * V]
  float* state; long long slot_stride;
  StateRef ref;
  const int* cu_q;
  int H, G, K, V;
  float q_scale;
};

template <typename T>
__device__ __forceinline__ void delta_ring(const DeltaParams<T>& p, const T* rows, int slot, int past, int n, int h, int p0, int np, int tid,
                                           int threads) {
  T* ring = p.conv.ring + static_cast<long long>(slot) * p.conv.slot_stride;
  ring_store(p.conv, rows, ring, past, n, 2 * p.G * p.K + h * p.V + p0, np, tid, threads);
  const int per = p.H / p.G, g = h / per;
  if (h % per == 0 && p0 == 0) {
    ring_store(p.conv, rows, ring, past, n, g * p.K, p.K, tid, threads);
    ring_store(p.conv, rows, ring, past, n, (p.G + g) * p.K, p.K, tid, threads);
  }
}

// Scans of several new tokens per sequence on the tensor cores (state_chunk.cu): -100 where the sizes are not covered.
int space_chunks(const SpaceParams<bf16>& p, int B, cudaStream_t st);
int delta_chunks(const DeltaParams<bf16>& p, int B, cudaStream_t st);

}  // namespace ksana
