// Gated linear recurrence over the new tokens of a step, for recurrent layers whose gates do not depend on the state:
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
#include "f32x2.cuh"
#include "guards.cuh"
#include "pdl.cuh"
#include "vec8.cuh"
#include <cuda_runtime.h>

namespace ksana {

// consecutive tokens per thread and chunk, and the staging area of two chunks: every thread stages its own vectors (no
// barrier), 16 bytes of consecutive threads side by side
template <typename T> constexpr int kScanPer = sizeof(T) == 2 ? 4 : 2;
template <typename T> constexpr int kScanPieces = sizeof(T) / 2;                       // 16-byte pieces of 8 elements
template <typename T, int THREADS> constexpr int kScanStage = 3 * kScanPer<T> * kScanPieces<T> * THREADS * 16;

template <typename T>
struct ScanParams {
  const T* z; const T* u; const T* g; long long ld;      // columns of one projection's rows, ld elements apart
  T* out; long long ldo;
  float* state; long long block_stride;                  // state row of block 0 of the layer; floats between blocks
  int block_tokens, num_blocks;
  const int* block_table; int table_stride;
  const int* cu_q; const int* kv_lens;
  const int* slots;                                      // one row per sequence: its cache slot (cu_q is not read)
  int W;                                                 // channels (a multiple of 8)
  float offset;
  int* err;
};

// 1 + exp(-x) of a pair
__device__ __forceinline__ F2 one_plus_exp_neg(F2 x) {
  float a, b;
  split(x * f2(-1.44269504f), a, b);
  return f2(exp2f(a), exp2f(b)) + f2(1.f);
}
__device__ __forceinline__ F2 reciprocal(F2 x) {
  float a, b;
  split(x, a, b);
  return f2(1.f / a, 1.f / b);
}

constexpr float kGateMin = -40.f;      // arguments of sigmoids are cut here (4e-18): products of two denominators stay finite

// decays and increments of a pair; both sigmoids of an element from one reciprocal
__device__ __forceinline__ void gate_pair(F2 z, F2 u, F2 offset, F2& a, F2& b) {
  const F2 dz = one_plus_exp_neg(z), du = one_plus_exp_neg(u), r = reciprocal(dz * du), gate = du * r;
  float u0, u1, p0, p1, n0, n1;
  split(u, u0, u1);
  split(u + offset, p0, p1);
  split(dz * r, n0, n1);
  a = fma2(gate, f2(-1.f), f2(1.f));
  b = gate * f2(u0 >= 0.f ? p0 : n0, u1 >= 0.f ? p1 : n1);
}
// S g sigmoid(g), one reciprocal for the pair
__device__ __forceinline__ F2 gated_out(F2 S, F2 g) {
  float a, b;
  split(one_plus_exp_neg(g), a, b);
  const float r = 1.f / (a * b);
  return (S * g) * (f2(b, a) * f2(r));
}

__device__ __forceinline__ void load8(const float* p, F2 (&f)[4]) {
  const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(p), y = *reinterpret_cast<const ulonglong2*>(p + 4);
  f[0].v = x.x; f[1].v = x.y; f[2].v = y.x; f[3].v = y.y;
}
__device__ __forceinline__ void load8(const bf16* p, F2 (&f)[4]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) f[i] = f2(__uint_as_float(w[i] << 16), __uint_as_float(w[i] & 0xffff0000u));
}
__device__ __forceinline__ void store8(float* p, const F2 (&f)[4]) {
  *reinterpret_cast<ulonglong2*>(p) = make_ulonglong2(f[0].v, f[1].v);
  *reinterpret_cast<ulonglong2*>(p + 4) = make_ulonglong2(f[2].v, f[3].v);
}
__device__ __forceinline__ void store8(bf16* p, const F2 (&f)[4]) {
  float g[8];
#pragma unroll
  for (int i = 0; i < 4; ++i) split(f[i], g[2 * i], g[2 * i + 1]);
  store8(p, g);
}
// the sigmoids' arguments: cut from below
__device__ __forceinline__ void load8_cut(const float* p, F2 (&f)[4]) {
  float g[8];
  load8(p, g);
#pragma unroll
  for (int i = 0; i < 4; ++i) f[i] = f2(fmaxf(g[2 * i], kGateMin), fmaxf(g[2 * i + 1], kGateMin));
}
__device__ __forceinline__ void load8_cut(const bf16* p, F2 (&f)[4]) {
  __align__(16) __nv_bfloat162 v[4];
  *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(p);
#pragma unroll
  for (int i = 0; i < 4; ++i) v[i] = __hmax2(v[i], __float2bfloat162_rn(kGateMin));
  load8(reinterpret_cast<const bf16*>(v), f);
}

__device__ __forceinline__ void copy16_async(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src));
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// State row of the block that holds position `pos` of a sequence, or null for an id outside the cache.
template <typename T>
__device__ __forceinline__ float* state_row(const ScanParams<T>& p, const int* table, int pos) {
  const int blk = table[pos / p.block_tokens];
  if (blk < 0 || blk >= p.num_blocks) { guard_report(p.err, kGuardBlockId, blk); return nullptr; }
  return p.state + static_cast<long long>(blk) * p.block_stride;
}

// TPR threads cover the channels of one token (8 each); the others take later tokens of the chunk.
template <typename T, int TPR, int THREADS>
__global__ void __launch_bounds__(THREADS, 512 / THREADS) gated_scan_kernel(const ScanParams<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float tot[2][THREADS / 32][2][TPR * 8];      // per warp: product of the decays, state from zero
  __shared__ __align__(16) float carry[2][TPR * 8];                    // state after the chunk before
  const int s = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cl = (threadIdx.x % TPR) * 8, c = blockIdx.x * TPR * 8 + cl;
  const bool live = c < p.W;
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.kv_lens[s] - n;
  if (n <= 0) return;
  if (past < 0) { if (threadIdx.x == 0) guard_report(p.err, kGuardQueryRow, q0 + n); return; }
  const int* table = p.block_table + static_cast<size_t>(s) * p.table_stride;
  constexpr int kPer = kScanPer<T>, kPieces = kScanPieces<T>, kLanes = THREADS / TPR, kChunk = kLanes * kPer;
  const int tl = threadIdx.x / TPR;
  extern __shared__ __align__(16) uint8_t staged[];
  // piece i of vector v (0 z, 1 u, 2 g) of this thread's token l
  auto slot = [&](int buf, int v, int l, int i) {
    return staged + buf * kScanStage<T, THREADS> + (((v * kPer + l) * kPieces + i) * THREADS + threadIdx.x) * 16;
  };
  auto fetch = [&](int buf, int v, int l, T (&raw)[8]) {
#pragma unroll
    for (int i = 0; i < kPieces; ++i) reinterpret_cast<uint4*>(raw)[i] = *reinterpret_cast<const uint4*>(slot(buf, v, l, i));
  };
  if (tl == 0) {
    float S[8] = {};
    if (past > 0 && live) {
      const float* row = state_row(p, table, past - 1);
      if (row) load8(row + c, S);
    }
    store8(&carry[0][cl], S);
  }
  const long long at = static_cast<long long>(q0) * p.ld + c;
  const T* zp = p.z + at;
  const T* up = p.u + at;
  const T* gp = p.g + at;
  T* op = p.out + static_cast<long long>(q0) * p.ldo + c;
  auto stage = [&](int t0, int buf) {
    if (!live) return;
#pragma unroll
    for (int l = 0; l < kPer; ++l) {
      const int t = t0 + tl * kPer + l;
      if (t >= n) break;
#pragma unroll
      for (int i = 0; i < kPieces; ++i) {
        copy16_async(slot(buf, 0, l, i), reinterpret_cast<const uint4*>(zp + t * p.ld) + i);
        copy16_async(slot(buf, 1, l, i), reinterpret_cast<const uint4*>(up + t * p.ld) + i);
        copy16_async(slot(buf, 2, l, i), reinterpret_cast<const uint4*>(gp + t * p.ld) + i);
      }
    }
  };
  stage(0, 0);
  copy_commit();
  for (int t0 = 0, buf = 0; t0 < n; t0 += kChunk, buf ^= 1) {
    const int first = t0 + tl * kPer, count = live ? min(kPer, n - first) : 0;      // tokens of this thread
    if (t0 + kChunk < n) stage(t0 + kChunk, buf ^ 1);
    copy_commit();
    copy_wait<1>();                     // this thread's vectors of this chunk have landed
    F2 a[kPer][4], b[kPer][4], A[4], B[4];                   // four pairs of channels
#pragma unroll
    for (int e = 0; e < 4; ++e) { A[e] = f2(1.f); B[e] = f2(0.f); }
#pragma unroll
    for (int l = 0; l < kPer; ++l) {
      if (l < count) {
        __align__(16) T zr[8], ur[8];
        F2 z[4], u[4];
        fetch(buf, 0, l, zr);
        fetch(buf, 1, l, ur);
        load8_cut(zr, z);
        load8_cut(ur, u);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          gate_pair(z[e], u[e], f2(p.offset), a[l][e], b[l][e]);
          B[e] = fma2(a[l][e], B[e], b[l][e]);
          A[e] = A[e] * a[l][e];
        }
      }
    }
    // inclusive prefixes over the warp's token lanes, then the exclusive one of this thread
#pragma unroll
    for (int o = TPR; o < 32; o <<= 1) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const F2 pa{__shfl_up_sync(0xffffffffu, A[e].v, o)}, pb{__shfl_up_sync(0xffffffffu, B[e].v, o)};
        if (lane >= o) { B[e] = fma2(A[e], pb, B[e]); A[e] = A[e] * pa; }
      }
    }
    if (lane >= 32 - TPR) {
      store8(&tot[buf][warp][0][cl], A);
      store8(&tot[buf][warp][1][cl], B);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const F2 pa{__shfl_up_sync(0xffffffffu, A[e].v, TPR)}, pb{__shfl_up_sync(0xffffffffu, B[e].v, TPR)};
      A[e] = lane >= TPR ? pa : f2(1.f);
      B[e] = lane >= TPR ? pb : f2(0.f);
    }
    __syncthreads();            // the other buffers are free again once every thread has passed the next chunk's barrier
    F2 S[4];
    load8(&carry[buf][cl], S);
    for (int w = 0; w < warp; ++w) {
      F2 wa[4], wb[4];
      load8(&tot[buf][w][0][cl], wa);
      load8(&tot[buf][w][1][cl], wb);
#pragma unroll
      for (int e = 0; e < 4; ++e) S[e] = fma2(wa[e], S[e], wb[e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) S[e] = fma2(A[e], S[e], B[e]);
    int block_end = p.block_tokens - 1 - (past + first) % p.block_tokens;      // the next token that ends a block
#pragma unroll
    for (int l = 0; l < kPer; ++l) {
      if (l < count) {
        __align__(16) T gr[8];
        F2 o[4];
        fetch(buf, 2, l, gr);
        load8_cut(gr, o);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[e] = fma2(a[l][e], S[e], b[l][e]);
          o[e] = gated_out(S[e], o[e]);
        }
        store8(op + (first + l) * p.ldo, o);
        if (l == block_end || first + l == n - 1) {
          float* row = state_row(p, table, past + first + l);
          if (row) store8(row + c, S);
          block_end += p.block_tokens;
        }
      }
    }
    if (tl == kLanes - 1) store8(&carry[buf ^ 1][cl], S);
  }
}

// One thread per 8 channels of a sequence's single new token, whose cache slot names the block that takes the state; only
// the first token of a block looks its predecessor's block up. slot < 0: a padding row, its output is zero.
template <typename T>
__global__ void gated_step_kernel(const ScanParams<T> p) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= p.W) return;
  const int slot = p.slots[s], pos = p.kv_lens[s] - 1;
  F2 z[4], u[4], o[4], S[4] = {};
  load8_cut(p.z + s * p.ld + c, z);                          // in flight together with the indices
  load8_cut(p.u + s * p.ld + c, u);
  load8_cut(p.g + s * p.ld + c, o);
  if (slot >= 0 && pos >= 0) {
    const int blk = slot / p.block_tokens;
    if (blk >= p.num_blocks) { guard_report(p.err, kGuardSlot, slot); return; }
    float* row = p.state + static_cast<long long>(blk) * p.block_stride + c;
    if (slot - blk * p.block_tokens > 0) {
      load8(row, S);
    } else if (pos > 0) {
      const float* before = state_row(p, p.block_table + static_cast<size_t>(s) * p.table_stride, pos - 1);
      if (before) load8(before + c, S);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      F2 a, b;
      gate_pair(z[e], u[e], f2(p.offset), a, b);
      S[e] = fma2(a, S[e], b);
      o[e] = gated_out(S[e], o[e]);
    }
    store8(row, S);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] = f2(0.f);
  }
  store8(p.out + s * p.ldo + c, o);
}

template <typename T, int TPR, int THREADS>
static int launch_tile(const ScanParams<T>& p, int B, cudaStream_t st) {
  constexpr int smem = 2 * kScanStage<T, THREADS>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(gated_scan_kernel<T, TPR, THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -3;
    set = true;
  }
  return launch_pdl(gated_scan_kernel<T, TPR, THREADS>, dim3((p.W + TPR * 8 - 1) / (TPR * 8), B), dim3(THREADS), smem, st, p) ==
                 cudaSuccess ? 0 : -4;
}
template <typename T>
static int launch_gated(const void* z, const void* u, const void* g, long long ld, void* out, long long ldo, float* state,
                        long long block_stride, int block_tokens, int num_blocks, const int* block_table, int table_stride,
                        const int* cu_q, const int* kv_lens, const int* slots, int B, int W, float offset, int* err,
                        cudaStream_t st) {
  ScanParams<T> p{};
  p.z = static_cast<const T*>(z); p.u = static_cast<const T*>(u); p.g = static_cast<const T*>(g); p.ld = ld;
  p.out = static_cast<T*>(out); p.ldo = ldo; p.state = state; p.block_stride = block_stride;
  p.block_tokens = block_tokens; p.num_blocks = num_blocks; p.block_table = block_table; p.table_stride = table_stride;
  p.cu_q = cu_q; p.kv_lens = kv_lens; p.slots = slots; p.W = W; p.offset = offset; p.err = err;
  cudaError_t e;
  if (slots) {
    const int vec = W / 8, threads = vec >= 128 ? 128 : (vec + 31) / 32 * 32;
    e = launch_pdl(gated_step_kernel<T>, dim3((vec + threads - 1) / threads, B), dim3(threads), 0, st, p);
  } else {
    // 32 channels per CTA where that fills the GPU two and a half times over, else 16, with few sequences over more threads
    const long long fill = 370, n = B;
    if (n * ((W + 31) / 32) >= fill) return launch_tile<T, 4, 128>(p, B, st);
    if (n * ((W + 15) / 16) >= fill) return launch_tile<T, 2, 128>(p, B, st);
    return launch_tile<T, 2, 256>(p, B, st);
  }
  return e == cudaSuccess ? 0 : -4;
}

}  // namespace ksana

using namespace ksana;

// z, u, g: columns of the projections' rows (ld elements apart), bf16 or (f32) fp32; out [rows, ldo]. slots given: every
// sequence has one row, with this cache slot. state: fp32 row of block 0 of the layer, block_stride floats between blocks.
extern "C" int ksana_gated_recurrence(const void* z, const void* u, const void* g, long long ld, void* out, long long ldo,
                                      float* state, long long block_stride, int block_tokens, int num_blocks,
                                      const int* block_table, int table_stride, const int* cu_q, const int* kv_lens,
                                      const int* slots, int B, int W, float offset, int f32, int* err, cudaStream_t st) {
  if (B <= 0) return 0;
  if (W <= 0 || W % 8 || ld % 8 || ldo % 8 || ldo < W || block_stride % 4 || block_tokens <= 0 || num_blocks <= 0 || B > 65535 ||
      (!slots && !cu_q))
    return -10;
  for (const void* q : {z, u, g, (const void*)out, (const void*)state})
    if (!aligned16(q)) return -11;
  return f32 ? launch_gated<float>(z, u, g, ld, out, ldo, state, block_stride, block_tokens, num_blocks, block_table, table_stride,
                                   cu_q, kv_lens, slots, B, W, offset, err, st)
             : launch_gated<bf16>(z, u, g, ld, out, ldo, state, block_stride, block_tokens, num_blocks, block_table, table_stride,
                                  cu_q, kv_lens, slots, B, W, offset, err, st);
}
