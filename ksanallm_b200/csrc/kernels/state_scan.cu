// Recurrent mixers whose state is a matrix per head, over the new tokens of a step. The state and everything that enters
// the recurrence besides projections and short convolutions is fp32. It lives in a slot per sequence:
//
//   matrix state  [heads][columns][keys] fp32 (transposed: the key dimension is contiguous)
//   ring          [taps][channels] of the activations' type: inputs of the short convolution, the one of position p in row
//                 p mod taps. A step of one token reads the rows before it and writes its own, so CTAs that share channels
//                 need no order among themselves
//
//   causal_conv     short convolution per channel (+ bias) and silu over several new tokens per sequence
//   state_space     S_t = exp(-A dt_t) S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t; dt = softplus(projection + bias); B
//                   and C belong to groups of heads
//   delta_rule      S' = diag(g_t) S_(t-1), u = beta_t (v_t - S'^T k_t), S_t = S' + k_t u^T, o_t = S_t^T q_t, with unit-length
//                   q (times dim^-1/2) and k per head, a decay g = exp(-A softplus(projection + bias)) per head and key channel
//                   and beta = sigmoid(projection)
//
// Both recurrences have a scan (several tokens per sequence, convolved inputs; in bf16 the tensor-core form of state_chunk.cu
// takes most sizes) and a step (one token per sequence, the convolution is part of it). Every column of a state is independent of
// the others: a CTA takes a slab of columns of one head, eight neighbouring lanes share a column and split its keys. Head and key
// sizes are multiples of 8 (padded with zeros). At position 0 the state is zero whatever the slot holds.
#include "f32x2.cuh"
#include "state_scan.cuh"

namespace ksana {

constexpr int kLanes = 8;                    // lanes that share a column
constexpr int kChunk = 16;                   // tokens staged at a time
constexpr int kCols = 2;                     // columns per thread in scans
constexpr int kScanThreads = 128;
constexpr int kSlab = kScanThreads / kLanes * kCols;
// silu(conv) of 8 channels of a single new token at position pos
template <typename T>
__device__ __forceinline__ void conv_one(const ConvRef<T>& v, const T* row, const T* ring, int pos, int c, float (&acc)[8]) {
  float f[8], w[8];
  load8(row + c, f);
  load8(v.w + static_cast<size_t>(v.taps - 1) * v.C + c, w);
  if (v.bias) load8(v.bias + c, acc);
#pragma unroll
  for (int e = 0; e < 8; ++e) acc[e] = fmaf(f[e], w[e], v.bias ? acc[e] : 0.f);
  for (int back = 1; back < v.taps && back <= pos; ++back) {
    load8(ring + static_cast<size_t>((pos - back) % v.taps) * v.C + c, f);
    load8(v.w + static_cast<size_t>(v.taps - 1 - back) * v.C + c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = fmaf(f[e], w[e], acc[e]);
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) acc[e] *= sigmoid_as<T>(acc[e]);
}

// ------------------------------------------------------------------------------------------------ convolution
// 4 consecutive elements as floats
__device__ __forceinline__ void load4(const bf16* p, float (&f)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void load4(const float* p, float (&f)[4]) { *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(bf16* p, const float (&f)[4]) {
  __nv_bfloat162 v[2] = {__floats2bfloat162_rn(f[0], f[1]), __floats2bfloat162_rn(f[2], f[3])};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(v);
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(f); }

// grid (channel tiles, row tiles, sequences); a thread walks the rows of its tile with 4 channels, the inputs before a row
// in registers (TAPS 0: any number of taps, reloaded).
constexpr int kConvRows = 16, kConvAhead = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) causal_conv_kernel(const ConvRef<T> v, const StateRef r, T* out, long long ldo, const int* cu_q) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, c = (blockIdx.x * blockDim.x + threadIdx.x) * 4, row0 = blockIdx.y * kConvRows;
  const int q0 = cu_q[s], n = cu_q[s + 1] - q0, past = r.kv_lens[s] - n;
  if (row0 >= n || c >= v.C) return;
  const int slot = slot_of(r, s);
  const T* ring = v.ring + static_cast<long long>(slot < 0 ? 0 : slot) * v.slot_stride + c;
  const T* x = v.x + static_cast<long long>(q0) * v.ld + c;
  auto input = [&](int t, float (&f)[4]) {             // of the row t (negative: from the ring, zero before the sequence)
    if (t >= 0) load4(x + t * v.ld, f);
    else if (past + t >= 0 && slot >= 0) load4(ring + static_cast<size_t>((past + t) % v.taps) * v.C, f);
    else f[0] = f[1] = f[2] = f[3] = 0.f;
  };
  float b[4] = {};
  if (v.bias) load4(v.bias + c, b);
  T* dst = out + static_cast<long long>(q0 + row0) * ldo + c;
  const int end = min(row0 + kConvRows, n);
  auto finish = [&](float (&acc)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[e] *= sigmoid_as<T>(acc[e]);
    store4(dst, acc);
    dst += ldo;
  };
  if constexpr (TAPS > 0) {
    float w[TAPS][4], hist[TAPS][4];                     // hist: the last TAPS inputs, the row's own last
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load4(v.w + static_cast<size_t>(j) * v.C + c, w[j]);
#pragma unroll
    for (int j = 1; j < TAPS; ++j) input(row0 - TAPS + j, hist[j]);
    for (int t = row0; t < end; t += kConvAhead) {
      float f[kConvAhead][4];                            // all loads of some rows before their stores
#pragma unroll
      for (int u = 0; u < kConvAhead; ++u) load4(x + min(t + u, n - 1) * v.ld, f[u]);
#pragma unroll
      for (int u = 0; u < kConvAhead; ++u) {
        if (t + u >= end) break;
        float acc[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
#pragma unroll
          for (int j = 0; j + 1 < TAPS; ++j) hist[j][e] = hist[j + 1][e];
          hist[TAPS - 1][e] = f[u][e];
          acc[e] = b[e];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(hist[j][e], w[j][e], acc[e]);
        }
        finish(acc);
      }
    }
  } else {
    for (int t = row0; t < end; ++t) {
      float acc[4] = {b[0], b[1], b[2], b[3]};
      for (int j = 0; j < v.taps; ++j) {
        float f[4], w[4];
        input(t - (v.taps - 1) + j, f);
        load4(v.w + static_cast<size_t>(j) * v.C + c, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(f[e], w[e], acc[e]);
      }
      finish(acc);
    }
  }
}

// ------------------------------------------------------------------------------------------------ columns of a state
// J float4 per thread and column: keys (j * 8 + lane) * 4 .. + 3, so eight lanes read 128 consecutive bytes.
template <int J>
__device__ __forceinline__ void load_column(const float* col, int keys, int lane, F2 (&S)[J][2]) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int k = (j * kLanes + lane) * 4;
    const ulonglong2 x = k < keys ? *reinterpret_cast<const ulonglong2*>(col + k) : make_ulonglong2(0, 0);
    S[j][0].v = x.x;
    S[j][1].v = x.y;
  }
}
template <int J>
__device__ __forceinline__ void store_column(float* col, int keys, int lane, const F2 (&S)[J][2]) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int k = (j * kLanes + lane) * 4;
    if (k < keys) *reinterpret_cast<ulonglong2*>(col + k) = make_ulonglong2(S[j][0].v, S[j][1].v);
  }
}
template <int J>
__device__ __forceinline__ void load_keys(const float* row, int lane, F2 (&f)[J][2]) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + (j * kLanes + lane) * 4);
    f[j][0].v = x.x;
    f[j][1].v = x.y;
  }
}
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = 1; o < kLanes; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ------------------------------------------------------------------------------------------------ state space
// One token for one column: decay, write, read-out (summed over this thread's keys)
template <int J>
__device__ __forceinline__ float space_token(F2 (&S)[J][2], const F2 (&B)[J][2], const F2 (&C)[J][2], F2 a, F2 dx) {
  F2 acc = f2(0.f);
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      S[j][i] = fma2(S[j][i], a, B[j][i] * dx);
      acc = fma2(S[j][i], C[j][i], acc);
    }
  }
  return sum2(acc);
}

// grid (slabs, H, sequences)
template <typename T, int J>
__global__ void __launch_bounds__(kScanThreads) space_scan_kernel(const SpaceParams<T> p) {
  pdl_trigger();
  pdl_wait();
  constexpr int KP = J * kLanes * 4;
  __shared__ __align__(16) float Bs[kChunk][KP], Cs[kChunk][KP];
  __shared__ float xs[kChunk][kSlab], ys[kChunk][kSlab], dts[kChunk], as[kChunk];
  const int s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * kSlab, np = min(kSlab, p.P - p0);
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.ref.kv_lens[s] - n;
  if (n <= 0) return;
  const int slot = slot_of(p.ref, s);
  if (slot < 0) return;
  const int lane = threadIdx.x & (kLanes - 1), tg = threadIdx.x / kLanes, g = h / (p.H / p.G);
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + static_cast<long long>(h) * p.P * p.N;
  F2 S[kCols][J][2];
#pragma unroll
  for (int c = 0; c < kCols; ++c) {
    const int col = tg + c * (kSlab / kCols);
    if (past > 0 && col < np) load_column<J>(state + static_cast<long long>(p0 + col) * p.N, p.N, lane, S[c]);
    else {
#pragma unroll
      for (int j = 0; j < J; ++j) S[c][j][0] = S[c][j][1] = f2(0.f);
    }
  }
  const float A = p.A[h], D = p.D[h], dtb = p.dt_bias[h];
  const T* crow = p.c + static_cast<long long>(q0) * p.ldc;
  const int xoff = h * p.P + p0, boff = p.H * p.P + g * p.N, coff = boff + p.G * p.N;
  for (int i = threadIdx.x; i < kChunk * KP; i += kScanThreads) (&Bs[0][0])[i] = (&Cs[0][0])[i] = 0.f;
  __syncthreads();
  for (int t0 = 0; t0 < n; t0 += kChunk) {
    const int m = min(kChunk, n - t0), nv = p.N >> 3, pv = np >> 3, per = 2 * nv + pv;
    for (int i = threadIdx.x; i < m * per; i += kScanThreads) {
      const int t = i / per, k = i % per;
      const T* row = crow + (t0 + t) * p.ldc;
      float f[8];
      float* dst = k < nv ? &Bs[t][k * 8] : k < 2 * nv ? &Cs[t][(k - nv) * 8] : &xs[t][(k - 2 * nv) * 8];
      load8(row + (k < nv ? boff + k * 8 : k < 2 * nv ? coff + (k - nv) * 8 : xoff + (k - 2 * nv) * 8), f);
#pragma unroll
      for (int e = 0; e < 8; ++e) dst[e] = f[e];
    }
    if (threadIdx.x < m) {
      const float dt = softplus_f(to_f(p.dt[static_cast<long long>(q0 + t0 + threadIdx.x) * p.ld_dt + h]) + dtb);
      dts[threadIdx.x] = dt;
      as[threadIdx.x] = decay_f(A * dt);
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < m; ++t) {
      F2 B[J][2], C[J][2];
      load_keys<J>(Bs[t], lane, B);
      load_keys<J>(Cs[t], lane, C);
      const F2 a = f2(as[t]);
#pragma unroll
      for (int c = 0; c < kCols; ++c) {
        const int col = tg + c * (kSlab / kCols);
        const float x = col < np ? xs[t][col] : 0.f;
        const float y = lanes_sum(space_token<J>(S[c], B, C, a, f2(dts[t] * x)));
        if (lane == 0) ys[t][col] = fmaf(D, x, y);
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < m * pv; i += kScanThreads) {
      const int t = i / pv, k = (i % pv) * 8;
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = ys[t][k + e];
      store8(p.y + static_cast<long long>(q0 + t0 + t) * p.ldy + xoff + k, f);
    }
  }
#pragma unroll
  for (int c = 0; c < kCols; ++c) {
    const int col = tg + c * (kSlab / kCols);
    if (col < np) store_column<J>(state + static_cast<long long>(p0 + col) * p.N, p.N, lane, S[c]);
  }
  space_ring(p, p.conv.x + static_cast<long long>(q0) * p.conv.ld, slot, past, n, h, p0, np, threadIdx.x, blockDim.x);
}

// One token per sequence: grid (slabs, H, sequences), blockDim = 8 lanes x columns of the slab (a multiple of 8).
template <typename T, int J>
__global__ void space_step_kernel(const SpaceParams<T> p) {
  pdl_trigger();
  pdl_wait();
  constexpr int KP = J * kLanes * 4;
  __shared__ __align__(16) float Bs[KP], Cs[KP], xs[32];
  __shared__ float step, decay;
  const int slab = blockDim.x / kLanes, s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * slab, np = min(slab, p.P - p0);
  const int slot = slot_of(p.ref, s), pos = p.ref.kv_lens[s] - 1;
  const int lane = threadIdx.x & (kLanes - 1), col = threadIdx.x / kLanes, g = h / (p.H / p.G);
  const int xoff = h * p.P + p0, boff = p.H * p.P + g * p.N, coff = boff + p.G * p.N;
  T* y = p.y + static_cast<long long>(s) * p.ldy + xoff;
  if (slot < 0 || pos < 0) {
    if (lane == 0 && col < np) y[col] = from_f<T>(0.f);
    return;
  }
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + (static_cast<long long>(h) * p.P + p0 + col) * p.N;
  F2 S[J][2];
  if (pos > 0 && col < np) load_column<J>(state, p.N, lane, S);
  else {
#pragma unroll
    for (int j = 0; j < J; ++j) S[j][0] = S[j][1] = f2(0.f);
  }
  const T* row = p.conv.x + static_cast<long long>(s) * p.conv.ld;
  const T* ring = p.conv.ring + static_cast<long long>(slot) * p.conv.slot_stride;
  const int nv = KP >> 3, rv = p.N >> 3, pv = np >> 3;
  for (int i = threadIdx.x; i < 2 * nv + pv; i += blockDim.x) {
    float f[8] = {};
    float* dst = i < nv ? Bs + i * 8 : i < 2 * nv ? Cs + (i - nv) * 8 : xs + (i - 2 * nv) * 8;
    const int k = i < nv ? i : i < 2 * nv ? i - nv : i - 2 * nv;
    if (i >= 2 * nv || k < rv) conv_one(p.conv, row, ring, pos, (i < nv ? boff : i < 2 * nv ? coff : xoff) + k * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) dst[e] = f[e];
  }
  if (threadIdx.x == blockDim.x - 1) {
    step = softplus_f(to_f(p.dt[static_cast<long long>(s) * p.ld_dt + h]) + p.dt_bias[h]);
    decay = decay_f(p.A[h] * step);
  }
  __syncthreads();
  F2 B[J][2], C[J][2];
  load_keys<J>(Bs, lane, B);
  load_keys<J>(Cs, lane, C);
  const float x = col < np ? xs[col] : 0.f;
  const float v = lanes_sum(space_token<J>(S, B, C, f2(decay), f2(step * x)));
  if (col < np) {
    store_column<J>(state, p.N, lane, S);
    if (lane == 0) y[col] = from_f<T>(fmaf(p.D[h], x, v));
  }
  space_ring(p, row, slot, pos, 1, h, p0, np, threadIdx.x, blockDim.x);
}

// ------------------------------------------------------------------------------------------------ delta rule
// One token for one column. qk = q . k
template <int J>
__device__ __forceinline__ float delta_token(F2 (&S)[J][2], const F2 (&q)[J][2], const F2 (&k)[J][2], const F2 (&g)[J][2], float qk,
                                             float v, float beta) {
  F2 kept = f2(0.f), seen = f2(0.f);
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      S[j][i] = S[j][i] * g[j][i];
      kept = fma2(S[j][i], k[j][i], kept);
      seen = fma2(S[j][i], q[j][i], seen);
    }
  }
  const float u = beta * (v - lanes_sum(sum2(kept))), o = fmaf(qk, u, lanes_sum(sum2(seen)));
  const F2 u2 = f2(u);
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < 2; ++i) S[j][i] = fma2(k[j][i], u2, S[j][i]);
  }
  return o;
}

// Unit vectors, their product, and decays of one token by one warp; rows in shared memory of KP floats (zeros behind K).
template <int KP, typename Load>
__device__ __forceinline__ void delta_operands(int K, float A, const float* decay_bias, float q_scale, Load load, float* qs, float* ks,
                                               float* gs, float* qk) {
  constexpr int E = KP / 32;
  const int lane = threadIdx.x & 31;
  float q[E], k[E], qq = 0.f, kk = 0.f, dot = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = lane + e * 32;
    float z = 0.f, b = 0.f;
    q[e] = k[e] = 0.f;
    if (i < K) { load(i, q[e], k[e], z); b = decay_bias[i]; }
    gs[i] = decay_f(A * softplus_f(z + b));
    qq = fmaf(q[e], q[e], qq);
    kk = fmaf(k[e], k[e], kk);
    dot = fmaf(q[e], k[e], dot);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    qq += __shfl_xor_sync(0xffffffffu, qq, o);
    kk += __shfl_xor_sync(0xffffffffu, kk, o);
    dot += __shfl_xor_sync(0xffffffffu, dot, o);
  }
  const float fq = q_scale / sqrtf(qq + kUnitEps), fk = 1.f / sqrtf(kk + kUnitEps);
#pragma unroll
  for (int e = 0; e < E; ++e) { qs[lane + e * 32] = q[e] * fq; ks[lane + e * 32] = k[e] * fk; }
  if (lane == 0) *qk = dot * fq * fk;
}

// grid (slabs, H, sequences)
template <typename T, int J>
__global__ void __launch_bounds__(kScanThreads) delta_scan_kernel(const DeltaParams<T> p) {
  pdl_trigger();
  pdl_wait();
  constexpr int KP = J * kLanes * 4, kTokens = J > 4 ? kChunk / 2 : kChunk;
  __shared__ __align__(16) float qs[kTokens][KP], ks[kTokens][KP], gs[kTokens][KP];
  __shared__ float vs[kTokens][kSlab], os[kTokens][kSlab], bs[kTokens], qks[kTokens];
  const int s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * kSlab, np = min(kSlab, p.V - p0);
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.ref.kv_lens[s] - n;
  if (n <= 0) return;
  const int slot = slot_of(p.ref, s);
  if (slot < 0) return;
  const int lane = threadIdx.x & (kLanes - 1), tg = threadIdx.x / kLanes, g = h / (p.H / p.G), warp = threadIdx.x >> 5;
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + static_cast<long long>(h) * p.V * p.K;
  F2 S[kCols][J][2];
#pragma unroll
  for (int c = 0; c < kCols; ++c) {
    const int col = tg + c * (kSlab / kCols);
    if (past > 0 && col < np) load_column<J>(state + static_cast<long long>(p0 + col) * p.K, p.K, lane, S[c]);
    else {
#pragma unroll
      for (int j = 0; j < J; ++j) S[c][j][0] = S[c][j][1] = f2(0.f);
    }
  }
  const float A = p.A[h];
  const int voff = 2 * p.G * p.K + h * p.V + p0, pv = np >> 3;
  for (int t0 = 0; t0 < n; t0 += kTokens) {
    const int m = min(kTokens, n - t0);
    for (int t = warp; t < m; t += kScanThreads / 32) {
      const T* row = p.c + static_cast<long long>(q0 + t0 + t) * p.ldc;
      const T* z = p.decay + static_cast<long long>(q0 + t0 + t) * p.ld_decay + h * p.K;
      delta_operands<KP>(p.K, A, p.decay_bias + h * p.K, p.q_scale, [&](int i, float& q, float& k, float& d) {
        q = to_f(row[g * p.K + i]);
        k = to_f(row[(p.G + g) * p.K + i]);
        d = to_f(z[i]);
      }, qs[t], ks[t], gs[t], &qks[t]);
    }
    for (int i = threadIdx.x; i < m * pv; i += kScanThreads) {
      const int t = i / pv, k = (i % pv) * 8;
      float f[8];
      load8(p.c + static_cast<long long>(q0 + t0 + t) * p.ldc + voff + k, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) vs[t][k + e] = f[e];
    }
    if (threadIdx.x < m) bs[threadIdx.x] = sigmoid_exact(to_f(p.beta[static_cast<long long>(q0 + t0 + threadIdx.x) * p.ld_beta + h]));
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      F2 q[J][2], k[J][2], d[J][2];
      load_keys<J>(qs[t], lane, q);
      load_keys<J>(ks[t], lane, k);
      load_keys<J>(gs[t], lane, d);
#pragma unroll
      for (int c = 0; c < kCols; ++c) {
        const int col = tg + c * (kSlab / kCols);
        const float o = delta_token<J>(S[c], q, k, d, qks[t], col < np ? vs[t][col] : 0.f, bs[t]);
        if (lane == 0) os[t][col] = o;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < m * pv; i += kScanThreads) {
      const int t = i / pv, k = (i % pv) * 8;
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = os[t][k + e];
      store8(p.o + static_cast<long long>(q0 + t0 + t) * p.ldo + h * p.V + p0 + k, f);
    }
  }
#pragma unroll
  for (int c = 0; c < kCols; ++c) {
    const int col = tg + c * (kSlab / kCols);
    if (col < np) store_column<J>(state + static_cast<long long>(p0 + col) * p.K, p.K, lane, S[c]);
  }
  delta_ring(p, p.conv.x + static_cast<long long>(q0) * p.conv.ld, slot, past, n, h, p0, np, threadIdx.x, blockDim.x);
}

// One token per sequence: grid (slabs, H, sequences), blockDim = 8 lanes x columns of the slab (a multiple of 8).
template <typename T, int J>
__global__ void delta_step_kernel(const DeltaParams<T> p) {
  pdl_trigger();
  pdl_wait();
  constexpr int KP = J * kLanes * 4;
  __shared__ __align__(16) float qs[KP], ks[KP], gs[KP], vs[32];
  const int slab = blockDim.x / kLanes, s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * slab, np = min(slab, p.V - p0);
  const int slot = slot_of(p.ref, s), pos = p.ref.kv_lens[s] - 1;
  const int lane = threadIdx.x & (kLanes - 1), col = threadIdx.x / kLanes, g = h / (p.H / p.G);
  T* o = p.o + static_cast<long long>(s) * p.ldo + h * p.V + p0;
  if (slot < 0 || pos < 0) {
    if (lane == 0 && col < np) o[col] = from_f<T>(0.f);
    return;
  }
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + (static_cast<long long>(h) * p.V + p0 + col) * p.K;
  F2 S[J][2];
  if (pos > 0 && col < np) load_column<J>(state, p.K, lane, S);
  else {
#pragma unroll
    for (int j = 0; j < J; ++j) S[j][0] = S[j][1] = f2(0.f);
  }
  const T* row = p.conv.x + static_cast<long long>(s) * p.conv.ld;
  const T* ring = p.conv.ring + static_cast<long long>(slot) * p.conv.slot_stride;
  const int kv = KP >> 3, rv = p.K >> 3, pv = np >> 3;
  for (int i = threadIdx.x; i < 2 * kv + pv; i += blockDim.x) {
    const int k = i < kv ? i : i < 2 * kv ? i - kv : i - 2 * kv;
    float f[8] = {};
    float* dst = i < kv ? qs + k * 8 : i < 2 * kv ? ks + k * 8 : vs + k * 8;
    if (i >= 2 * kv || k < rv)
      conv_one(p.conv, row, ring, pos, (i < kv ? g * p.K : i < 2 * kv ? (p.G + g) * p.K : 2 * p.G * p.K + h * p.V + p0) + k * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) dst[e] = f[e];
  }
  const float A = p.A[h];
  for (int i = blockDim.x - 1 - threadIdx.x; i < KP; i += blockDim.x)        // the other end of the CTA meanwhile
    gs[i] = i < p.K ? decay_f(A * softplus_f(to_f(p.decay[static_cast<long long>(s) * p.ld_decay + h * p.K + i]) + p.decay_bias[h * p.K + i])) : 1.f;
  const float beta = sigmoid_exact(to_f(p.beta[static_cast<long long>(s) * p.ld_beta + h]));
  __syncthreads();
  // lengths in every warp; the vectors stay as they are, their reciprocal lengths go into the sums
  float qq = 0.f, kk = 0.f, qk = 0.f;
  {
    const int l = threadIdx.x & 31;
#pragma unroll
    for (int e = 0; e < KP / 32; ++e) {
      const float a = qs[l + e * 32], b = ks[l + e * 32];
      qq = fmaf(a, a, qq);
      kk = fmaf(b, b, kk);
      qk = fmaf(a, b, qk);
    }
#pragma unroll
    for (int t = 16; t > 0; t >>= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, t);
      kk += __shfl_xor_sync(0xffffffffu, kk, t);
      qk += __shfl_xor_sync(0xffffffffu, qk, t);
    }
  }
  const float fq = p.q_scale / sqrtf(qq + kUnitEps), fk = 1.f / sqrtf(kk + kUnitEps);
  F2 q[J][2], k[J][2], d[J][2];
  load_keys<J>(qs, lane, q);
  load_keys<J>(ks, lane, k);
  load_keys<J>(gs, lane, d);
  F2 kept = f2(0.f), seen = f2(0.f);
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      S[j][i] = S[j][i] * d[j][i];
      kept = fma2(S[j][i], k[j][i], kept);
      seen = fma2(S[j][i], q[j][i], seen);
    }
  }
  const float u = beta * ((col < np ? vs[col] : 0.f) - fk * lanes_sum(sum2(kept))), v = fq * fmaf(qk * fk, u, lanes_sum(sum2(seen)));
  const F2 u2 = f2(u * fk);
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < 2; ++i) S[j][i] = fma2(k[j][i], u2, S[j][i]);
  }
  if (col < np) {
    store_column<J>(state, p.K, lane, S);
    if (lane == 0) o[col] = from_f<T>(v);
  }
  delta_ring(p, row, slot, pos, 1, h, p0, np, threadIdx.x, blockDim.x);
}

// ------------------------------------------------------------------------------------------------ host
static int launched(cudaError_t e) { return e == cudaSuccess ? 0 : -4; }
static int column_vectors(int keys) { const int j = (keys + 31) / 32; return j <= 1 ? 1 : j <= 2 ? 2 : j <= 4 ? 4 : j <= 8 ? 8 : 0; }
static int step_threads(int cols) { return (cols < 32 ? (cols + 7) / 8 * 8 : 32) * kLanes; }

template <typename T>
static int launch_conv(const ConvRef<T>& v, const StateRef& r, T* out, long long ldo, const int* cu_q, int B, int max_q, cudaStream_t st) {
  const int vec = v.C / 4, threads = vec < 256 ? (vec + 31) / 32 * 32 : 256;
  const dim3 grid((vec + threads - 1) / threads, (max_q + kConvRows - 1) / kConvRows, B);
  switch (v.taps) {
    case 1: return launched(launch_pdl(causal_conv_kernel<T, 1>, grid, dim3(threads), 0, st, v, r, out, ldo, cu_q));
    case 2: return launched(launch_pdl(causal_conv_kernel<T, 2>, grid, dim3(threads), 0, st, v, r, out, ldo, cu_q));
    case 3: return launched(launch_pdl(causal_conv_kernel<T, 3>, grid, dim3(threads), 0, st, v, r, out, ldo, cu_q));
    case 4: return launched(launch_pdl(causal_conv_kernel<T, 4>, grid, dim3(threads), 0, st, v, r, out, ldo, cu_q));
  }
  return launched(launch_pdl(causal_conv_kernel<T, 0>, grid, dim3(threads), 0, st, v, r, out, ldo, cu_q));
}

template <typename T, int J>
static int launch_space(const SpaceParams<T>& p, int B, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    const int rc = p.cu_q ? space_chunks(p, B, st) : -100;
    if (rc != -100) return rc;
  }
  if (p.cu_q) return launched(launch_pdl(space_scan_kernel<T, J>, dim3((p.P + kSlab - 1) / kSlab, p.H, B), dim3(kScanThreads), 0, st, p));
  const int threads = step_threads(p.P), slab = threads / kLanes;
  return launched(launch_pdl(space_step_kernel<T, J>, dim3((p.P + slab - 1) / slab, p.H, B), dim3(threads), 0, st, p));
}
template <typename T, int J>
static int launch_delta(const DeltaParams<T>& p, int B, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    const int rc = p.cu_q ? delta_chunks(p, B, st) : -100;
    if (rc != -100) return rc;
  }
  if (p.cu_q) return launched(launch_pdl(delta_scan_kernel<T, J>, dim3((p.V + kSlab - 1) / kSlab, p.H, B), dim3(kScanThreads), 0, st, p));
  const int threads = step_threads(p.V), slab = threads / kLanes;
  return launched(launch_pdl(delta_step_kernel<T, J>, dim3((p.V + slab - 1) / slab, p.H, B), dim3(threads), 0, st, p));
}

template <typename T>
static ConvRef<T> conv_ref(const void* x, long long ld, const void* w, const void* bias, void* ring, long long ring_stride, int taps, int C) {
  return {static_cast<const T*>(x), ld, static_cast<const T*>(w), static_cast<const T*>(bias), static_cast<T*>(ring), ring_stride, taps, C};
}

static bool bad_conv(const void* x, long long ld, const void* w, const void* bias, const void* ring, long long ring_stride, int taps, int C,
                     int f32) {
  return taps < 1 || taps > kMaxTaps || C <= 0 || C % 8 || ld % 8 || ring_stride % (f32 ? 4 : 8) || !aligned16(x) || !aligned16(w) ||
         !aligned16(bias) || !aligned16(ring);
}

}  // namespace ksana

using namespace ksana;

// x: raw rows (first channel), ld elements apart; w [taps][C], bias [C] or null; ring: [slots] of [taps][C], ring_stride
// elements between slots. Sequences of any number of new tokens. f32: everything fp32 instead of bf16.
extern "C" int ksana_causal_conv(const void* x, long long ld, const void* w, const void* bias, void* ring, long long ring_stride, int taps,
                                 int C, void* out, long long ldo, const int* cu_q, const int* kv_lens, const int* slots, int num_slots,
                                 int B, int max_q, int f32, int* err, cudaStream_t st) {
  if (B <= 0 || max_q <= 0) return 0;
  if (bad_conv(x, ld, w, bias, ring, ring_stride, taps, C, f32) || ldo % 8 || !aligned16(out) || B > 65535 || !cu_q) return -10;
  const StateRef r{slots, num_slots, kv_lens, err};
  return f32 ? launch_conv<float>(conv_ref<float>(x, ld, w, bias, ring, ring_stride, taps, C), r, static_cast<float*>(out), ldo, cu_q, B, max_q, st)
             : launch_conv<bf16>(conv_ref<bf16>(x, ld, w, bias, ring, ring_stride, taps, C), r, static_cast<bf16*>(out), ldo, cu_q, B, max_q, st);
}

// cu_q given: a scan over convolved rows c; null: one token per sequence, c is not read. state: fp32 [H][P][N] of slot 0.
extern "C" int ksana_state_space(const void* x, long long ld, const void* w, const void* bias, void* ring, long long ring_stride, int taps,
                                 const void* c, long long ldc, const void* dt, long long ld_dt, const float* dt_bias, const float* A,
                                 const float* D, void* y, long long ldy, float* state, long long slot_stride, const int* cu_q,
                                 const int* kv_lens, const int* slots, int num_slots, int B, int H, int G, int P, int N, int f32,
                                 int* err, cudaStream_t st) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || P <= 0 || N <= 0 || P % 8 || N % 8 || H > 65535 || B > 65535 || slot_stride % 4 || ldy % 8 || !aligned16(y) ||
      !aligned16(state) || (cu_q && (!c || ldc % 8 || !aligned16(c))) ||
      bad_conv(x, ld, w, bias, ring, ring_stride, taps, H * P + 2 * G * N, f32))
    return -10;
  auto run = [&](auto tag) {
    typedef decltype(tag) T;
    SpaceParams<T> p{};
    p.conv = conv_ref<T>(x, ld, w, bias, ring, ring_stride, taps, H * P + 2 * G * N);
    p.c = static_cast<const T*>(c); p.ldc = ldc; p.dt = static_cast<const T*>(dt); p.ld_dt = ld_dt;
    p.dt_bias = dt_bias; p.A = A; p.D = D; p.y = static_cast<T*>(y); p.ldy = ldy;
    p.state = state; p.slot_stride = slot_stride; p.ref = {slots, num_slots, kv_lens, err}; p.cu_q = cu_q;
    p.H = H; p.G = G; p.P = P; p.N = N;
    switch (column_vectors(N)) {
      case 1: return launch_space<T, 1>(p, B, st);
      case 2: return launch_space<T, 2>(p, B, st);
      case 4: return launch_space<T, 4>(p, B, st);
      case 8: return launch_space<T, 8>(p, B, st);
    }
    return -11;
  };
  return f32 ? run(0.f) : run(bf16());
}

// As above; state: fp32 [H][V][K] of slot 0.
extern "C" int ksana_delta_rule(const void* x, long long ld, const void* w, void* ring, long long ring_stride, int taps, const void* c,
                                long long ldc, const void* beta, long long ld_beta, const void* decay, long long ld_decay,
                                const float* decay_bias, const float* A, void* o, long long ldo, float* state, long long slot_stride,
                                const int* cu_q, const int* kv_lens, const int* slots, int num_slots, int B, int H, int G, int K, int V,
                                float q_scale, int f32, int* err, cudaStream_t st) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || K <= 0 || V <= 0 || K % 8 || V % 8 || H > 65535 || B > 65535 || slot_stride % 4 || ldo % 8 || !aligned16(o) ||
      !aligned16(state) || (cu_q && (!c || ldc % 8 || !aligned16(c))) ||
      bad_conv(x, ld, w, nullptr, ring, ring_stride, taps, 2 * G * K + H * V, f32))
    return -10;
  auto run = [&](auto tag) {
    typedef decltype(tag) T;
    DeltaParams<T> p{};
    p.conv = conv_ref<T>(x, ld, w, nullptr, ring, ring_stride, taps, 2 * G * K + H * V);
    p.c = static_cast<const T*>(c); p.ldc = ldc; p.beta = static_cast<const T*>(beta); p.ld_beta = ld_beta;
    p.decay = static_cast<const T*>(decay); p.ld_decay = ld_decay; p.decay_bias = decay_bias; p.A = A;
    p.o = static_cast<T*>(o); p.ldo = ldo; p.state = state; p.slot_stride = slot_stride; p.ref = {slots, num_slots, kv_lens, err};
    p.cu_q = cu_q; p.H = H; p.G = G; p.K = K; p.V = V; p.q_scale = q_scale;
    switch (column_vectors(K)) {
      case 1: return launch_delta<T, 1>(p, B, st);
      case 2: return launch_delta<T, 2>(p, B, st);
      case 4: return launch_delta<T, 4>(p, B, st);
      case 8: return launch_delta<T, 8>(p, B, st);
    }
    return -11;
  };
  return f32 ? run(0.f) : run(bf16());
}
