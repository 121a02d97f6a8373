// Scans of matrix-state recurrences (state_scan.cu has the equations) by chunks of tokens on the tensor cores: inside a chunk the
// recurrence is a product of small matrices, between chunks the state is carried in fp32 accumulators. Operands that are bf16
// anyway (convolved inputs) enter as they are; everything that belongs to the recurrence (states, decayed weights) is fp32 and enters
// a product as the sum of two bf16 numbers (16 bits of mantissa), accumulated in fp32.
//
// space_chunk_kernel: one CTA per (sequence, head, 64 columns), chunks of 64 tokens. With G_t = -A (dt_1 + .. + dt_t) in the chunk:
//   Y   = exp(G_t) C S + M X,  M_ts = (C_t . B_s) exp(G_t - G_s) dt_s for s <= t (+ D on the diagonal)
//   S  <- exp(G_L) S + sum_s exp(G_L - G_s) dt_s B_s x_s^T
// A warp owns 16 columns: its part of S stays in registers in the accumulator layout of the update (rows: columns of the state,
// columns: keys), which is the operand layout of C S. The weights M are computed by rows, 16 per warp, and shared.
//
// delta_chunk_kernel: one CTA per (sequence, head, 64 or 128 columns), chunks of 16 tokens. With P_t = g_1 .. g_t per key channel:
//   (I + A) U = beta (V - (k P) S),  A_ts = beta_t sum_c k_tc k_sc (g_(s+1) .. g_t)_c for s < t
//   O = (q P) S + Q U,  Q_ts likewise with q_t, for s <= t;   S <- P_L S + sum_s (k_s g_(s+1) .. g_L) u_s^T
// Decays enter as products of factors <= 1 only, never as quotients, so no decay is too strong. Three groups of four warps prepare the
// operands of the chunks in turn (unit vectors, decays, A and the inverse of I + A, Q) in a ring of four buffers; four warps apply
// them, each to 16 or 32 columns, whose state never leaves their registers.
#include "f32x2.cuh"
#include "state_scan.cuh"

namespace ksana {

__device__ __forceinline__ uint32_t sc_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void sc_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sc_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sc_copy16(uint32_t dst, const void* src, bool there) {     // zeros where nothing is there
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ uint32_t pair(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpair(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float log2_fast(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// a, b as the sum of two pairs of bf16
__device__ __forceinline__ void pair_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pair(a, b);
  const float2 h = unpair(hi);
  lo = pair(a - h.x, b - h.y);
}

// ------------------------------------------------------------------------------------------------ state space
constexpr int kSpaceTokens = 64, kSpaceCols = 64, kSpaceThreads = 128;
constexpr int kXPitch = (kSpaceCols + 8) * 2;            // bytes between rows of X and M: ldmatrix rows fall into different banks
template <int NK> constexpr int kBPitch = (NK * 16 + 8) * 2;
template <int NK> constexpr int kSpaceStage = kSpaceTokens * (2 * kBPitch<NK> + kXPitch);
template <int NK> constexpr int kSpaceSmem = 2 * kSpaceStage<NK> + 2 * kSpaceTokens * kXPitch + 8 * kSpaceTokens * 4;

// NK: steps of 16 keys. grid (column slabs, H, sequences)
template <int NK>
__global__ void __launch_bounds__(kSpaceThreads, 2) space_chunk_kernel(const SpaceParams<bf16> p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int PB = kBPitch<NK>, L = kSpaceTokens;
  uint8_t* mh = smem + 2 * kSpaceStage<NK>;
  uint8_t* ml = mh + L * kXPitch;
  float* scalars = reinterpret_cast<float*>(ml + L * kXPitch);  // per stage: G_t, dt_t, dt_s exp(G_L - G_s), exp(G_t)
  const int s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * kSpaceCols, np = min(kSpaceCols, p.P - p0);
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.ref.kv_lens[s] - n;
  if (n <= 0) return;
  const int slot = slot_of(p.ref, s);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (p.H / p.G);
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + (static_cast<long long>(h) * p.P + p0) * p.N;
  const bf16* rows = p.c + static_cast<long long>(q0) * p.ldc;
  const int xoff = h * p.P + p0, boff = p.H * p.P + g * p.N, coff = boff + p.G * p.N;
  const float A = p.A[h], D = p.D[h], dtb = p.dt_bias[h];

  float S[2 * NK][4];
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int col = warp * 16 + r4 + half * 8, key = j * 8 + c2;
      const float2 v = past > 0 && col < np && key < p.N ? *reinterpret_cast<const float2*>(state + static_cast<long long>(col) * p.N + key)
                                                         : make_float2(0.f, 0.f);
      S[j][2 * half] = v.x;
      S[j][2 * half + 1] = v.y;
    }
  }
  auto stage = [&](int buf) { return smem + buf * kSpaceStage<NK>; };
  auto issue = [&](int t0, int buf) {
    // a thread has one 16-byte piece of every STEP-th row of B and C, and one of every 16th row of X
    constexpr int V = NK * 2, STEP = kSpaceThreads / V, XV = kSpaceCols / 8, XSTEP = kSpaceThreads / XV;
    const uint32_t b = sc_addr(stage(buf));
    {
      const int v = threadIdx.x % V, t = threadIdx.x / V;
      const bool in = v * 8 < p.N;
      const bf16* src = rows + static_cast<long long>(t0 + t) * p.ldc + (in ? v * 8 : 0);
      const uint32_t dst = b + t * PB + v * 16;
#pragma unroll
      for (int i = 0; i < (L + STEP - 1) / STEP; ++i) {
        const bool there = in && t0 + t + i * STEP < n;
        const bf16* at = there ? src + i * STEP * p.ldc : rows;
        if (L % STEP == 0 || t + i * STEP < L) {
          sc_copy16(dst + i * STEP * PB, at + (there ? boff : 0), there);
          sc_copy16(dst + L * PB + i * STEP * PB, at + (there ? coff : 0), there);
        }
      }
    }
    {
      const int v = threadIdx.x % XV, t = threadIdx.x / XV;
      const bool in = v * 8 < np;
      const bf16* src = rows + static_cast<long long>(t0 + t) * p.ldc + xoff + (in ? v * 8 : 0);
      const uint32_t dst = b + 2 * L * PB + t * kXPitch + v * 16;
#pragma unroll
      for (int i = 0; i < L / XSTEP; ++i) {
        const bool there = in && t0 + t + i * XSTEP < n;
        sc_copy16(dst + i * XSTEP * kXPitch, there ? src + i * XSTEP * p.ldc : rows, there);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto raw_dt = [&](int t) { return t < n ? to_f(p.dt[static_cast<long long>(q0 + t) * p.ld_dt + h]) : 0.f; };
  float d0 = 0.f, d1 = 0.f;
  // step sizes of the chunk at t0 (raw ones in d0, d1), their running sums, decays; then the raw ones of the chunk behind it
  auto decays = [&](int t0, float* out) {
    const float a = t0 + 2 * lane < n ? softplus_f(d0 + dtb) : 0.f, b = t0 + 2 * lane + 1 < n ? softplus_f(d1 + dtb) : 0.f;
    float sum = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    const float total = __shfl_sync(0xffffffffu, sum, 31), g1 = -A * sum, g0 = -A * (sum - b), gl = -A * total;
    *reinterpret_cast<float2*>(out + 2 * lane) = make_float2(g0, g1);
    *reinterpret_cast<float2*>(out + L + 2 * lane) = make_float2(a, b);
    *reinterpret_cast<float2*>(out + 2 * L + 2 * lane) = make_float2(a * expf(gl - g0), b * expf(gl - g1));
    *reinterpret_cast<float2*>(out + 3 * L + 2 * lane) = make_float2(expf(g0), expf(g1));
    d0 = raw_dt(t0 + L + 2 * lane);
    d1 = raw_dt(t0 + L + 2 * lane + 1);
  };
  issue(0, 0);
  if (warp == 0) {
    d0 = raw_dt(2 * lane);
    d1 = raw_dt(2 * lane + 1);
    decays(0, scalars);
  }
  for (int t0 = 0, buf = 0; t0 < n; t0 += L, buf ^= 1) {
    if (t0 + L < n) issue(t0 + L, buf ^ 1);
    else asm volatile("cp.async.commit_group;" ::: "memory");
    const float *cum = scalars + buf * 4 * L, *dts = cum + L, *wend = dts + L, *edec = wend + L;
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t bs = sc_addr(stage(buf)), cs = bs + L * PB, xs = bs + 2 * L * PB;
    // M, rows 16 * warp ..
    {
      float acc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t a[4];
        sc_ldsm(a, cs + (warp * 16 + (lane & 15)) * PB + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int jp = 0; jp < 4; ++jp) {
          if (jp > warp) break;
          uint32_t b[4];
          sc_ldsm(b, bs + (jp * 16 + (lane & 7) + ((lane >> 4) << 3)) * PB + kk * 32 + ((lane >> 3) & 1) * 16);
          sc_mma(acc[2 * jp], a, b[0], b[1]);
          sc_mma(acc[2 * jp + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = warp * 16 + r4 + half * 8;
        const float gt = cum[t];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (j > 2 * warp + 1) break;
          float v[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int u = j * 8 + c2 + e;
            v[e] = u <= t ? acc[j][2 * half + e] * exp2_fast((gt - cum[u]) * 1.44269504f) * dts[u] : 0.f;
            if (u == t) v[e] += D;
          }
          uint32_t hi, lo;
          pair_split(v[0], v[1], hi, lo);
          *reinterpret_cast<uint32_t*>(mh + t * kXPitch + (j * 8 + c2) * 2) = hi;
          *reinterpret_cast<uint32_t*>(ml + t * kXPitch + (j * 8 + c2) * 2) = lo;
        }
      }
    }
    if (warp == 0 && t0 + L < n) decays(t0 + L, scalars + (buf ^ 1) * 4 * L);      // this warp had the fewest weights
    // the state as an operand
    uint32_t sh[2 * NK][2], sl[2 * NK][2];
#pragma unroll
    for (int j = 0; j < 2 * NK; ++j) {
      pair_split(S[j][0], S[j][1], sh[j][0], sl[j][0]);
      pair_split(S[j][2], S[j][3], sh[j][1], sl[j][1]);
    }
    uint32_t x[4][4];                                    // X: 16 tokens x this warp's 16 columns each
#pragma unroll
    for (int k = 0; k < 4; ++k) sc_ldsm_t(x[k], xs + (k * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * kXPitch + (warp * 2 + (lane >> 4)) * 16);
    __syncthreads();
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      float y[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t a[4];
        sc_ldsm(a, cs + (m * 16 + (lane & 15)) * PB + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          sc_mma(y[c], a, sh[2 * kk][c], sh[2 * kk + 1][c]);
          sc_mma(y[c], a, sl[2 * kk][c], sl[2 * kk + 1][c]);
        }
      }
      const float e0 = edec[m * 16 + r4], e1 = edec[m * 16 + r4 + 8];
#pragma unroll
      for (int c = 0; c < 2; ++c) { y[c][0] *= e0; y[c][1] *= e0; y[c][2] *= e1; y[c][3] *= e1; }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k > m) break;
        uint32_t a[4], b[4];
        const uint32_t at = (m * 16 + (lane & 15)) * kXPitch + k * 32 + (lane >> 4) * 16;
        sc_ldsm(a, sc_addr(mh) + at);
        sc_ldsm(b, sc_addr(ml) + at);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          sc_mma(y[c], a, x[k][2 * c], x[k][2 * c + 1]);
          sc_mma(y[c], b, x[k][2 * c], x[k][2 * c + 1]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = t0 + m * 16 + r4 + half * 8;
        if (t >= n) continue;
        bf16* dst = p.y + static_cast<long long>(q0 + t) * p.ldy + xoff;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int col = warp * 16 + c * 8 + c2;
          if (col < np) *reinterpret_cast<uint32_t*>(dst + col) = pair(y[c][2 * half], y[c][2 * half + 1]);
        }
      }
    }
    // the state after the chunk
    const float el = edec[L - 1];
#pragma unroll
    for (int j = 0; j < 2 * NK; ++j) { S[j][0] *= el; S[j][1] *= el; S[j][2] *= el; S[j][3] *= el; }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 w0 = *reinterpret_cast<const float2*>(wend + k * 16 + c2), w1 = *reinterpret_cast<const float2*>(wend + k * 16 + 8 + c2);
      uint32_t ah[4], al[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        // operand order: (columns 0-7, tokens 0-7), (columns 8-15, tokens 0-7), (columns 0-7, tokens 8-15), the rest
        const float2 v = unpair(x[k][(i & 1) * 2 + (i >> 1)]), w = i < 2 ? w0 : w1;
        pair_split(v.x * w.x, v.y * w.y, ah[i], al[i]);
      }
#pragma unroll
      for (int j = 0; j < NK; ++j) {
        uint32_t b[4];
        sc_ldsm_t(b, bs + (k * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * PB + (j * 2 + (lane >> 4)) * 16);
        sc_mma(S[2 * j], ah, b[0], b[1]);
        sc_mma(S[2 * j], al, b[0], b[1]);
        sc_mma(S[2 * j + 1], ah, b[2], b[3]);
        sc_mma(S[2 * j + 1], al, b[2], b[3]);
      }
    }
    __syncthreads();                                     // the stage, M and the decays may be overwritten
  }
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int col = warp * 16 + r4 + half * 8, key = j * 8 + c2;
      if (col < np && key < p.N)
        *reinterpret_cast<float2*>(state + static_cast<long long>(col) * p.N + key) = make_float2(S[j][2 * half], S[j][2 * half + 1]);
    }
  }
  space_ring(p, p.conv.x + static_cast<long long>(q0) * p.conv.ld, slot, past, n, h, p0, np, threadIdx.x, blockDim.x);
}

template <int NK>
static int launch_space_chunks(const SpaceParams<bf16>& p, int B, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(space_chunk_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSpaceSmem<NK>) != cudaSuccess) return -3;
    set = true;
  }
  return launch_pdl(space_chunk_kernel<NK>, dim3((p.P + kSpaceCols - 1) / kSpaceCols, p.H, B), dim3(kSpaceThreads), kSpaceSmem<NK>, st, p) ==
                 cudaSuccess ? 0 : -4;
}

int space_chunks(const SpaceParams<bf16>& p, int B, cudaStream_t st) {
  const int steps = (p.N + 15) / 16;
  if (steps > 8 || p.ldc % 8 || !aligned16(p.c) || p.ldy % 2) return -100;
  if (steps <= 1) return launch_space_chunks<1>(p, B, st);
  if (steps <= 2) return launch_space_chunks<2>(p, B, st);
  if (steps <= 4) return launch_space_chunks<4>(p, B, st);
  return launch_space_chunks<8>(p, B, st);
}

// ------------------------------------------------------------------------------------------------ delta rule
constexpr int kDeltaTokens = 16, kDeltaGroups = 3, kDeltaBuffers = 4, kDeltaThreads = 128 * (1 + kDeltaGroups);
constexpr int kMPitch = (kDeltaTokens + 8) * 2;
// NK: steps of 16 keys, CT: 16-column tiles per warp that applies
template <int NK, int CT> struct DeltaSmem {
  static constexpr int KP = NK * 16, cols = 64 * CT, pitch = (KP + 8) * 2, rows = kDeltaTokens * pitch, vpitch = (cols + 8) * 2, fpitch = KP + 4;
  // operands of one chunk
  static constexpr int kt = 0, qt = 2 * rows, kh = 4 * rows, inv = 6 * rows, qk = inv + 2 * kDeltaTokens * kMPitch,
                       v = qk + 2 * kDeltaTokens * kMPitch, beta = v + kDeltaTokens * vpitch, total = beta + kDeltaTokens * 4,
                       operands = total + KP * 4;
  // what a preparing group works on: raw rows (q, k, decay), decays, A, reciprocal lengths
  static constexpr int raw = 3 * kDeltaTokens * KP * 2,
                       work = raw + (kDeltaTokens * fpitch + kDeltaTokens * (kDeltaTokens + 4) + 2 * kDeltaTokens) * 4;
  static constexpr int out = kDeltaBuffers * operands + kDeltaGroups * work, bytes = out + kDeltaTokens * vpitch;
};

__device__ __forceinline__ void sc_stsm_t(uint32_t addr, const uint32_t (&r)[4]) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3])
               : "memory");
}
// barriers: 1 the applying warps, 2 .. the preparing groups, then per buffer "full" and "empty" (a group and the applying warps)
constexpr int kBarGroup = 2, kBarFull = kBarGroup + kDeltaGroups, kBarEmpty = kBarFull + kDeltaBuffers;
__device__ __forceinline__ void bar_wait(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void bar_signal(int id, int threads) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
template <int N> __device__ __forceinline__ void registers_up() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(N)); }
template <int N> __device__ __forceinline__ void registers_down() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(N)); }
template <int CT> constexpr int kApplyRegs = CT == 1 ? 200 : 248;       // 128 * these + 384 * the others = 512 * 128, the launch's
template <int CT> constexpr int kPrepareRegs = CT == 1 ? 104 : 88;
constexpr int kLaunchRegs = 128;
static_assert(128 * kApplyRegs<1> + 384 * kPrepareRegs<1> <= kDeltaThreads * kLaunchRegs, "register split");
static_assert(128 * kApplyRegs<2> + 384 * kPrepareRegs<2> <= kDeltaThreads * kLaunchRegs, "register split");
__device__ __forceinline__ void put_split(uint8_t* hi, uint8_t* lo, float v) {
  const bf16 h = __float2bfloat16(v);
  *reinterpret_cast<bf16*>(hi) = h;
  *reinterpret_cast<bf16*>(lo) = __float2bfloat16(v - __bfloat162float(h));
}
__device__ __forceinline__ F2 wide2(uint32_t v) { return f2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }    // two bf16
// accumulators of two 8-column tiles as a 16 x 16 operand
__device__ __forceinline__ void operand_split(const float (&t0)[4], const float (&t1)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  pair_split(t0[0], t0[1], hi[0], lo[0]);
  pair_split(t0[2], t0[3], hi[1], lo[1]);
  pair_split(t1[0], t1[1], hi[2], lo[2]);
  pair_split(t1[2], t1[3], hi[3], lo[3]);
}
// c += a b with both operands as sums of two bf16 (the product of the small parts is left out)
__device__ __forceinline__ void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1,
                                          uint32_t bl0, uint32_t bl1) {
  sc_mma(c, ah, bh0, bh1);
  sc_mma(c, al, bh0, bh1);
  sc_mma(c, ah, bl0, bl1);
}

// One chunk's operands from its raw rows, by a group of 128 threads (tid 0 .. 127); m of its 16 tokens exist.
template <int NK, int CT>
__device__ __forceinline__ void delta_prepare(const DeltaParams<bf16>& p, uint8_t* op, uint8_t* work, int tid, int group, int m, float A,
                                              float bias, const bf16* beta) {
  typedef DeltaSmem<NK, CT> Sm;
  constexpr int KP = Sm::KP, T = kDeltaTokens, FP = Sm::fpitch;
  const int warp = tid >> 5, lane = tid & 31, bar = kBarGroup + group;
  const bf16* rq = reinterpret_cast<const bf16*>(work);
  const bf16* rk = rq + T * KP;
  const bf16* rz = rk + T * KP;
  float* gf = reinterpret_cast<float*>(work + Sm::raw);
  float* am = gf + T * FP;                       // A, [T][T + 4]
  float* iq = am + T * (T + 4);                  // reciprocal lengths
  float* ik = iq + T;
  float* bt = reinterpret_cast<float*>(op + Sm::beta);
  // lengths: four tokens per warp, eight lanes per token
  {
    const int t = warp * 4 + (lane >> 3);
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int c = (lane & 7) * 2; c < KP; c += 16) {
      const float2 q = unpair(*reinterpret_cast<const uint32_t*>(rq + t * KP + c)), k = unpair(*reinterpret_cast<const uint32_t*>(rk + t * KP + c));
      qq = fmaf(q.x, q.x, fmaf(q.y, q.y, qq));
      kk = fmaf(k.x, k.x, fmaf(k.y, k.y, kk));
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
    }
    if ((lane & 7) == 0) {
      iq[t] = p.q_scale * rsqrtf(qq + kUnitEps);
      ik[t] = rsqrtf(kk + kUnitEps);
      bt[t] = t < m ? sigmoid_exact(to_f(beta[static_cast<long long>(t) * p.ld_beta])) : 0.f;
    }
  }
  bar_wait(bar, 128);
  if (tid < KP) {                                // one key channel per thread
    const int c = tid;
    float g[T], P = 1.f;
#pragma unroll
    for (int t = 0; t < T; ++t) {
      // exp(-A softplus(z)) = 2^(-A log2(1 + e^z))
      const float z = (to_f(rz[t * KP + c]) + bias) * 1.44269504f;
      g[t] = t < m && c < p.K ? exp2_fast(-A * (z > 30.f ? z : log2_fast(1.f + exp2_fast(z)))) : 1.f;
      gf[t * FP + ((c >> 2) & 1) * (KP / 2) + (c >> 3) * 4 + (c & 3)] = g[t];       // halves of the pieces of 8 apart
    }
#pragma unroll
    for (int t = 0; t < T; ++t) {
      P *= g[t];
      uint8_t* at = op + t * Sm::pitch + c * 2;
      put_split(at + Sm::kt, at + Sm::kt + Sm::rows, to_f(rk[t * KP + c]) * ik[t] * P);
      put_split(at + Sm::qt, at + Sm::qt + Sm::rows, to_f(rq[t * KP + c]) * iq[t] * P);
    }
    reinterpret_cast<float*>(op + Sm::total)[c] = P;
    P = 1.f;
#pragma unroll
    for (int t = T - 1; t >= 0; --t) {
      uint8_t* at = op + Sm::kh + t * Sm::pitch + c * 2;
      put_split(at, at + Sm::rows, to_f(rk[t * KP + c]) * ik[t] * P);
      P *= g[t];
    }
  }
  bar_wait(bar, 128);
  // A and Q by columns s, four per warp: eight lanes share a column, each with pieces of 8 key channels; lengths enter at the end.
  // Columns with more rows go to another warp in every group
  {
    constexpr int PIECES = KP >= 64 ? KP / 64 : 1;
    const int block = (warp + group) & 3, l = lane & 7, s = block * 4 + (lane >> 3);
    float v[2 * T];
    F2 d[PIECES][4];
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
#pragma unroll
      for (int e = 0; e < 4; ++e) d[i][e] = f2(0.f);
    }
#pragma unroll
    for (int t = 0; t < T; ++t) {
      v[t] = v[T + t] = 0.f;
      if (t < block * 4) continue;
      const F2 first = f2(t == s ? 1.f : 0.f);
      F2 kk = f2(0.f), qk = f2(0.f);
#pragma unroll
      for (int i = 0; i < PIECES; ++i) {
        const int piece = l + 8 * i;
        if (KP < 64 && piece * 8 >= KP) break;
        const uint4 kr = *reinterpret_cast<const uint4*>(rk + t * KP + piece * 8), qr = *reinterpret_cast<const uint4*>(rq + t * KP + piece * 8);
        const ulonglong2 g0 = *reinterpret_cast<const ulonglong2*>(gf + t * FP + piece * 4),
                         g1 = *reinterpret_cast<const ulonglong2*>(gf + t * FP + KP / 2 + piece * 4);
        const uint32_t kw[4] = {kr.x, kr.y, kr.z, kr.w}, qw[4] = {qr.x, qr.y, qr.z, qr.w};
        const unsigned long long gw[4] = {g0.x, g0.y, g1.x, g1.y};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const F2 k = wide2(kw[e]);
          d[i][e] = fma2(k, first, d[i][e] * F2{gw[e]});
          kk = fma2(d[i][e], k, kk);
          qk = fma2(d[i][e], wide2(qw[e]), qk);
        }
      }
      v[t] = sum2(kk);
      v[T + t] = sum2(qk);
    }
    // sums over the eight lanes; each keeps four entries
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
#pragma unroll
      for (int j = 0; j < 4 * o; ++j) {
        const bool up = l & o;
        const float send = up ? v[j] : v[j + 4 * o], keep = up ? v[j + 4 * o] : v[j];
        v[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    const float mine = ik[s];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = (l & 3) * 4 + j;
      if (l < 4) am[t * (T + 4) + s] = t > s ? bt[t] * ik[t] * mine * v[j] : 0.f;
      else {
        uint8_t* at = op + Sm::qk + t * kMPitch + s * 2;
        put_split(at, at + T * kMPitch, t >= s ? iq[t] * mine * v[j] : 0.f);
      }
    }
  }
  bar_wait(bar, 128);
  if (warp == ((group + 1) & 3) && lane < T) {   // column `lane` of the inverse of I + A
    float x[T];
#pragma unroll
    for (int t = 0; t < T; ++t) {
      float a = t == lane ? 1.f : 0.f, b = 0.f;
#pragma unroll
      for (int s4 = 0; s4 < t; s4 += 4) {
        const float4 r = *reinterpret_cast<const float4*>(am + t * (T + 4) + s4);
        a = fmaf(-r.x, x[s4], a);
        if (s4 + 1 < t) b = fmaf(-r.y, x[s4 + 1], b);
        if (s4 + 2 < t) a = fmaf(-r.z, x[s4 + 2], a);
        if (s4 + 3 < t) b = fmaf(-r.w, x[s4 + 3], b);
      }
      x[t] = a + b;
      uint8_t* at = op + Sm::inv + t * kMPitch + lane * 2;
      put_split(at, at + T * kMPitch, x[t]);
    }
  }
}

// grid (column slabs, H, sequences); warps 0 - 3 apply, the others prepare: group r the chunks r, r + 3, ..
template <int NK, int CT>
__global__ void __launch_bounds__(kDeltaThreads, 1) delta_chunk_kernel(const DeltaParams<bf16> p) {
  pdl_trigger();
  pdl_wait();
  typedef DeltaSmem<NK, CT> Sm;
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int KP = Sm::KP, T = kDeltaTokens, NB = kDeltaBuffers;
  const int s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * Sm::cols, np = min(Sm::cols, p.V - p0);
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.ref.kv_lens[s] - n;
  if (n <= 0) return;
  const int slot = slot_of(p.ref, s);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (p.H / p.G), chunks = (n + T - 1) / T;
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + (static_cast<long long>(h) * p.V + p0) * p.K;
  const bf16* rows = p.c + static_cast<long long>(q0) * p.ldc;
  if (warp >= 4) {
    registers_down<kPrepareRegs<CT>>();
    const int group = (warp >> 2) - 1, tid = threadIdx.x & 127;
    uint8_t* work = smem + NB * Sm::operands + group * Sm::work;
    const float A = p.A[h], bias = tid < p.K ? p.decay_bias[h * p.K + tid] : 0.f;
    const bf16* z = p.decay + static_cast<long long>(q0) * p.ld_decay + h * p.K;
    const bf16* beta = p.beta + static_cast<long long>(q0) * p.ld_beta + h;
    // a thread copies one 16-byte piece of some rows
    constexpr int V = KP / 8, STEP = 128 / V, VV = Sm::cols / 8, VSTEP = 128 / VV;
    auto fetch = [&](int i) {                    // raw rows of chunk i
      const int c = tid % V * 8;
      const bool in = c < p.K;
#pragma unroll
      for (int j = 0; j < (T + STEP - 1) / STEP; ++j) {
        const int t = tid / V + j * STEP, row = i * T + t;
        if (STEP > T && t >= T) break;
        const bool there = in && row < n;
        const long long r = there ? row : 0;
        const uint32_t dst = sc_addr(work) + (t * KP + c) * 2;
        const bf16* src = rows + r * p.ldc + (there ? g * p.K + c : 0);
        sc_copy16(dst, src, there);
        sc_copy16(dst + T * KP * 2, src + (there ? p.G * p.K : 0), there);
        sc_copy16(dst + 2 * T * KP * 2, z + r * p.ld_decay + (there ? c : 0), there);
      }
    };
    auto fetch_v = [&](int i, uint8_t* op) {
      const int c = tid % VV * 8;
#pragma unroll
      for (int j = 0; j < T / VSTEP; ++j) {
        const int t = tid / VV + j * VSTEP, row = i * T + t;
        const bool there = row < n && c < np;
        sc_copy16(sc_addr(op + Sm::v) + t * Sm::vpitch + c * 2,
                  rows + static_cast<long long>(there ? row : 0) * p.ldc + (there ? 2 * p.G * p.K + h * p.V + p0 + c : 0), there);
      }
    };
    auto landed = [&]() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory"); };
    if (group < chunks) fetch(group);
    for (int i = group; i < chunks; i += kDeltaGroups) {
      uint8_t* op = smem + (i % NB) * Sm::operands;
      landed();
      if (i >= NB) bar_wait(kBarEmpty + i % NB, 256);
      bar_wait(kBarGroup + group, 128);          // every thread's raw rows are here
      fetch_v(i, op);
      delta_prepare<NK, CT>(p, op, work, tid, group, min(T, n - i * T), A, bias, beta + static_cast<long long>(i * T) * p.ld_beta);
      landed();
      bar_signal(kBarFull + i % NB, 256);
      // the group's last barrier inside lies behind the last read of its raw rows
      if (i + kDeltaGroups < chunks) fetch(i + kDeltaGroups);
    }
    if (group == 0) delta_ring(p, p.conv.x + static_cast<long long>(q0) * p.conv.ld, slot, past, n, h, p0, np, tid, 128);
    return;
  }
  registers_up<kApplyRegs<CT>>();
  float S[CT][2 * NK][4];
#pragma unroll
  for (int ct = 0; ct < CT; ++ct) {
#pragma unroll
    for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int col = (warp * CT + ct) * 16 + r4 + half * 8, key = j * 8 + c2;
        const float2 v = past > 0 && col < np && key < p.K ? *reinterpret_cast<const float2*>(state + static_cast<long long>(col) * p.K + key)
                                                           : make_float2(0.f, 0.f);
        S[ct][j][2 * half] = v.x;
        S[ct][j][2 * half + 1] = v.y;
      }
    }
  }
  const uint32_t out = sc_addr(smem + Sm::out);
  const uint32_t flat = ((lane & 7) + ((lane >> 4) << 3)), side = ((lane >> 3) & 1) * 16;        // 16 rows x 16 columns, rows as columns of B
  const uint32_t across = (lane & 7) + (((lane >> 3) & 1) << 3), part = lane >> 4;               // transposed reads
  for (int i = 0; i < chunks; ++i) {
    const uint8_t* op = smem + (i % NB) * Sm::operands;
    const uint32_t ob = sc_addr(op);
    bar_wait(kBarFull + i % NB, 256);
    float w[CT][2][4] = {}, o[CT][2][4] = {};
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t bh[4], bl[4], dh[4], dl[4];
      const uint32_t at = ob + flat * Sm::pitch + kk * 32 + side;
      sc_ldsm(bh, at + Sm::kt);
      sc_ldsm(bl, at + Sm::kt + Sm::rows);
      sc_ldsm(dh, at + Sm::qt);
      sc_ldsm(dl, at + Sm::qt + Sm::rows);
#pragma unroll
      for (int ct = 0; ct < CT; ++ct) {
        uint32_t ah[4], al[4];
        operand_split(S[ct][2 * kk], S[ct][2 * kk + 1], ah, al);
        mma_split(w[ct][0], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_split(w[ct][1], ah, al, bh[2], bh[3], bl[2], bl[3]);
        mma_split(o[ct][0], ah, al, dh[0], dh[1], dl[0], dl[1]);
        mma_split(o[ct][1], ah, al, dh[2], dh[3], dl[2], dl[3]);
      }
    }
    const float* bt = reinterpret_cast<const float*>(op + Sm::beta);
    const uint32_t mat = ob + flat * kMPitch + side;
    uint32_t uh[CT][4], ul[CT][4];
#pragma unroll
    for (int ct = 0; ct < CT; ++ct) {
      uint32_t v[4];                             // (tokens 0-7, columns 0-7), (tokens 8-15, columns 0-7), then columns 8-15
      sc_ldsm_t(v, ob + Sm::v + across * Sm::vpitch + ((warp * CT + ct) * 2 + part) * 16);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float2 b = *reinterpret_cast<const float2*>(bt + j * 8 + c2), v0 = unpair(v[j]), v1 = unpair(v[2 + j]);
        w[ct][j][0] = b.x * (v0.x - w[ct][j][0]);
        w[ct][j][1] = b.y * (v0.y - w[ct][j][1]);
        w[ct][j][2] = b.x * (v1.x - w[ct][j][2]);
        w[ct][j][3] = b.y * (v1.y - w[ct][j][3]);
      }
      uint32_t ah[4], al[4], bh[4], bl[4];
      operand_split(w[ct][0], w[ct][1], ah, al);
      float u[2][4] = {};
      sc_ldsm(bh, mat + Sm::inv);
      sc_ldsm(bl, mat + Sm::inv + T * kMPitch);
      mma_split(u[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(u[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      operand_split(u[0], u[1], uh[ct], ul[ct]);
    }
    const float* total = reinterpret_cast<const float*>(op + Sm::total);
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t bh[4], bl[4];
      const uint32_t at = ob + Sm::kh + across * Sm::pitch + (kk * 2 + part) * 16;
      sc_ldsm_t(bh, at);
      sc_ldsm_t(bl, at + Sm::rows);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float2 d = *reinterpret_cast<const float2*>(total + kk * 16 + j * 8 + c2);
#pragma unroll
        for (int ct = 0; ct < CT; ++ct) {
          float (&t)[4] = S[ct][2 * kk + j];
          t[0] *= d.x; t[1] *= d.y; t[2] *= d.x; t[3] *= d.y;
          mma_split(t, uh[ct], ul[ct], bh[2 * j], bh[2 * j + 1], bl[2 * j], bl[2 * j + 1]);
        }
      }
    }
    {
      uint32_t bh[4], bl[4];
      sc_ldsm(bh, mat + Sm::qk);
      sc_ldsm(bl, mat + Sm::qk + T * kMPitch);
      if (i > 0) bar_wait(1, 128);               // the rows of the chunk before have been stored
#pragma unroll
      for (int ct = 0; ct < CT; ++ct) {
        mma_split(o[ct][0], uh[ct], ul[ct], bh[0], bh[1], bl[0], bl[1]);
        mma_split(o[ct][1], uh[ct], ul[ct], bh[2], bh[3], bl[2], bl[3]);
        const uint32_t packed[4] = {pair(o[ct][0][0], o[ct][0][1]), pair(o[ct][1][0], o[ct][1][1]), pair(o[ct][0][2], o[ct][0][3]),
                                    pair(o[ct][1][2], o[ct][1][3])};
        sc_stsm_t(out + across * Sm::vpitch + ((warp * CT + ct) * 2 + part) * 16, packed);
      }
    }
    if (i + NB < chunks) bar_signal(kBarEmpty + i % NB, 256);
    bar_wait(1, 128);                            // the chunk's output rows are complete
#pragma unroll
    for (int j = 0; j < CT; ++j) {
      const int at = threadIdx.x + j * 128, t = at / (8 * CT), c = at % (8 * CT) * 8;
      if (i * T + t < n && c < np)
        *reinterpret_cast<uint4*>(p.o + static_cast<long long>(q0 + i * T + t) * p.ldo + h * p.V + p0 + c) =
            *reinterpret_cast<const uint4*>(smem + Sm::out + t * Sm::vpitch + c * 2);
    }
  }
#pragma unroll
  for (int ct = 0; ct < CT; ++ct) {
#pragma unroll
    for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int col = (warp * CT + ct) * 16 + r4 + half * 8, key = j * 8 + c2;
        if (col < np && key < p.K)
          *reinterpret_cast<float2*>(state + static_cast<long long>(col) * p.K + key) = make_float2(S[ct][j][2 * half], S[ct][j][2 * half + 1]);
      }
    }
  }
}

template <int NK, int CT>
static int launch_delta_chunks(const DeltaParams<bf16>& p, int B, cudaStream_t st) {
  typedef DeltaSmem<NK, CT> Sm;
  static int ok = 0;                             // 1: ready, -1: not with the registers that the kernel was compiled to
  if (ok == 0) {
    cudaFuncAttributes a;
    if (cudaFuncGetAttributes(&a, delta_chunk_kernel<NK, CT>) != cudaSuccess ||
        cudaFuncSetAttribute(delta_chunk_kernel<NK, CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sm::bytes) != cudaSuccess) return -3;
    ok = a.numRegs == kLaunchRegs ? 1 : -1;
  }
  if (ok < 0) return -100;
  return launch_pdl(delta_chunk_kernel<NK, CT>, dim3((p.V + Sm::cols - 1) / Sm::cols, p.H, B), dim3(kDeltaThreads), Sm::bytes, st, p) ==
                 cudaSuccess ? 0 : -4;
}

int delta_chunks(const DeltaParams<bf16>& p, int B, cudaStream_t st) {
  const int steps = (p.K + 15) / 16;
  if (steps > 8 || p.ldc % 8 || p.ld_decay % 8 || !aligned16(p.c) || !aligned16(p.decay) || p.ldo % 8) return -100;
  // 64 columns per CTA while these fill at most one wave, else 128
  const bool wide = p.V > 64 && static_cast<long long>((p.V + 63) / 64) * p.H * B > 148;
  if (steps <= 1) return wide ? launch_delta_chunks<1, 2>(p, B, st) : launch_delta_chunks<1, 1>(p, B, st);
  if (steps <= 2) return wide ? launch_delta_chunks<2, 2>(p, B, st) : launch_delta_chunks<2, 1>(p, B, st);
  if (steps <= 4) return wide ? launch_delta_chunks<4, 2>(p, B, st) : launch_delta_chunks<4, 1>(p, B, st);
  return wide ? launch_delta_chunks<8, 2>(p, B, st) : launch_delta_chunks<8, 1>(p, B, st);
}

}  // namespace ksana
