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
// delta_chunk_kernel: one CTA per (sequence, head, 64 columns), chunks of 16 tokens. With P_t = g_1 .. g_t per key channel:
//   (I + A) U = beta (V - (k P) S),  A_ts = beta_t sum_c k_tc k_sc (g_(s+1) .. g_t)_c for s < t
//   O = (q P) S + Q U,  Q_ts likewise with q_t, for s <= t;   S <- P_L S + sum_s (k_s g_(s+1) .. g_L) u_s^T
// Decays enter as products of factors <= 1 only, never as quotients, so no decay is too strong. Four warps prepare the operands of
// the next chunk (unit vectors, decays, A and its unit-triangular inverse, Q), four warps with 16 columns each apply them; U and the
// state never leave their registers.
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
template <int NK> constexpr int kSpaceSmem = 2 * kSpaceStage<NK> + 2 * kSpaceTokens * kXPitch + 4 * kSpaceTokens * 4;

// NK: steps of 16 keys. grid (column slabs, H, sequences)
template <int NK>
__global__ void __launch_bounds__(kSpaceThreads, 2) space_chunk_kernel(const SpaceParams<bf16> p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int PB = kBPitch<NK>, L = kSpaceTokens;
  uint8_t* mh = smem + 2 * kSpaceStage<NK>;
  uint8_t* ml = mh + L * kXPitch;
  float* cum = reinterpret_cast<float*>(ml + L * kXPitch);      // G_t
  float* dts = cum + L;
  float* wend = dts + L;                                        // dt_s exp(G_L - G_s)
  float* edec = wend + L;                                       // exp(G_t)
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
    uint8_t* b = stage(buf);
    constexpr int V = NK * 2, W = 2 * V + kSpaceCols / 8;       // 16-byte pieces of a row
    for (int i = threadIdx.x; i < L * W; i += kSpaceThreads) {
      const int t = i / W, k = i % W;
      const bool is_x = k >= 2 * V, is_c = !is_x && k >= V;
      const int v = is_x ? k - 2 * V : is_c ? k - V : k;
      const bool there = t0 + t < n && (is_x ? v * 8 < np : v * 8 < p.N);
      uint8_t* dst = is_x ? b + 2 * L * PB + t * kXPitch : b + (is_c ? L * PB : 0) + t * PB;
      const bf16* src = rows + static_cast<long long>(there ? t0 + t : 0) * p.ldc + (there ? (is_x ? xoff : is_c ? coff : boff) + v * 8 : 0);
      sc_copy16(sc_addr(dst + v * 16), src, there);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto raw_dt = [&](int t) { return t < n ? to_f(p.dt[static_cast<long long>(q0 + t) * p.ld_dt + h]) : 0.f; };
  issue(0, 0);
  float d0 = warp == 0 ? raw_dt(2 * lane) : 0.f, d1 = warp == 0 ? raw_dt(2 * lane + 1) : 0.f;
  for (int t0 = 0, buf = 0; t0 < n; t0 += L, buf ^= 1) {
    if (t0 + L < n) issue(t0 + L, buf ^ 1);
    else asm volatile("cp.async.commit_group;" ::: "memory");
    if (warp == 0) {                                     // step sizes, their running sums, decays
      const float a = t0 + 2 * lane < n ? softplus_f(d0 + dtb) : 0.f, b = t0 + 2 * lane + 1 < n ? softplus_f(d1 + dtb) : 0.f;
      float sum = a + b;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      const float total = __shfl_sync(0xffffffffu, sum, 31), g1 = -A * sum, g0 = -A * (sum - b), gl = -A * total;
      cum[2 * lane] = g0;
      cum[2 * lane + 1] = g1;
      dts[2 * lane] = a;
      dts[2 * lane + 1] = b;
      edec[2 * lane] = expf(g0);
      edec[2 * lane + 1] = expf(g1);
      wend[2 * lane] = a * expf(gl - g0);
      wend[2 * lane + 1] = b * expf(gl - g1);
      d0 = raw_dt(t0 + L + 2 * lane);
      d1 = raw_dt(t0 + L + 2 * lane + 1);
    }
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
            v[e] = u <= t ? acc[j][2 * half + e] * __expf(gt - cum[u]) * dts[u] : 0.f;
            if (u == t) v[e] += D;
          }
          uint32_t hi, lo;
          pair_split(v[0], v[1], hi, lo);
          *reinterpret_cast<uint32_t*>(mh + t * kXPitch + (j * 8 + c2) * 2) = hi;
          *reinterpret_cast<uint32_t*>(ml + t * kXPitch + (j * 8 + c2) * 2) = lo;
        }
      }
    }
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
constexpr int kDeltaTokens = 16, kDeltaCols = 64, kDeltaThreads = 256, kMPitch = (kDeltaTokens + 8) * 2;
template <int NK> struct DeltaSmem {
  static constexpr int KP = NK * 16, pitch = (KP + 8) * 2, rows = kDeltaTokens * pitch, fpitch = KP + 4;
  // operands of one chunk
  static constexpr int kt = 0, qt = 2 * rows, kh = 4 * rows, inv = 6 * rows, qk = inv + 2 * kDeltaTokens * kMPitch,
                       v = qk + 2 * kDeltaTokens * kMPitch, beta = v + kDeltaTokens * kXPitch, total = beta + kDeltaTokens * 4,
                       operands = total + KP * 4;
  // raw rows of one chunk: q, k, decay
  static constexpr int raw = 3 * kDeltaTokens * KP * 2;
  static constexpr int out = 2 * operands + 2 * raw, f32 = out + kDeltaTokens * kXPitch,
                       bytes = f32 + (3 * kDeltaTokens * fpitch + kDeltaTokens * (kDeltaTokens + 4) + 2 * kDeltaTokens) * 4;
};

__device__ __forceinline__ void sc_stsm_t(uint32_t addr, const uint32_t (&r)[4]) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3])
               : "memory");
}
__device__ __forceinline__ void half_barrier(int id) { asm volatile("bar.sync %0, 128;" ::"r"(id) : "memory"); }
__device__ __forceinline__ void put_split(uint8_t* hi, uint8_t* lo, float v) {
  const bf16 h = __float2bfloat16(v);
  *reinterpret_cast<bf16*>(hi) = h;
  *reinterpret_cast<bf16*>(lo) = __float2bfloat16(v - __bfloat162float(h));
}
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

// One chunk's operands from its raw rows, by 128 threads (tid 0 .. 127); m of its 16 tokens exist.
template <int NK>
__device__ __forceinline__ void delta_prepare(const DeltaParams<bf16>& p, uint8_t* op, const uint8_t* raw, float* f, int tid, int m, float A,
                                              float bias, const bf16* beta) {
  typedef DeltaSmem<NK> Sm;
  constexpr int KP = Sm::KP, T = kDeltaTokens, FP = Sm::fpitch;
  const int warp = tid >> 5, lane = tid & 31;
  const bf16* rq = reinterpret_cast<const bf16*>(raw);
  const bf16* rk = rq + T * KP;
  const bf16* rz = rk + T * KP;
  float* kf = f;
  float* qf = kf + T * FP;
  float* gf = qf + T * FP;
  float* am = gf + T * FP;                       // A, [T][T + 4]
  float* iq = am + T * (T + 4);                  // reciprocal lengths
  float* ik = iq + T;
  float* bt = reinterpret_cast<float*>(op + Sm::beta);
  // lengths: four tokens per warp
#pragma unroll
  for (int i = 0; i < T / 4; ++i) {
    const int t = warp * (T / 4) + i;
    float qq = 0.f, kk = 0.f;
    for (int c = lane * 2; c < KP; c += 64) {
      const float2 q = unpair(*reinterpret_cast<const uint32_t*>(rq + t * KP + c)), k = unpair(*reinterpret_cast<const uint32_t*>(rk + t * KP + c));
      qq = fmaf(q.x, q.x, fmaf(q.y, q.y, qq));
      kk = fmaf(k.x, k.x, fmaf(k.y, k.y, kk));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
    }
    if (lane == 0) {
      iq[t] = p.q_scale * rsqrtf(qq + kUnitEps);
      ik[t] = rsqrtf(kk + kUnitEps);
      bt[t] = t < m ? sigmoid_exact(to_f(beta[static_cast<long long>(t) * p.ld_beta])) : 0.f;
    }
  }
  half_barrier(2);
  if (tid < KP) {                                // one key channel per thread
    const int c = tid;
    float k[T], g[T], P = 1.f;
#pragma unroll
    for (int t = 0; t < T; ++t) {
      k[t] = to_f(rk[t * KP + c]) * ik[t];
      const float q = to_f(rq[t * KP + c]) * iq[t], z = to_f(rz[t * KP + c]) + bias;
      const float soft = fmaxf(z, 0.f) + __logf(1.f + __expf(-fabsf(z)));
      g[t] = t < m && c < p.K ? __expf(-A * soft) : 1.f;
      P *= g[t];
      kf[t * FP + c] = k[t];
      qf[t * FP + c] = q;
      gf[t * FP + c] = g[t];
      uint8_t* at = op + t * Sm::pitch + c * 2;
      put_split(at + Sm::kt, at + Sm::kt + Sm::rows, k[t] * P);
      put_split(at + Sm::qt, at + Sm::qt + Sm::rows, q * P);
    }
    reinterpret_cast<float*>(op + Sm::total)[c] = P;
    P = 1.f;
#pragma unroll
    for (int t = T - 1; t >= 0; --t) {
      uint8_t* at = op + Sm::kh + t * Sm::pitch + c * 2;
      put_split(at, at + Sm::rows, k[t] * P);
      P *= g[t];
    }
  }
  half_barrier(2);
  // A and Q by columns s, four per warp; a lane has four key channels
#pragma unroll
  for (int i = 0; i < T / 4; ++i) {
    const int s = i * 4 + (i & 1 ? 3 - warp : warp);
    float v[2 * T];
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool on = lane * 4 < KP;
#pragma unroll
    for (int t = 0; t < T; ++t) {
      v[t] = v[T + t] = 0.f;
      if (t < s) continue;
      if (!on) continue;
      const float4 k = *reinterpret_cast<const float4*>(kf + t * FP + lane * 4), q = *reinterpret_cast<const float4*>(qf + t * FP + lane * 4);
      if (t == s) {
        d = k;
      } else {
        const float4 g = *reinterpret_cast<const float4*>(gf + t * FP + lane * 4);
        d.x *= g.x; d.y *= g.y; d.z *= g.z; d.w *= g.w;
        v[t] = fmaf(d.x, k.x, fmaf(d.y, k.y, fmaf(d.z, k.z, d.w * k.w)));
      }
      v[T + t] = fmaf(d.x, q.x, fmaf(d.y, q.y, fmaf(d.z, q.z, d.w * q.w)));
    }
    // sums over the lanes; lane l keeps entry l
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
      for (int j = 0; j < o; ++j) {
        const bool up = lane & o;
        const float send = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
        v[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    const int t = lane & 15;
    if (lane < T) am[t * (T + 4) + s] = t > s ? bt[t] * v[0] : 0.f;
    else {
      uint8_t* at = op + Sm::qk + t * kMPitch + s * 2;
      put_split(at, at + T * kMPitch, t >= s ? v[0] : 0.f);
    }
  }
  half_barrier(2);
  if (tid < T) {                                 // column tid of the inverse of I + A
    float x[T];
#pragma unroll
    for (int t = 0; t < T; ++t) {
      float a = t == tid ? 1.f : 0.f, b = 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) {
        if (s & 1) b = fmaf(-am[t * (T + 4) + s], x[s], b);
        else a = fmaf(-am[t * (T + 4) + s], x[s], a);
      }
      x[t] = a + b;
      uint8_t* at = op + Sm::inv + t * kMPitch + tid * 2;
      put_split(at, at + T * kMPitch, x[t]);
    }
  }
}

// grid (column slabs, H, sequences); warps 0 - 3 apply, warps 4 - 7 prepare
template <int NK>
__global__ void __launch_bounds__(kDeltaThreads, 1) delta_chunk_kernel(const DeltaParams<bf16> p) {
  pdl_trigger();
  pdl_wait();
  typedef DeltaSmem<NK> Sm;
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int KP = Sm::KP, T = kDeltaTokens;
  const int s = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * kDeltaCols, np = min(kDeltaCols, p.V - p0);
  const int q0 = p.cu_q[s], n = p.cu_q[s + 1] - q0, past = p.ref.kv_lens[s] - n;
  if (n <= 0) return;
  const int slot = slot_of(p.ref, s);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (p.H / p.G), chunks = (n + T - 1) / T;
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;
  float* state = p.state + static_cast<long long>(slot) * p.slot_stride + (static_cast<long long>(h) * p.V + p0) * p.K;
  const bf16* rows = p.c + static_cast<long long>(q0) * p.ldc;
  if (warp >= 4) {
    const int tid = threadIdx.x - 128;
    const float A = p.A[h], bias = tid < p.K ? p.decay_bias[h * p.K + tid] : 0.f;
    const bf16* z = p.decay + static_cast<long long>(q0) * p.ld_decay + h * p.K;
    const bf16* beta = p.beta + static_cast<long long>(q0) * p.ld_beta + h;
    auto fetch = [&](int i) {                    // raw rows of chunk i
      uint8_t* dst = smem + 2 * Sm::operands + (i & 1) * Sm::raw;
      for (int j = tid; j < 3 * T * (KP / 8); j += 128) {
        const int what = j / (T * (KP / 8)), t = j / (KP / 8) % T, c = j % (KP / 8) * 8, row = i * T + t;
        const bool there = row < n && c < p.K;
        const bf16* src = what == 2 ? z + static_cast<long long>(there ? row : 0) * p.ld_decay
                                    : rows + static_cast<long long>(there ? row : 0) * p.ldc + (what ? p.G + g : g) * p.K;
        sc_copy16(sc_addr(dst + (what * T * KP + t * KP + c) * 2), src + (there ? c : 0), there);
      }
    };
    auto fetch_v = [&](int i) {
      uint8_t* dst = smem + (i & 1) * Sm::operands + Sm::v;
      const int t = tid >> 3, c = (tid & 7) * 8, row = i * T + t;                          // 16 rows of 8 pieces
      const bool there = row < n && c < np;
      sc_copy16(sc_addr(dst + t * kXPitch + c * 2),
                rows + static_cast<long long>(there ? row : 0) * p.ldc + 2 * p.G * p.K + h * p.V + p0 + (there ? c : 0), there);
    };
    auto landed = [&]() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory"); };
    float* f = reinterpret_cast<float*>(smem + Sm::f32);
    fetch(0);
    fetch_v(0);
    landed();
    half_barrier(2);
    if (chunks > 1) fetch(1);
    delta_prepare<NK>(p, smem, smem + 2 * Sm::operands, f, tid, min(T, n), A, bias, beta);
    landed();
    __syncthreads();
    for (int i = 0; i < chunks; ++i) {
      if (i + 1 < chunks) {
        fetch_v(i + 1);
        if (i + 2 < chunks) fetch(i + 2);
        delta_prepare<NK>(p, smem + ((i + 1) & 1) * Sm::operands, smem + 2 * Sm::operands + ((i + 1) & 1) * Sm::raw, f, tid,
                          min(T, n - (i + 1) * T), A, bias, beta + static_cast<long long>((i + 1) * T) * p.ld_beta);
        landed();
      }
      __syncthreads();
    }
    delta_ring(p, p.conv.x + static_cast<long long>(q0) * p.conv.ld, slot, past, n, h, p0, np, tid, 128);
    return;
  }
  float S[2 * NK][4];
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int col = warp * 16 + r4 + half * 8, key = j * 8 + c2;
      const float2 v = past > 0 && col < np && key < p.K ? *reinterpret_cast<const float2*>(state + static_cast<long long>(col) * p.K + key)
                                                         : make_float2(0.f, 0.f);
      S[j][2 * half] = v.x;
      S[j][2 * half + 1] = v.y;
    }
  }
  __syncthreads();
  const uint32_t out = sc_addr(smem + Sm::out);
  const uint32_t flat = ((lane & 7) + ((lane >> 4) << 3)), side = ((lane >> 3) & 1) * 16;        // 16 rows x 16 columns, rows as columns of B
  const uint32_t across = (lane & 7) + (((lane >> 3) & 1) << 3), part = lane >> 4;               // transposed reads
  for (int i = 0; i < chunks; ++i) {
    const uint8_t* op = smem + (i & 1) * Sm::operands;
    const uint32_t ob = sc_addr(op);
    float w[2][4] = {}, o[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      operand_split(S[2 * kk], S[2 * kk + 1], ah, al);
      const uint32_t at = ob + flat * Sm::pitch + kk * 32 + side;
      sc_ldsm(bh, at + Sm::kt);
      sc_ldsm(bl, at + Sm::kt + Sm::rows);
      mma_split(w[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(w[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      sc_ldsm(bh, at + Sm::qt);
      sc_ldsm(bl, at + Sm::qt + Sm::rows);
      mma_split(o[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(o[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    }
    uint32_t v[4];                               // (tokens 0-7, columns 0-7), (tokens 8-15, columns 0-7), then columns 8-15
    sc_ldsm_t(v, ob + Sm::v + across * kXPitch + (warp * 2 + part) * 16);
    const float* bt = reinterpret_cast<const float*>(op + Sm::beta);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float2 b = *reinterpret_cast<const float2*>(bt + j * 8 + c2), v0 = unpair(v[j]), v1 = unpair(v[2 + j]);
      w[j][0] = b.x * (v0.x - w[j][0]);
      w[j][1] = b.y * (v0.y - w[j][1]);
      w[j][2] = b.x * (v1.x - w[j][2]);
      w[j][3] = b.y * (v1.y - w[j][3]);
    }
    uint32_t ah[4], al[4], bh[4], bl[4];
    operand_split(w[0], w[1], ah, al);
    float u[2][4] = {};
    const uint32_t mat = ob + flat * kMPitch + side;
    sc_ldsm(bh, mat + Sm::inv);
    sc_ldsm(bl, mat + Sm::inv + T * kMPitch);
    mma_split(u[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
    mma_split(u[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    operand_split(u[0], u[1], ah, al);
    sc_ldsm(bh, mat + Sm::qk);
    sc_ldsm(bl, mat + Sm::qk + T * kMPitch);
    mma_split(o[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
    mma_split(o[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    const uint32_t packed[4] = {pair(o[0][0], o[0][1]), pair(o[1][0], o[1][1]), pair(o[0][2], o[0][3]), pair(o[1][2], o[1][3])};
    sc_stsm_t(out + across * kXPitch + (warp * 2 + part) * 16, packed);
    const float* total = reinterpret_cast<const float*>(op + Sm::total);
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      const uint32_t at = ob + Sm::kh + across * Sm::pitch + (kk * 2 + part) * 16;
      sc_ldsm_t(bh, at);
      sc_ldsm_t(bl, at + Sm::rows);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float2 d = *reinterpret_cast<const float2*>(total + kk * 16 + j * 8 + c2);
        float (&t)[4] = S[2 * kk + j];
        t[0] *= d.x; t[1] *= d.y; t[2] *= d.x; t[3] *= d.y;
        mma_split(t, ah, al, bh[2 * j], bh[2 * j + 1], bl[2 * j], bl[2 * j + 1]);
      }
    }
    half_barrier(1);                             // the chunk's output rows are complete
    {
      const int t = threadIdx.x >> 3, c = (threadIdx.x & 7) * 8;
      if (i * T + t < n && c < np)
        *reinterpret_cast<uint4*>(p.o + static_cast<long long>(q0 + i * T + t) * p.ldo + h * p.V + p0 + c) =
            *reinterpret_cast<const uint4*>(smem + Sm::out + t * kXPitch + c * 2);
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int col = warp * 16 + r4 + half * 8, key = j * 8 + c2;
      if (col < np && key < p.K)
        *reinterpret_cast<float2*>(state + static_cast<long long>(col) * p.K + key) = make_float2(S[j][2 * half], S[j][2 * half + 1]);
    }
  }
}

template <int NK>
static int launch_delta_chunks(const DeltaParams<bf16>& p, int B, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaSmem<NK>::bytes) != cudaSuccess) return -3;
    set = true;
  }
  return launch_pdl(delta_chunk_kernel<NK>, dim3((p.V + kDeltaCols - 1) / kDeltaCols, p.H, B), dim3(kDeltaThreads), DeltaSmem<NK>::bytes, st,
                    p) == cudaSuccess ? 0 : -4;
}

int delta_chunks(const DeltaParams<bf16>& p, int B, cudaStream_t st) {
  const int steps = (p.K + 15) / 16;
  if (steps > 8 || p.ldc % 8 || p.ld_decay % 8 || !aligned16(p.c) || !aligned16(p.decay) || p.ldo % 8) return -100;
  if (steps <= 1) return launch_delta_chunks<1>(p, B, st);
  if (steps <= 2) return launch_delta_chunks<2>(p, B, st);
  if (steps <= 4) return launch_delta_chunks<4>(p, B, st);
  return launch_delta_chunks<8>(p, B, st);
}

}  // namespace ksana
