// Prefill (and chunked-prefill) attention on the tcgen05 tensor cores: causal attention of new query rows
// against the paged KV cache, head sizes up to 128 (query/key and value sizes may differ; both padded with zeros in shared
// memory only), bf16 cache, optionally a sliding window with kept first tokens and a per-head sink logit.
//
// One CTA owns up to 128 packed query rows of one KV head group: row = (token, head inside the group), so the G query
// heads that share a KV head reuse every staged K/V tile (whole tokens only: 128 / G of them, the rows behind stay idle). Per 128-token KV tile:
//   S = Q K^T      tcgen05.mma, both operands K-major in shared memory (TMA, 128-byte swizzle), S in TMEM
//   softmax        4 warps, one thread per row (TMEM lane): no cross-thread reductions; online max with a
//                  lazy rescale of O (only when a row's maximum grew by more than 2^8)
//   O += P V       tcgen05.mma with P read from TMEM (bf16 pairs written over S's columns by the softmax warps)
//                  and V as an MN-major shared-memory operand, O accumulating in TMEM
// Warp roles: warp 0 TMA producer (Q once; K and V tiles through the block table, one box per cache block and
// 64-column panel), warp 1 MMA issuer + TMEM owner, warps 2..5 softmax + epilogue. Two CTAs share an SM
// (96 KB of shared memory, 256 TMEM columns each), so one CTA's softmax overlaps the other's MMAs.
// With sigmoid weights (SIG) a key's weight is sigmoid(score + bias[head][distance]): no maximum, no sum, no rescale; the
// heads' bias rows are staged in shared memory where they fit. Outputs may be multiplied by the sigmoid of a gate.
// Every wait is bounded; a timeout sets the error word and leaves the output untouched.
//
// Same operator as the reference's flash-attention prefill call plus its separate prefix-cache gather
// (src/ksana_llm/layers/flash_attention_layer.cpp, 3rdparty/LLM_kernels/csrc/kernels/nvidia/paged_attention):
// here K/V are read in place from the paged cache.
#include "sm100_ptx.cuh"
#include <cuda_bf16.h>
#include <math_constants.h>
#include <stdio.h>

namespace ksana {

typedef __nv_bfloat16 bf16;
constexpr int kFaThreads = 192;
constexpr int kFaTile = 128;                 // query rows per CTA and KV tokens per tile
constexpr int kFaD = 128;                    // padded head size
constexpr int kFaPanelBytes = kFaTile * 128; // one 64-column panel of a 128-row tile
constexpr int kFaTileBytes = 2 * kFaPanelBytes;
constexpr int kFaSmemBytes = 3 * kFaTileBytes + 1024 + 256;
constexpr int kFaBiasBytes = 14 * 1024;      // distance biases of a head group that still let two CTAs share an SM
constexpr uint32_t kFaTmemCols = 256;        // S / P at columns [0,128), O at [128,256)
constexpr float kFaRescaleLog2 = 8.f;        // O is rescaled only when a row maximum grew by more than this

struct FaParams {
  bf16* out; long long out_stride;
  const int* block_table; int table_stride;
  const int* cu_q; const int* kv_lens; const float* alibi;
  const float* sinks;                        // [Hq] logits added to the softmax denominator, or null
  int Hq, Hkv, G, block_tokens;
  int shared;                                // the values are the keys: one tile per step, two in flight
  int rows;                                  // query rows of a CTA: the largest multiple of G up to 128
  int D, Dv;                                 // real head sizes
  int window, keep;                          // sliding window in tokens (0: none), first tokens every row sees
  const float* bias; int bias_len;           // sigmoid weights: [Hq][bias_len] by distance (the last entry holds beyond)
  // floats between the heads' rows in shared memory (there times -log2 e, with kFaTile entries in front for keys behind the
  // row and kFaTile repetitions of the last entry behind, so that a tile's distances need no clamping); 0: read from global memory
  int bias_ld;
  const bf16* gate; long long gate_stride; float out_factor;     // sigmoid weights: optional gate rows like out's, and a factor
  float scale_log2;
  int* err;
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// WIN: sliding window (p.window > 0); without it the window's tests are not compiled in
template <bool WIN, bool SIG>
__global__ void __launch_bounds__(kFaThreads, 2)
prefill_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                  const __grid_constant__ CUtensorMap v_map, const FaParams p) {
  extern __shared__ uint8_t fa_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(fa_smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* k_s = smem + kFaTileBytes;
  uint8_t* v_s = smem + 2 * kFaTileBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 3 * kFaTileBytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 2;
  uint64_t* v_full = bars + 3;
  uint64_t* v_empty = bars + 4;
  uint64_t* s_full = bars + 5;
  uint64_t* p_full = bars + 6;
  uint64_t* o_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  float* bias_s = reinterpret_cast<float*>(smem + 3 * kFaTileBytes + 256);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int s = blockIdx.z, g = blockIdx.y;
  const int G = p.G;
  const int q0 = p.cu_q[s], q_len = p.cu_q[s + 1] - q0;
  const int kv_len = p.kv_lens[s];
  const int qtile = static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x);   // longest rows first
  const int row0 = qtile * p.rows;
  if (row0 >= q_len * G) return;
  const int past = kv_len - q_len;
  const int last_row = min(row0 + p.rows - 1, q_len * G - 1);
  const int kv_end = min(kv_len, past + last_row / G + 1);
  // tiles visited: those with kept first tokens, then from the first position in the window of this CTA's first row on
  const int first_lo = WIN ? past + row0 / G - p.window + 1 : 0;
  const int win_tile = WIN ? max(first_lo, 0) / kFaTile : 0;
  const int keep_tiles = WIN ? min((p.keep + kFaTile - 1) / kFaTile, win_tile) : 0;
  const int ntiles = keep_tiles + (kv_end + kFaTile - 1) / kFaTile - win_tile;
  auto tile_start = [&](int j) { return (j < keep_tiles ? j : win_tile + j - keep_tiles) * kFaTile; };
  const int kpanels = (p.D + 63) >> 6, vpanels = (p.Dv + 63) >> 6;
  const int* table = p.block_table + static_cast<size_t>(s) * p.table_stride;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1); mbar_init(k_full, 1); mbar_init(k_empty, 1); mbar_init(v_full, 1); mbar_init(v_empty, 1);
    mbar_init(s_full, 1); mbar_init(p_full, 4); mbar_init(o_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, kFaTmemCols); tmem_relinquish(); }
  if (SIG && p.bias_ld > 0)
    for (int i = threadIdx.x; i < G * p.bias_ld; i += kFaThreads) {
      const int at = min(max(i % p.bias_ld - kFaTile, 0), p.bias_len - 1);
      bias_s[i] = -1.44269504f * p.bias[static_cast<size_t>(g * G + i / p.bias_ld) * p.bias_len + at];
    }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 128;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      tma_prefetch_desc(&q_map);
      tma_prefetch_desc(&k_map);
      tma_prefetch_desc(&v_map);
      mbar_expect_tx(q_full, kpanels * p.rows * 128);
      const int tok0 = q0 + row0 / G;
      for (int h = 0; h < kpanels; ++h) tma_load_3d(q_s + h * kFaPanelBytes, &q_map, q_full, h * 64, g * G, tok0);
      const int bt = p.block_tokens;
      bool ok = true;
      for (int j = 0; p.shared && j < ntiles && ok; ++j) {       // key tiles alternate between the two places
        const int t0 = tile_start(j), nblk = min(kFaTile / bt, (kv_len - t0 + bt - 1) / bt);
        uint8_t* dst = j & 1 ? v_s : k_s;
        uint64_t* full = j & 1 ? v_full : k_full;
        if (!mbar_wait(j & 1 ? v_empty : k_empty, ((j >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_expect_tx(full, static_cast<uint32_t>(nblk) * kpanels * bt * 128);
        for (int b = 0; b < nblk; ++b) {
          const int blk = table[t0 / bt + b];
          for (int h = 0; h < kpanels; ++h) tma_load_3d(dst + h * kFaPanelBytes + b * bt * 128, &k_map, full, h * 64, g * bt, blk);
        }
      }
      for (int j = 0; !p.shared && j < ntiles && ok; ++j) {
        const int t0 = tile_start(j);
        const int nblk = min(kFaTile / bt, (kv_len - t0 + bt - 1) / bt);
#pragma unroll
        for (int which = 0; which < 2; ++which) {
          uint64_t* full = which ? v_full : k_full;
          uint64_t* empty = which ? v_empty : k_empty;
          uint8_t* dst = which ? v_s : k_s;
          if (!mbar_wait(empty, (j & 1) ^ 1, abort_flag)) { ok = false; break; }
          const int panels = which ? vpanels : kpanels;
          mbar_expect_tx(full, static_cast<uint32_t>(nblk) * panels * bt * 128);
          for (int b = 0; b < nblk; ++b) {
            const int blk = table[t0 / bt + b];
            for (int h = 0; h < panels; ++h)               // columns past the row's end arrive as zeros
              tma_load_3d(dst + h * kFaPanelBytes + b * bt * 128, which ? &v_map : &k_map, full, h * 64, g * bt, blk);
          }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc(128, 128, 1, 1);
      const uint32_t idesc_pv = make_idesc(128, vpanels * 64, 1, 1) | (1u << 16);     // B (= V) is MN-major
      const int ksteps = (p.D + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, abort_flag);
      for (int j = 0; j < ntiles && ok; ++j) {
        const uint32_t par = j & 1;
        const bool second = p.shared && (j & 1);
        uint8_t* kt = second ? v_s : k_s;
        uint8_t* vt = p.shared ? kt : v_s;
        if (!mbar_wait(second ? v_full : k_full, p.shared ? (j >> 1) & 1 : par, abort_flag)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (k >= ksteps) break;
          const uint32_t off = (k >> 2) * kFaPanelBytes;
          const uint64_t adesc = make_smem_desc_sw128(smem_u32(q_s) + off) + 2 * (k & 3);
          const uint64_t bdesc = make_smem_desc_sw128(smem_u32(kt) + off) + 2 * (k & 3);
          mma_f16(tmem_s, adesc, bdesc, idesc_qk, k != 0);
        }
        tc_commit(s_full);
        if (!p.shared) {
          tc_commit(k_empty);
          if (!mbar_wait(v_full, par, abort_flag)) { ok = false; break; }
        }
        if (!mbar_wait(p_full, par, abort_flag)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          // 16 tokens per MMA: 8 TMEM columns of P (two bf16 each), 16 rows (2 KB) of the V tile
          const uint64_t bdesc = make_smem_desc_mn_sw128(smem_u32(vt) + k * 2048, kFaPanelBytes);
          mma_f16_ts(tmem_o, tmem_s + 8 * k, bdesc, idesc_pv, (j | k) != 0);
        }
        tc_commit(p.shared && !second ? k_empty : v_empty);
        if (j == ntiles - 1) tc_commit(o_full);
      }
    }
    __syncwarp();
  } else {
    // ------------------------------------------------------------------ softmax + epilogue (one thread per row)
    const int qd = warp & 3;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const int vr = row0 + qd * 32 + lane;                  // packed row index inside the sequence
    const bool active = qd * 32 + lane < p.rows && vr < q_len * G;
    const int tok = vr / G, head = g * G + vr % G;
    const int limit = active ? past + tok : -1;            // last visible KV position
    const int lo = WIN ? limit - p.window + 1 : 0;            // first position inside the window
    const int keep = WIN ? p.keep : 0;
    auto sees = [&](int pos) { return pos <= limit && (!WIN || pos >= lo || pos < keep); };
    const float slope2 = (p.alibi && active) ? p.alibi[head] * 1.44269504f : 0.f;
    const float* near = SIG ? bias_s + (vr % G) * p.bias_ld + kFaTile : nullptr;
    const float* tab = SIG ? p.bias + static_cast<size_t>(head) * p.bias_len : nullptr;
    const int bias_last = SIG ? p.bias_len - 1 : 0;
    float m_used = -CUDART_INF_F, l = 0.f;
    bool ok = true;
    for (int j = 0; j < ntiles; ++j) {
      const uint32_t par = j & 1;
      const int t0 = tile_start(j);
      if (!mbar_wait(s_full, par, abort_flag)) { ok = false; break; }
      tc_fence_after();
      const bool biased = slope2 != 0.f || p.scale_log2 <= 0.f;
      const bool need_mask = (t0 + kFaTile - 1 > limit) ||
                             (WIN && t0 < lo && t0 + kFaTile > keep);
      // lazy rescale of O: keep the old reference maximum unless the row's maximum grew by more than 2^8
      auto update_reference = [&](float mx) {
        float m_new = m_used;
        if (mx > m_used + kFaRescaleLog2 || m_used == -CUDART_INF_F) m_new = (mx == -CUDART_INF_F) ? m_used : mx;
        const bool grow = j > 0 && m_new != m_used && m_used != -CUDART_INF_F;
        if (__any_sync(0xffffffffu, grow)) {
          const float f = grow ? exp2f(m_used - m_new) : 1.f;
          l *= f;
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t o[32];
            tmem_ld32(tmem_o + lane_off + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
            tmem_st32(tmem_o + lane_off + c * 32, o);
          }
        }
        m_used = m_new;
        return (m_used == -CUDART_INF_F) ? 0.f : m_used;
      };
      if constexpr (SIG) {
        uint32_t r[128];
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_ld32(tmem_s + lane_off + c * 32, *reinterpret_cast<uint32_t(*)[32]>(&r[c * 32]));
        tmem_ld_wait();
        const int from = limit - t0;                       // distance of the tile's first key
        // the row's visible keys as bits
        uint32_t seen[4] = {~0u, ~0u, ~0u, ~0u};
        const bool masked = __any_sync(0xffffffffu, need_mask);
        if (masked) {
          const int last = from, first = lo - t0, kept = keep - t0;
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            auto below = [&](int n) { return n - c * 32 >= 32 ? ~0u : n - c * 32 <= 0 ? 0u : (1u << (n - c * 32)) - 1u; };   // keys before n
            seen[c] = below(last + 1);
            if (WIN) seen[c] &= ~below(first) | below(kept);
          }
        }
        auto weigh = [&](auto bias_at) {                   // -log2(e) times the bias of the tile's key i
#pragma unroll
          for (int i = 0; i < 128; i += 2) {
            float w2[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const float v = fast_rcp(1.f + fast_exp2(fmaf(__uint_as_float(r[i + e]), -p.scale_log2, bias_at(i + e))));
              w2[e] = seen[(i + e) >> 5] >> ((i + e) & 31) & 1u ? v : 0.f;
            }
            __nv_bfloat162 pb = __floats2bfloat162_rn(w2[0], w2[1]);
            r[i >> 1] = *reinterpret_cast<uint32_t*>(&pb);
          }
        };
        const bool far = from - (kFaTile - 1) >= bias_last;      // every distance of the row has the last bias
        if (__all_sync(0xffffffffu, far || !active)) {
          const float b = tab[bias_last] * -1.44269504f;
          weigh([&](int) { return b; });
        } else if (p.bias_ld > 0) {
          // (a row that is far, or that does not exist, in a warp that is not: any entry inside the table, then the last one)
          const float* at = near + min(max(from, -1), bias_last + kFaTile - 1);
          weigh([&](int i) { return at[-i]; });
        } else {
          weigh([&](int i) { return tab[min(max(from - i, 0), bias_last)] * -1.44269504f; });
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_st16(tmem_s + lane_off + c * 16, *reinterpret_cast<uint32_t(*)[16]>(&r[c * 16]));
      } else if (!__any_sync(0xffffffffu, biased)) {
        // the whole row in registers with a single TMEM round trip; hidden keys (window, diagonal) become -inf there
        uint32_t r[128];
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_ld32(tmem_s + lane_off + c * 32, *reinterpret_cast<uint32_t(*)[32]>(&r[c * 32]));
        tmem_ld_wait();
        if (__any_sync(0xffffffffu, need_mask)) {
          const int last = limit - t0, first = lo - t0, kept = keep - t0;       // column bounds of this row
#pragma unroll
          for (int i = 0; i < 128; ++i)
            if (i > last || (WIN && i < first && i >= kept)) r[i] = 0xff800000u;
        }
        float mx4[4] = {-CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F};
#pragma unroll
        for (int i = 0; i < 128; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(r[i]));
        const float mref = update_reference(fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2);
        float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 128; i += 2) {
          const float p0 = fast_exp2(fmaf(__uint_as_float(r[i]), p.scale_log2, -mref));
          const float p1 = fast_exp2(fmaf(__uint_as_float(r[i + 1]), p.scale_log2, -mref));
          l4[(i >> 1) & 3] += p0 + p1;
          __nv_bfloat162 pb = __floats2bfloat162_rn(p0, p1);
          r[i >> 1] = *reinterpret_cast<uint32_t*>(&pb);        // in place: slot i/2 has already been consumed
        }
        l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_st16(tmem_s + lane_off + c * 16, *reinterpret_cast<uint32_t(*)[16]>(&r[c * 16]));
      } else {
        // ALiBi (or a scale that is not positive): masked two-pass form
        float mx = -CUDART_INF_F;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t r[32];
          tmem_ld32(tmem_s + lane_off + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int pos = t0 + c * 32 + i;
            const float v = __uint_as_float(r[i]) * p.scale_log2 + slope2 * static_cast<float>(pos - limit);
            mx = fmaxf(mx, sees(pos) ? v : -CUDART_INF_F);
          }
        }
        const float mref = update_reference(mx);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t r[32];
          tmem_ld32(tmem_s + lane_off + c * 32, r);
          tmem_ld_wait();
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const int pos = t0 + c * 32 + i;
            const float v0 = __uint_as_float(r[i]) * p.scale_log2 + slope2 * static_cast<float>(pos - limit) - mref;
            const float v1 = __uint_as_float(r[i + 1]) * p.scale_log2 + slope2 * static_cast<float>(pos + 1 - limit) - mref;
            const float p0 = sees(pos) ? fast_exp2(v0) : 0.f;
            const float p1 = sees(pos + 1) ? fast_exp2(v1) : 0.f;
            l += p0 + p1;
            __nv_bfloat162 pb = __floats2bfloat162_rn(p0, p1);
            pk[i >> 1] = *reinterpret_cast<uint32_t*>(&pb);
          }
          tmem_st16(tmem_s + lane_off + c * 16, pk);
        }
      }
      tmem_st_wait();
      if (t0 + kFaTile > kv_len) {
        // last tile of the sequence: V rows past the sequence end hold stale shared memory or whatever the cache
        // has there; their probabilities are 0, but 0 x NaN would poison O. Zero them before the PV MMA reads.
        // (the keys' product is complete here, so a shared tile is free to be changed)
        if (!p.shared && !mbar_wait(v_full, par, abort_flag)) { ok = false; break; }
        uint8_t* vt = p.shared && !(j & 1) ? k_s : v_s;
        const int first_bad = kv_len - t0;
        const int nchunks = (kFaTile - first_bad) * 16;       // 16-byte chunks per row: 2 panels x 8
        for (int i = threadIdx.x - 64; i < nchunks; i += 128) {
          const int r = first_bad + (i >> 4), ch = i & 15;
          *reinterpret_cast<uint4*>(vt + (ch >> 3) * kFaPanelBytes + r * 128 + (((ch & 7) ^ (r & 7)) << 4)) =
              make_uint4(0, 0, 0, 0);
        }
        fence_async_smem();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    if (ok && mbar_wait(o_full, 0, abort_flag)) {
      tc_fence_after();
      if (p.sinks && active) l += exp2f(p.sinks[head] * 1.44269504f - m_used);
      const float inv = SIG ? 1.f : l > 0.f ? 1.f / l : 0.f;
      bf16* dst = p.out + static_cast<size_t>(q0 + tok) * p.out_stride + head * p.Dv;
      const bf16* gate = SIG && p.gate ? p.gate + static_cast<size_t>(q0 + tok) * p.gate_stride + head * p.Dv : nullptr;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        if (c * 32 >= p.Dv) break;
        uint32_t r[32];
        tmem_ld32(tmem_o + lane_off + c * 32, r);
        tmem_ld_wait();
        if (active) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c * 32 + i >= p.Dv) break;
            if (SIG && gate) {
              const uint4 gv = *reinterpret_cast<const uint4*>(gate + c * 32 + i);
              const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 z = __bfloat1622float2(g2[e]);
                r[i + 2 * e] = __float_as_uint(__uint_as_float(r[i + 2 * e]) * p.out_factor / (1.f + fast_exp2(z.x * -1.44269504f)));
                r[i + 2 * e + 1] = __float_as_uint(__uint_as_float(r[i + 2 * e + 1]) * p.out_factor / (1.f + fast_exp2(z.y * -1.44269504f)));
              }
            }
            uint4 ov;
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&ov);
#pragma unroll
            for (int e = 0; e < 4; ++e)
              o2[e] = __floats2bfloat162_rn(__uint_as_float(r[i + 2 * e]) * inv, __uint_as_float(r[i + 2 * e + 1]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + i) = ov;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    if (threadIdx.x == 0 && p.err) atomicExch(p.err, 7);
    for (int i = 0; i < 1000; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, kFaTmemCols); }
}

typedef CUresult (*FaEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                               const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static FaEncodeFn fa_encode_fn() {
  static FaEncodeFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess ||
        q != cudaDriverEntryPointSuccess) return nullptr;
    fn = reinterpret_cast<FaEncodeFn>(ptr);
  }
  return fn;
}

}  // namespace ksana

using namespace ksana;

// Returns 0 when launched, -100 when this kernel does not cover the configuration (the caller then uses the
// general kernel of attention.cu), other negatives on setup errors.
// q: [T, q_stride] bf16 with head h at column h*D (T = rows addressable from q); kc / vc: the layer's K and V panels of
// block 0, [Hkv][block_tokens][D] and [Hkv][block_tokens][Dv] bf16, blocks block_stride elements apart, num_blocks of them.
// window 0: no sliding window. sinks: [Hq] fp32 or null. bias [Hq][bias_len] fp32 switches to sigmoid weights; gate: optional
// rows like out's (16-byte aligned), with a common factor.
extern "C" int ksana_paged_prefill_tc(const void* q, long long q_stride, long long q_rows, void* out, long long out_stride,
                                      const void* kc, const void* vc, long long block_stride, int block_tokens,
                                      const int* block_table, int table_stride, const int* cu_q, const int* kv_lens,
                                      const float* alibi, const float* sinks, int B, int max_q_len, int Hq, int Hkv, int D,
                                      int Dv, int window, int keep, float scale, int num_blocks, const float* bias, int bias_len,
                                      const void* gate, long long gate_stride, float out_factor, int* err, cudaStream_t st) {
  if (B <= 0 || max_q_len <= 0) return 0;
  if (bias ? (bias_len <= 0 || sinks || alibi) : gate != nullptr) return -14;
  if (gate && ((reinterpret_cast<uintptr_t>(gate) & 15) || gate_stride % 8)) return -100;
  if (D <= 0 || Dv <= 0 || D > kFaD || Dv > kFaD || D % 8 || Dv % 8 || Hkv <= 0 || Hq % Hkv) return -100;
  const int G = Hq / Hkv;
  const int bt = block_tokens;
  if (G > kFaTile || !(bt == 8 || bt == 16 || bt == 32 || bt == 64 || bt == 128)) return -100;
  if (block_stride % 8 || num_blocks <= 0 || q_rows <= 0 || (out_stride % 8)) return -100;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kc) | reinterpret_cast<uintptr_t>(vc) |
       reinterpret_cast<uintptr_t>(out)) & 15 || (q_stride % 8)) return -100;
  FaEncodeFn enc = fa_encode_fn();
  if (!enc) return -100;
  CUtensorMap q_map, k_map, v_map;
  {
    cuuint64_t dims[3] = {static_cast<cuuint64_t>(D), static_cast<cuuint64_t>(Hq), static_cast<cuuint64_t>(q_rows)};
    cuuint64_t strides[2] = {static_cast<cuuint64_t>(D) * 2, static_cast<cuuint64_t>(q_stride) * 2};
    cuuint32_t box[3] = {64, static_cast<cuuint32_t>(G), static_cast<cuuint32_t>(kFaTile / G)};
    cuuint32_t estr[3] = {1, 1, 1};
    if (enc(&q_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS) return -100;
  }
  for (int which = 0; which < 2; ++which) {
    const int d = which ? Dv : D;
    cuuint64_t dims[3] = {static_cast<cuuint64_t>(d), static_cast<cuuint64_t>(Hkv) * bt, static_cast<cuuint64_t>(num_blocks)};
    cuuint64_t strides[2] = {static_cast<cuuint64_t>(d) * 2, static_cast<cuuint64_t>(block_stride) * 2};
    cuuint32_t box[3] = {64, static_cast<cuuint32_t>(bt), 1};
    cuuint32_t estr[3] = {1, 1, 1};
    if (enc(which ? &v_map : &k_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(which ? vc : kc), dims, strides, box,
            estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS) return -100;
  }
  static bool set = false;
  if (!set) {
    for (auto* k : {prefill_tc_kernel<false, false>, prefill_tc_kernel<true, false>, prefill_tc_kernel<false, true>, prefill_tc_kernel<true, true>})
      if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kFaSmemBytes + kFaBiasBytes) != cudaSuccess) return -3;
    set = true;
  }
  FaParams p{};
  p.out = static_cast<bf16*>(out); p.out_stride = out_stride;
  p.block_table = block_table; p.table_stride = table_stride; p.cu_q = cu_q; p.kv_lens = kv_lens; p.alibi = alibi;
  p.shared = kc == vc && D == Dv;
  p.sinks = sinks; p.D = D; p.Dv = Dv; p.window = window; p.keep = window > 0 ? keep : 0;
  p.Hq = Hq; p.Hkv = Hkv; p.G = G; p.block_tokens = bt; p.rows = kFaTile / G * G;
  p.scale_log2 = scale * 1.44269504f;
  p.err = err;
  p.bias = bias; p.bias_len = bias_len; p.gate = static_cast<const bf16*>(gate); p.gate_stride = gate_stride; p.out_factor = out_factor;
  const int pitch = (bias_len + 2 * kFaTile) | 1;                                          // odd: heads in different banks
  const long long table = bias ? static_cast<long long>(G) * pitch * 4 : 0;
  p.bias_ld = table > 0 && table <= kFaBiasBytes ? pitch : 0;
  const int smem = kFaSmemBytes + (p.bias_ld ? static_cast<int>(table) : 0);
  dim3 grid((max_q_len * G + p.rows - 1) / p.rows, Hkv, B);
  auto* kernel = bias ? (window > 0 ? prefill_tc_kernel<true, true> : prefill_tc_kernel<false, true>)
                      : (window > 0 ? prefill_tc_kernel<true, false> : prefill_tc_kernel<false, false>);
  kernel<<<grid, kFaThreads, smem, st>>>(q_map, k_map, v_map, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
