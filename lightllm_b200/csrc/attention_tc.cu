// Prefill attention on the 5th-generation tensor cores (tcgen05 + tensor memory), causal, varlen, aware of an already cached
// prefix, K/V read through the token-granular slot table of the KV pool.  Head size 128, and a windowed form with key sizes
// up to 256, any multiple of 64 as value size, chunks of positions, kept first positions, biases by distance, soft-capped scores, and
// a sigmoid gate on the output.
//
// One CTA computes 128 query rows of one (request, query head).  Per 128-key tile (64 keys for key sizes above 128):
//   S  = Q . K^T            tcgen05.mma into one of two tensor-memory buffers
//   P  = exp2(S - m)        the eight softmax warps (two threads per query row) read S back, keep the running
//                           maximum / sum and write P as bf16 into shared memory in the operand layout
//   PV = P . V              tcgen05.mma into a third buffer, started from zero for every tile; the softmax
//                           threads add it to their fp32 output row in registers, rescaled when the maximum moves
// The MMA thread issues S of tile j + 1 before it waits for P of tile j, so the tensor core works on the next
// scores while the softmax of the current tile runs.  K and V tiles are gathered row by row (one row per
// token and KV head) with 16-byte asynchronous copies straight into the 128-byte-swizzled operand layout; each
// of the two stages has its own K warp and V warp, so two tiles are always in flight.  V is consumed in the
// layout it has in memory (keys x head-dim, head-dim contiguous) as an MN-major B operand, 64 head-dim columns
// per instruction so that one swizzle atom spans the whole MN extent.
//
// Behavioural counterpart in the reference: lightllm/common/basemodel/triton_kernel/att/prefill_att/
// context_flashattention_nopad.py and the FlashInfer paged prefill wrapper
// (lightllm/common/basemodel/attention/flashinfer/).
#include "sm100_ptx.cuh"

using namespace llb;
using namespace llb::sm100;
LLB_DEBUG_BOUNDS_STORAGE(attention_tc)


namespace {

constexpr int BM = 128;
constexpr int BLOCK_BYTES = 128 * 128;      // 128 rows x 64 bf16 (one swizzle-wide column block)
constexpr int THREADS = 11 * 32;  // warp 0, 10: K/V gather of stage 0, 1; warp 1: MMA; warps 2..9: softmax
// shared memory: Q | P (high part, low part) | 2 stages x (K, V) | barriers | row-maximum / row-sum exchange
template <int DK, int DV, int BN, bool SPLIT_P>
struct PrefillLayout {
  static constexpr int KV_BLOCK = BN * 128;  // BN rows x 64 bf16
  static constexpr int Q_BYTES = DK / 64 * BLOCK_BYTES, P_BYTES = BN / 64 * BLOCK_BYTES;
  static constexpr int K_BYTES = DK / 64 * KV_BLOCK, V_BYTES = DV / 64 * KV_BLOCK, STAGE = K_BYTES + V_BYTES;
  static constexpr int OFF_Q = 0, OFF_P = Q_BYTES, OFF_KV = OFF_P + (SPLIT_P ? 2 : 1) * P_BYTES;
  static constexpr int OFF_BAR = OFF_KV + 2 * STAGE;
  static constexpr int OFF_XCH = OFF_BAR + 256;  // float [2 tile parities][2 halves][128 rows]
  // the dynamic shared memory starts on a 1024-byte boundary (checked in the kernel), so no slack is added
  static constexpr int BYTES = OFF_XCH + 2 * 2 * 128 * 4;
};
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint64_t kIssueWaitNs = 2000000000ull;

__device__ int g_attn_tc_status = 0;

// byte offset of 16-byte chunk `ch` (8 head-dim / key elements each) of row `r` inside a tile of 64-column blocks
template <int BLOCK>
__device__ __forceinline__ uint32_t tile_off(int r, int ch) {
  return (uint32_t)((ch >> 3) * BLOCK + r * 128 + (((ch & 7) ^ (r & 7)) << 4));
}

__device__ __forceinline__ float ex2_fast(float x) {  // 2^x, one MUFU instruction (x = -inf gives 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// v[e] (fp32 bits) = top * tanh(v[e] * in).  Where all of a warp's arguments x are small, the Taylor series
// x - x^3/3 + 2x^5/15 (|x| < 1/8), or up to 62x^9/2835 (|x| < 0.35), with a relative error below 3e-7; else top - 2 top / (1 + e^2x),
// whose absolute error (a few 1e-7 top) is that of rounding values of the cap's size.
template <int N>
__device__ __forceinline__ void cap_scores(uint32_t* v, float in, float top) {
  float big = 0.f;
#pragma unroll
  for (int e = 0; e < N; ++e) big = fmaxf(big, fabsf(__uint_as_float(v[e])));
  const float i2 = in * in, k1 = top * in;  // the series in powers of the score itself
  const float c3 = k1 * i2 * (-1.f / 3.f), c5 = k1 * i2 * i2 * (2.f / 15.f);
  if (__all_sync(0xffffffffu, big * in < 0.125f)) {
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const float x = __uint_as_float(v[e]), x2 = x * x;
      v[e] = __float_as_uint(x * fmaf(x2, fmaf(x2, c5, c3), k1));
    }
  } else if (__all_sync(0xffffffffu, big * in < 0.35f)) {
    const float c7 = k1 * i2 * i2 * i2 * (-17.f / 315.f), c9 = k1 * i2 * i2 * i2 * i2 * (62.f / 2835.f);
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const float x = __uint_as_float(v[e]), x2 = x * x;
      v[e] = __float_as_uint(x * fmaf(x2, fmaf(x2, fmaf(x2, fmaf(x2, c9, c7), c5), c3), k1));
    }
  } else {
    const float to2 = 2.f * kLog2e * in;
#pragma unroll
    for (int e = 0; e < N; ++e)
      v[e] = __float_as_uint(fmaf(-2.f * top, __fdividef(1.f, 1.f + ex2_fast(__uint_as_float(v[e]) * to2)), top));
  }
}

__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const bf162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// DK, DV: key size and the value columns of one CTA (a wider value head is shared out over CTAs: v_blocks per head).
// rule.window, rule.chunk: the positions a query sees (see KeyRule).  SPLIT_P: the weights enter P . V as the sum of two bf16
// tiles.  EXT: positions below rule.keep are seen at any distance (the tiles that hold them come ahead of the window's), scores
// are capped (rule.cap) and get the biases of rule.rel.  gate: factor on the output (OutGate, bf16).
template <int DK, int DV, int BN, bool SPLIT_P, bool EXT>
__global__ void __launch_bounds__(THREADS, 1)
gqa_prefill_tc_kernel(const bf16* __restrict__ q, int64_t q_stride, const bf16* __restrict__ kv_layer,
                      const int* __restrict__ req_to_token, int64_t r2t_stride, const int* __restrict__ b_req_idx,
                      const int* __restrict__ cu_q, const int* __restrict__ b_ready_len, bf16* __restrict__ out,
                      int64_t out_stride, int Hq, int Hkv, float scale_log2, int v_blocks, const KeyRule rule,
                      const OutGate gate) {
  using L = PrefillLayout<DK, DV, BN, SPLIT_P>;
  constexpr int HK = BN / 2;   // keys of a score tile per softmax thread
  constexpr int OC = DV / 2;   // value columns per softmax thread
  extern __shared__ __align__(1024) uint8_t smem_gen[];
  const uint32_t smem_base = smem_u32(smem_gen);
  const uint32_t bar_base = smem_base + L::OFF_BAR;
  auto k_full = [&](int s) { return bar_base + 8 * s; };
  auto v_full = [&](int s) { return bar_base + 8 * (2 + s); };
  auto k_empty = [&](int s) { return bar_base + 8 * (4 + s); };
  auto v_empty = [&](int s) { return bar_base + 8 * (6 + s); };
  auto s_full = [&](int b) { return bar_base + 8 * (8 + b); };
  const uint32_t p_full = bar_base + 8 * 10, pv_full = bar_base + 8 * 11, q_full = bar_base + 8 * 12;
  float* xch = reinterpret_cast<float*>(smem_gen + L::OFF_XCH);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem_gen + L::OFF_BAR + 128);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem_gen + L::OFF_BAR + 132);

  const int b = blockIdx.z, h = blockIdx.y / v_blocks, vb = blockIdx.y - h * v_blocks;
  const int kvh = h / (Hq / Hkv);
  const int q_begin = cu_q[b];
  const int q_len = cu_q[b + 1] - q_begin;
  const int tile = gridDim.x - 1 - blockIdx.x;  // heavy (late) tiles first
  const int q0 = tile * BM;
  if (q0 >= q_len) return;  // whole CTA: nothing allocated yet
  const int ready = b_ready_len[b];
  const int req = LLB_CHECK_REQ(b_req_idx[b]);
  const int rows_valid = min(BM, q_len - q0);
  const int kv_end = ready + q0 + rows_valid;  // exclusive bound on the keys any row of this tile may see
  const int kv0 = rule.first_seen(ready + q0);
  const int kept = EXT ? min(rule.keep, kv0) : 0;      // kept positions ahead of the window
  const int kept_tiles = EXT ? (kept + BN - 1) / BN : 0;
  const int n_tiles = kept_tiles + (kv_end - kv0 + BN - 1) / BN;
  // first position of tile j, and the exclusive bound on the positions it holds
  auto tile_pos = [&](int j) { return EXT && j < kept_tiles ? j * BN : kv0 + (j - kept_tiles) * BN; };
  auto tile_bound = [&](int j) { return EXT && j < kept_tiles ? kept : kv_end; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t r2t_base = (int64_t)req * r2t_stride;
  int* status = &g_attn_tc_status;
  if (smem_base & 1023u) {
    if (threadIdx.x == 0) atomicCAS(status, 0, 50);
    return;
  }

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int s = 0; s < 2; ++s) {
      mbar_init(k_full(s), 1);
      mbar_init(v_full(s), 1);
      mbar_init(k_empty(s), 1);
      mbar_init(v_empty(s), 1);
      mbar_init(s_full(s), 1);
    }
    mbar_init(p_full, 8);
    mbar_init(pv_full, 1);
    mbar_init(q_full, 8);
    fence_barrier_init();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  if (warp >= 2 && warp <= 9) {
    // Q tile -> shared memory in operand layout (rows beyond the request's tokens are zero), by the softmax warps
    // while the gather warps already fetch the first K / V tiles
    constexpr int CH = DK / 8;
    for (int c = threadIdx.x - 64; c < BM * CH; c += 256) {
      const int r = c / CH, ch = c % CH;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < rows_valid)
        v = *reinterpret_cast<const uint4*>(q + (int64_t)(q_begin + q0 + r) * q_stride + (int64_t)h * DK + ch * 8);
      *reinterpret_cast<uint4*>(smem_gen + L::OFF_Q + tile_off<BLOCK_BYTES>(r, ch)) = v;
    }
    fence_proxy_async();  // the tensor core reads Q through the async proxy
    __syncwarp();
    if (lane == 0) mbar_arrive(q_full);
  }

  if (warp == 0 || warp == 10) {
    // ---- K / V gather of one stage: tiles stage, stage + 2, ...  K is released as soon as its scores are done,
    // V after P.V, so the K copy of tile j + 2 is in flight while tile j + 1 is being worked on ----
    const int stage = warp == 0 ? 0 : 1;
    const uint32_t k_dst = smem_base + L::OFF_KV + stage * L::STAGE, v_dst = k_dst + L::K_BYTES;
    const int64_t row = (int64_t)Hkv * (DK + DV * v_blocks);
    const bf16* k_src = kv_layer + (int64_t)kvh * DK;
    const bf16* v_src = kv_layer + (int64_t)Hkv * DK + ((int64_t)kvh * v_blocks + vb) * DV;
    for (int j = stage; j < n_tiles; j += 2) {
      const uint32_t par = (((uint32_t)j >> 1) & 1u) ^ 1u;
      const int kt = tile_pos(j), bound = tile_bound(j);
      int slots[BN / 32];
#pragma unroll
      for (int u = 0; u < BN / 32; ++u) {
        const int pos = kt + u * 32 + lane;
        slots[u] = pos < bound ? LLB_CHECK_SLOT(req_to_token[r2t_base + pos]) : -1;
      }
      mbar_wait(k_empty(stage), par, abort_flag, status, 41);
#pragma unroll
      for (int u = 0; u < BN / 32; ++u) {  // keys 32 u .. 32 u + 31, one row after the other in 16-byte chunks
#pragma unroll 4
        for (int i = 0; i < DK / 8; ++i) {
          const int kk = (i * 32 + lane) / (DK / 8), ch = (i * 32 + lane) % (DK / 8);
          const int sl = __shfl_sync(0xffffffffu, slots[u], kk);
          cp_async16(k_dst + tile_off<L::KV_BLOCK>(u * 32 + kk, ch), k_src + (int64_t)(sl >= 0 ? sl : 0) * row + ch * 8,
                     sl >= 0);
        }
      }
      cp_async_commit();
      mbar_wait(v_empty(stage), par, abort_flag, status, 48);
#pragma unroll
      for (int u = 0; u < BN / 32; ++u) {
#pragma unroll 4
        for (int i = 0; i < DV / 8; ++i) {
          const int kk = (i * 32 + lane) / (DV / 8), ch = (i * 32 + lane) % (DV / 8);
          const int sl = __shfl_sync(0xffffffffu, slots[u], kk);
          cp_async16(v_dst + tile_off<L::KV_BLOCK>(u * 32 + kk, ch), v_src + (int64_t)(sl >= 0 ? sl : 0) * row + ch * 8,
                     sl >= 0);
        }
      }
      cp_async_commit();
      cp_async_wait<1>();  // K landed
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(k_full(stage));
      cp_async_wait<0>();  // V landed
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(v_full(stage));
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // ---- MMA issuer: scores of tile s and P.V of tile t are issued in whichever order their inputs arrive ----
      constexpr uint32_t IDESC_S = umma_idesc(BM, BN, 1);
      constexpr uint32_t IDESC_PV = umma_idesc(BM, 64, 1) | (1u << 16);  // B operand MN-major
      const uint32_t q_addr = smem_base + L::OFF_Q;
      int s_next = 0, pv_next = 0;
      mbar_wait(q_full, 0, abort_flag, status, 40);
      uint64_t t0 = 0;
      uint32_t spins = 0;
      while (pv_next < n_tiles) {
        // score buffer s_next & 1 was last read for tile s_next - 2: free once that tile's P has been seen
        if (s_next < n_tiles && s_next < pv_next + 2 && mbar_test_wait(k_full(s_next & 1), ((uint32_t)s_next >> 1) & 1u)) {
          tc_fence_after();
          const uint32_t k_addr = smem_base + L::OFF_KV + (s_next & 1) * L::STAGE;
#pragma unroll
          for (int ks = 0; ks < DK / 16; ++ks) {
            umma_bf16(tmem_base + (s_next & 1) * BN,
                      umma_smem_desc_sw128(q_addr + (ks >> 2) * BLOCK_BYTES + (ks & 3) * 32),
                      umma_smem_desc_sw128(k_addr + (ks >> 2) * L::KV_BLOCK + (ks & 3) * 32), IDESC_S, ks != 0);
          }
          umma_commit(s_full(s_next & 1));
          umma_commit(k_empty(s_next & 1));
          ++s_next;
          spins = 0;
          t0 = 0;
          continue;
        }
        if (pv_next < s_next && mbar_test_wait(p_full, (uint32_t)pv_next & 1u) &&
            mbar_test_wait(v_full(pv_next & 1), ((uint32_t)pv_next >> 1) & 1u)) {
          tc_fence_after();
          const uint32_t v_addr = smem_base + L::OFF_KV + (pv_next & 1) * L::STAGE + L::K_BYTES;
#pragma unroll
          for (int hb = 0; hb < DV / 64; ++hb) {  // value columns 64 hb .. 64 hb + 63
#pragma unroll
            for (int part = 0; part < (SPLIT_P ? 2 : 1); ++part) {  // high, then low part of the weights
              const uint32_t p_addr = smem_base + L::OFF_P + part * L::P_BYTES;
#pragma unroll
              for (int ks = 0; ks < BN / 16; ++ks) {  // 16 keys per instruction
                const uint32_t a_off = (ks >> 2) * BLOCK_BYTES + (ks & 3) * 32;
                umma_bf16(tmem_base + 2 * BN + hb * 64, umma_smem_desc_sw128(p_addr + a_off),
                          umma_smem_desc_sw128_mn(v_addr + hb * L::KV_BLOCK + ks * 2048), IDESC_PV, (part | ks) != 0);
              }
            }
          }
          umma_commit(pv_full);
          umma_commit(v_empty(pv_next & 1));
          ++pv_next;
          spins = 0;
          t0 = 0;
          continue;
        }
        if ((++spins & 0xff) == 0) {  // bounded: give up after two seconds without progress
          if (*abort_flag) break;
          const uint64_t now = global_timer_ns();
          if (t0 == 0) {
            t0 = now;
          } else if (now - t0 > kIssueWaitNs) {
            *abort_flag = 1;
            atomicCAS(status, 0, 49);
            break;
          }
        }
      }
    }
  } else {
    // ---- softmax + output accumulation: warps 2..9.  Two threads per query row: `half` 0 owns the first half of the
    // keys of every score tile and of the output columns, half 1 the rest; they exchange the row maximum ----
    const int lane_grp = warp & 3;
    const int half = (warp - 2) >> 2;
    const int erow = lane_grp * 32 + lane;
    const int prow = ready + q0 + erow;  // absolute position of this row's token
    const int row_first = rule.first_seen(prow);
    const uint32_t t_lane = tmem_base + ((uint32_t)(lane_grp * 32) << 16);
    const uint32_t t_s = t_lane + half * HK, t_o = t_lane + 2 * BN + half * OC;
    uint8_t* p_tile = smem_gen + L::OFF_P;
    float o[OC];
#pragma unroll
    for (int i = 0; i < OC; ++i) o[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    const float* rel = EXT && rule.rel != nullptr ? rule.rel + h * rule.rel_stride : nullptr;
    const float far_bias = EXT && rel != nullptr ? rel[rule.far] * kLog2e : 0.f;
    for (int j = 0; j < n_tiles; ++j) {
      const int kt = tile_pos(j) + half * HK;
      mbar_wait(s_full(j & 1), ((uint32_t)j >> 1) & 1u, abort_flag, status, 45);
      tc_fence_after();
      uint32_t sr[HK];
#pragma unroll
      for (int c = 0; c < HK; c += 32) tmem_ld_32x32(t_s + (j & 1) * BN + c, sr + c);
      tmem_wait_ld();
      const int lim = min(prow, tile_bound(j) - 1) - kt;  // my columns lo..lim (and those below `first`) are visible to this row
      const int lo = row_first - kt;
      const int first = EXT ? rule.keep - kt : 0;
      auto seen = [&](int c) { return c <= lim && (c >= lo || (EXT && c < first)); };
      // whole tile (every tile but those at the diagonal and the edges)
      const bool all_visible = lim >= HK - 1 && (lo <= 0 || (EXT && first >= HK));
      float to_log2 = scale_log2, shift = 0.f;  // score in log2 units = sr * to_log2 + shift
      if (EXT && rule.cap > 0.f) {
        cap_scores<HK>(sr, scale_log2 * (1.f / kLog2e) / rule.cap, rule.cap * kLog2e);
        to_log2 = 1.f;
      }
      if (EXT && rel != nullptr) {
        const int dist = prow - kt;  // of my first column; the last one is HK - 1 nearer
        if (dist - (HK - 1) >= rule.far) {
          shift = far_bias;
        } else {  // columns of a negative distance are not seen, whatever they are added
          const float* at = rel + max(dist, 0);
          const float scale = to_log2 * (1.f / kLog2e);
          to_log2 = kLog2e;
#pragma unroll
          for (int e = 0; e < HK; ++e) sr[e] = __float_as_uint(fmaf(__uint_as_float(sr[e]), scale, at[-e]));
        }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (!all_visible) {  // scores that are not seen: -inf, whose weight comes out as 0
#pragma unroll
        for (int e = 0; e < HK; ++e)
          if (!seen(e)) sr[e] = 0xff800000u;
      }
#pragma unroll
      for (int e = 0; e < HK; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], __uint_as_float(sr[e]));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      if (EXT) mx = fmaf(mx, to_log2, shift);
      float* x = xch + (j & 1) * 256;
      x[half * 128 + erow] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      mx = fmaxf(mx, x[(half ^ 1) * 128 + erow]);
      const float m_new = fmaxf(m_run, EXT ? mx : mx * to_log2);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = ex2_fast(m_run - m_use);
      m_run = m_new;
      if (j > 0) {  // o = (o + P V of the previous tile), then rescaled to the new maximum
        mbar_wait(pv_full, (uint32_t)(j - 1) & 1u, abort_flag, status, 46);
        tc_fence_after();
        uint32_t r[OC];
#pragma unroll
        for (int c = 0; c < OC; c += 32) tmem_ld_32x32(t_o + c, r + c);
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < OC; ++e) o[e] = (o[e] + __uint_as_float(r[e])) * alpha;
      }
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int g = 0; g < HK / 8; ++g) {
        float pv[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int c = g * 8 + e;
          pv[e] = ex2_fast(fmaf(__uint_as_float(sr[c]), to_log2, EXT ? shift - m_use : -m_use));
          rs4[e & 3] += pv[e];
        }
        const uint32_t off = tile_off<BLOCK_BYTES>(erow, half * (HK / 8) + g);
        uint32_t ph[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) ph[e] = pack2(pv[2 * e], pv[2 * e + 1]);
        *reinterpret_cast<uint4*>(p_tile + off) = make_uint4(ph[0], ph[1], ph[2], ph[3]);
        if (SPLIT_P) {
          uint32_t pl[4];
#pragma unroll
          for (int e = 0; e < 4; ++e)
            pl[e] = pack2(pv[2 * e] - __uint_as_float(ph[e] << 16), pv[2 * e + 1] - __uint_as_float(ph[e] & 0xffff0000u));
          *reinterpret_cast<uint4*>(p_tile + L::P_BYTES + off) = make_uint4(pl[0], pl[1], pl[2], pl[3]);
        }
      }
      l_run = l_run * alpha + (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);
      tc_fence_before();    // my reads of S and of the previous P V are done
      fence_proxy_async();  // my P stores are visible to the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    mbar_wait(pv_full, (uint32_t)(n_tiles - 1) & 1u, abort_flag, status, 47);
    tc_fence_after();
    // total row sum = my keys + the other half's keys
    float* x = xch + (n_tiles & 1) * 256;
    x[half * 128 + erow] = l_run;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float l_tot = l_run + x[(half ^ 1) * 128 + erow];
    float inv = l_tot > 0.f ? gate.scale / l_tot : 0.f;
    const bf16* gt = reinterpret_cast<const bf16*>(gate.gate);
    if (gt != nullptr && !gate.elem && erow < rows_valid)
      inv = __fdividef(inv, 1.f + __expf(-__bfloat162float(gt[(int64_t)(q_begin + q0 + erow) * gate.stride + h])));
    // output: every warp parks its 32 rows x OC columns in its own part of the (now idle) Q / P buffers and
    // writes whole lines
    constexpr int PITCH = OC * 2 + 16, SEGS = OC / 8;
    static_assert(8 * 32 * PITCH <= L::OFF_KV, "output staging fits the Q / P buffers");
    uint8_t* stg = smem_gen + L::OFF_Q + (warp - 2) * (32 * PITCH);
    {
      uint32_t r[OC];
#pragma unroll
      for (int c = 0; c < OC; c += 32) tmem_ld_32x32(t_o + c, r + c);
      tmem_wait_ld();
#pragma unroll
      for (int g = 0; g < SEGS; ++g) {
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = (o[g * 8 + e] + __uint_as_float(r[g * 8 + e])) * inv;
        *reinterpret_cast<uint4*>(stg + lane * PITCH + g * 16) =
            make_uint4(pack2(v[0], v[1]), pack2(v[2], v[3]), pack2(v[4], v[5]), pack2(v[6], v[7]));
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < SEGS; ++i) {
      const int id = i * 32 + lane, r = id / SEGS, seg = id % SEGS;
      const int lr = lane_grp * 32 + r;
      if (lr < rows_valid) {
        const int64_t row = q_begin + q0 + lr, col = ((int64_t)h * v_blocks + vb) * DV + half * OC + seg * 8;
        bf16x8 v = *reinterpret_cast<const bf16x8*>(stg + r * PITCH + seg * 16);
        if (gt != nullptr && gate.elem) {
          float f[8], gv[8];
          unpack8(v, f);
          unpack8(*reinterpret_cast<const bf16x8*>(gt + row * gate.stride + col), gv);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = __fdividef(f[e], 1.f + __expf(-gv[e]));
          v = pack8(f);
        }
        *reinterpret_cast<bf16x8*>(out + row * out_stride + col) = v;
      }
    }
    tc_fence_before();
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DK, int DV, int BN, bool SPLIT_P, bool EXT>
int launch_tc(const bf16* q, int64_t q_stride, const bf16* kv_layer, const int* req_to_token, int64_t r2t_stride,
              const int* b_req_idx, const int* cu_q, const int* b_ready_len, bf16* out, int64_t out_stride, int B,
              int max_q_len, int Hq, int Hkv, float sm_scale, int v_blocks, const KeyRule& rule, const OutGate& gate,
              cudaStream_t st) {
  using L = PrefillLayout<DK, DV, BN, SPLIT_P>;
  static_assert(L::BYTES <= 227 * 1024, "shared memory");
  static DeviceOnce configured;
  if (!configured.done()) {
    cudaError_t e = cudaFuncSetAttribute(gqa_prefill_tc_kernel<DK, DV, BN, SPLIT_P, EXT>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, L::BYTES);
    if (e != cudaSuccess) return (int)e;
    configured.set();
  }
  const dim3 grid((max_q_len + BM - 1) / BM, Hq * v_blocks, B);
  gqa_prefill_tc_kernel<DK, DV, BN, SPLIT_P, EXT><<<grid, THREADS, L::BYTES, st>>>(
      q, q_stride, kv_layer, req_to_token, r2t_stride, b_req_idx, cu_q, b_ready_len, out, out_stride, Hq, Hkv,
      sm_scale * kLog2e, v_blocks, rule, gate);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

}  // namespace

LLB_EXPORT int llb_attn_tc_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_attn_tc_status, sizeof(int));
  return v;
}

// Same contract as llb_gqa_prefill (head size 128 only): q [T, Hq, 128] new tokens of all requests back to back.
LLB_EXPORT int llb_gqa_prefill_tc(const void* q, int64_t q_stride, const void* kv_layer, const int* req_to_token,
                                  int64_t r2t_stride, const int* b_req_idx, const int* cu_q, const int* b_ready_len,
                                  void* out, int64_t out_stride, int B, int max_q_len, int Hq, int Hkv, float sm_scale,
                                  cudaStream_t st) {
  if (B <= 0 || max_q_len <= 0) return LLB_OK;
  if (!(sm_scale > 0.f) || Hkv <= 0 || Hq % Hkv != 0 || (q_stride % 8) || (out_stride % 8) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15))
    return LLB_ERR_BAD_ARG;
  return launch_tc<128, 128, 128, false, false>((const bf16*)q, q_stride, (const bf16*)kv_layer, req_to_token, r2t_stride, b_req_idx,
                                         cu_q, b_ready_len, (bf16*)out, out_stride, B, max_q_len, Hq, Hkv, sm_scale, 1, KeyRule{},
                                         OutGate{nullptr, 0, 1.f, 0}, st);
}

// Key size dk (64, 128, 192, 256), value size dv (a multiple of 64), window or chunk (0: none), first `keep` positions always seen,
// biases by distance rel [Hq, far + 1] (or null), cap on the scores (0: none; see KeyRule): pool rows [Hkv * dk | Hkv * dv], q
// [T, >= Hq * dk], out [T, >= Hq * dv].  gate [T, >= Hq], with gate_elem [T, >= Hq * dv], or null: the output times
// out_scale * sigmoid(gate).
LLB_EXPORT int llb_window_gqa_prefill_tc(const void* q, int64_t q_stride, const void* kv_layer, const int* req_to_token,
                                         int64_t r2t_stride, const int* b_req_idx, const int* cu_q, const int* b_ready_len,
                                         void* out, int64_t out_stride, int B, int max_q_len, int Hq, int Hkv, int dk,
                                         int dv, float sm_scale, int window, int keep, const float* rel, int far,
                                         int64_t rel_stride, int chunk, float cap, const void* gate, int64_t gate_stride,
                                         int gate_elem, float out_scale, cudaStream_t st) {
  if (B <= 0 || max_q_len <= 0) return LLB_OK;
  if (!(sm_scale > 0.f) || Hkv <= 0 || Hq % Hkv != 0 || (q_stride % 8) || (out_stride % 8) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15) ||
      window < 0 || keep < 0 || (rel != nullptr && far < 0) || dv <= 0 || chunk < 0 || (chunk > 0 && window > 0) || !(cap >= 0.f) ||
      (gate_elem && ((gate_stride % 8) || ((uintptr_t)gate & 15))))
    return LLB_ERR_BAD_ARG;
  const KeyRule rule{window, keep, rel, far, rel_stride, chunk, cap};
  const OutGate og{gate, gate_stride, out_scale, gate_elem};
  const bool ext = ((window > 0 || chunk > 0) && keep > 0) || rel != nullptr || cap > 0.f;
  if ((dv % 64) || (dk != 64 && dk != 128 && dk != 192 && dk != 256) || Hq * (dv / 64) > 65535 || B > 65535)
    return LLB_ERR_UNSUPPORTED;
#define LLB_WINDOW_TC(DK, DV, BN)                                                                                         \
  return (ext ? launch_tc<DK, DV, BN, true, true> : launch_tc<DK, DV, BN, true, false>)(                                  \
      (const bf16*)q, q_stride, (const bf16*)kv_layer, req_to_token, r2t_stride, b_req_idx, cu_q, b_ready_len, (bf16*)out, \
      out_stride, B, max_q_len, Hq, Hkv, sm_scale, dv / DV, rule, og, st)
  if (dv % 128 == 0) {
    if (dk == 64) LLB_WINDOW_TC(64, 128, 128);
    if (dk == 128) LLB_WINDOW_TC(128, 128, 128);
    if (dk == 192) LLB_WINDOW_TC(192, 128, 64);
    LLB_WINDOW_TC(256, 128, 64);
  }
  if (dk == 64) LLB_WINDOW_TC(64, 64, 128);
  if (dk == 128) LLB_WINDOW_TC(128, 64, 128);
  if (dk == 192) LLB_WINDOW_TC(192, 64, 64);
  LLB_WINDOW_TC(256, 64, 64);
#undef LLB_WINDOW_TC
}
