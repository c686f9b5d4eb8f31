// Prompt attention through a sliding window on the 5th-generation tensor cores, over keys and values that were formed
// for this pass (latent attention in its expanded form): causal, varlen, aware of cached positions before the new ones.
// Key sizes up to 256 and value sizes up to 128, multiples of 64; every query head has its own keys and values.  An optional gate
// [T, H * DV] multiplies the result element by element with its sigmoid.
//
//   kv [rows, H * DK | H * DV]: request b's keys are rows cu_kv[b] .., position kv_start[b] first
//   a query sees its own position and the window - 1 before it  (window 0: all before it)
//
// One CTA computes 128 query rows of one (request, head), as in attention_tc.cu: per tile of 128 keys (64 for key sizes above 128) S = Q . K^T into one of
// two tensor-memory buffers, softmax by eight warps (two threads per query row), P . V into a third buffer that the
// softmax threads add to their fp32 rows.  What differs:
//   * the tiles are rows of a dense matrix, so one thread fetches them with TMA (64 columns x BN rows per box, 128-byte
//     swizzle); only the tiles the window reaches are visited
//   * the weights enter P . V as the sum of two bf16 tiles (high and low part): they keep fp32-like precision
#include "sm100_ptx.cuh"

using namespace llb;
using namespace llb::sm100;

namespace {

constexpr int BM = 128;
constexpr int BLOCK_BYTES = 128 * 128;  // 128 rows x 64 bf16
constexpr int THREADS = 10 * 32;        // warp 0: TMA, warp 1: MMA, warps 2..9: softmax
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint64_t kIssueWaitNs = 2000000000ull;

__device__ int g_window_tc_status = 0;

template <int DK, int DV, int BN>
struct Layout {
  static constexpr int KV_BLOCK = BN * 128;  // BN rows x 64 bf16
  static constexpr int Q_BYTES = DK / 64 * BLOCK_BYTES, P_BYTES = BN / 64 * BLOCK_BYTES;
  static constexpr int K_BYTES = DK / 64 * KV_BLOCK, V_BYTES = DV / 64 * KV_BLOCK;
  static constexpr int OFF_Q = 0, OFF_PH = Q_BYTES, OFF_PL = OFF_PH + P_BYTES, OFF_KV = OFF_PL + P_BYTES;
  static constexpr int STAGE = K_BYTES + V_BYTES;
  static constexpr int OFF_BAR = OFF_KV + 2 * STAGE;
  static constexpr int OFF_XCH = OFF_BAR + 256;  // float [2 tile parities][2 halves][128 rows]
  // the dynamic shared memory starts on a 1024-byte boundary (checked in the kernel), so no slack is added
  static constexpr int BYTES = OFF_XCH + 2 * 2 * 128 * 4;
};

// byte offset of 16-byte chunk `ch` of row `r` inside a tile of 64-column blocks
__device__ __forceinline__ uint32_t tile_off(int r, int ch) {
  return (uint32_t)((ch >> 3) * BLOCK_BYTES + r * 128 + (((ch & 7) ^ (r & 7)) << 4));
}
__device__ __forceinline__ float ex2_fast(float x) {  // 2^x, one MUFU instruction (x = -inf gives 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct Params {
  const int *cu_q, *cu_kv, *kv_start, *b_ready_len;
  bf16* out;
  int64_t out_stride;
  const bf16* gate;  // [T, >= H * DV] or null
  int64_t gate_stride;
  int H, window;
  float scale_log2;
};

template <int DK, int DV, int BN>
__global__ void __launch_bounds__(THREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV, const Params p) {
  using L = Layout<DK, DV, BN>;
  constexpr int HK = BN / 2;  // keys of a score tile per softmax thread
  extern __shared__ __align__(1024) uint8_t smem[];
  const uint32_t smem_base = smem_u32(smem);
  const uint32_t bar_base = smem_base + L::OFF_BAR;
  auto k_full = [&](int s) { return bar_base + 8 * s; };
  auto v_full = [&](int s) { return bar_base + 8 * (2 + s); };
  auto k_empty = [&](int s) { return bar_base + 8 * (4 + s); };
  auto v_empty = [&](int s) { return bar_base + 8 * (6 + s); };
  auto s_full = [&](int b) { return bar_base + 8 * (8 + b); };
  const uint32_t p_full = bar_base + 8 * 10, pv_full = bar_base + 8 * 11, q_full = bar_base + 8 * 12;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::OFF_BAR + 128);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::OFF_BAR + 132);
  float* xch = reinterpret_cast<float*>(smem + L::OFF_XCH);
  int* status = &g_window_tc_status;

  const int b = blockIdx.z, h = blockIdx.y;
  const int q_begin = p.cu_q[b];
  const int q_len = p.cu_q[b + 1] - q_begin;
  const int q0 = (int)(gridDim.x - 1 - blockIdx.x) * BM;  // late tiles first
  if (q0 >= q_len) return;                                // whole CTA: nothing allocated yet
  if (smem_base & 1023u) {
    if (threadIdx.x == 0) atomicCAS(status, 0, 60);
    return;
  }
  const int ready = p.b_ready_len[b];
  const int rows_valid = min(BM, q_len - q0);
  const int kv_end = ready + q0 + rows_valid;  // exclusive bound on the keys any row of this tile may see
  const int kv0 = p.window > 0 ? max(p.kv_start[b], ready + q0 - p.window + 1) : p.kv_start[b];
  const int row0 = p.cu_kv[b] + kv0 - p.kv_start[b];
  const int n_tiles = (kv_end - kv0 + BN - 1) / BN;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

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
    mbar_init(q_full, 1);
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

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmKV);
      mbar_expect_tx(q_full, L::Q_BYTES);
#pragma unroll
      for (int c = 0; c < DK / 64; ++c)
        tma_load_2d(smem_base + L::OFF_Q + c * BLOCK_BYTES, &tmQ, q_full, h * DK + c * 64, q_begin + q0);
      for (int j = 0; j < n_tiles; ++j) {
        const int stage = j & 1;
        const uint32_t par = (((uint32_t)j >> 1) & 1u) ^ 1u;
        const uint32_t k_dst = smem_base + L::OFF_KV + stage * L::STAGE, v_dst = k_dst + L::K_BYTES;
        if (!mbar_wait(k_empty(stage), par, abort_flag, status, 61)) break;
        mbar_expect_tx(k_full(stage), L::K_BYTES);
#pragma unroll
        for (int c = 0; c < DK / 64; ++c)
          tma_load_2d(k_dst + c * L::KV_BLOCK, &tmKV, k_full(stage), h * DK + c * 64, row0 + j * BN);
        if (!mbar_wait(v_empty(stage), par, abort_flag, status, 62)) break;
        mbar_expect_tx(v_full(stage), L::V_BYTES);
#pragma unroll
        for (int c = 0; c < DV / 64; ++c)
          tma_load_2d(v_dst + c * L::KV_BLOCK, &tmKV, v_full(stage), p.H * DK + h * DV + c * 64, row0 + j * BN);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      // ---- MMA issuer: scores of tile s and P.V of tile t are issued in whichever order their inputs arrive ----
      constexpr uint32_t IDESC_S = umma_idesc(BM, BN, 1);
      constexpr uint32_t IDESC_PV = umma_idesc(BM, 64, 1) | (1u << 16);  // B operand MN-major
      int s_next = 0, pv_next = 0;
      mbar_wait(q_full, 0, abort_flag, status, 63);
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
                      umma_smem_desc_sw128(smem_base + L::OFF_Q + (ks >> 2) * BLOCK_BYTES + (ks & 3) * 32),
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
            for (int part = 0; part < 2; ++part) {  // high, then low part of the weights
              const uint32_t p_addr = smem_base + (part == 0 ? L::OFF_PH : L::OFF_PL);
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
            atomicCAS(status, 0, 64);
            break;
          }
        }
      }
    }
    __syncwarp();
  } else {
    // ---- softmax + output accumulation.  Two threads per query row: `half` 0 owns the first half of the keys of every score
    // tile and of the value columns, half 1 the rest; they exchange the row maximum ----
    constexpr int OC = DV / 2;  // value columns per thread
    const int lane_grp = warp & 3;
    const int half = (warp - 2) >> 2;
    const int erow = lane_grp * 32 + lane;
    const int prow = ready + q0 + erow;  // absolute position of this row's token
    const uint32_t t_lane = tmem_base + ((uint32_t)(lane_grp * 32) << 16);
    const uint32_t t_s = t_lane + half * HK, t_o = t_lane + 2 * BN + half * OC;
    float o[OC];
#pragma unroll
    for (int i = 0; i < OC; ++i) o[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    for (int j = 0; j < n_tiles; ++j) {
      const int kt = kv0 + j * BN + half * HK;  // position of my first key
      mbar_wait(s_full(j & 1), ((uint32_t)j >> 1) & 1u, abort_flag, status, 65);
      tc_fence_after();
      uint32_t sr[HK];
#pragma unroll
      for (int c = 0; c < HK; c += 32) tmem_ld_32x32(t_s + (j & 1) * BN + c, sr + c);
      tmem_wait_ld();
      // my columns lo..hi are visible to this row
      const int hi = min(prow, kv_end - 1) - kt;
      const int lo = p.window > 0 ? prow - p.window + 1 - kt : 0;
      const bool all_visible = hi >= HK - 1 && lo <= 0;
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (!all_visible) {  // scores that are not seen: -inf, whose weight comes out as 0
#pragma unroll
        for (int e = 0; e < HK; ++e)
          if (e < lo || e > hi) sr[e] = 0xff800000u;
      }
#pragma unroll
      for (int e = 0; e < HK; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], __uint_as_float(sr[e]));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      float* x = xch + (j & 1) * 256;
      x[half * 128 + erow] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      mx = fmaxf(mx, x[(half ^ 1) * 128 + erow]);
      const float m_new = fmaxf(m_run, mx * p.scale_log2);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = ex2_fast(m_run - m_use);
      m_run = m_new;
      if (j > 0) {  // o = (o + P V of the previous tile), then rescaled to the new maximum
        mbar_wait(pv_full, (uint32_t)(j - 1) & 1u, abort_flag, status, 66);
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
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
          float pv[2];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int c = g * 8 + e + u;
            pv[u] = ex2_fast(fmaf(__uint_as_float(sr[c]), p.scale_log2, -m_use));
            rs4[(e + u) & 3] += pv[u];
          }
          ph[e / 2] = pack_bf16x2(pv[0], pv[1]);
          pl[e / 2] = pack_bf16x2(pv[0] - __uint_as_float(ph[e / 2] << 16),
                                  pv[1] - __uint_as_float(ph[e / 2] & 0xffff0000u));
        }
        const uint32_t off = tile_off(erow, half * (HK / 8) + g);
        *reinterpret_cast<uint4*>(smem + L::OFF_PH + off) = make_uint4(ph[0], ph[1], ph[2], ph[3]);
        *reinterpret_cast<uint4*>(smem + L::OFF_PL + off) = make_uint4(pl[0], pl[1], pl[2], pl[3]);
      }
      l_run = l_run * alpha + (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);
      tc_fence_before();    // my reads of S and of the previous P V are done
      fence_proxy_async();  // my P stores are visible to the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    mbar_wait(pv_full, (uint32_t)(n_tiles - 1) & 1u, abort_flag, status, 67);
    tc_fence_after();
    // total row sum = my keys + the other half's keys
    float* x = xch + (n_tiles & 1) * 256;
    x[half * 128 + erow] = l_run;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float l_tot = l_run + x[(half ^ 1) * 128 + erow];
    const float inv = l_tot > 0.f ? 1.f / l_tot : 0.f;
    // output: every warp parks its 32 rows x OC columns in its own part of the (now idle) Q / P buffers and writes
    // whole lines
    constexpr int PITCH = OC * 2 + 16;  // bytes per parked row
    constexpr int SEGS = OC / 8;
    uint8_t* stg = smem + L::OFF_Q + (warp - 2) * (32 * PITCH);
    {
      uint32_t r[OC];
#pragma unroll
      for (int c = 0; c < OC; c += 32) tmem_ld_32x32(t_o + c, r + c);
      tmem_wait_ld();
#pragma unroll
      for (int g = 0; g < SEGS; ++g) {
        uint32_t w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = g * 8 + 2 * e;
          w[e] = pack_bf16x2((o[c] + __uint_as_float(r[c])) * inv, (o[c + 1] + __uint_as_float(r[c + 1])) * inv);
        }
        *reinterpret_cast<uint4*>(stg + lane * PITCH + g * 16) = make_uint4(w[0], w[1], w[2], w[3]);
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < SEGS; ++i) {
      const int id = i * 32 + lane, r = id / SEGS, seg = id % SEGS;
      const int lr = lane_grp * 32 + r;
      if (lr < rows_valid) {
        const int64_t row = q_begin + q0 + lr;
        const int col = h * DV + half * OC + seg * 8;
        bf16x8 v = *reinterpret_cast<const bf16x8*>(stg + r * PITCH + seg * 16);
        if (p.gate != nullptr) {
          float f[8], g[8];
          unpack8(v, f);
          unpack8(*reinterpret_cast<const bf16x8*>(p.gate + row * p.gate_stride + col), g);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = __fdividef(f[e], 1.f + __expf(-g[e]));
          v = pack8(f);
        }
        *reinterpret_cast<bf16x8*>(p.out + row * p.out_stride + col) = v;
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

template <int DK, int DV, int BN>
int launch(const CUtensorMap& tq, const CUtensorMap& tkv, const Params& p, int B, int max_q_len, cudaStream_t st) {
  using L = Layout<DK, DV, BN>;
  static_assert(L::BYTES <= 227 * 1024, "shared memory");
  static_assert(8 * 32 * (DV + 16) <= L::OFF_KV, "output staging fits the Q / P buffers");
  static DeviceOnce configured;
  if (!configured.done()) {
    cudaError_t e = cudaFuncSetAttribute(window_prefill_kernel<DK, DV, BN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         L::BYTES);
    if (e != cudaSuccess) return (int)e;
    configured.set();
  }
  const dim3 grid((max_q_len + BM - 1) / BM, p.H, B);
  window_prefill_kernel<DK, DV, BN><<<grid, THREADS, L::BYTES, st>>>(tq, tkv, p);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

}  // namespace

// 0 while every bounded wait of the kernel was met; 60: shared memory not where the layout needs it.
LLB_EXPORT int llb_window_tc_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_window_tc_status, sizeof(int));
  return v;
}

// q [T, >= H * DK] bf16 (row pitch q_stride), kv [kv_rows, H * (DK + DV)] (pitch kv_stride), out [T, H * DV]; gate
// [T, >= H * DV] or null: out *= sigmoid(gate).
LLB_EXPORT int llb_window_prefill_tc(const void* q, int64_t q_stride, const void* kv, int64_t kv_stride, int kv_rows,
                                     const int* cu_q, const int* cu_kv, const int* kv_start, const int* b_ready_len,
                                     void* out, int64_t out_stride, int B, int T, int max_q_len, int H, int dk, int dv,
                                     float sm_scale, int window, const void* gate, int64_t gate_stride,
                                     cudaStream_t st) {
  if (B <= 0 || max_q_len <= 0 || T <= 0) return LLB_OK;
  if (!(sm_scale > 0.f) || H <= 0 || H > 65535 || B > 65535 || kv_rows <= 0 || window < 0) return LLB_ERR_BAD_ARG;
  if ((dk != 64 && dk != 128 && dk != 192 && dk != 256) || (dv != 64 && dv != 128)) return LLB_ERR_UNSUPPORTED;
  if (gate != nullptr && ((gate_stride % 8) || ((uintptr_t)gate & 15))) return LLB_ERR_BAD_ARG;
  const int bn = dk > 128 ? 64 : 128;
  if ((out_stride % 8) || ((uintptr_t)out & 15)) return LLB_ERR_BAD_ARG;
  CUtensorMap tq, tkv;
  int rc = make_tmap_2d(&tq, q, 2, (uint64_t)T, (uint64_t)H * dk, (uint64_t)q_stride, BM, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tkv, kv, 2, (uint64_t)kv_rows, (uint64_t)H * (dk + dv), (uint64_t)kv_stride, bn, 64);
  if (rc) return rc;
  const Params p{cu_q, cu_kv, kv_start, b_ready_len, (bf16*)out, out_stride, (const bf16*)gate, gate_stride, H, window,
                 sm_scale * kLog2e};
#define LLB_WINDOW(DK, BN)                                                                                        \
  if (dk == DK)                                                                                                   \
    return dv == 64 ? launch<DK, 64, BN>(tq, tkv, p, B, max_q_len, st) : launch<DK, 128, BN>(tq, tkv, p, B, max_q_len, st);
  LLB_WINDOW(64, 128)
  LLB_WINDOW(128, 128)
  LLB_WINDOW(192, 64)
  LLB_WINDOW(256, 64)
#undef LLB_WINDOW
  return LLB_ERR_UNSUPPORTED;
}
