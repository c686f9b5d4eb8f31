// Paged causal attention for the layer shapes the tensor-core kernels do not cover: any head size up to
// 256 (Gemma 256, Phi-3 96, StableLM 80 ...; up to 512 in the form with its own value size, in bf16 or fp32),
// sliding windows (with kept first positions), chunks of positions, ALiBi slopes, tables of biases by distance, logit soft-capping, attention sinks and a sigmoid output gate (per head or per element).  One CTA per (query token, query head); its four warps stride over the keys, each
// keeps an online-softmax state with the head vector spread over the lanes, and the states are merged
// in shared memory.  Prefill and decode use the same kernel: a query is described by its position and
// the request row it belongs to.
//
// KV pool row layout (one layer): [slot][Hkv * D | Hkv * DV], K heads first, then V heads.
#include "common.cuh"

using namespace llb;

constexpr int GEN_WARPS = 4;
constexpr int GEN_MAX_EPL = 8;  // elements per lane: D <= 256

namespace {
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float v, float* p) { *p = v; }
__device__ __forceinline__ void from_f(float v, bf16* p) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float exp_for(float v, const float*) { return expf(v); }
__device__ __forceinline__ float exp_for(float v, const bf16*) { return __expf(v); }
}  // namespace

// EPL: elements per lane (sizes up to 32 * EPL).  gate: factor on the output (OutGate, format E).
template <typename E, int EPL>
__global__ void __launch_bounds__(GEN_WARPS * 32)
attn_generic_kernel(const E* __restrict__ q, int64_t q_stride, const E* __restrict__ kv,
                    const int* __restrict__ req_to_token, int64_t r2t_stride, const int* __restrict__ b_req_idx,
                    const int* __restrict__ pos, const int* __restrict__ batch_of, E* __restrict__ out,
                    int64_t out_stride, int Hq, int Hkv, int D, int DV, float sm_scale, const KeyRule rule,
                    const float* __restrict__ alibi, const float* __restrict__ sinks, const OutGate gate) {
  const int t = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = batch_of ? batch_of[t] : t;
  const int qpos = pos[t];
  const int kvh = h / (Hq / Hkv);
  const int* slots = req_to_token + (int64_t)b_req_idx[b] * r2t_stride;
  const int64_t row = (int64_t)Hkv * (D + DV);

  float qv[EPL], acc[EPL];
#pragma unroll
  for (int e = 0; e < EPL; ++e) {
    int d = lane + e * 32;
    qv[e] = d < D ? to_f(q[(int64_t)t * q_stride + (int64_t)h * D + d]) * sm_scale : 0.f;
    acc[e] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int j0 = rule.first_seen(qpos);
  const int kept = min(rule.keep, j0), n = kept + qpos + 1 - j0;  // kept first positions, then the window
  const float slope = alibi ? alibi[h] : 0.f;
  const float* rel = rule.rel ? rule.rel + h * rule.rel_stride : nullptr;
  for (int i = warp; i < n; i += GEN_WARPS) {
    const int j = i < kept ? i : j0 + i - kept;
    const E* kr = kv + (int64_t)slots[j] * row + (int64_t)kvh * D;
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      int d = lane + e * 32;
      if (d < D) s += qv[e] * to_f(kr[d]);
    }
    s = warp_sum(s);
    if (rule.cap > 0.f) s = rule.cap * tanhf(s / rule.cap);
    s += slope * (float)(j - qpos);
    if (rel) s += rel[min(qpos - j, rule.far)];
    const float mn = fmaxf(m, s);
    const float corr = exp_for(m - mn, q), p = exp_for(s - mn, q);
    l = l * corr + p;
    const E* vr = kv + (int64_t)slots[j] * row + (int64_t)Hkv * D + (int64_t)kvh * DV;
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      int d = lane + e * 32;
      if (d < DV) acc[e] = acc[e] * corr + p * to_f(vr[d]);
    }
    m = mn;
  }
  __shared__ float s_m[GEN_WARPS], s_l[GEN_WARPS];
  __shared__ float s_acc[GEN_WARPS][EPL * 32];
  if (lane == 0) {
    s_m[warp] = m;
    s_l[warp] = l;
  }
#pragma unroll
  for (int e = 0; e < EPL; ++e) s_acc[warp][lane + e * 32] = acc[e];
  __syncthreads();
  if (warp == 0) {
    float M = sinks ? sinks[h] : -INFINITY;
#pragma unroll
    for (int w = 0; w < GEN_WARPS; ++w) M = fmaxf(M, s_m[w]);
    float L = sinks ? exp_for(sinks[h] - M, q) : 0.f;
    float o[EPL];
#pragma unroll
    for (int e = 0; e < EPL; ++e) o[e] = 0.f;
#pragma unroll
    for (int w = 0; w < GEN_WARPS; ++w) {
      if (s_m[w] == -INFINITY) continue;
      const float c = exp_for(s_m[w] - M, q);
      L += s_l[w] * c;
#pragma unroll
      for (int e = 0; e < EPL; ++e) o[e] += s_acc[w][lane + e * 32] * c;
    }
    float inv = L > 0.f ? gate.scale / L : 0.f;
    const E* gt = gate.gate != nullptr ? (const E*)gate.gate + (int64_t)t * gate.stride : nullptr;
    if (gt != nullptr && !gate.elem) inv /= 1.f + exp_for(-to_f(gt[h]), q);
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      int d = lane + e * 32;
      if (d >= DV) continue;
      float r = o[e] * inv;
      if (gt != nullptr && gate.elem) r /= 1.f + exp_for(-to_f(gt[h * DV + d]), q);
      from_f(r, &out[(int64_t)t * out_stride + (int64_t)h * DV + d]);
    }
  }
}

LLB_EXPORT int llb_attn_generic(const void* q, int64_t q_stride, const void* kv_layer, const int* req_to_token,
                                int64_t r2t_stride, const int* b_req_idx, const int* pos, const int* batch_of, void* out,
                                int64_t out_stride, int T, int Hq, int Hkv, int D, float sm_scale, int window,
                                float softcap, const float* alibi_slopes, const float* sinks, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (D <= 0 || D > 32 * GEN_MAX_EPL || Hkv <= 0 || Hq % Hkv != 0) return LLB_ERR_UNSUPPORTED;
  dim3 grid(T, Hq);
  attn_generic_kernel<bf16, GEN_MAX_EPL><<<grid, GEN_WARPS * 32, 0, st>>>(
      (const bf16*)q, q_stride, (const bf16*)kv_layer, req_to_token, r2t_stride, b_req_idx, pos, batch_of, (bf16*)out,
      out_stride, Hq, Hkv, D, D, sm_scale, KeyRule{window, 0, nullptr, 0, 0, 0, softcap}, alibi_slopes, sinks,
      OutGate{nullptr, 0, 1.f, 0});
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// The form with a value size of its own, chunks, kept first positions, biases by distance, capped scores (see KeyRule), an output
// gate per head or (gate_elem) per element, and fp32 (dt 0) beside bf16 (dt 1).
LLB_EXPORT int llb_attn_generic_kv(const void* q, int dt, int64_t q_stride, const void* kv_layer, const int* req_to_token,
                                   int64_t r2t_stride, const int* b_req_idx, const int* pos, const int* batch_of,
                                   void* out, int64_t out_stride, int T, int Hq, int Hkv, int D, int DV, float sm_scale,
                                   int window, int keep, const float* rel, int far, int64_t rel_stride, int chunk,
                                   float cap, const void* gate, int64_t gate_stride, int gate_elem, float out_scale,
                                   cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (window < 0 || keep < 0 || (rel != nullptr && far < 0) || chunk < 0 || (chunk > 0 && window > 0) || !(cap >= 0.f))
    return LLB_ERR_BAD_ARG;
  const KeyRule rule{window, keep, rel, far, rel_stride, chunk, cap};
  const OutGate og{gate, gate_stride, out_scale, gate_elem};
  if (D <= 0 || DV <= 0 || D > 512 || DV > 512 || Hkv <= 0 || Hq % Hkv != 0 || Hq > 65535) return LLB_ERR_UNSUPPORTED;
  const dim3 grid(T, Hq);
#define LLB_GENERIC(E, EPL)                                                                                           \
  attn_generic_kernel<E, EPL><<<grid, GEN_WARPS * 32, 0, st>>>(                                                       \
      (const E*)q, q_stride, (const E*)kv_layer, req_to_token, r2t_stride, b_req_idx, pos, batch_of, (E*)out,         \
      out_stride, Hq, Hkv, D, DV, sm_scale, rule, nullptr, nullptr, og)
  if (D <= 128 && DV <= 128) {
    if (dt == 0)
      LLB_GENERIC(float, 4);
    else
      LLB_GENERIC(bf16, 4);
  } else if (dt == 0) {
    LLB_GENERIC(float, 16);
  } else {
    LLB_GENERIC(bf16, 16);
  }
#undef LLB_GENERIC
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// RoPE + KV scatter for head sizes / rotary widths the vectorised kernel does not take (head size not 64, 128
// or 256, rotary width not a multiple of 16).  One CTA per token: the token's qkv row is staged in shared
// memory so that rotation partners are read before anything is overwritten.  Same contract as
// llb_rope_kv_scatter (half-split rotary layout, q rotated in place, K and V written to kv_layer[slot]).
__global__ void __launch_bounds__(256) rope_kv_scatter_generic_kernel(bf16* __restrict__ qkv, bf16* __restrict__ kv_layer,
                                                                      const float* __restrict__ cos_t,
                                                                      const float* __restrict__ sin_t,
                                                                      const int* __restrict__ pos,
                                                                      const int* __restrict__ slot, int Hq, int Hkv,
                                                                      int D, int rot_dim, int64_t qkv_stride) {
  extern __shared__ float srow[];
  const int t = blockIdx.x;
  const int n = (Hq + 2 * Hkv) * D;
  bf16* row = qkv + (int64_t)t * qkv_stride;
  for (int i = threadIdx.x; i < n; i += blockDim.x) srow[i] = __bfloat162float(row[i]);
  __syncthreads();
  const int half = rot_dim >> 1;
  const int p = pos[t], s = slot[t];
  const float* cr = cos_t + (int64_t)p * half;
  const float* sr = sin_t + (int64_t)p * half;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int head = i / D, d = i - head * D;
    const int kind = head < Hq ? 0 : (head < Hq + Hkv ? 1 : 2);
    float x = srow[i];
    if (kind != 2 && d < rot_dim) {
      if (d < half)
        x = x * cr[d] - srow[i + half] * sr[d];
      else
        x = x * cr[d - half] + srow[i - half] * sr[d - half];
    }
    const bf16 o = __float2bfloat16(x);
    if (kind == 0)
      row[i] = o;
    else
      kv_layer[((int64_t)s * (2 * Hkv) + (head - Hq)) * D + d] = o;
  }
}

LLB_EXPORT int llb_rope_kv_scatter_generic(void* qkv, void* kv_layer, const float* cos_t, const float* sin_t,
                                           const int* pos, const int* slot, int T, int Hq, int Hkv, int D, int rot_dim,
                                           int64_t qkv_stride, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  const size_t smem = (size_t)(Hq + 2 * Hkv) * D * sizeof(float);
  if ((rot_dim & 1) || rot_dim > D || smem > 200 * 1024) return LLB_ERR_UNSUPPORTED;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(rope_kv_scatter_generic_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  rope_kv_scatter_generic_kernel<<<T, 256, smem, st>>>((bf16*)qkv, (bf16*)kv_layer, cos_t, sin_t, pos, slot, Hq, Hkv, D,
                                                      rot_dim, qkv_stride);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// Per-head RMS norm of q and k over the first `dim` of their D elements (a null weight is all ones; norm 0: none), a factor per
// query head (q_scale fp32 [Hq] or null), rotary positions on the first rot_dim, and the cache write, for layers whose value size DV differs from the key size D.  A norm without a weight
// commutes with the rotation.  qkv row: [Hq * D | Hkv * D | Hkv * DV]; q is rewritten in place, K and V go to kv_layer[slot].
// Hkv = 0: queries only (a layer that reads another layer's cache).  Sizes are multiples of 8; a group of 2^k lanes works on one head, a lane
// on 8 elements of it (NIT times, 8 * lanes apart); rotation partners meet in shared memory.
__device__ __forceinline__ void load8(const bf16* p, float* f) { unpack8(*reinterpret_cast<const bf16x8*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(bf16* p, const float* f) { *reinterpret_cast<bf16x8*>(p) = pack8(f); }
__device__ __forceinline__ void store8(float* p, const float* f) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

// FAST (NIT = 1, rot_dim a multiple of 16): a lane's 8 elements lie in one half, their partners in one other lane.
template <typename E, int NIT, bool FAST>
__global__ void __launch_bounds__(256)
qk_norm_rope_scatter_kernel(E* __restrict__ qkv, int64_t qkv_stride, E* __restrict__ kv_layer,
                            const float* __restrict__ cos_t, const float* __restrict__ sin_t, const int* __restrict__ pos,
                            const int* __restrict__ slot, const float* __restrict__ qw, const float* __restrict__ kw,
                            float eps, int norm, const float* __restrict__ q_scale, unsigned items, int Hq, int Hkv, int D, int dim, int DV, int rot_dim, int lanes_log2) {
  pdl_wait();
  extern __shared__ float srow[];  // [groups][rot_dim]
  const int lanes = 1 << lanes_log2;
  const int gl = threadIdx.x & (lanes - 1), grp = threadIdx.x >> lanes_log2;
  const unsigned heads = Hq + 2 * Hkv;
  const unsigned item = blockIdx.x * (256u >> lanes_log2) + grp;
  const bool live = item < items;
  const unsigned t = live ? item / heads : 0;
  const int head = live ? (int)(item - t * heads) : Hq + Hkv;
  E* row = qkv + (int64_t)t * qkv_stride;
  const int half = rot_dim >> 1;
  float* sh = srow + grp * rot_dim;
  const bool qk = live && head < Hq + Hkv;
  E* x = row + (int64_t)head * D;
  E* kv_row = Hkv > 0 ? kv_layer + (int64_t)slot[t] * Hkv * (D + DV) : nullptr;
  if (live && !qk) {  // V
    const int g = head - Hq - Hkv;
    const uint4* src = reinterpret_cast<const uint4*>(row + (int64_t)(Hq + Hkv) * D + (int64_t)g * DV);
    uint4* dst = reinterpret_cast<uint4*>(kv_row + (int64_t)Hkv * D + (int64_t)g * DV);
    for (int v = gl; v < DV * (int)sizeof(E) / 16; v += lanes) dst[v] = src[v];
  }
  float f[NIT][8] = {};
  float ss = 0.f;
  if (qk) {
#pragma unroll
    for (int n = 0; n < NIT; ++n) {
      const int d = (gl + n * lanes) * 8;
      if (d >= D) continue;
      load8(x + d, f[n]);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss = fmaf(f[n][i], f[n][i], ss);
    }
  }
  for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  float inv = norm ? rsqrtf(ss / (float)dim + eps) : 1.f;
  if (q_scale != nullptr && head < Hq) inv *= q_scale[head];
  const float* w = head < Hq ? qw : kw;
  if (qk) {
#pragma unroll
    for (int n = 0; n < NIT; ++n) {
      const int d = (gl + n * lanes) * 8;
      if (d >= D) continue;
      float wv[8];
      if (w != nullptr) load8(w + d, wv);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[n][i] *= w != nullptr ? inv * wv[i] : inv;
      if (!FAST && d < rot_dim) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (d + i < rot_dim) sh[d + i] = f[n][i];
      }
    }
  }
  E* dst = head < Hq ? x : kv_row + (int64_t)(head - Hq) * D;
  if (FAST) {
    const int d = gl * 8, step = half >> 3;
    const bool turns = d < rot_dim, upper = d >= half;
    float o[8];
    const int lane = threadIdx.x & 31, src = turns ? (upper ? lane - step : lane + step) : lane;
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = __shfl_sync(0xffffffffu, f[0][i], src);
    if (!qk || d >= D) return;
    if (turns) {
      const int64_t at = (int64_t)pos[t] * half + (upper ? d - half : d);
      float c[8], s[8];
      load8(cos_t + at, c);
      load8(sin_t + at, s);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[0][i] = f[0][i] * c[i] + (upper ? o[i] : -o[i]) * s[i];
    }
    store8(dst + d, f[0]);
    return;
  }
  __syncwarp();
  if (!qk) return;
  const float *cr = cos_t + (int64_t)pos[t] * half, *sr = sin_t + (int64_t)pos[t] * half;
#pragma unroll
  for (int n = 0; n < NIT; ++n) {
    const int d = (gl + n * lanes) * 8;
    if (d >= D) continue;
    if (d < rot_dim) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int e = d + i;
        if (e < half)
          f[n][i] = f[n][i] * cr[e] - sh[e + half] * sr[e];
        else if (e < rot_dim)
          f[n][i] = f[n][i] * cr[e - half] + sh[e - half] * sr[e - half];
      }
    }
    store8(dst + d, f[n]);
  }
}

// qw, kw: fp32 [D], zero beyond dim, or null.  norm 0: no norm (qw, kw null).  q_scale: fp32 [Hq] or null.  dt: 0 = fp32, 1 = bf16.
LLB_EXPORT int llb_qk_norm_rope_scatter(void* qkv, int dt, int64_t qkv_stride, void* kv_layer, const float* cos_t,
                                        const float* sin_t, const int* pos, const int* slot, const float* qw,
                                        const float* kw, float eps, int norm, const float* q_scale, int T, int Hq, int Hkv, int D, int dim, int DV,
                                        int rot_dim, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (D <= 0 || (D % 8) || DV <= 0 || (DV % 8) || D > 512 || dim <= 0 || dim > D || (rot_dim & 1) || rot_dim > dim ||
      (qkv_stride % 8) || Hq < 0 || Hkv < 0 || (!norm && (qw != nullptr || kw != nullptr)))
    return LLB_ERR_UNSUPPORTED;
  int lg = 2;
  while (lg < 5 && (8 << lg) < D) ++lg;
  const int64_t items = (int64_t)T * (Hq + 2 * Hkv);
  const int groups = 256 >> lg;
  const size_t smem = (size_t)groups * rot_dim * sizeof(float);
  if (smem > 48 * 1024 || items > 0x7fffff00) return LLB_ERR_UNSUPPORTED;
  const dim3 grid((unsigned)cdiv64(items, groups));
#define LLB_QK(E, NIT, FAST)                                                                                              \
  launch_pdl(qk_norm_rope_scatter_kernel<E, NIT, FAST>, grid, dim3(256), FAST ? 0 : smem, st, (E*)qkv, qkv_stride,        \
             (E*)kv_layer, cos_t, sin_t, pos, slot, qw, kw, eps, norm, q_scale, (unsigned)items, Hq, Hkv, D, dim, DV, rot_dim, lg)
  if (D <= 256 && rot_dim > 0 && rot_dim % 16 == 0) {
    if (dt == 0)
      LLB_QK(float, 1, true);
    else
      LLB_QK(bf16, 1, true);
  } else if (D <= 256) {
    if (dt == 0)
      LLB_QK(float, 1, false);
    else
      LLB_QK(bf16, 1, false);
  } else if (dt == 0) {
    LLB_QK(float, 2, false);
  } else {
    LLB_QK(bf16, 2, false);
  }
#undef LLB_QK
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}
