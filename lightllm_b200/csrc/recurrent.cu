// Matrix-state recurrences with decays: per head a state S [dk, dv] in fp32,
//
//   S_t = diag(a_t) S_(t-1) + b_t k_t v_t^T,   o_t = S_t^T q_t * dim^(-1/2)
//
//   gated linear attention (GLA)  a_t = sigmoid(z_t)^(1/tau) per key channel, b_t = 1;  z = A2 (A1 h) + bias
//   mLSTM                         a_t = exp(f + m_(t-1) - m_t), b_t = exp(i - m_t) per head, m_t = max(f + m_(t-1), i),
//                                 i = cap tanh(zi / cap), f = logsigmoid(cap tanh(zf / cap)); a second state n takes k alone
//                                 and o_t is divided by max(|n_t . q_t dim^(-1/2)|, exp(-m_t)) + 1e-6.  m starts at 0.
//
// followed by the head's output step: RMS norm over dv, times a weight, times silu(g) (GLA) or sigmoid(g) (mLSTM).
//
// recurrent_scan   token by token: decode steps, and prompts in fp32.  A CTA owns one (request, head); a thread keeps the
//                  same four columns of every 256 / (dv / 4)-th state row, which it reads and writes once per token.
// chunked form     prompts in bf16, 64 tokens at a time on tensor cores:
//   *_prep         decays summed within every chunk (GLA: per channel, with the low-rank product; mLSTM: F, m, i)
//   chunk_local    what every chunk adds to the state, decayed to the chunk's end: K'^T V, all chunks side by side
//   chunk_scan     the recurrence over chunks, elementwise; leaves the state before every chunk as the sum of two bf16
//                  planes and the last one in the request's row
//   chunk_output   per (chunk, head): pairs inside the chunk plus the state before it, then the output step
// Decay factors are only formed between positions where they are at most 1 (or in a range checked to be small), so nothing
// overflows however strong the decay; fp32 quantities enter tensor-core products as two bf16 planes (high and low part).
//
// Sizes: dk, dv multiples of 16 (zero-padded); state row of a request: S [H][dk][dv], then for mLSTM n [H][dk], m [H].
#include "common.cuh"

using namespace llb;

namespace {

constexpr int GLA = 0, MLSTM = 1;
constexpr int C = 64;  // tokens per chunk

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// q, k, v, g: heads side by side, row pitch ld.  GLA: a1 (pitch ld) [rank], a2 [H * dk, rank], a2b [H * dk]; mLSTM: zi, zf
// [T, H] (pitch ldz).  w: output weight, w_stride elements between heads (0: shared).
struct Mix {
  const void *q, *k, *v, *g, *a1, *a2;
  const float *a2b, *zi, *zf, *w;
  void* out;
  float* state;
  int64_t ld, ldz, out_ld, state_row;
  const int *req, *cu_q, *first_pos;
  int H, dk, dv, dim, vdim, rank, w_stride;
  float inv_tau, cap, eps, out_scale;
};

// ------------------------------------------------------------------------------------------------ token by token
template <typename E, int MODE>
__global__ void __launch_bounds__(256) recurrent_scan_kernel(const Mix p) {
  pdl_wait();
  constexpr int U = 16;  // state rows in flight per thread
  extern __shared__ float sm[];
  __shared__ float red33[33];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int dk = p.dk, dv = p.dv;
  float *qs = sm, *ks = qs + dk, *as = ks + dk, *ns = as + dk, *vs = ns + dk, *os = vs + dv, *red = os + dv;
  const int ncol = dv >> 2, rgroups = 256 / ncol;
  const int cg = tid % ncol, rg = tid / ncol;
  const bool active = rg < rgroups;
  const int t0 = p.cu_q != nullptr ? p.cu_q[b] : b, t1 = p.cu_q != nullptr ? p.cu_q[b + 1] : b + 1;
  if (t0 >= t1) return;
  float* row = p.state + (int64_t)p.req[b] * p.state_row;
  float4* S = reinterpret_cast<float4*>(row + (int64_t)h * dk * dv) + cg;
  float* n_st = row + (int64_t)p.H * dk * dv + (int64_t)h * dk;
  float* m_st = row + (int64_t)p.H * dk * (dv + 1) + h;
  bool fresh = p.first_pos[b] == 0;
  float m = 0.f;
  if (MODE == MLSTM) {
    if (!fresh) m = *m_st;
    for (int d = tid; d < dk; d += 256) ns[d] = fresh ? 0.f : n_st[d];
  }
  const float scale = rsqrtf((float)p.dim);
  for (int t = t0; t < t1; ++t, fresh = false) {
    float4 s[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int r = rg + u * rgroups;
      s[u] = (active && !fresh && r < dk) ? S[(int64_t)r * ncol] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const E *q = (const E*)p.q + t * p.ld + h * dk, *k = (const E*)p.k + t * p.ld + h * dk,
            *v = (const E*)p.v + t * p.ld + h * dv, *g = (const E*)p.g + t * p.ld + h * dv;
    float nq = 0.f, bt = 1.f, at = 1.f;
    if (MODE == MLSTM) {
      const float i = soft_cap(p.zi[t * p.ldz + h], p.cap), f = logsigmoid(soft_cap(p.zf[t * p.ldz + h], p.cap));
      const float m1 = fmaxf(f + m, i);
      at = expf(f + m - m1);
      bt = expf(i - m1);
      m = m1;
    }
    for (int d = tid; d < dk; d += 256) {
      const float qd = ldf(q + d) * scale, kd = ldf(k + d);
      qs[d] = qd;
      if (MODE == GLA) {
        const E *a1 = (const E*)p.a1 + t * p.ld, *a2 = (const E*)p.a2 + (int64_t)(h * dk + d) * p.rank;
        float z = p.a2b[h * dk + d];
        for (int r = 0; r < p.rank; ++r) z = fmaf(ldf(a2 + r), ldf(a1 + r), z);
        as[d] = expf(logsigmoid(z) * p.inv_tau);
        ks[d] = kd;
      } else {
        const float kb = bt * kd, n1 = at * ns[d] + kb;
        ks[d] = kb;
        ns[d] = n1;
        nq = fmaf(n1, qd, nq);
      }
    }
    for (int c = tid; c < dv; c += 256) vs[c] = ldf(v + c);
    if (MODE == MLSTM) nq = block_sum(nq, red33);
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active) {
      const float4 vv = *reinterpret_cast<const float4*>(vs + cg * 4);
      for (int r0 = rg; r0 < dk; r0 += U * rgroups) {
        if (r0 != rg) {
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int r = r0 + u * rgroups;
            s[u] = (!fresh && r < dk) ? S[(int64_t)r * ncol] : make_float4(0.f, 0.f, 0.f, 0.f);
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * rgroups;
          if (r < dk) {
            const float a = MODE == GLA ? as[r] : at, kr = ks[r], qr = qs[r];
            float4 x = s[u];
            x.x = fmaf(a, x.x, kr * vv.x);
            x.y = fmaf(a, x.y, kr * vv.y);
            x.z = fmaf(a, x.z, kr * vv.z);
            x.w = fmaf(a, x.w, kr * vv.w);
            S[(int64_t)r * ncol] = x;
            o.x = fmaf(x.x, qr, o.x);
            o.y = fmaf(x.y, qr, o.y);
            o.z = fmaf(x.z, qr, o.z);
            o.w = fmaf(x.w, qr, o.w);
          }
        }
      }
      *reinterpret_cast<float4*>(red + rg * dv + cg * 4) = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < dv; c += 256) {
      float x = 0.f;
      for (int r = 0; r < rgroups; ++r) x += red[r * dv + c];
      if (MODE == MLSTM) x /= fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
      os[c] = x;
      ss = fmaf(x, x, ss);
    }
    ss = block_sum(ss, red33);
    const float inv = rsqrtf(ss / (float)p.vdim + p.eps) * p.out_scale;
    E* out = (E*)p.out + t * p.out_ld + h * dv;
    const float* w = p.w + (int64_t)h * p.w_stride;
    for (int c = tid; c < dv; c += 256) {
      const float gv = ldf(g + c), sg = 1.f / (1.f + expf(-gv));
      stf(out + c, os[c] * inv * w[c] * (MODE == GLA ? gv * sg : sg));
    }
    __syncthreads();
  }
  if (MODE == MLSTM) {
    for (int d = tid; d < dk; d += 256) n_st[d] = ns[d];
    if (tid == 0) *m_st = m;
  }
}

// ------------------------------------------------------------------------------------------------ chunked form
// chunk c: tokens tok0[c] .. tok0[c] + len[c] - 1 of one request; request b owns chunks cu_chunk[b] .. cu_chunk[b + 1] - 1.
struct Chunks {
  const int *tok0, *len, *cu_chunk;
  float* decay;            // GLA: [T, H * dk] log decays summed from the chunk's start; mLSTM: F, i, m [3][T, H]
  float* total;            // decay over the whole chunk: GLA [chunks, H, dk], mLSTM [chunks, H]
  float *m_prev, *n_prev;  // mLSTM: [chunks, H], [chunks, H, dk] before the chunk
  float* s_loc;            // [chunks, H, dk, dv] what the chunk adds
  float* n_loc;            // mLSTM: [chunks, H, dk]
  bf16 *s_hi, *s_lo;       // [chunks, H, dk, dv] state before the chunk
  int T;
};

// Two threads per key channel, one for either half of the chunk's tokens.
__global__ void __launch_bounds__(512) gla_prep_kernel(const Mix p, const Chunks c) {
  pdl_wait();
  constexpr int HC = C / 2;
  extern __shared__ float a1s[];  // [C][rank]
  __shared__ float first[256];    // the first half's sums
  const int ch = blockIdx.x, h = blockIdx.y;
  const int t0 = c.tok0[ch], len = c.len[ch];
  const int rank = p.rank, per = rank >> 3;
  for (int i = threadIdx.x; i < C * per; i += blockDim.x) {
    const int t = i / per, r = (i - t * per) * 8;
    float f[8] = {};
    if (t < len) unpack8(*reinterpret_cast<const bf16x8*>((const bf16*)p.a1 + (int64_t)(t0 + t) * p.ld + r), f);
#pragma unroll
    for (int e = 0; e < 8; ++e) a1s[t * rank + r + e] = f[e];
  }
  __syncthreads();
  const int half = blockDim.x >> 1;
  const int d = threadIdx.x % half, hf = threadIdx.x / half;
  const bool live = d < p.dk;
  float z[HC];
  if (live) {
    const float bias = p.a2b[h * p.dk + d];
#pragma unroll
    for (int t = 0; t < HC; ++t) z[t] = bias;
    const bf16* a2 = (const bf16*)p.a2 + (int64_t)(h * p.dk + d) * rank;
    for (int r0 = 0; r0 < rank; r0 += 8) {
      float a[8];
      unpack8(*reinterpret_cast<const bf16x8*>(a2 + r0), a);
#pragma unroll
      for (int t = 0; t < HC; ++t) {
        const float4* x = reinterpret_cast<const float4*>(a1s + (hf * HC + t) * rank + r0);
        const float4 u = x[0], v = x[1];
        z[t] = fmaf(a[0], u.x, fmaf(a[1], u.y, fmaf(a[2], u.z, fmaf(a[3], u.w, z[t]))));
        z[t] = fmaf(a[4], v.x, fmaf(a[5], v.y, fmaf(a[6], v.z, fmaf(a[7], v.w, z[t]))));
      }
    }
    float sum = 0.f;
#pragma unroll
    for (int t = 0; t < HC; ++t) {
      sum += (fminf(z[t], 0.f) - log1pf(__expf(-fabsf(z[t])))) * p.inv_tau;
      z[t] = sum;
    }
    if (hf == 0) first[d] = sum;
  }
  __syncthreads();
  if (!live) return;
  const float before = hf == 0 ? 0.f : first[d];
  float* dst = c.decay + (int64_t)t0 * p.H * p.dk + h * p.dk + d;
#pragma unroll
  for (int t = 0; t < HC; ++t) {
    const int tt = hf * HC + t;
    const float v = before + z[t];
    if (tt < len) dst[(int64_t)tt * p.H * p.dk] = v;
    if (tt == len - 1) c.total[((int64_t)ch * p.H + h) * p.dk + d] = __expf(v);
  }
}

// A warp takes one chunk (two tokens per lane), 16 chunks at a time.  (F, M) of a run of tokens: the sum of the log forget
// gates and the largest input gate after decay to the run's end; runs compose, so m_t = max(F_t + m before, M_t).
__global__ void __launch_bounds__(512) mlstm_prep_kernel(const Mix p, const Chunks c) {
  pdl_wait();
  __shared__ float sF[16], sM[16];
  const int h = blockIdx.x, b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = c.cu_chunk[b], c1 = c.cu_chunk[b + 1];
  if (c0 >= c1) return;
  float* m_st = p.state + (int64_t)p.req[b] * p.state_row + (int64_t)p.H * p.dk * (p.dv + 1) + h;
  float m_run = p.first_pos[b] == 0 ? 0.f : *m_st;
  float *oF = c.decay, *oI = oF + (int64_t)c.T * p.H, *oM = oI + (int64_t)c.T * p.H;
  for (int cb = c0; cb < c1; cb += 16) {
    const int ch = cb + warp;
    const int len = ch < c1 ? c.len[ch] : 0, t0 = ch < c1 ? c.tok0[ch] : 0;
    float f[2], in[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = 2 * lane + u;
      f[u] = 0.f;
      in[u] = -INFINITY;
      if (t < len) {
        in[u] = soft_cap(p.zi[(int64_t)(t0 + t) * p.ldz + h], p.cap);
        f[u] = logsigmoid(soft_cap(p.zf[(int64_t)(t0 + t) * p.ldz + h], p.cap));
      }
    }
    float F = f[0] + f[1], M = fmaxf(in[0] + f[1], in[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float F0 = __shfl_up_sync(0xffffffffu, F, o), M0 = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(M0 + F, M);
        F += F0;
      }
    }
    float Fx = __shfl_up_sync(0xffffffffu, F, 1), Mx = __shfl_up_sync(0xffffffffu, M, 1);
    if (lane == 0) Fx = 0.f, Mx = -INFINITY;
    if (lane == 31) sF[warp] = F, sM[warp] = M;
    __syncthreads();
    float mp = m_run, m_end = m_run;
    for (int w = 0; w < 16; ++w) {
      if (w == warp) mp = m_end;
      m_end = fmaxf(sF[w] + m_end, sM[w]);  // chunks past the end: (0, -inf)
    }
    m_run = m_end;
    if (lane == 0 && ch < c1) {
      c.m_prev[(int64_t)ch * p.H + h] = mp;
      c.total[(int64_t)ch * p.H + h] = __expf(sF[warp] + mp - fmaxf(sF[warp] + mp, sM[warp]));
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      Mx = fmaxf(Mx + f[u], in[u]);
      Fx += f[u];
      const int t = 2 * lane + u;
      if (t < len) {
        const int64_t o = (int64_t)(t0 + t) * p.H + h;
        oF[o] = Fx;
        oI[o] = in[u];
        oM[o] = fmaxf(Fx + mp, Mx);
      }
    }
    __syncthreads();
  }
  if (threadIdx.x == 0) *m_st = m_run;
}

constexpr int TP = 72;  // pitch of 64-column bf16 tiles: 144 bytes, ldmatrix rows fall on distinct banks

// 64 rows (tokens, `len` valid) x 64 columns from col0 (`cols` valid in all) of a bf16 matrix, zero beyond
template <int THREADS>
__device__ __forceinline__ void load_tile(bf16* dst, const bf16* src, int64_t ld, int rows, int len, int col0, int cols) {
  for (int i = threadIdx.x; i < rows * 8; i += THREADS) {
    const int r = i >> 3, x = (i & 7) * 8;
    const bool ok = r < len && col0 + x < cols;
    cp_async16(smem_u32(dst + r * TP + x), ok ? src + (int64_t)r * ld + col0 + x : src, ok);
  }
}

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  lo = pack_bf16x2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

struct LocalSmem {
  bf16 k[C * TP], kh[C * TP], kl[C * TP], v[2][C * TP];
  float b[C][64];
  float wt[C];
};

// NV: 64-column value tiles per CTA (a warp works on 16 key channels x 64 values)
template <int MODE, int NV>
__global__ void __launch_bounds__(128 * NV) chunk_local_kernel(const Mix p, const Chunks c) {
  pdl_wait();
  constexpr int THREADS = 128 * NV;
  extern __shared__ __align__(16) uint8_t raw[];
  LocalSmem& s = *reinterpret_cast<LocalSmem*>(raw);
  const int vt = (p.dv + 64 * NV - 1) / (64 * NV);
  const int d0 = (blockIdx.z / vt) * 64, v0 = (blockIdx.z % vt) * 64 * NV;
  const int ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, tig = lane & 3, wr = warp & 3, wv = warp >> 2;
  const int t0 = c.tok0[ch], len = c.len[ch];
  load_tile<THREADS>(s.k, (const bf16*)p.k + (int64_t)t0 * p.ld + h * p.dk, p.ld, C, len, d0, p.dk);
  if (MODE == GLA) {
    const float* src = c.decay + (int64_t)t0 * p.H * p.dk + h * p.dk;
    for (int i = tid; i < C * 16; i += THREADS) {
      const int r = i >> 4, x = (i & 15) * 4;
      const bool ok = r < len && d0 + x < p.dk;
      cp_async16(smem_u32(&s.b[r][x]), ok ? src + (int64_t)r * p.H * p.dk + d0 + x : src, ok);
    }
  }
  cp_async_commit();
#pragma unroll
  for (int j = 0; j < NV; ++j)
    load_tile<THREADS>(s.v[j], (const bf16*)p.v + (int64_t)t0 * p.ld + h * p.dv, p.ld, C, len, v0 + j * 64, p.dv);
  cp_async_commit();
  if (MODE == MLSTM && tid < C) {
    const float *F = c.decay, *I = F + (int64_t)c.T * p.H, *M = I + (int64_t)c.T * p.H;
    const int64_t oe = (int64_t)(t0 + len - 1) * p.H + h, o = (int64_t)(t0 + tid) * p.H + h;
    s.wt[tid] = tid < len ? __expf(F[oe] - F[o] + I[o] - M[oe]) : 0.f;
  }
  cp_async_wait<1>();
  __syncthreads();
  {  // keys times their decay to the chunk's end, as two planes: two channels per thread
    const int d = (tid & 31) * 2, part = tid >> 5;
    constexpr int TOK = C / (THREADS / 32);
    float2 be = make_float2(0.f, 0.f);
    if (MODE == GLA) be = *reinterpret_cast<const float2*>(&s.b[len - 1][d]);
    float2 ns = make_float2(0.f, 0.f);
#pragma unroll 8
    for (int t = part * TOK; t < part * TOK + TOK; ++t) {
      const uint32_t kk = *reinterpret_cast<const uint32_t*>(s.k + t * TP + d);
      float x = __uint_as_float(kk << 16), y = __uint_as_float(kk & 0xffff0000u);
      if (MODE == GLA) {
        const float2 bb = *reinterpret_cast<const float2*>(&s.b[t][d]);
        x *= __expf(be.x - bb.x);
        y *= __expf(be.y - bb.y);
      } else {
        x *= s.wt[t];
        y *= s.wt[t];
        ns.x += x;
        ns.y += y;
      }
      uint32_t hi, lo;
      split2(x, y, hi, lo);
      *reinterpret_cast<uint32_t*>(s.kh + t * TP + d) = hi;
      *reinterpret_cast<uint32_t*>(s.kl + t * TP + d) = lo;
    }
    if (MODE == MLSTM && v0 == 0) {  // sums over the tokens through the (now idle) decay tile, in a fixed order
      s.b[part][d] = ns.x;
      s.b[part][d + 1] = ns.y;
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  if (MODE == MLSTM && v0 == 0 && tid < 64 && d0 + tid < p.dk) {
    float n = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) n += s.b[i][tid];
    c.n_loc[((int64_t)ch * p.H + h) * p.dk + d0 + tid] = n;
  }
  float acc[8][4] = {};
#pragma unroll
  for (int ks = 0; ks < C / 16; ++ks) {
    if (ks * 16 >= len) break;
    uint32_t ah[4], al[4];
    const int at = ks * 16 + (lane >> 4) * 8 + (lane & 7), ad = wr * 16 + ((lane >> 3) & 1) * 8;
    ldmatrix_x4_trans(ah[0], ah[1], ah[2], ah[3], smem_u32(s.kh + at * TP + ad));
    ldmatrix_x4_trans(al[0], al[1], al[2], al[3], smem_u32(s.kl + at * TP + ad));
    const int bt = ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int n2 = 0; n2 < 4; ++n2) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(b0, b1, b2, b3, smem_u32(s.v[wv] + bt * TP + n2 * 16 + (lane >> 4) * 8));
      mma_bf16_16816(acc[2 * n2], ah[0], ah[1], ah[2], ah[3], b0, b1);
      mma_bf16_16816(acc[2 * n2 + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
      mma_bf16_16816(acc[2 * n2], al[0], al[1], al[2], al[3], b0, b1);
      mma_bf16_16816(acc[2 * n2 + 1], al[0], al[1], al[2], al[3], b2, b3);
    }
  }
  float* dst = c.s_loc + ((int64_t)ch * p.H + h) * p.dk * p.dv;
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + wr * 16 + g + r * 8, v = v0 + wv * 64 + j * 8 + tig * 2;
      if (d < p.dk && v < p.dv)
        *reinterpret_cast<float2*>(dst + (int64_t)d * p.dv + v) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
    }
}

// A thread carries four neighbouring values of one state row through the request's chunks.
template <int MODE>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const Mix p, const Chunks c) {
  pdl_wait();
  constexpr int U = 8;  // chunks in flight
  const int h = blockIdx.y, b = blockIdx.z;
  const int c0 = c.cu_chunk[b], c1 = c.cu_chunk[b + 1];
  if (c0 >= c1) return;
  const int n4 = p.dk * p.dv / 4;
  const int i = blockIdx.x * 256 + threadIdx.x;
  float* row = p.state + (int64_t)p.req[b] * p.state_row;
  const bool fresh = p.first_pos[b] == 0;
  auto decay = [&](int ch, int d) {
    return MODE == GLA ? c.total[((int64_t)ch * p.H + h) * p.dk + d] : c.total[(int64_t)ch * p.H + h];
  };
  if (i < n4) {
    const int d = i / (p.dv / 4);
    float4* S = reinterpret_cast<float4*>(row + (int64_t)h * p.dk * p.dv) + i;
    float4 x = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *S;
    for (int cb = c0; cb < c1; cb += U) {
      float4 a[U];
      float e[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (cb + u < c1) {
          a[u] = reinterpret_cast<const float4*>(c.s_loc + ((int64_t)(cb + u) * p.H + h) * p.dk * p.dv)[i];
          e[u] = decay(cb + u, d);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (cb + u < c1) {
          uint2 hi, lo;
          split2(x.x, x.y, hi.x, lo.x);
          split2(x.z, x.w, hi.y, lo.y);
          const int64_t o = ((int64_t)(cb + u) * p.H + h) * n4 + i;
          reinterpret_cast<uint2*>(c.s_hi)[o] = hi;
          reinterpret_cast<uint2*>(c.s_lo)[o] = lo;
          x = make_float4(fmaf(e[u], x.x, a[u].x), fmaf(e[u], x.y, a[u].y), fmaf(e[u], x.z, a[u].z), fmaf(e[u], x.w, a[u].w));
        }
      }
    }
    *S = x;
  }
  if (MODE == MLSTM && blockIdx.x == 0) {
    float* n_st = row + (int64_t)p.H * p.dk * p.dv + (int64_t)h * p.dk;
    for (int d = threadIdx.x; d < p.dk; d += 256) {
      float n = fresh ? 0.f : n_st[d];
      for (int cb = c0; cb < c1; cb += U) {
        float a[U], e[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          if (cb + u < c1) a[u] = c.n_loc[((int64_t)(cb + u) * p.H + h) * p.dk + d], e[u] = decay(cb + u, d);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          if (cb + u < c1) {
            c.n_prev[((int64_t)(cb + u) * p.H + h) * p.dk + d] = n;
            n = fmaf(e[u], n, a[u]);
          }
        }
      }
      n_st[d] = n;
    }
  }
}

// shared memory of chunk_output, in bytes, for key size dk
struct OutSmem {
  int qp, bp, off_r, off_a, total;  // pitches (elements) of the query / key tiles and of the decay tile; offsets
  __host__ __device__ OutSmem(int mode, int dk) {
    qp = dk + 8;
    bp = dk + 4;
    off_r = (mode == GLA ? 2 : 1) * C * qp * 2;
    const int keys = C * qp * 2 + (mode == GLA ? C * bp * 4 : 0);
    const int tiles = 2 * dk * TP * 2 + C * TP * 2;
    off_a = off_r + (keys > tiles ? keys : tiles);
    total = off_a + 2 * C * TP * 2;
  }
};

template <int MODE, int VT>
__global__ void __launch_bounds__(256) chunk_output_kernel(const Mix p, const Chunks c) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t raw[];
  __shared__ float sF[C], sI[C], sM[C], s_nq[C], s_rs[C][4], s_ss[2][C];
  const OutSmem L(MODE, p.dk);
  bf16 *qh = reinterpret_cast<bf16*>(raw), *ql = qh + C * L.qp;
  bf16* kt = reinterpret_cast<bf16*>(raw + L.off_r);
  float* bt = reinterpret_cast<float*>(raw + L.off_r + C * L.qp * 2);
  bf16 *sh = kt, *sl = sh + p.dk * TP, *vt_s = sl + p.dk * TP;
  bf16 *ah_s = reinterpret_cast<bf16*>(raw + L.off_a), *al_s = ah_s + C * TP;
  const int ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, tig = lane & 3;
  const int t0 = c.tok0[ch], len = c.len[ch], dk = p.dk;
  const float scale = rsqrtf((float)p.dim);

  {
    const bf16 *q = (const bf16*)p.q + (int64_t)t0 * p.ld + h * dk, *k = (const bf16*)p.k + (int64_t)t0 * p.ld + h * dk;
    const int per = dk >> 3;
    for (int i = tid; i < C * per; i += 256) {
      const int r = i / per, x = (i - r * per) * 8;
      const bool ok = r < len;
      cp_async16(smem_u32(qh + r * L.qp + x), ok ? q + (int64_t)r * p.ld + x : q, ok);
      cp_async16(smem_u32(kt + r * L.qp + x), ok ? k + (int64_t)r * p.ld + x : k, ok);
    }
    if (MODE == GLA) {
      const float* d = c.decay + (int64_t)t0 * p.H * dk + h * dk;
      const int pb = dk >> 2;
      for (int i = tid; i < C * pb; i += 256) {
        const int r = i / pb, x = (i - r * pb) * 4;
        const bool ok = r < len;
        cp_async16(smem_u32(bt + r * L.bp + x), ok ? d + (int64_t)r * p.H * dk + x : d, ok);
      }
    } else if (tid < C) {
      const int64_t o = (int64_t)(t0 + tid) * p.H + h, st = (int64_t)c.T * p.H;
      sF[tid] = tid < len ? c.decay[o] : 0.f;
      sI[tid] = tid < len ? c.decay[o + st] : -INFINITY;
      sM[tid] = tid < len ? c.decay[o + 2 * st] : 0.f;
    }
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
  }
  const float m_prev = MODE == MLSTM ? c.m_prev[(int64_t)ch * p.H + h] : 0.f;
  if (MODE == MLSTM) {  // q . n of the state before the chunk: four threads per row
    const int r = tid >> 2;
    const float* n = c.n_prev + ((int64_t)ch * p.H + h) * dk;
    float x = 0.f;
    for (int d = (tid & 3) * 8; d < dk; d += 32) {
      float qf[8];
      unpack8(*reinterpret_cast<const bf16x8*>(qh + r * L.qp + d), qf);
      const float4 n0 = *reinterpret_cast<const float4*>(n + d), n1 = *reinterpret_cast<const float4*>(n + d + 4);
      x = fmaf(qf[0], n0.x, fmaf(qf[1], n0.y, fmaf(qf[2], n0.z, fmaf(qf[3], n0.w, x))));
      x = fmaf(qf[4], n1.x, fmaf(qf[5], n1.y, fmaf(qf[6], n1.z, fmaf(qf[7], n1.w, x))));
    }
    x += __shfl_xor_sync(0xffffffffu, x, 1);
    x += __shfl_xor_sync(0xffffffffu, x, 2);
    if ((tid & 3) == 0) s_nq[r] = x;
  }

  // ---- weights of the pairs inside the chunk, in 16 x 16 blocks on and below the diagonal ----
  for (int blk = warp; blk < 10; blk += 8) {
    int I = blk, J = blk;
    if (blk >= 4) {
      const int e = blk - 4;
      I = e == 0 ? 1 : (e < 3 ? 2 : 3);
      J = e == 0 ? 0 : (e < 3 ? e - 1 : e - 3);
    }
    const int i0 = I * 16, j0 = J * 16;
    float x[2][4] = {};
    if (i0 < len) {
      if (MODE == MLSTM) {
        for (int ks = 0; ks < dk; ks += 16) {
          uint32_t a[4], b0, b1, b2, b3;
          ldmatrix_x4(a[0], a[1], a[2], a[3],
                      smem_u32(qh + (i0 + (lane & 7) + ((lane >> 3) & 1) * 8) * L.qp + ks + (lane >> 4) * 8));
          ldmatrix_x4(b0, b1, b2, b3,
                      smem_u32(kt + (j0 + (lane & 7) + (lane >> 4) * 8) * L.qp + ks + ((lane >> 3) & 1) * 8));
          mma_bf16_16816(x[0], a[0], a[1], a[2], a[3], b0, b1);
          mma_bf16_16816(x[1], a[0], a[1], a[2], a[3], b2, b3);
        }
      } else {
        bool direct = false;
        float top = 0.f;  // largest exponent that may occur on either side of the reference row
        if (I == J) {
          const int last = min(i0 + 15, len - 1);
          float range = 0.f;
          for (int d = lane; d < dk; d += 32) range = fmaxf(range, bt[i0 * L.bp + d] - bt[last * L.bp + d]);
          direct = warp_max(range) > 40.f;
          top = 40.f;
        }
        if (!direct) {
          // exp(b_i - b_j) = exp(b_i - ref) exp(ref - b_j); below the diagonal ref is the row before block I, so that
          // neither factor exceeds 1; on it the block's middle row (the range was checked).  Rows past the end are zero.
          const int rr = I == J ? min(i0 + 7, len - 1) : i0 - 1;
          const float* ref = bt + rr * L.bp;
          for (int ks = 0; ks < dk; ks += 16) {
            uint32_t ahi[4], alo[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              const int r = i0 + g + (u & 1) * 8, d = ks + tig * 2 + (u >> 1) * 8;
              const float2 bb = *reinterpret_cast<const float2*>(bt + r * L.bp + d);
              const float2 rf = *reinterpret_cast<const float2*>(ref + d);
              const uint32_t qq = *reinterpret_cast<const uint32_t*>(qh + r * L.qp + d);
              split2(__uint_as_float(qq << 16) * __expf(fminf(bb.x - rf.x, top)),
                     __uint_as_float(qq & 0xffff0000u) * __expf(fminf(bb.y - rf.y, top)), ahi[u], alo[u]);
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
              uint32_t bhi[2], blo[2];
#pragma unroll
              for (int u = 0; u < 2; ++u) {
                const int r = j0 + nt * 8 + g, d = ks + tig * 2 + u * 8;
                const float2 bb = *reinterpret_cast<const float2*>(bt + r * L.bp + d);
                const float2 rf = *reinterpret_cast<const float2*>(ref + d);
                const uint32_t kk = *reinterpret_cast<const uint32_t*>(kt + r * L.qp + d);
                split2(__uint_as_float(kk << 16) * __expf(fminf(rf.x - bb.x, top)),
                       __uint_as_float(kk & 0xffff0000u) * __expf(fminf(rf.y - bb.y, top)), bhi[u], blo[u]);
              }
              mma_bf16_16816(x[nt], ahi[0], ahi[1], ahi[2], ahi[3], bhi[0], bhi[1]);
              mma_bf16_16816(x[nt], ahi[0], ahi[1], ahi[2], ahi[3], blo[0], blo[1]);
              mma_bf16_16816(x[nt], alo[0], alo[1], alo[2], alo[3], bhi[0], bhi[1]);
            }
          }
        } else {  // strong decay inside the block: pair by pair
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int i = i0 + g + (e >> 1) * 8, j = j0 + nt * 8 + tig * 2 + (e & 1);
              if (j > i || i >= len) continue;
              float y = 0.f;
              for (int d = 0; d < dk; ++d)
                y = fmaf(__bfloat162float(qh[i * L.qp + d]) * __bfloat162float(kt[j * L.qp + d]),
                         __expf(bt[i * L.bp + d] - bt[j * L.bp + d]), y);
              x[nt][e] = y;
            }
        }
      }
    }
    float rs[2] = {0.f, 0.f};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = i0 + g + hf * 8, j = j0 + nt * 8 + tig * 2;
        float y[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float v = j + e <= i && i < len ? x[nt][2 * hf + e] * scale : 0.f;
          if (MODE == MLSTM && v != 0.f) v *= __expf(sF[i] - sF[j + e] + sI[j + e] - sM[i]);
          y[e] = v;
        }
        rs[hf] += y[0] + y[1];
        uint32_t hi, lo;
        split2(y[0], y[1], hi, lo);
        *reinterpret_cast<uint32_t*>(ah_s + i * TP + j) = hi;
        *reinterpret_cast<uint32_t*>(al_s + i * TP + j) = lo;
      }
    if (MODE == MLSTM) {
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        rs[hf] += __shfl_xor_sync(0xffffffffu, rs[hf], 1);
        rs[hf] += __shfl_xor_sync(0xffffffffu, rs[hf], 2);
        if (tig == 0) s_rs[i0 + g + hf * 8][J] = rs[hf];
      }
    }
  }
  __syncthreads();
  if (MODE == GLA) {  // queries times their decay from the chunk's start, as two planes
    for (int i = tid; i < C * (dk >> 1); i += 256) {
      const int r = i / (dk >> 1), d = (i - r * (dk >> 1)) * 2;
      const float2 bb = *reinterpret_cast<const float2*>(bt + r * L.bp + d);
      const uint32_t qq = *reinterpret_cast<const uint32_t*>(qh + r * L.qp + d);
      uint32_t hi, lo;
      split2(__uint_as_float(qq << 16) * (scale * __expf(bb.x)), __uint_as_float(qq & 0xffff0000u) * (scale * __expf(bb.y)),
             hi, lo);
      *reinterpret_cast<uint32_t*>(qh + r * L.qp + d) = hi;
      *reinterpret_cast<uint32_t*>(ql + r * L.qp + d) = lo;
    }
    __syncthreads();
  }

  // ---- output rows: state before the chunk, then the pairs ----
  const int wr = warp & 3, wc = warp >> 2;
  const int64_t sbase = ((int64_t)ch * p.H + h) * dk * p.dv;
  const int rows[2] = {wr * 16 + g, wr * 16 + g + 8};
  float rf[2] = {1.f, 1.f};
  if (MODE == MLSTM) {
#pragma unroll
    for (int r = 0; r < 2; ++r) rf[r] = scale * __expf(sF[rows[r]] + m_prev - sM[rows[r]]);
  }
  float acc[VT][4][4];
#pragma unroll
  for (int vt = 0; vt < VT; ++vt) {
    if (vt > 0) __syncthreads();
    load_tile<256>(sh, c.s_hi + sbase, p.dv, dk, dk, vt * 64, p.dv);
    load_tile<256>(sl, c.s_lo + sbase, p.dv, dk, dk, vt * 64, p.dv);
    load_tile<256>(vt_s, (const bf16*)p.v + (int64_t)t0 * p.ld + h * p.dv, p.ld, C, len, vt * 64, p.dv);
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int n = 0; n < 4; ++n) acc[vt][n][0] = acc[vt][n][1] = acc[vt][n][2] = acc[vt][n][3] = 0.f;
    const int ar = wr * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ac = (lane >> 4) * 8;
    const int br = (lane & 7) + ((lane >> 3) & 1) * 8, bc = wc * 32 + (lane >> 4) * 8;
    for (int ks = 0; ks < dk; ks += 16) {
      uint32_t a[4], al[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], smem_u32(qh + ar * L.qp + ks + ac));
      if (MODE == GLA) ldmatrix_x4(al[0], al[1], al[2], al[3], smem_u32(ql + ar * L.qp + ks + ac));
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t b[4], bl[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], smem_u32(sh + (ks + br) * TP + bc + n2 * 16));
        ldmatrix_x4_trans(bl[0], bl[1], bl[2], bl[3], smem_u32(sl + (ks + br) * TP + bc + n2 * 16));
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float* o = acc[vt][2 * n2 + e];
          mma_bf16_16816(o, a[0], a[1], a[2], a[3], b[2 * e], b[2 * e + 1]);
          mma_bf16_16816(o, a[0], a[1], a[2], a[3], bl[2 * e], bl[2 * e + 1]);
          if (MODE == GLA) mma_bf16_16816(o, al[0], al[1], al[2], al[3], b[2 * e], b[2 * e + 1]);
        }
      }
    }
    if (MODE == MLSTM) {
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        acc[vt][n][0] *= rf[0];
        acc[vt][n][1] *= rf[0];
        acc[vt][n][2] *= rf[1];
        acc[vt][n][3] *= rf[1];
      }
    }
    for (int ks = 0; ks <= wr; ++ks) {
      uint32_t a[4], al[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], smem_u32(ah_s + ar * TP + ks * 16 + ac));
      ldmatrix_x4(al[0], al[1], al[2], al[3], smem_u32(al_s + ar * TP + ks * 16 + ac));
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t b[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], smem_u32(vt_s + (ks * 16 + br) * TP + bc + n2 * 16));
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float* o = acc[vt][2 * n2 + e];
          mma_bf16_16816(o, a[0], a[1], a[2], a[3], b[2 * e], b[2 * e + 1]);
          mma_bf16_16816(o, al[0], al[1], al[2], al[3], b[2 * e], b[2 * e + 1]);
        }
      }
    }
  }

  // ---- output step ----
  float dn[2] = {1.f, 1.f};
  if (MODE == MLSTM) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = rows[r];
      float nq = s_nq[i] * rf[r];
      for (int J = 0; J <= (i >> 4); ++J) nq += s_rs[i][J];
      dn[r] = 1.f / (fmaxf(fabsf(nq), __expf(-sM[i])) + 1e-6f);
    }
  }
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int vt = 0; vt < VT; ++vt)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        acc[vt][n][e] *= dn[e >> 1];
        ss[e >> 1] = fmaf(acc[vt][n][e], acc[vt][n][e], ss[e >> 1]);
      }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
    ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
    if (tig == 0) s_ss[wc][rows[r]] = ss[r];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = rows[r];
    if (i >= len) continue;
    const float inv = rsqrtf((s_ss[0][i] + s_ss[1][i]) / (float)p.vdim + p.eps) * p.out_scale;
    const bf16* gr = (const bf16*)p.g + (int64_t)(t0 + i) * p.ld + h * p.dv;
    bf16* orow = (bf16*)p.out + (int64_t)(t0 + i) * p.out_ld + h * p.dv;
    const float* w = p.w + (int64_t)h * p.w_stride;
#pragma unroll
    for (int vt = 0; vt < VT; ++vt)
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int v = vt * 64 + wc * 32 + n * 8 + tig * 2;
        if (v >= p.dv) continue;
        const uint32_t gg = *reinterpret_cast<const uint32_t*>(gr + v);
        float o[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float gv = __uint_as_float(e == 0 ? gg << 16 : gg & 0xffff0000u);
          const float sg = __fdividef(1.f, 1.f + __expf(-gv));
          o[e] = acc[vt][n][2 * r + e] * inv * w[v + e] * (MODE == GLA ? gv * sg : sg);
        }
        *reinterpret_cast<uint32_t*>(orow + v) = pack_bf16x2(o[0], o[1]);
      }
  }
}

template <typename K>
int opt_in(K kernel, int bytes, DeviceOnce& once) {
  if (!once.done()) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    once.set();
  }
  return LLB_OK;
}

template <int MODE, int VT>
int launch_output(const Mix& p, const Chunks& c, int n_chunks, cudaStream_t st) {
  static DeviceOnce once;
  int rc = opt_in(chunk_output_kernel<MODE, VT>, 220 * 1024, once);
  if (rc) return rc;
  launch_pdl(chunk_output_kernel<MODE, VT>, dim3(n_chunks, p.H), dim3(256), OutSmem(MODE, p.dk).total, st, p, c);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

template <int MODE>
int launch_chunks(const Mix& p, const Chunks& c, int B, int n_chunks, cudaStream_t st) {
  if (MODE == GLA) {
    launch_pdl(gla_prep_kernel, dim3(n_chunks, p.H), dim3(2 * cdiv(p.dk, 32) * 32), (size_t)C * p.rank * sizeof(float), st,
               p, c);
  } else {
    launch_pdl(mlstm_prep_kernel, dim3(p.H, B), dim3(512), 0, st, p, c);
  }
  LLB_LAUNCH_CHECK();
  if (p.dv > 64) {
    static DeviceOnce once;
    int rc = opt_in(chunk_local_kernel<MODE, 2>, (int)sizeof(LocalSmem), once);
    if (rc) return rc;
    launch_pdl(chunk_local_kernel<MODE, 2>, dim3(n_chunks, p.H, cdiv(p.dk, 64) * cdiv(p.dv, 128)), dim3(256),
               sizeof(LocalSmem), st, p, c);
  } else {
    static DeviceOnce once;
    int rc = opt_in(chunk_local_kernel<MODE, 1>, (int)sizeof(LocalSmem), once);
    if (rc) return rc;
    launch_pdl(chunk_local_kernel<MODE, 1>, dim3(n_chunks, p.H, cdiv(p.dk, 64)), dim3(128), sizeof(LocalSmem), st, p, c);
  }
  LLB_LAUNCH_CHECK();
  launch_pdl(chunk_scan_kernel<MODE>, dim3(cdiv(p.dk * p.dv / 4, 256), p.H, B), dim3(256), 0, st, p, c);
  LLB_LAUNCH_CHECK();
  const int vt = cdiv(p.dv, 64);
  if (vt == 1) return launch_output<MODE, 1>(p, c, n_chunks, st);
  if (vt == 2) return launch_output<MODE, 2>(p, c, n_chunks, st);
  if (vt <= 4) return launch_output<MODE, 4>(p, c, n_chunks, st);
  return launch_output<MODE, 8>(p, c, n_chunks, st);
}

bool sizes_ok(const Mix& p, int B) {
  return p.H > 0 && p.H <= 65535 && B <= 65535 && p.dk > 0 && p.dv > 0 && (p.dk % 16) == 0 && (p.dv % 16) == 0 &&
         p.dim > 0 && p.dim <= p.dk && p.vdim > 0 && p.vdim <= p.dv && (p.state_row % 4) == 0 &&
         ((uintptr_t)p.state & 15) == 0;
}

}  // namespace

// kind 0: GLA, 1: mLSTM; dt 0: fp32, 1: bf16 (q, k, v, g, a1, a2, out).  cu_q null: one token per request (row b).
// first_pos[b]: position of the request's first token in this pass; 0 starts from a zero state.
LLB_EXPORT int llb_recurrent_scan(int kind, int dt, const void* q, const void* k, const void* v, const void* g, int64_t ld,
                                  const void* a1, const void* a2, const float* a2b, int rank, float inv_tau,
                                  const float* zi, const float* zf, int64_t ldz, float cap, float* state,
                                  int64_t state_row, const float* w, int w_stride, float eps, void* out, int64_t out_ld,
                                  float out_scale, const int* req, const int* cu_q, const int* first_pos, int B, int H,
                                  int dk, int dv, int dim, int vdim, cudaStream_t st) {
  if (B <= 0) return LLB_OK;
  const Mix p{q,  k,  v,   g,     a1,   a2,        a2b,  zi,     zf,        w, out, state, ld,  ldz, out_ld,
              state_row, req, cu_q, first_pos, H,   dk,   dv, dim, vdim, rank, w_stride, inv_tau, cap, eps, out_scale};
  if (!sizes_ok(p, B) || dv > 1024 || dk > 1024 || kind < 0 || kind > 1) return LLB_ERR_UNSUPPORTED;
  const int ncol = dv / 4, rgroups = 256 / ncol;
  const size_t smem = (size_t)(4 * dk + 2 * dv + rgroups * dv) * sizeof(float);
  const dim3 grid(H, B);
  if (kind == GLA) {
    if (dt == 0)
      launch_pdl(recurrent_scan_kernel<float, GLA>, grid, dim3(256), smem, st, p);
    else
      launch_pdl(recurrent_scan_kernel<bf16, GLA>, grid, dim3(256), smem, st, p);
  } else {
    if (dt == 0)
      launch_pdl(recurrent_scan_kernel<float, MLSTM>, grid, dim3(256), smem, st, p);
    else
      launch_pdl(recurrent_scan_kernel<bf16, MLSTM>, grid, dim3(256), smem, st, p);
  }
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// bf16 prompts.  tok0, len [n_chunks], cu_chunk [B + 1]; decay: fp32 scratch [T, H * dk] (GLA) or [3, T, H] (mLSTM);
// total: fp32 scratch [n_chunks, H * dk] (GLA) or [n_chunks, H]; m_prev [n_chunks, H], n_prev and n_loc [n_chunks, H, dk] (mLSTM); s_loc: fp32, s_hi, s_lo: bf16 scratch
// [n_chunks, H, dk, dv].
LLB_EXPORT int llb_recurrent_chunks(int kind, const void* q, const void* k, const void* v, const void* g, int64_t ld,
                                    const void* a1, const void* a2, const float* a2b, int rank, float inv_tau,
                                    const float* zi, const float* zf, int64_t ldz, float cap, float* state,
                                    int64_t state_row, const float* w, int w_stride, float eps, void* out, int64_t out_ld,
                                    float out_scale, const int* req, const int* first_pos, const int* tok0, const int* len,
                                    const int* cu_chunk, float* decay, float* total, float* m_prev, float* n_prev, float* n_loc, float* s_loc,
                                    void* s_hi, void* s_lo,
                                    int T, int n_chunks, int B, int H, int dk, int dv, int dim, int vdim,
                                    cudaStream_t st) {
  if (B <= 0 || n_chunks <= 0) return LLB_OK;
  const Mix p{q,  k,  v,   g,     a1,   a2,        a2b,  zi,     zf,        w, out, state, ld,  ldz, out_ld,
              state_row, req, nullptr, first_pos, H,   dk,   dv, dim, vdim, rank, w_stride, inv_tau, cap, eps, out_scale};
  if (!sizes_ok(p, B) || dk > 256 || dv > 512 || (kind == GLA && (rank > 128 || rank % 8 || ((uintptr_t)a1 & 15) || ((uintptr_t)a2 & 15))))
    return LLB_ERR_UNSUPPORTED;
  if ((ld % 8) || (out_ld % 2) || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15) || (((uintptr_t)g | (uintptr_t)out) & 3))
    return LLB_ERR_BAD_ARG;
  const Chunks c{tok0, len, cu_chunk, decay, total, m_prev, n_prev, s_loc, n_loc, (bf16*)s_hi, (bf16*)s_lo, T};
  if (kind == GLA) return launch_chunks<GLA>(p, c, B, n_chunks, st);
  if (kind == MLSTM) return launch_chunks<MLSTM>(p, c, B, n_chunks, st);
  return LLB_ERR_UNSUPPORTED;
}
