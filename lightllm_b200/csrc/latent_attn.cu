// Latent attention over a paged pool of latents, with an optional rotary part and an optional sliding window.
//
// Pool row of a token: [the RMS-normalised latent c, zero-padded to `rank` values | rotated key part], `keys` values in all,
// one "head" shared by all query heads.  The query of a head is taken into the latent space with the key up-projection and
// followed by its own rotated part (q_lat = [q . W_uk | q_rot]), scores are q_lat . row, the value read is c, and the value
// up-projection follows the attention.
// A query sees its own position and the window - 1 positions before it (window 0: all of them).  Scores, weights and
// their sums are fp32.
//
//   latent_prepare         RMSNorm of new latents and rotation of their key parts, written to their pool slots; RMSNorm of the
//                          queries' own latents
//   rope_heads             rotation of a range of columns of every query head, in place
//   latent_gather          rows of a range of positions of every request, back to back (for the expanded prefill form)
//   latent_attn_generic    up to 1024 values per row, fp32 or bf16; one CTA per (query token, head), warps stride over the keys
//   latent_attn_mma        bf16, up to 576 values per row, 512 of them latent: one CTA per (query token, 16 heads, share of the keys).  The 16 query rows
//                          live in registers as MMA fragments; 64-key tiles of the pool are gathered through the slot
//                          table into a three-stage shared-memory ring and used for both products.  The weights enter
//                          P . c as a sum of two bf16 values (high and low part), so that they keep fp32-like
//                          precision.  With more than one share per query the partial results are merged by
//   latent_attn_merge
#include "common.cuh"

using namespace llb;
LLB_DEBUG_BOUNDS_STORAGE(latent_attn)

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void from_f(bf16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ void ld8(const float* p, float* f) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void ld8(const bf16* p, float* f) { unpack8(*reinterpret_cast<const bf16x8*>(p), f); }
__device__ __forceinline__ void st8(float* p, const float* f) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void st8(bf16* p, const float* f) { *reinterpret_cast<bf16x8*>(p) = pack8(f); }

// A warp writes RMSNorm(s[0 .. rank)) * w to d[0 .. cols), zero beyond rank; cols is a multiple of 8.
template <typename T>
__device__ __forceinline__ void norm_row(const T* s, T* d, const float* w, int rank, int cols, float eps, int lane) {
  float ss = 0.f;
  for (int c = lane * 8; c < rank; c += 256) {
    float f[8];
    ld8(s + c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c + i < rank) ss = fmaf(f[i], f[i], ss);
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)rank + eps);
  for (int c = lane * 8; c < cols; c += 256) {
    float f[8] = {}, wv[8];
    if (c < rank) ld8(s + c, f);
    if (c + 8 <= rank) {
      ld8(w + c, wv);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) wv[i] = c + i < rank ? w[c + i] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = c + i < rank ? f[i] * r * wv[i] : 0.f;
    st8(d + c, f);
  }
}

// Rotation of the pairs of `dims` columns: neighbours (2 i, 2 i + 1), or halves (i, i + dims / 2).  Tables [positions, dims / 2].
struct Rotation {
  const float *cos_t, *sin_t;
  const int* pos;
  int dims, neighbours;
};
template <typename T>
__device__ __forceinline__ void rotate_pair(const Rotation& r, const T* s, T* d, int p, int i) {
  const int half = r.dims >> 1, a = r.neighbours ? 2 * i : i, b = r.neighbours ? 2 * i + 1 : i + half;
  const float c = r.cos_t[(int64_t)p * half + i], n = r.sin_t[(int64_t)p * half + i];
  const float u = to_f(s[a]), v = to_f(s[b]);
  from_f(d + a, u * c - v * n);
  from_f(d + b, v * c + u * n);
}

template <typename T>
struct PrepareArgs {
  const T* src;  // [T, [latent, padded to cols | rotated part]]
  int64_t src_stride;
  T* pool;
  int row_elems, rank, cols;
  const float* w;
  const int* slot;
  Rotation rot;
  const T* q_src;  // [T, q_cols] latents of the queries (null: none)
  int64_t q_stride;
  T* q_out;
  int q_rank, q_cols;
  const float* q_w;
  int Tn;
  float eps;
};

// One warp per token and latent.
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const PrepareArgs<T> a) {
  pdl_wait();
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= a.Tn) {
    const int t = item - a.Tn;
    if (a.q_src != nullptr && t < a.Tn)
      norm_row(a.q_src + (int64_t)t * a.q_stride, a.q_out + (int64_t)t * a.q_cols, a.q_w, a.q_rank, a.q_cols, a.eps, lane);
    return;
  }
  const int t = item;
  const T* s = a.src + (int64_t)t * a.src_stride;
  T* d = a.pool + (int64_t)LLB_CHECK_SLOT(a.slot[t]) * a.row_elems;
  norm_row(s, d, a.w, a.rank, a.cols, a.eps, lane);
  if (a.rot.dims > 0) {
    const int p = a.rot.pos[t];
    for (int i = lane; i < (a.rot.dims >> 1); i += 32) rotate_pair(a.rot, s + a.cols, d + a.cols, p, i);
  }
  for (int i = a.cols + a.rot.dims + lane; i < a.row_elems; i += 32) from_f(d + i, 0.f);
}

// x [T, heads]: columns off .. off + dims of every head (pitch elements apart) rotated in place.  VEC: neighbours, four pairs per
// thread.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
rope_heads_kernel(T* __restrict__ x, int64_t stride, const Rotation r, int64_t items, int H, int pitch, int off) {
  pdl_wait();
  const int per = VEC ? r.dims >> 3 : r.dims >> 1;  // threads per head
  const int64_t id = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (id >= items) return;
  const int i = (int)(id % per);
  const int64_t th = id / per;
  const int h = (int)(th % H);
  const int64_t t = th / H;
  T* p = x + t * stride + (int64_t)h * pitch + off;
  if (VEC) {
    const int64_t at = (int64_t)r.pos[t] * (r.dims >> 1) + i * 4;
    float f[8], o[8];
    ld8(p + i * 8, f);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float c = r.cos_t[at + k], n = r.sin_t[at + k];
      o[2 * k] = f[2 * k] * c - f[2 * k + 1] * n;
      o[2 * k + 1] = f[2 * k + 1] * c + f[2 * k] * n;
    }
    st8(p + i * 8, o);
  } else {
    rotate_pair(r, p, p, r.pos[t], i);
  }
}

// out row cu_kv[b] + i = latent of position kv_start[b] + i of request b.  One warp per row, 16-byte pieces.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pool, int row_vec, const int* __restrict__ req_to_token,
                     int64_t r2t_stride, const int* __restrict__ b_req_idx, const int* __restrict__ cu_kv,
                     const int* __restrict__ kv_start, uint4* __restrict__ out, int B) {
  const int rows = cu_kv[B];
  const int lane = threadIdx.x & 31;
  for (int r = blockIdx.x * 8 + (threadIdx.x >> 5); r < rows; r += gridDim.x * 8) {
    int lo = 0, hi = B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (cu_kv[mid] <= r) lo = mid; else hi = mid - 1;
    }
    const int pos = kv_start[lo] + r - cu_kv[lo];
    const int sl = LLB_CHECK_SLOT(req_to_token[(int64_t)LLB_CHECK_REQ(b_req_idx[lo]) * r2t_stride + LLB_CHECK_POS(pos)]);
    for (int v = lane; v < row_vec; v += 32) out[(int64_t)r * row_vec + v] = pool[(int64_t)sl * row_vec + v];
  }
}

// ---------------------------------------------------------------------------------------------- any rank, any type
constexpr int GW = 8;  // warps

template <typename T, int EPL>
__global__ void __launch_bounds__(GW * 32)
latent_attn_generic_kernel(const T* __restrict__ q_lat, const T* __restrict__ pool, int row_elems,
                           const int* __restrict__ req_to_token, int64_t r2t_stride, const int* __restrict__ b_req_idx,
                           const int* __restrict__ pos, const int* __restrict__ batch_of, T* __restrict__ out, int H,
                           int keys, int rank, float scale, int window) {
  extern __shared__ float sm[];  // [GW][rank] partial outputs, then [GW] maxima, [GW] sums
  const int t = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = batch_of ? batch_of[t] : t;
  const int p = pos[t];
  const int* slots = req_to_token + (int64_t)LLB_CHECK_REQ(b_req_idx[b]) * r2t_stride;
  float q[EPL], acc[EPL];
#pragma unroll
  for (int e = 0; e < EPL; ++e) {
    const int d = lane + e * 32;
    q[e] = d < keys ? to_f(q_lat[((int64_t)t * H + h) * keys + d]) * scale : 0.f;
    acc[e] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int j0 = window > 0 ? max(0, p - window + 1) : 0;
  for (int j = j0 + warp; j <= p; j += GW) {
    const T* c = pool + (int64_t)LLB_CHECK_SLOT(slots[j]) * row_elems;
    float cv[EPL];
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      const int d = lane + e * 32;
      cv[e] = d < keys ? to_f(c[d]) : 0.f;
      s += q[e] * cv[e];
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float corr = expf(m - mn), w = expf(s - mn);
    l = l * corr + w;
#pragma unroll
    for (int e = 0; e < EPL; ++e) acc[e] = acc[e] * corr + w * cv[e];
    m = mn;
  }
  float* s_m = sm + GW * rank;
  float* s_l = s_m + GW;
  if (lane == 0) {
    s_m[warp] = m;
    s_l[warp] = l;
  }
#pragma unroll
  for (int e = 0; e < EPL; ++e) {
    const int d = lane + e * 32;
    if (d < rank) sm[warp * rank + d] = acc[e];
  }
  __syncthreads();
  float M = -INFINITY;
#pragma unroll
  for (int w = 0; w < GW; ++w) M = fmaxf(M, s_m[w]);
  float L = 0.f, c[GW];
#pragma unroll
  for (int w = 0; w < GW; ++w) {
    c[w] = s_m[w] == -INFINITY ? 0.f : expf(s_m[w] - M);
    L += s_l[w] * c[w];
  }
  const float inv = 1.f / L;
  for (int d = threadIdx.x; d < rank; d += blockDim.x) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < GW; ++w) o += sm[w * rank + d] * c[w];
    from_f(out + ((int64_t)t * H + h) * rank + d, o * inv);
  }
}

template <typename T>
int launch_generic(const void* q_lat, const void* pool, int row_elems, const int* r2t, int64_t r2t_stride,
                   const int* b_req_idx, const int* pos, const int* batch_of, void* out, int T_n, int H, int keys,
                   int rank, float scale, int window, cudaStream_t st) {
  const dim3 grid(T_n, H);
  const size_t smem = (size_t)(GW * rank + 2 * GW) * sizeof(float);
#define LLB_GENERIC(EPL)                                                                                              \
  latent_attn_generic_kernel<T, EPL><<<grid, GW * 32, smem, st>>>((const T*)q_lat, (const T*)pool, row_elems, r2t,    \
                                                                  r2t_stride, b_req_idx, pos, batch_of, (T*)out, H,   \
                                                                  keys, rank, scale, window)
  if (keys <= 128)
    LLB_GENERIC(4);
  else if (keys <= 512)
    LLB_GENERIC(16);
  else
    LLB_GENERIC(32);
#undef LLB_GENERIC
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// ---------------------------------------------------------------------------------------------- tensor cores, bf16
constexpr int KT = 64;       // keys per tile
constexpr int STAGES = 3;
constexpr int S_PITCH = KT + 8;  // floats per score row in shared memory

template <int LAT>
constexpr int mma_smem() {
  return STAGES * KT * LAT * 2 + 2 * 16 * S_PITCH * 4 + 2 * KT * 4;
}

// byte offset of 16-byte chunk `ch` of key `row` inside a tile
template <int LAT>
__device__ __forceinline__ uint32_t tile_off(int row, int ch) {
  return (uint32_t)(row * (LAT * 2) + ((ch ^ (row & 7)) << 4));
}

// LAT: columns of a tile, at least `keys` (tile columns beyond the row pitch are zero-filled); LATV: columns read as values, at
// least `rank`.
// Partial results (splits > 1): part_o [split][token][head][rank] unnormalised, part_ml [split][token][head] (max, sum).
template <int LAT, int LATV>
__global__ void __launch_bounds__(256, 1)
latent_attn_mma_kernel(const bf16* __restrict__ q_lat, const bf16* __restrict__ pool, int row_elems,
                       const int* __restrict__ req_to_token, int64_t r2t_stride, const int* __restrict__ b_req_idx,
                       const int* __restrict__ pos, const int* __restrict__ batch_of, bf16* __restrict__ out,
                       float* __restrict__ part_o, float2* __restrict__ part_ml, int Tn, int H, int keys, int rank,
                       float scale_log2, int window) {
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int CH = LAT / 8;            // 16-byte chunks per tile row
  constexpr int KSTEPS = LAT / 16;
  constexpr int N2 = LATV / 128;         // pairs of 8-column output blocks per warp
  const uint32_t kv_base = smem_u32(smem);
  float* s_sm = reinterpret_cast<float*>(smem + STAGES * KT * LAT * 2);
  int* slot_sm = reinterpret_cast<int*>(s_sm + 2 * 16 * S_PITCH);

  const int t = blockIdx.x, head0 = blockIdx.y * 16;
  const int split = blockIdx.z, splits = gridDim.z;
  const int b = batch_of ? batch_of[t] : t;
  const int p = pos[t];
  const int* slots = req_to_token + (int64_t)LLB_CHECK_REQ(b_req_idx[b]) * r2t_stride;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tig = lane & 3;
  const int row_ch = row_elems >> 3;

  const int k_begin = window > 0 ? max(0, p - window + 1) : 0;
  const int k_end = p + 1;
  const int all_tiles = (k_end - k_begin + KT - 1) / KT;
  const int tile0 = (int)((int64_t)split * all_tiles / splits), tile1 = (int)((int64_t)(split + 1) * all_tiles / splits);
  const int n_tiles = tile1 - tile0;
  const int key0 = k_begin + tile0 * KT;

  // slots of tile `i` -> slot_sm[i & 1] (-1 beyond the last visible key)
  auto fetch_slot = [&](int i) {
    const int kp = key0 + i * KT + (int)threadIdx.x;
    return (i < n_tiles && kp < k_end) ? LLB_CHECK_SLOT(slots[LLB_CHECK_POS(kp)]) : -1;
  };
  auto issue = [&](int i) {
    if (i < n_tiles) {
      const uint32_t sb = kv_base + (uint32_t)(i % STAGES) * (KT * LAT * 2);
      const int* sl_sm = slot_sm + (i & 1) * KT;
#pragma unroll 4
      for (int c = threadIdx.x; c < KT * CH; c += 256) {
        const int tok = c / CH, ch = c % CH;
        const int sl = sl_sm[tok];
        const bool ok = sl >= 0 && ch < row_ch;
        cp_async16(sb + tile_off<LAT>(tok, ch), pool + (ok ? (int64_t)sl * row_elems + ch * 8 : 0), ok);
      }
    }
    cp_async_commit();
  };

  if (threadIdx.x < KT) {
    slot_sm[threadIdx.x] = fetch_slot(0);
    slot_sm[KT + threadIdx.x] = fetch_slot(1);
  }
  // query rows as MMA fragments
  uint32_t qf[KSTEPS][4];
  {
    const bf16* q0 = q_lat + ((int64_t)t * H + head0 + g) * keys;
    const bf16* q1 = q0 + (int64_t)8 * keys;
    const bool ok0 = head0 + g < H, ok1 = head0 + g + 8 < H;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
      const int d = ks * 16 + tig * 2;
      qf[ks][0] = ok0 && d < keys ? *reinterpret_cast<const uint32_t*>(q0 + d) : 0u;
      qf[ks][1] = ok1 && d < keys ? *reinterpret_cast<const uint32_t*>(q1 + d) : 0u;
      qf[ks][2] = ok0 && d + 8 < keys ? *reinterpret_cast<const uint32_t*>(q0 + d + 8) : 0u;
      qf[ks][3] = ok1 && d + 8 < keys ? *reinterpret_cast<const uint32_t*>(q1 + d + 8) : 0u;
    }
  }
  // scores of this warp's 8 keys of tile i over the whole latent, scaled and masked: columns (warp * 8 + tig * 2, + 1) of
  // rows g and g + 8
  auto scores = [&](int i, float* s) {
    const uint32_t kb = kv_base + (uint32_t)(i % STAGES) * (KT * LAT * 2);
    float sc[4][4];
#pragma unroll
    for (int a = 0; a < 4; ++a) sc[a][0] = sc[a][1] = sc[a][2] = sc[a][3] = 0.f;
#pragma unroll
    for (int k2 = 0; k2 < KSTEPS / 2; ++k2) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, kb + tile_off<LAT>(warp * 8 + (lane & 7), k2 * 4 + (lane >> 3)));
      mma_bf16_16816(sc[(2 * k2) & 3], qf[2 * k2][0], qf[2 * k2][1], qf[2 * k2][2], qf[2 * k2][3], b0, b1);
      mma_bf16_16816(sc[(2 * k2 + 1) & 3], qf[2 * k2 + 1][0], qf[2 * k2 + 1][1], qf[2 * k2 + 1][2], qf[2 * k2 + 1][3],
                     b2, b3);
    }
    const int kp = key0 + i * KT + warp * 8 + tig * 2;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      s[e] = kp + (e & 1) < k_end ? ((sc[0][e] + sc[1][e]) + (sc[2][e] + sc[3][e])) * scale_log2 : -INFINITY;
  };
  auto store_scores = [&](int i, const float* s) {
    float* dst = s_sm + (i & 1) * 16 * S_PITCH + warp * 8 + tig * 2;
    *reinterpret_cast<float2*>(dst + g * S_PITCH) = make_float2(s[0], s[1]);
    *reinterpret_cast<float2*>(dst + (g + 8) * S_PITCH) = make_float2(s[2], s[3]);
  };

  __syncthreads();
  issue(0);
  issue(1);
  __syncthreads();  // both slot buffers read
  if (threadIdx.x < KT) slot_sm[threadIdx.x] = fetch_slot(2);

  float o[2 * N2][4];
#pragma unroll
  for (int i = 0; i < 2 * N2; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  if (n_tiles > 0) {
    cp_async_wait<1>();  // tile 0 landed
    __syncthreads();
    float s0[4];
    scores(0, s0);
    store_scores(0, s0);
  }
  // One barrier per tile: between two of them every warp computes the scores of tile i + 1 and the softmax and P . c of
  // tile i, which do not depend on each other.
  for (int i = 0; i < n_tiles; ++i) {
    cp_async_wait<0>();  // tile i + 1 landed
    __syncthreads();     // ... for all threads; scores of tile i and slots of tile i + 2 visible; tile i - 1 free
    issue(i + 2);
    const int next_slot = threadIdx.x < KT ? fetch_slot(i + 3) : 0;
    const uint32_t kb = kv_base + (uint32_t)(i % STAGES) * (KT * LAT * 2);
    const float* s_cur = s_sm + (i & 1) * 16 * S_PITCH;
    float s_next[4];
    if (i + 1 < n_tiles) scores(i + 1, s_next);

    // ---- softmax bookkeeping, the same in all warps ----
    float s[KT / 8][4];
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < KT / 8; ++j) {
      const float2 lo = *reinterpret_cast<const float2*>(s_cur + g * S_PITCH + j * 8 + tig * 2);
      const float2 hi = *reinterpret_cast<const float2*>(s_cur + (g + 8) * S_PITCH + j * 8 + tig * 2);
      s[j][0] = lo.x; s[j][1] = lo.y; s[j][2] = hi.x; s[j][3] = hi.y;
      mx[0] = fmaxf(mx[0], fmaxf(lo.x, lo.y));
      mx[1] = fmaxf(mx[1], fmaxf(hi.x, hi.y));
    }
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float m_new = fmaxf(m_run[r], mx[r]);  // finite: every tile has a visible key
      alpha[r] = exp2f(m_run[r] - m_new);
      m_run[r] = m_new;
      float rs = 0.f;
#pragma unroll
      for (int j = 0; j < KT / 8; ++j) {
        s[j][2 * r] = exp2f(s[j][2 * r] - m_new);
        s[j][2 * r + 1] = exp2f(s[j][2 * r + 1] - m_new);
        rs += s[j][2 * r] + s[j][2 * r + 1];
      }
      l_run[r] = l_run[r] * alpha[r] + rs;
    }
#pragma unroll
    for (int n = 0; n < 2 * N2; ++n) {
      o[n][0] *= alpha[0];
      o[n][1] *= alpha[0];
      o[n][2] *= alpha[1];
      o[n][3] *= alpha[1];
    }
    // ---- o[:, this warp's columns] += P . c, P = high + low bf16 parts ----
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int q4 = 0; q4 < 4; ++q4) {  // a0: row g, a1: row g + 8, a2 / a3: the same rows, keys + 8
        const float x = s[2 * kk + (q4 >> 1)][(q4 & 1) * 2], y = s[2 * kk + (q4 >> 1)][(q4 & 1) * 2 + 1];
        ah[q4] = pack_bf16x2(x, y);
        const float xh = __uint_as_float(ah[q4] << 16), yh = __uint_as_float(ah[q4] & 0xffff0000u);
        al[q4] = pack_bf16x2(x - xh, y - yh);
      }
      const int tok = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int n = 0; n < N2; ++n) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, kb + tile_off<LAT>(tok, warp * (LATV / 64) + n * 2 + (lane >> 4)));
        mma_bf16_16816(o[2 * n], ah[0], ah[1], ah[2], ah[3], b0, b1);
        mma_bf16_16816(o[2 * n + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
        mma_bf16_16816(o[2 * n], al[0], al[1], al[2], al[3], b0, b1);
        mma_bf16_16816(o[2 * n + 1], al[0], al[1], al[2], al[3], b2, b3);
      }
    }
    if (i + 1 < n_tiles) store_scores(i + 1, s_next);
    if (threadIdx.x < KT) slot_sm[((i + 1) & 1) * KT + threadIdx.x] = next_slot;
  }

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    const int h = head0 + g + 8 * r;
    if (h >= H) continue;
    const int64_t row = (int64_t)t * H + h;
    const int col0 = warp * (LATV / 8) + tig * 2;
    if (splits == 1) {
      const float inv = 1.f / l_run[r];
#pragma unroll
      for (int n = 0; n < 2 * N2; ++n) {
        const int col = col0 + n * 8;
        if (col < rank)
          *reinterpret_cast<bf162*>(out + row * rank + col) =
              __floats2bfloat162_rn(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
      }
    } else {
      const int64_t prow = (int64_t)split * Tn * H + row;
#pragma unroll
      for (int n = 0; n < 2 * N2; ++n) {
        const int col = col0 + n * 8;
        if (col < rank)
          *reinterpret_cast<float2*>(part_o + prow * rank + col) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
      }
      if (warp == 0 && tig == 0) part_ml[prow] = make_float2(m_run[r], l_run[r]);
    }
  }
  cp_async_wait<0>();
}

// One warp per (token, head): merges the partial results of the shares.
__global__ void __launch_bounds__(256)
latent_attn_merge_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, bf16* __restrict__ out,
                         int rows, int rank, int splits) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, part_ml[(int64_t)s * rows + row].x);
  float L = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float2 ml = part_ml[(int64_t)s * rows + row];
    if (ml.x != -INFINITY) L += ml.y * exp2f(ml.x - M);
  }
  const float inv = 1.f / L;
  for (int d = lane * 2; d < rank; d += 64) {
    float2 acc = make_float2(0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float m = part_ml[(int64_t)s * rows + row].x;
      if (m == -INFINITY) continue;
      const float w = exp2f(m - M);
      const float2 v = *reinterpret_cast<const float2*>(part_o + ((int64_t)s * rows + row) * rank + d);
      acc.x += w * v.x;
      acc.y += w * v.y;
    }
    *reinterpret_cast<bf162*>(out + (int64_t)row * rank + d) = __floats2bfloat162_rn(acc.x * inv, acc.y * inv);
  }
}

struct MmaArgs {
  const bf16 *q_lat, *pool;
  bf16* out;
  const int *r2t, *b_req_idx, *pos, *batch_of;
  float* part_o;
  float2* part_ml;
  int64_t r2t_stride;
  int row_elems, T, H, keys, rank, window, splits;
  float scale_log2;
};

template <int LAT, int LATV>
int launch_mma(const MmaArgs& a, cudaStream_t st) {
  static DeviceOnce configured;
  if (!configured.done()) {
    cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<LAT, LATV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         mma_smem<LAT>());
    if (e != cudaSuccess) return (int)e;
    configured.set();
  }
  const dim3 grid(a.T, (a.H + 15) / 16, a.splits);
  latent_attn_mma_kernel<LAT, LATV><<<grid, 256, mma_smem<LAT>(), st>>>(
      a.q_lat, a.pool, a.row_elems, a.r2t, a.r2t_stride, a.b_req_idx, a.pos, a.batch_of, a.out, a.part_o, a.part_ml, a.T,
      a.H, a.keys, a.rank, a.scale_log2, a.window);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

}  // namespace

// dtype: 0 = fp32, 1 = bf16.  src row: [latent, `rank` values in `cols` columns | rot_dims values to rotate]; the pool row gets
// [RMSNorm(latent) * w, zero to cols | rotated part, zero to row_elems].  q_src (or null): rows of q_rank values in q_cols columns,
// normalised into q_out [T, q_cols].  Columns and pitches are multiples of 8.
LLB_EXPORT int llb_latent_prepare(const void* src, int dtype, int64_t src_stride, void* pool, int row_elems, const float* w,
                                  const int* slot, int T, int rank, int cols, const float* cos_t, const float* sin_t,
                                  const int* pos, int rot_dims, int neighbours, const void* q_src, int64_t q_stride,
                                  void* q_out, int q_rank, int q_cols, const float* q_w, float eps, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (rank <= 0 || rank > cols || cols + rot_dims > row_elems || (cols % 8) || (row_elems % 8) || (src_stride % 8) ||
      rot_dims < 0 || (rot_dims & 1) || ((uintptr_t)src & 15) || ((uintptr_t)pool & 15) || ((uintptr_t)w & 15) ||
      (rot_dims > 0 && (cos_t == nullptr || sin_t == nullptr || pos == nullptr)))
    return LLB_ERR_BAD_ARG;
  if (q_src != nullptr && (q_rank <= 0 || q_rank > q_cols || (q_cols % 8) || (q_stride % 8) || q_out == nullptr ||
                           q_w == nullptr || (((uintptr_t)q_src | (uintptr_t)q_out | (uintptr_t)q_w) & 15)))
    return LLB_ERR_BAD_ARG;
  const Rotation rot{cos_t, sin_t, pos, rot_dims, neighbours};
  const dim3 grid(cdiv(q_src != nullptr ? 2 * T : T, 4));
#define LLB_PREPARE(E)                                                                                                     \
  launch_pdl(latent_prepare_kernel<E>, grid, dim3(128), 0, st,                                                             \
             PrepareArgs<E>{(const E*)src, src_stride, (E*)pool, row_elems, rank, cols, w, slot, rot, (const E*)q_src,     \
                            q_stride, (E*)q_out, q_rank, q_cols, q_w, T, eps})
  if (dtype == 0)
    LLB_PREPARE(float);
  else
    LLB_PREPARE(bf16);
#undef LLB_PREPARE
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// x [T, H heads, `pitch` elements apart] (row pitch `stride`): columns off .. off + dims of every head rotated in place.
LLB_EXPORT int llb_rope_heads(void* x, int dtype, int64_t stride, const float* cos_t, const float* sin_t, const int* pos, int T,
                              int H, int pitch, int off, int dims, int neighbours, cudaStream_t st) {
  if (T <= 0 || dims <= 0) return LLB_OK;
  if (H <= 0 || off < 0 || off + dims > pitch || (dims & 1)) return LLB_ERR_BAD_ARG;
  const Rotation rot{cos_t, sin_t, pos, dims, neighbours};
  const bool vec = neighbours && dims % 8 == 0 && off % 8 == 0 && pitch % 8 == 0 && stride % 8 == 0 && ((uintptr_t)x & 15) == 0;
  const int64_t items = (int64_t)T * H * (vec ? dims / 8 : dims / 2);
  const dim3 grid((unsigned)cdiv64(items, 256));
#define LLB_ROPE(E, V) launch_pdl(rope_heads_kernel<E, V>, grid, dim3(256), 0, st, (E*)x, stride, rot, items, H, pitch, off)
  if (dtype == 0) {
    if (vec)
      LLB_ROPE(float, true);
    else
      LLB_ROPE(float, false);
  } else if (vec) {
    LLB_ROPE(bf16, true);
  } else {
    LLB_ROPE(bf16, false);
  }
#undef LLB_ROPE
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

LLB_EXPORT int llb_latent_gather(const void* pool, int row_bytes, const int* req_to_token, int64_t r2t_stride,
                                 const int* b_req_idx, const int* cu_kv, const int* kv_start, void* out, int B, int rows,
                                 cudaStream_t st) {
  if (B <= 0 || rows <= 0) return LLB_OK;
  if ((row_bytes & 15) || ((uintptr_t)pool & 15) || ((uintptr_t)out & 15)) return LLB_ERR_BAD_ARG;
  const int grid = cdiv(rows, 8) < 148 * 8 ? cdiv(rows, 8) : 148 * 8;
  latent_gather_kernel<<<grid, 256, 0, st>>>((const uint4*)pool, row_bytes / 16, req_to_token, r2t_stride, b_req_idx,
                                             cu_kv, kv_start, (uint4*)out, B);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// q_lat [T, H, keys], out [T, H, rank], contiguous (padding columns of q_lat are zero); the pool row has row_elems >= keys values.
// pos: position of every query token; batch_of: its request (null: token i belongs to request i).
LLB_EXPORT int llb_latent_attn_generic(const void* q_lat, int dtype, const void* pool, int row_elems,
                                       const int* req_to_token, int64_t r2t_stride, const int* b_req_idx, const int* pos,
                                       const int* batch_of, void* out, int T, int H, int keys, int rank, float scale,
                                       int window, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (rank <= 0 || rank > keys || keys > 1024 || keys > row_elems || H <= 0 || H > 65535) return LLB_ERR_UNSUPPORTED;
  return dtype == 0 ? launch_generic<float>(q_lat, pool, row_elems, req_to_token, r2t_stride, b_req_idx, pos, batch_of,
                                            out, T, H, keys, rank, scale, window, st)
                    : launch_generic<bf16>(q_lat, pool, row_elems, req_to_token, r2t_stride, b_req_idx, pos, batch_of,
                                           out, T, H, keys, rank, scale, window, st);
}

// bf16; keys and rank multiples of 8, at most 576 and 512.  splits > 1: part_o [splits * T * H * rank] and part_ml [splits * T * H * 2]
// floats of scratch.
LLB_EXPORT int llb_latent_attn_mma(const void* q_lat, const void* pool, int row_elems, const int* req_to_token,
                                   int64_t r2t_stride, const int* b_req_idx, const int* pos, const int* batch_of,
                                   void* out, float* part_o, float* part_ml, int T, int H, int keys, int rank,
                                   int splits, float scale, int window, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (rank <= 0 || rank > 512 || rank > keys || keys > 576 || (rank % 8) || (keys % 8) || (row_elems % 8) ||
      keys > row_elems || H <= 0)
    return LLB_ERR_UNSUPPORTED;
  if (splits < 1 || splits > 256 || (splits > 1 && (part_o == nullptr || part_ml == nullptr))) return LLB_ERR_BAD_ARG;
  if (((uintptr_t)q_lat & 15) || ((uintptr_t)pool & 15) || ((uintptr_t)out & 3)) return LLB_ERR_BAD_ARG;
  MmaArgs a{(const bf16*)q_lat, (const bf16*)pool, (bf16*)out, req_to_token, b_req_idx, pos, batch_of, part_o,
            (float2*)part_ml, r2t_stride, row_elems, T, H, keys, rank, window, splits, scale * kLog2e};
  int rc;
  if (rank <= 128 && keys <= 128)
    rc = launch_mma<128, 128>(a, st);
  else if (rank <= 128 && keys <= 192)
    rc = launch_mma<192, 128>(a, st);
  else if (rank <= 256 && keys <= 256)
    rc = launch_mma<256, 256>(a, st);
  else if (rank <= 256 && keys <= 320)
    rc = launch_mma<320, 256>(a, st);
  else if (rank <= 384 && keys <= 384)
    rc = launch_mma<384, 384>(a, st);
  else if (rank <= 384 && keys <= 448)
    rc = launch_mma<448, 384>(a, st);
  else if (keys <= 512)
    rc = launch_mma<512, 512>(a, st);
  else
    rc = launch_mma<576, 512>(a, st);
  if (rc || splits == 1) return rc;
  latent_attn_merge_kernel<<<cdiv(T * H, 8), 256, 0, st>>>(part_o, (const float2*)part_ml, (bf16*)out, T * H, rank, splits);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}
