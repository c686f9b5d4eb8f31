// RMS norms around an fp32 residual stream: sublayers that read the stream itself and are normalised on the way out (w), and
// sublayers that read a norm of the stream (w_next) and are added as they are (no w):
//
//   embedding_pair    x[t] = table[id] + table2[(prev * mul_prev + id * mul_cur) mod buckets]   (second table optional; a
//                     sequence's first token takes row `buckets`);  h[t] = x[t], or rms(x[t]) * w_next
//   add_rms           x += rms(y) * w, or x += y;  h = x, or rms(x) * w_next when a next norm is given
//   moe_combine_rms   y[t] = sum_k weight[t,k] * expert_out[row of (t,k)] + shared[t], then add_rms; or, when a tensor-
//                     parallel reduction follows, y[t] is written out in fp32
//
// with rms(v) = v / sqrt(mean(v^2) + eps).  The stream x, the norms and the sums are fp32; h has the number format of the
// layer's matrix products (bf16 or fp32).  Rows are W elements apart (a multiple of 8, zero beyond `width`, over which the
// mean is taken); one CTA per row keeps the row in registers, so every operand is read once.
#include "common.cuh"

using namespace llb;
LLB_DEBUG_BOUNDS_STORAGE(rms_stream)

namespace {

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

struct Bigram {
  int64_t buckets, mul_prev, mul_cur;
  int* slot_token;  // token id of every pool slot
  const int *mem_index, *pos, *batch_of, *b_req_idx, *req_to_token;
  int64_t r2t_stride;
};

template <typename TH>
__global__ void __launch_bounds__(256) embedding_pair_kernel(const int64_t* __restrict__ ids, const TH* __restrict__ table,
                                                             const TH* __restrict__ table2, const Bigram g,
                                                             float* __restrict__ x, TH* __restrict__ h, int64_t vocab,
                                                             int W, const float* __restrict__ w_next, int width,
                                                             float eps) {
  pdl_wait();
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int64_t id = ids[t];
  const TH* r1 = table + (id >= 0 && id < vocab ? id : 0) * W;
  const TH* r2 = nullptr;
  if (table2 != nullptr) {
    const int p = g.pos[t];
    int64_t row = g.buckets;
    if (p > 0) {
      // the previous token is the row before in this pass, or sits in the pool slot of the position before
      int64_t prev;
      if (g.batch_of != nullptr && t > 0 && g.batch_of[t - 1] == g.batch_of[t]) {
        prev = ids[t - 1];
      } else {
        const int req = LLB_CHECK_REQ(g.b_req_idx[g.batch_of != nullptr ? g.batch_of[t] : t]);
        prev = g.slot_token[LLB_CHECK_SLOT(g.req_to_token[(int64_t)req * g.r2t_stride + LLB_CHECK_POS(p - 1)])];
      }
      row = (prev * g.mul_prev + id * g.mul_cur) % g.buckets;
      if (row < 0) row = 0;
    }
    r2 = table2 + row * W;
    if (threadIdx.x == 0) g.slot_token[LLB_CHECK_SLOT(g.mem_index[t])] = (int)id;
  }
  float ss = 0.f;
  for (int v = threadIdx.x * 8; v < W; v += blockDim.x * 8) {
    float a[8];
    ld8(r1 + v, a);
    if (r2 != nullptr) {
      float b[8];
      ld8(r2 + v, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] += b[i];
    }
    st8(x + (int64_t)t * W + v, a);
    if (w_next == nullptr) st8(h + (int64_t)t * W + v, a);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(a[i], a[i], ss);
  }
  if (w_next == nullptr) return;
  const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
  for (int v = threadIdx.x * 8; v < W; v += blockDim.x * 8) {  // a thread reads back what it wrote
    float a[8], wv[8];
    ld8(x + (int64_t)t * W + v, a);
    ld8(w_next + v, wv);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] *= inv * wv[i];
    st8(h + (int64_t)t * W + v, a);
  }
}

struct Combine {
  const int* pair_row;
  const float* weights;
  int k;
};

// COMBINE: the row y[t] is the weighted sum of the token's expert rows (y holds them) plus shared[t].
template <typename TY, typename TH, int VPT, bool COMBINE>
__global__ void __launch_bounds__(256) add_rms_kernel(const TY* __restrict__ y, const Combine c, const TY* __restrict__ shared,
                                                      float* __restrict__ x, TH* __restrict__ h, float* __restrict__ y_out,
                                                      const float* __restrict__ w, const float* __restrict__ w_next,
                                                      int width, int W, float eps) {
  pdl_wait();
  __shared__ float red[33];
  const int64_t t = blockIdx.x, base = t * W;
  const int nv = W >> 3;
  float yv[VPT][8], xv[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int v = threadIdx.x + j * blockDim.x;
    if (v >= nv) continue;
    if (x != nullptr) ld8(x + base + v * 8, xv[j]);
    if (COMBINE) {
      if (shared != nullptr) {
        ld8(shared + base + v * 8, yv[j]);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) yv[j][i] = 0.f;
      }
      for (int s = 0; s < c.k; ++s) {
        const int r = c.pair_row[t * c.k + s];
        if (r < 0) continue;
        const float wt = c.weights[t * c.k + s];
        float f[8];
        ld8(y + (int64_t)r * W + v * 8, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) yv[j][i] = fmaf(wt, f[i], yv[j][i]);
      }
      if (y_out != nullptr) st8(y_out + base + v * 8, yv[j]);
    } else {
      ld8(y + base + v * 8, yv[j]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(yv[j][i], yv[j][i], ss);
  }
  if (x == nullptr) return;
  const float inv = w != nullptr ? rsqrtf(block_sum(ss, red) / (float)width + eps) : 1.f;
  float sx = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int v = threadIdx.x + j * blockDim.x;
    if (v >= nv) continue;
    float wv[8];
    if (w != nullptr) {
      ld8(w + v * 8, wv);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) wv[i] = 1.f;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      xv[j][i] += yv[j][i] * inv * wv[i];
      sx = fmaf(xv[j][i], xv[j][i], sx);
    }
    st8(x + base + v * 8, xv[j]);
    if (w_next == nullptr) st8(h + base + v * 8, xv[j]);
  }
  if (w_next == nullptr) return;
  const float inv2 = rsqrtf(block_sum(sx, red) / (float)width + eps);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int v = threadIdx.x + j * blockDim.x;
    if (v >= nv) continue;
    float wv[8], o[8];
    ld8(w_next + v * 8, wv);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = xv[j][i] * inv2 * wv[i];
    st8(h + base + v * 8, o);
  }
}

template <typename TY, typename TH, bool COMBINE>
int launch_add(const void* y, const Combine& c, const void* shared, float* x, void* h, float* y_out, const float* w,
               const float* w_next, int T, int width, int W, float eps, cudaStream_t st) {
  const int nv = W / 8;
  const int threads = nv >= 256 ? 256 : cdiv(nv, 32) * 32;
  const int vpt = cdiv(nv, threads);
#define LLB_ADD_RMS(V)                                                                                                  \
  launch_pdl(add_rms_kernel<TY, TH, V, COMBINE>, dim3(T), dim3(threads), 0, st, (const TY*)y, c, (const TY*)shared, x, \
             (TH*)h, y_out, w, w_next, width, W, eps)
  if (vpt == 1)
    LLB_ADD_RMS(1);
  else if (vpt == 2)
    LLB_ADD_RMS(2);
  else if (vpt <= 4)
    LLB_ADD_RMS(4);
  else if (vpt <= 8)
    LLB_ADD_RMS(8);
  else
    return LLB_ERR_UNSUPPORTED;
#undef LLB_ADD_RMS
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

template <bool COMBINE>
int dispatch_add(const void* y, int y_dt, const Combine& c, const void* shared, float* x, void* h, int h_dt, float* y_out,
                 const float* w, const float* w_next, int T, int width, int W, float eps, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8) || width <= 0 || width > W) return LLB_ERR_BAD_ARG;
  if (x == nullptr ? y_out == nullptr : h == nullptr) return LLB_ERR_BAD_ARG;
  if (y_dt == 0)
    return h_dt == 0 ? launch_add<float, float, COMBINE>(y, c, shared, x, h, y_out, w, w_next, T, width, W, eps, st)
                     : launch_add<float, bf16, COMBINE>(y, c, shared, x, h, y_out, w, w_next, T, width, W, eps, st);
  return h_dt == 0 ? launch_add<bf16, float, COMBINE>(y, c, shared, x, h, y_out, w, w_next, T, width, W, eps, st)
                   : launch_add<bf16, bf16, COMBINE>(y, c, shared, x, h, y_out, w, w_next, T, width, W, eps, st);
}

}  // namespace

// Number formats: 0 = fp32, 1 = bf16.  table [vocab, W], table2 [buckets + 1, W] or null; batch_of null: row t belongs to
// request t (decode).  slot_token [pool slots] receives the token id of every new token at mem_index[t].  w_next (or null):
// fp32 [W], zero beyond `width`.
LLB_EXPORT int llb_embedding_pair(const int64_t* ids, const void* table, int dt, int64_t vocab, const void* table2,
                                  int64_t buckets, int64_t mul_prev, int64_t mul_cur, int* slot_token,
                                  const int* mem_index, const int* pos, const int* batch_of, const int* b_req_idx,
                                  const int* req_to_token, int64_t r2t_stride, float* x, void* h, int T, int W,
                                  const float* w_next, int width, float eps, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8) || width <= 0 || width > W) return LLB_ERR_BAD_ARG;
  if (table2 != nullptr && (buckets <= 0 || slot_token == nullptr)) return LLB_ERR_BAD_ARG;
  const Bigram g{buckets, mul_prev, mul_cur, slot_token, mem_index, pos, batch_of, b_req_idx, req_to_token, r2t_stride};
  const int threads = W / 8 >= 256 ? 256 : cdiv(W / 8, 32) * 32;
  if (dt == 0)
    launch_pdl(embedding_pair_kernel<float>, dim3(T), dim3(threads), 0, st, ids, (const float*)table, (const float*)table2, g,
               x, (float*)h, vocab, W, w_next, width, eps);
  else
    launch_pdl(embedding_pair_kernel<bf16>, dim3(T), dim3(threads), 0, st, ids, (const bf16*)table, (const bf16*)table2, g, x,
               (bf16*)h, vocab, W, w_next, width, eps);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// y [T, W] (y_dt), x fp32 [T, W] in place, h [T, W] (h_dt), w and w_next (either may be null) fp32 [W].
LLB_EXPORT int llb_add_rms(const void* y, int y_dt, float* x, void* h, int h_dt, const float* w, const float* w_next, int T,
                           int width, int W, float eps, cudaStream_t st) {
  return dispatch_add<false>(y, y_dt, Combine{nullptr, nullptr, 0}, nullptr, x, h, h_dt, nullptr, w, w_next, T, width, W, eps,
                             st);
}

// y [rows, W]: expert outputs in expert-sorted order; shared [T, W] in the same format, or null.  x null: only y_out.
LLB_EXPORT int llb_moe_combine_rms(const void* y, int y_dt, const int* pair_row, const float* weights, int k,
                                   const void* shared, float* x, void* h, int h_dt, float* y_out, const float* w,
                                   const float* w_next, int T, int width, int W, float eps, cudaStream_t st) {
  if (k <= 0) return LLB_ERR_BAD_ARG;
  return dispatch_add<true>(y, y_dt, Combine{pair_row, weights, k}, shared, x, h, h_dt, y_out, w, w_next, T, width, W, eps,
                            st);
}
