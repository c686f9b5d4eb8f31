// Dynamic-tanh normalisation over an fp32 residual stream, and the row passes it is fused with.
//
//   dyt(x) = tanh(alpha * x) * w + b          elementwise: no row statistics, so it also fits a GEMM epilogue
//
//   embedding_dyt     x[t] = table[id[t]];  h[t] = dyt(x[t])
//   dyt               h = dyt(x)
//   add_dyt           x += dyt_post(y);  h = dyt_next(x)        (sandwich norm: the sublayer's output is normalised
//                                                                before it joins the stream)
//   moe_combine_dyt   y[t] = scale * sum_k expert_out[row of (t,k)] + sigmoid(h[t] . w_gate) * shared[t], then add_dyt;
//                     or, when a tensor-parallel reduction follows, y[t] is written out in fp32
//
// The stream x and all arithmetic are fp32; h has the number format of the layer's matrix products (bf16 or fp32).
// Rows are `W` elements, a multiple of 8.
#include "common.cuh"

using namespace llb;

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

struct Dyt {
  const float* w;
  const float* b;
  float alpha;
};

__device__ __forceinline__ float tanh_for(float x, const float*) { return tanhf(x); }
__device__ __forceinline__ float tanh_for(float x, const bf16*) { return tanh_fast(x); }

// TH: the number format the pass writes
template <typename TH>
__device__ __forceinline__ void dyt8(const Dyt& n, int col, const float* in, float* out) {
  float w[8], b[8];
  ld8(n.w + col, w);
  ld8(n.b + col, b);
#pragma unroll
  for (int i = 0; i < 8; ++i) out[i] = tanh_for(n.alpha * in[i], (const TH*)nullptr) * w[i] + b[i];
}

template <typename TE, typename TH>
__global__ void __launch_bounds__(256) embedding_dyt_kernel(const int64_t* __restrict__ ids, const TE* __restrict__ table,
                                                            int64_t rows, float* __restrict__ x, TH* __restrict__ h,
                                                            int T, int W, Dyt n) {
  const int wv = W >> 3;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < (int64_t)T * wv; i += (int64_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / wv), c = (int)(i - (int64_t)t * wv) * 8;
    const int64_t id = ids[t];
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, o[8];
    if (id >= 0 && id < rows) ld8(table + id * W + c, v);
    st8(x + (int64_t)t * W + c, v);
    dyt8<TH>(n, c, v, o);
    st8(h + (int64_t)t * W + c, o);
  }
}

template <typename TH>
__global__ void __launch_bounds__(256) dyt_kernel(const float* __restrict__ x, TH* __restrict__ h, int64_t n_vec, int wv,
                                                  Dyt n) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n_vec; i += (int64_t)gridDim.x * blockDim.x) {
    float v[8], o[8];
    ld8(x + i * 8, v);
    dyt8<TH>(n, (int)(i % wv) * 8, v, o);
    st8(h + i * 8, o);
  }
}

template <typename TY, typename TH>
__global__ void __launch_bounds__(256) add_dyt_kernel(float* __restrict__ x, const TY* __restrict__ y, TH* __restrict__ h,
                                                      int64_t n_vec, int wv, Dyt post, Dyt next) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n_vec; i += (int64_t)gridDim.x * blockDim.x) {
    const int c = (int)(i % wv) * 8;
    float v[8], a[8], o[8];
    ld8(y + i * 8, v);
    dyt8<TH>(post, c, v, a);
    ld8(x + i * 8, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += a[e];
    st8(x + i * 8, v);
    dyt8<TH>(next, c, v, o);
    st8(h + i * 8, o);
  }
}

// One CTA per token.  `shared` / `gate_w` may be null (no shared expert / a shared expert without a gate).
template <typename T>
__global__ void __launch_bounds__(256)
moe_combine_dyt_kernel(const T* __restrict__ y, const int* __restrict__ pair_row, int k, float scale,
                       const T* __restrict__ shared, const T* __restrict__ h_in, const float* __restrict__ gate_w,
                       float* __restrict__ x, T* __restrict__ h_out, float* __restrict__ y_out, int W, Dyt post,
                       Dyt next) {
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int64_t row = (int64_t)t * W;
  float g = 1.f;
  if (shared != nullptr && gate_w != nullptr) {
    float s = 0.f;
    for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
      float hv[8], gv[8];
      ld8(h_in + row + c, hv);
      ld8(gate_w + c, gv);
#pragma unroll
      for (int e = 0; e < 8; ++e) s += hv[e] * gv[e];
    }
    g = 1.f / (1.f + expf(-block_sum(s, red)));
  }
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, f[8];
    for (int s = 0; s < k; ++s) {
      const int r = pair_row[(int64_t)t * k + s];
      if (r < 0) continue;
      ld8(y + (int64_t)r * W + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] += f[e];
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] *= scale;
    if (shared != nullptr) {
      ld8(shared + row + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] += g * f[e];
    }
    if (y_out != nullptr) {
      st8(y_out + row + c, acc);
      continue;
    }
    float a[8], v[8], o[8];
    dyt8<T>(post, c, acc, a);
    ld8(x + row + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += a[e];
    st8(x + row + c, v);
    dyt8<T>(next, c, v, o);
    st8(h_out + row + c, o);
  }
}

int grid_for(int64_t n_vec) {
  const int64_t g = cdiv64(n_vec, 256);
  return (int)(g < 148 * 16 ? g : 148 * 16);
}

}  // namespace

// dtype codes: 0 = fp32, 1 = bf16
LLB_EXPORT int llb_embedding_dyt(const int64_t* ids, const void* table, int dtype, int64_t rows, float* x, void* h, int T,
                                 int W, const float* w, const float* b, float alpha, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8)) return LLB_ERR_UNSUPPORTED;
  const Dyt n{w, b, alpha};
  const int grid = grid_for((int64_t)T * (W / 8));
  if (dtype == 0)
    embedding_dyt_kernel<float, float><<<grid, 256, 0, st>>>(ids, (const float*)table, rows, x, (float*)h, T, W, n);
  else
    embedding_dyt_kernel<bf16, bf16><<<grid, 256, 0, st>>>(ids, (const bf16*)table, rows, x, (bf16*)h, T, W, n);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

LLB_EXPORT int llb_dyt(const float* x, void* h, int h_dtype, int T, int W, const float* w, const float* b, float alpha,
                       cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8)) return LLB_ERR_UNSUPPORTED;
  const Dyt n{w, b, alpha};
  const int64_t nv = (int64_t)T * (W / 8);
  if (h_dtype == 0)
    dyt_kernel<float><<<grid_for(nv), 256, 0, st>>>(x, (float*)h, nv, W / 8, n);
  else
    dyt_kernel<bf16><<<grid_for(nv), 256, 0, st>>>(x, (bf16*)h, nv, W / 8, n);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

LLB_EXPORT int llb_add_dyt(float* x, const void* y, int y_dtype, void* h, int h_dtype, int T, int W, const float* w1,
                           const float* b1, float alpha1, const float* w2, const float* b2, float alpha2,
                           cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8)) return LLB_ERR_UNSUPPORTED;
  const Dyt post{w1, b1, alpha1}, next{w2, b2, alpha2};
  const int64_t nv = (int64_t)T * (W / 8);
  if (y_dtype == 0 && h_dtype == 0)
    add_dyt_kernel<float, float><<<grid_for(nv), 256, 0, st>>>(x, (const float*)y, (float*)h, nv, W / 8, post, next);
  else if (y_dtype == 0)
    add_dyt_kernel<float, bf16><<<grid_for(nv), 256, 0, st>>>(x, (const float*)y, (bf16*)h, nv, W / 8, post, next);
  else if (h_dtype == 1)
    add_dyt_kernel<bf16, bf16><<<grid_for(nv), 256, 0, st>>>(x, (const bf16*)y, (bf16*)h, nv, W / 8, post, next);
  else
    return LLB_ERR_UNSUPPORTED;
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// y_out != null: only the fp32 sum is written (x / h_out unused).
LLB_EXPORT int llb_moe_combine_dyt(const void* y, int dtype, const int* pair_row, int k, float scale, const void* shared,
                                   const void* h_in, const float* gate_w, float* x, void* h_out, float* y_out, int T,
                                   int W, const float* w1, const float* b1, float alpha1, const float* w2, const float* b2,
                                   float alpha2, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8)) return LLB_ERR_UNSUPPORTED;
  const Dyt post{w1, b1, alpha1}, next{w2, b2, alpha2};
  const int threads = W >= 2048 ? 256 : 128;
  if (dtype == 0)
    moe_combine_dyt_kernel<float><<<T, threads, 0, st>>>((const float*)y, pair_row, k, scale, (const float*)shared,
                                                         (const float*)h_in, gate_w, x, (float*)h_out, y_out, W, post,
                                                         next);
  else
    moe_combine_dyt_kernel<bf16><<<T, threads, 0, st>>>((const bf16*)y, pair_row, k, scale, (const bf16*)shared,
                                                        (const bf16*)h_in, gate_w, x, (bf16*)h_out, y_out, W, post,
                                                        next);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}
