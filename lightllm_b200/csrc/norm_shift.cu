// Norm ahead of a sublayer around an fp32 residual stream, with an optional token shift:
//
//   x'[t] = x[t] + y[t]          (x null: x' = y, the embedding's rows, found through ids)
//   n[t]  = (x'[t] - mean) / sqrt(var + eps) * w      (centred; or without the mean: x' / sqrt(mean(x'^2) + eps) * w)
//   h[t]  = n[t], or n[t] + (n[t - 1] - n[t]) * mu    with n[t - 1] of the same sequence, zero ahead of its first token
//
// x', n and the shift are fp32; h has the number format of the sublayer's matrix products.  Rows are W elements apart (a multiple
// of 8, zero beyond `width`, over which the statistics are taken).  The n of a sequence's last token is part of its state: one fp32
// row per request slot.
//
//   norm_row     one row per CTA, in registers: passes without a shift, and decode steps (every row has its own state row)
//   norm_rows    prompts with a shift: a CTA takes a run of rows, the loads of the next one under way (asynchronous copies, every
//                thread its own columns), and carries n in registers.  It starts with the row before its own, formed again: x' is
//                therefore written to another buffer than x.  The CTA of a request's first row in the pass reads the request's state
//                and, after that, leaves there the n of the request's last row, which it forms once more unless it is the same row:
//                so nobody else touches the state row.
#include "common.cuh"

using namespace llb;
LLB_DEBUG_BOUNDS_STORAGE(norm_shift)

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

struct Norm {
  const void* y;
  const int64_t* ids;  // row of y per token, or null (row t)
  int64_t y_rows;
  const float* x;      // or null
  float* x_out;
  void* h;
  const float* w;
  int T, width, W, centred;
  float eps;
  // token shift
  const float* mu;     // or null: no shift
  float* state;        // [slots, W], row pitch state_row
  int64_t state_row;
  const int *req, *cu_q, *first_pos, *batch_of;  // cu_q, batch_of null: row t is the one token of request t
};

// Sum over the CTA.  red: 16 floats, those beyond the CTA's warps zero, that nobody writes until the next __syncthreads after this.
__device__ __forceinline__ float sum_all(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const float4 *r = reinterpret_cast<const float4*>(red), a = r[0], b = r[1];
  float s = ((a.x + a.y) + (a.z + a.w)) + ((b.x + b.y) + (b.z + b.w));
  if (blockDim.x > 256) {
    const float4 c = r[2], d = r[3];
    s += ((c.x + c.y) + (c.z + c.w)) + ((d.x + d.y) + (d.z + d.w));
  }
  return s;
}

// row of y that belongs to token t
__device__ __forceinline__ int64_t source_row(const Norm& p, int t) {
  if (p.ids == nullptr) return t;
  const int64_t id = p.ids[t];
  return id >= 0 && id < p.y_rows ? id : 0;
}

// v = x + y of row t
template <typename TY, int VPT>
__device__ __forceinline__ void load_row(const Norm& p, int t, float (*v)[8]) {
  const TY* y = (const TY*)p.y + source_row(p, t) * p.W;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int c = threadIdx.x + j * blockDim.x;
#pragma unroll
    for (int i = 0; i < 8; ++i) v[j][i] = 0.f;
    if (c >= p.W >> 3) continue;
    ld8(y + c * 8, v[j]);
    if (p.x != nullptr) {
      float x[8];
      ld8(p.x + (int64_t)t * p.W + c * 8, x);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[j][i] += x[i];
    }
  }
}

// v -> its norm (zero beyond `width`).  red: 32 floats, zero at first; consecutive calls may share them.
template <int VPT>
__device__ __forceinline__ void norm_values(const Norm& p, float (*v)[8], float* red) {
  float mean = 0.f;
  if (p.centred) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) s += v[j][i];
    mean = sum_all(s, red) / (float)p.width;
  }
  float q = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int left = p.width - (int)(threadIdx.x + j * blockDim.x) * 8;  // columns from here on
    if (left >= 8) {
#pragma unroll
      for (int i = 0; i < 8; ++i) v[j][i] -= mean;
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) v[j][i] = i < left ? v[j][i] - mean : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) q = fmaf(v[j][i], v[j][i], q);
  }
  if (!p.centred) __syncthreads();  // the last call's readers are done
  const float inv = rsqrtf(sum_all(q, red + 16) / (float)p.width + p.eps);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int c = threadIdx.x + j * blockDim.x;
    if (c >= p.W >> 3) continue;
    float w[8];
    ld8(p.w + c * 8, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[j][i] *= inv * w[i];
  }
}

// o = n + (before - n) mu of the 8 columns at c
__device__ __forceinline__ void shifted(const Norm& p, int c, const float* n, const float* before, float* o) {
  float mu[8];
  ld8(p.mu + c * 8, mu);
#pragma unroll
  for (int i = 0; i < 8; ++i) o[i] = fmaf(before[i] - n[i], mu[i], n[i]);
}

template <typename TY, typename TH, int VPT, bool SHIFT>
__global__ void __launch_bounds__(512) norm_row_kernel(const Norm p) {
  pdl_wait();
  __shared__ __align__(16) float red[32];
  if (threadIdx.x < 32) red[threadIdx.x] = 0.f;
  __syncthreads();
  const int nv = p.W >> 3, t = blockIdx.x;
  float v[VPT][8];
  load_row<TY, VPT>(p, t, v);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int c = threadIdx.x + j * blockDim.x;
    if (c < nv) st8(p.x_out + (int64_t)t * p.W + c * 8, v[j]);
  }
  norm_values<VPT>(p, v, red);
  float* st = SHIFT ? p.state + (int64_t)LLB_CHECK_REQ(p.req[t]) * p.state_row : nullptr;
  const bool fresh = SHIFT && p.first_pos[t] == 0;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int c = threadIdx.x + j * blockDim.x;
    if (c >= nv) continue;
    TH* h = (TH*)p.h + (int64_t)t * p.W + c * 8;
    if (!SHIFT) {
      st8(h, v[j]);
      continue;
    }
    float before[8] = {}, o[8];
    if (!fresh) ld8(st + c * 8, before);
    shifted(p, c, v[j], before, o);
    st8(h, o);
    st8(st + c * 8, v[j]);
  }
}

constexpr int kMaxRows = 32;  // rows of one CTA

// S: rows in flight (1: none ahead).  Dynamic shared memory: S rows of x and of y.
template <typename TY, typename TH, int VPT, int S>
__global__ void __launch_bounds__(512, VPT == 2 ? 2 : 1) norm_rows_kernel(const Norm p, int rows) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t ring[];
  __shared__ __align__(16) float red[32];
  __shared__ int64_t src[kMaxRows + 1];  // rows of y, from the row before the first
  __shared__ int rq[kMaxRows + 2];       // requests of rows t0 - 2 ..; -1 ahead of the first row
  const int nv = p.W >> 3, t0 = blockIdx.x * rows, t1 = min(t0 + rows, p.T);
  if (threadIdx.x < 32) red[threadIdx.x] = 0.f;
  for (int i = threadIdx.x; i < rows + 2; i += blockDim.x) {
    const int t = t0 - 2 + i;
    rq[i] = t >= 0 && t < p.T ? p.batch_of[t] : -1;
    if (i > 0) src[i - 1] = t >= 0 && t < p.T ? source_row(p, t) : 0;
  }
  __syncthreads();
  const int begin = rq[1] >= 0 && rq[1] == rq[2] ? t0 - 1 : t0;  // the row before, if it is of the same request
  const uint32_t row_bytes = p.W * (4 + (uint32_t)sizeof(TY));
  auto issue = [&](int t) {
    if (t < t1) {
      uint8_t* dst = ring + (uint32_t)((t - begin) % S) * row_bytes;
      const TY* y = (const TY*)p.y + src[t - t0 + 1] * p.W;
#pragma unroll
      for (int j = 0; j < VPT; ++j) {
        const int c = threadIdx.x + j * blockDim.x;
        if (c >= nv) continue;
        if (p.x != nullptr) {
          const float* x = p.x + (int64_t)t * p.W + c * 8;
          cp_async16(smem_u32(dst + c * 32), x, true);
          cp_async16(smem_u32(dst + c * 32 + 16), x + 4, true);
        }
        TY* d = reinterpret_cast<TY*>(dst + p.W * 4) + c * 8;
#pragma unroll
        for (int k = 0; k < (int)sizeof(TY) / 2; ++k)
          cp_async16(smem_u32(d) + 16 * k, reinterpret_cast<const uint8_t*>(y + c * 8) + 16 * k, true);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < S - 1; ++i) issue(begin + i);
  float before[VPT][8];
  for (int t = begin; t < t1; ++t) {
    issue(t + S - 1);
    cp_async_wait<S - 1>();
    const uint8_t* from = ring + (uint32_t)((t - begin) % S) * row_bytes;
    float v[VPT][8];
    const bool own = t >= t0;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {  // a thread reads the columns it copied
      const int c = threadIdx.x + j * blockDim.x;
#pragma unroll
      for (int i = 0; i < 8; ++i) v[j][i] = 0.f;
      if (c >= nv) continue;
      ld8(reinterpret_cast<const TY*>(from + p.W * 4) + c * 8, v[j]);
      if (p.x != nullptr) {
        float x[8];
        ld8(reinterpret_cast<const float*>(from) + c * 8, x);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[j][i] += x[i];
      }
      if (own) st8(p.x_out + (int64_t)t * p.W + c * 8, v[j]);
    }
    norm_values<VPT>(p, v, red);
    float* st = nullptr;  // the request's state row, when this is its first row in the pass
    bool fresh = false, last_too = false;
    const int q = rq[t - t0 + 2];
    if (own && q != rq[t - t0 + 1]) {
      st = p.state + (int64_t)LLB_CHECK_REQ(p.req[q]) * p.state_row;
      fresh = p.first_pos[q] == 0;
      last_too = p.cu_q[q + 1] - 1 == t;
    }
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
      if (c >= nv) continue;
      if (own) {
        if (st != nullptr) {
          if (fresh) {
#pragma unroll
            for (int i = 0; i < 8; ++i) before[j][i] = 0.f;
          } else {
            ld8(st + c * 8, before[j]);
          }
        }
        float o[8];
        shifted(p, c, v[j], before[j], o);
        st8((TH*)p.h + (int64_t)t * p.W + c * 8, o);
        if (last_too) st8(st + c * 8, v[j]);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) before[j][i] = v[j][i];
    }
  }
  // requests that start here and end on a later row: their last row once more, for the state
  for (int t = t0; t < t1; ++t) {
    const int q = rq[t - t0 + 2];
    if (q == rq[t - t0 + 1]) continue;
    const int last = p.cu_q[q + 1] - 1;
    if (last == t) continue;
    float v[VPT][8];
    load_row<TY, VPT>(p, last, v);
    norm_values<VPT>(p, v, red);
    float* st = p.state + (int64_t)LLB_CHECK_REQ(p.req[q]) * p.state_row;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
      if (c < nv) st8(st + c * 8, v[j]);
    }
  }
}

template <typename TY, typename TH, int VPT, int S>
int launch_rows(const Norm& p, int threads, cudaStream_t st) {
  static DeviceOnce configured;
  constexpr int kMaxSmem = 220 * 1024;
  const int smem = S * p.W * (4 + (int)sizeof(TY));
  if (!configured.done()) {
    cudaError_t e = cudaFuncSetAttribute(norm_rows_kernel<TY, TH, VPT, S>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
    if (e != cudaSuccess) return (int)e;
    configured.set();
  }
  if (smem > kMaxSmem) return LLB_ERR_UNSUPPORTED;
  const int per_sm = VPT == 2 ? max(1, min(1024 / threads, kMaxSmem / (smem + 1024))) : 1;
  const int rows = min(kMaxRows, cdiv(p.T, 148 * per_sm));
  launch_pdl(norm_rows_kernel<TY, TH, VPT, S>, dim3(cdiv(p.T, rows)), dim3(threads), (size_t)smem, st, p, rows);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

template <typename TY, typename TH, bool SHIFT>
int launch_row(const Norm& p, int threads, int vpt, cudaStream_t st) {
  if (vpt == 1)
    launch_pdl(norm_row_kernel<TY, TH, 1, SHIFT>, dim3(p.T), dim3(threads), 0, st, p);
  else if (vpt == 2)
    launch_pdl(norm_row_kernel<TY, TH, 2, SHIFT>, dim3(p.T), dim3(threads), 0, st, p);
  else
    launch_pdl(norm_row_kernel<TY, TH, 4, SHIFT>, dim3(p.T), dim3(threads), 0, st, p);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

template <typename TY, typename TH>
int launch_norm(const Norm& p, cudaStream_t st) {
  const int nv = p.W / 8;
  const int threads = nv >= 512 ? 512 : cdiv(nv, 32) * 32;
  const int vpt = cdiv(nv, threads);
  if (vpt > 4) return LLB_ERR_UNSUPPORTED;
  if (p.mu == nullptr) return launch_row<TY, TH, false>(p, threads, vpt, st);
  if (p.cu_q == nullptr) return launch_row<TY, TH, true>(p, threads, vpt, st);
  if (nv <= 1024) return launch_rows<TY, TH, 2, 2>(p, cdiv(cdiv(nv, 2), 32) * 32, st);
  return launch_rows<TY, TH, 4, 1>(p, threads, st);
}

}  // namespace

// Number formats: 0 = fp32, 1 = bf16.  y [T, W], or a table [y_rows, W] with ids [T]; x fp32 [T, W] or null; x_out fp32 [T, W]: may
// be x, unless there is a shift over rows of several tokens (cu_q given); h [T, W]; w fp32 [W], zero beyond `width`.  centred 0: no
// mean is taken off.  Shift: mu fp32 [W] or null; state fp32 rows; req [B], first_pos [B] (position of the request's first token in
// this pass), cu_q [B + 1] and batch_of [T], both null when row t is the one token of request t.
LLB_EXPORT int llb_norm_shift(const void* y, int y_dt, const int64_t* ids, int64_t y_rows, const float* x, float* x_out, void* h,
                              int h_dt, const float* w, int T, int width, int W, int centred, float eps, const float* mu,
                              float* state, int64_t state_row, const int* req, const int* cu_q, const int* first_pos,
                              const int* batch_of, cudaStream_t st) {
  if (T <= 0) return LLB_OK;
  if (W <= 0 || (W % 8) || width <= 0 || width > W || y_rows <= 0 || x_out == nullptr || h == nullptr || w == nullptr)
    return LLB_ERR_BAD_ARG;
  if (ids == nullptr && y_rows < T) return LLB_ERR_BAD_ARG;
  if (mu != nullptr && (state == nullptr || (state_row % 4) || ((uintptr_t)state & 15) || req == nullptr || first_pos == nullptr ||
                        (cu_q == nullptr) != (batch_of == nullptr) || (cu_q != nullptr && x == x_out)))
    return LLB_ERR_BAD_ARG;
  const Norm p{y,  ids,   y_rows, x,         x_out, h,    w,         T,       width, W, centred, eps,
               mu, state, state_row, req, cu_q, first_pos, batch_of};
  if (y_dt == 0) return h_dt == 0 ? launch_norm<float, float>(p, st) : launch_norm<float, bf16>(p, st);
  return h_dt == 0 ? launch_norm<bf16, float>(p, st) : launch_norm<bf16, bf16>(p, st);
}
