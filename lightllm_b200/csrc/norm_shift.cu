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
// A CTA keeps ROWS rows in registers, and with a shift the row before them (formed again: x' is therefore written to another
// buffer than x in prompt passes).  The CTA of a request's first row in the pass reads the request's state and, after that, leaves
// there the n of the request's last row, which it forms once more unless it is the same row: so nobody else touches the state row.
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

// Sums of N values over the CTA, the same order for every N.  red: N * 16 floats nobody else uses until the next __syncthreads
// after this call.
template <int N>
__device__ __forceinline__ void block_sums(float* v, float* red) {
  const int lane = threadIdx.x & 31, wp = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) red[i * 16 + wp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) {
    float s = 0.f;
    for (int k = 0; k < nw; ++k) s += red[i * 16 + k];
    v[i] = s;
  }
}

// v[r] = n of row t[r] (t < 0: skipped, zero); x' of the rows from `store_from` on is written out.
template <typename TY, int VPT, int N>
__device__ __forceinline__ void norm_rows(const Norm& p, const int* t, int store_from, float (*v)[VPT][8], float* red) {
  const int nv = p.W >> 3;
  float s[N];
#pragma unroll
  for (int r = 0; r < N; ++r) {
    s[r] = 0.f;
    const bool live = t[r] >= 0;
    const int64_t id = live && p.ids != nullptr ? p.ids[t[r]] : t[r];
    const int64_t yr = id >= 0 && id < p.y_rows ? id : 0;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
#pragma unroll
      for (int i = 0; i < 8; ++i) v[r][j][i] = 0.f;
      if (!live || c >= nv) continue;
      ld8((const TY*)p.y + yr * p.W + c * 8, v[r][j]);
      if (p.x != nullptr) {
        float a[8];
        ld8(p.x + (int64_t)t[r] * p.W + c * 8, a);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[r][j][i] += a[i];
      }
    }
  }
#pragma unroll
  for (int r = 0; r < N; ++r) {
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
      if (r >= store_from && t[r] >= 0 && c < nv) st8(p.x_out + (int64_t)t[r] * p.W + c * 8, v[r][j]);
#pragma unroll
      for (int i = 0; i < 8; ++i) s[r] += v[r][j][i];
    }
  }
  float mean[N];
  if (p.centred) {
    block_sums<N>(s, red);
#pragma unroll
    for (int r = 0; r < N; ++r) mean[r] = s[r] / (float)p.width;
  } else {
#pragma unroll
    for (int r = 0; r < N; ++r) mean[r] = 0.f;
  }
#pragma unroll
  for (int r = 0; r < N; ++r) {
    s[r] = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = (threadIdx.x + j * blockDim.x) * 8;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (c + i < p.width) v[r][j][i] -= mean[r];
        s[r] = fmaf(v[r][j][i], v[r][j][i], s[r]);
      }
    }
  }
  block_sums<N>(s, red + N * 16);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int c = threadIdx.x + j * blockDim.x;
    if (c >= nv) continue;
    float wv[8];
    ld8(p.w + c * 8, wv);
#pragma unroll
    for (int r = 0; r < N; ++r) {
      const float inv = rsqrtf(s[r] / (float)p.width + p.eps);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[r][j][i] *= inv * wv[i];
    }
  }
}

template <typename TY, typename TH, int VPT, int ROWS, bool SHIFT>
__global__ void __launch_bounds__(512) norm_shift_kernel(const Norm p) {
  pdl_wait();
  constexpr int N = ROWS + (SHIFT ? 1 : 0), F = SHIFT ? 1 : 0;  // F: index of the CTA's first own row
  __shared__ float red[2 * N * 16], red1[2 * 16];
  const int nv = p.W >> 3, t0 = blockIdx.x * ROWS;
  int t[N];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) t[F + r] = t0 + r < p.T ? t0 + r : -1;
  // request of the CTA's rows (-1 ahead of the first and behind the last row)
  int b[N];
  if (SHIFT) {
    auto request = [&](int i) { return i < 0 || i >= p.T ? -1 : (p.batch_of != nullptr ? p.batch_of[i] : i); };
#pragma unroll
    for (int r = 0; r < N; ++r) b[r] = request(t0 + r - 1);
    t[0] = b[0] >= 0 && b[0] == b[1] ? t0 - 1 : -1;
  }
  float v[N][VPT][8];
  norm_rows<TY, VPT, N>(p, t, F, v, red);
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    if (t[F + r] < 0) continue;
    const int row = t[F + r];
    float* st = nullptr;  // the request's state row, when this is its first row in the pass
    bool fresh = false, last_too = false;
    if (SHIFT && b[r] != b[r + 1]) {
      const int q = b[r + 1];
      st = p.state + (int64_t)LLB_CHECK_REQ(p.req[q]) * p.state_row;
      fresh = p.first_pos[q] == 0;
      last_too = p.cu_q == nullptr || p.cu_q[q + 1] - 1 == row;
    }
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
      if (c >= nv) continue;
      if (!SHIFT) {
        st8((TH*)p.h + (int64_t)row * p.W + c * 8, v[r][j]);
        continue;
      }
      float before[8], m[8], o[8];
      if (st == nullptr) {
#pragma unroll
        for (int i = 0; i < 8; ++i) before[i] = v[r][j][i];
      } else if (fresh) {
#pragma unroll
        for (int i = 0; i < 8; ++i) before[i] = 0.f;
      } else {
        ld8(st + c * 8, before);
      }
      ld8(p.mu + c * 8, m);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float n = v[F + r][j][i];
        o[i] = fmaf(before[i] - n, m[i], n);
      }
      st8((TH*)p.h + (int64_t)row * p.W + c * 8, o);
      if (st != nullptr && last_too) st8(st + c * 8, v[F + r][j]);
    }
  }
  if (!SHIFT || p.cu_q == nullptr) return;
  // requests that start here and end on a later row: their last row once more, for the state
  for (int r = 0; r < ROWS; ++r) {
    const int row = t0 + r;
    if (row >= p.T) break;
    const int q = p.batch_of[row];
    const int last = p.cu_q[q + 1] - 1;
    if (p.cu_q[q] != row || last == row) continue;
    float e[1][VPT][8];
    __syncthreads();
    norm_rows<TY, VPT, 1>(p, &last, 1, e, red1);
    float* st = p.state + (int64_t)LLB_CHECK_REQ(p.req[q]) * p.state_row;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      const int c = threadIdx.x + j * blockDim.x;
      if (c < nv) st8(st + c * 8, e[0][j]);
    }
  }
}

template <typename TY, typename TH, bool SHIFT>
int launch_norm(const Norm& p, cudaStream_t st) {
  const int nv = p.W / 8;
  const int threads = nv >= 512 ? 512 : cdiv(nv, 32) * 32;
  const int vpt = cdiv(nv, threads);
  // a shift forms the row before a CTA's rows again: several rows per CTA once there are enough of them
  const bool many = SHIFT && p.cu_q != nullptr && p.T >= 1024;
#define LLB_NORM(V, R) \
  launch_pdl(norm_shift_kernel<TY, TH, V, R, SHIFT>, dim3(cdiv(p.T, R)), dim3(threads), 0, st, p)
  if (vpt == 1) {
    if (SHIFT && many)
      LLB_NORM(1, (SHIFT ? 4 : 1));
    else
      LLB_NORM(1, 1);
  } else if (vpt == 2) {
    if (SHIFT && many)
      LLB_NORM(2, (SHIFT ? 2 : 1));
    else
      LLB_NORM(2, 1);
  } else if (vpt <= 4) {
    LLB_NORM(4, 1);
  } else {
    return LLB_ERR_UNSUPPORTED;
  }
#undef LLB_NORM
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

template <typename TY, typename TH>
int launch_norm(const Norm& p, cudaStream_t st) {
  return p.mu != nullptr ? launch_norm<TY, TH, true>(p, st) : launch_norm<TY, TH, false>(p, st);
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
