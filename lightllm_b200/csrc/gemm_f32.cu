// fp32 GEMM on the CUDA cores:  C[M, N] = A[M, K] . W[N, K]^T  with the epilogues of the bf16 tensor-core GEMM, for
// models that run in 32-bit (the tensor cores have no fp32 input format; TF32 keeps 10 bits of the mantissa).
//
// 64 x 64 output tile per CTA, 256 threads, 4 x 4 results per thread, K in steps of 16 through shared memory.  The sum
// over a K step is formed apart and added to the running total, so that the error grows with K / 16.
// Batched (per-head) and grouped (expert-sorted rows) forms as in the bf16 GEMM.
#include "common.cuh"

using namespace llb;

namespace {

enum Epi { F_STORE = 0, F_RESIDUAL = 1, F_GATED_SILU = 2, F_F32 = 3, F_GATED_GELU = 4, F_RELU2 = 5, F_DYT = 6, F_GATED_CLAMP = 7 };
__host__ __device__ constexpr bool gated_epi(int e) { return e == F_GATED_SILU || e == F_GATED_GELU || e == F_GATED_CLAMP; }

struct DytPair {
  float* x;  // residual stream, same pitch as C
  const float *w1, *b1, *w2, *b2;
  float alpha1, alpha2;
};

struct F32Params {
  const float* A;
  const float* W;
  float* C;
  const float* residual;
  const float* bias;
  const int* mblock_expert;  // grouped: expert of every 128-row block (-1: skip)
  int64_t lda, ldw, ldc, a_batch, w_batch, c_batch;
  int M, N, K;
  float alpha;
  DytPair d;
  float act_alpha, act_limit;  // F_GATED_CLAMP
  float softcap;               // F_F32: > 0 stores softcap * tanh(value / softcap)
};

constexpr int TM = 64, TN = 64, TK = 16;

__device__ __forceinline__ float act_silu(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float act_gelu_tanh(float v) {
  return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
}

template <int EPI>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const F32Params p) {
  __shared__ float As[TK][TM + 4], Ws[TK][TN + 4];
  constexpr bool GATED = gated_epi(EPI);
  __shared__ float gate_tile[GATED ? TM : 1][GATED ? TN + 1 : 1];
  const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
  const float* A = p.A + blockIdx.z * p.a_batch;
  const float* W = p.W + blockIdx.z * p.w_batch;
  if (p.mblock_expert != nullptr) {
    const int e = p.mblock_expert[m0 >> 7];
    if (e < 0) return;
    W += (int64_t)e * p.N * p.ldw;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (threadIdx.x >> 4) + 16 * i, k = threadIdx.x & 15;
      As[k][r] = (m0 + r < p.M && k0 + k < p.K) ? A[(int64_t)(m0 + r) * p.lda + k0 + k] : 0.f;
      Ws[k][r] = (n0 + r < p.N && k0 + k < p.K) ? W[(int64_t)(n0 + r) * p.ldw + k0 + k] : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) w[j] = Ws[k][tx + 16 * j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(a[i], w[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
  float* C = p.C + blockIdx.z * p.c_batch;
  if constexpr (GATED) {  // columns n0 .. n0 + 31 are gate rows, n0 + 32 .. n0 + 63 up rows
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) gate_tile[ty * 4 + i][tx + 16 * j] = acc[i][j];
    __syncthreads();
    for (int i = threadIdx.x; i < TM * 32; i += 256) {
      const int r = i >> 5, c = i & 31;
      if (m0 + r < p.M && n0 + c < p.N) {
        float g = gate_tile[r][c], u = gate_tile[r][c + 32], v;
        if (EPI == F_GATED_CLAMP) {
          g = fminf(g, p.act_limit);
          u = fminf(fmaxf(u, -p.act_limit), p.act_limit);
          v = g / (1.f + expf(-p.act_alpha * g)) * (u + 1.f);
        } else {
          v = (EPI == F_GATED_SILU ? act_silu(g) : act_gelu_tanh(g)) * u;
        }
        C[(int64_t)(m0 + r) * p.ldc + n0 / 2 + c] = v;
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int row = m0 + ty * 4 + i;
      if (row >= p.M) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = n0 + tx + 16 * j;
        if (col >= p.N) continue;
        const int64_t off = (int64_t)row * p.ldc + col;
        float v = acc[i][j];
        if (p.bias) v += p.bias[col];
        if (EPI == F_RESIDUAL) v += p.residual[off];
        if (EPI == F_RELU2) {
          v = fmaxf(v, 0.f);
          v *= v;
        }
        if (EPI == F_F32) {
          v *= p.alpha;
          if (p.softcap > 0.f) v = p.softcap * tanhf(v / p.softcap);
        }
        if (EPI == F_DYT) {
          const float x = p.d.x[off] + tanhf(p.d.alpha1 * v) * p.d.w1[col] + p.d.b1[col];
          p.d.x[off] = x;
          v = tanhf(p.d.alpha2 * x) * p.d.w2[col] + p.d.b2[col];
        }
        C[off] = v;
      }
    }
  }
}

template <int EPI>
int launch(const F32Params& p, int batch, cudaStream_t st) {
  const dim3 grid(cdiv(p.N, TN), cdiv(p.M, TM), batch);
  gemm_f32_kernel<EPI><<<grid, 256, 0, st>>>(p);
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

}  // namespace

// `batch` matrices: element strides a_batch / w_batch / c_batch.  mblock_expert: grouped form (batch 1), W stacks the
// experts' [N, K] matrices.  x, w1 .. alpha2: the dynamic-tanh epilogue (x += dyt1(acc); C = dyt2(x)).
LLB_EXPORT int llb_gemm_f32(const float* A, int64_t lda, int64_t a_batch, const float* W, int64_t ldw, int64_t w_batch,
                            float* C, int64_t ldc, int64_t c_batch, const float* residual, const float* bias, float* x,
                            const float* w1, const float* b1, float alpha1, const float* w2, const float* b2,
                            float alpha2, const int* mblock_expert, int M, int N, int K, int batch, int epi,
                            float alpha, float act_alpha, float act_limit, float softcap, cudaStream_t st) {
  if (M <= 0 || N <= 0 || batch <= 0) return LLB_OK;
  if (K <= 0 || cdiv(M, TM) > 65535 || batch > 65535) return LLB_ERR_UNSUPPORTED;
  if (gated_epi(epi) && (N % 64)) return LLB_ERR_UNSUPPORTED;
  if (mblock_expert != nullptr && (batch != 1 || (M % 128))) return LLB_ERR_BAD_ARG;
  if (epi == F_RESIDUAL && residual == nullptr) return LLB_ERR_BAD_ARG;
  if (epi == F_DYT && (x == nullptr || w1 == nullptr || b1 == nullptr || w2 == nullptr || b2 == nullptr || batch != 1))
    return LLB_ERR_BAD_ARG;
  F32Params p;
  p.A = A;
  p.W = W;
  p.C = C;
  p.residual = residual;
  p.bias = bias;
  p.mblock_expert = mblock_expert;
  p.lda = lda;
  p.ldw = ldw;
  p.ldc = ldc;
  p.a_batch = a_batch;
  p.w_batch = w_batch;
  p.c_batch = c_batch;
  p.M = M;
  p.N = N;
  p.K = K;
  p.alpha = alpha;
  p.act_alpha = act_alpha;
  p.act_limit = act_limit;
  p.softcap = softcap;
  p.d = DytPair{x, w1, b1, w2, b2, alpha1, alpha2};
  switch (epi) {
    case F_STORE: return launch<F_STORE>(p, batch, st);
    case F_RESIDUAL: return launch<F_RESIDUAL>(p, batch, st);
    case F_GATED_SILU: return launch<F_GATED_SILU>(p, batch, st);
    case F_F32: return launch<F_F32>(p, batch, st);
    case F_GATED_GELU: return launch<F_GATED_GELU>(p, batch, st);
    case F_RELU2: return launch<F_RELU2>(p, batch, st);
    case F_DYT: return launch<F_DYT>(p, batch, st);
    case F_GATED_CLAMP: return launch<F_GATED_CLAMP>(p, batch, st);
  }
  return LLB_ERR_UNSUPPORTED;
}
