// Elementwise gated recurrences over fp32 states, one value per channel:
//
//   S_t = (1 - z_t) S_(t-1) + z_t c_t,   o_t = S_t * silu(g_t),   z = sigmoid(zr),   c = xr + 1/2 where xr >= 0, else sigmoid(xr)
//
// (minGRU: gate and candidate read the current token alone.)  zr, xr and g are columns of one projection, its biases already added.
//
//   gated_scan      token by token: decode steps, and passes of short portions.  A thread owns four channels of one request.
//   gated_chunks    longer prompts, a chunk of tokens at a time:
//     chunk_sums    every chunk as one step S -> a S + b: a = product of (1 - z), b = the state that starts from zero; the states at
//                   the start of the pass are copied aside, since the last kernel writes the new ones
//     chunk_output  composes the steps of the request's earlier chunks, then runs through the chunk's tokens again and writes o
#include "common.cuh"

using namespace llb;

namespace {

constexpr int V = 4;    // channels per thread
constexpr int U = 8;    // tokens in flight

__device__ __forceinline__ void ld4(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
__device__ __forceinline__ void ld4(const bf16* p, float* f) {
  const uint2 a = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(a.x << 16); f[1] = __uint_as_float(a.x & 0xffff0000u);
  f[2] = __uint_as_float(a.y << 16); f[3] = __uint_as_float(a.y & 0xffff0000u);
}
__device__ __forceinline__ void st4(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void st4(bf16* p, const float* f) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
}
// FAST: the bf16 path, where the inputs are rounded to 8 bits
template <bool FAST>
__device__ __forceinline__ float sigmoid(float v) {
  return FAST ? __fdividef(1.f, 1.f + __expf(-v)) : 1.f / (1.f + expf(-v));
}

struct Scan {
  const void *z, *x, *g;  // row pitch ld
  void* out;              // row pitch out_ld
  float* state;           // [slots, n], row pitch state_row
  int64_t ld, out_ld, state_row;
  const int *req, *cu_q, *first_pos;
  int n;
};
struct Steps {
  const int *tok0, *len, *cu_chunk, *chunk_req;  // chunk c: len[c] tokens from row tok0[c] on, of request chunk_req[c]
  float *a, *b, *start;                          // [chunks, n], [chunks, n], [requests, n]
};

// keep = 1 - z, formed as sigmoid(-z): no cancellation where the state hardly decays
template <bool FAST>
__device__ __forceinline__ void step(float zr, float xr, float& keep, float& add) {
  keep = sigmoid<FAST>(-zr);
  add = sigmoid<FAST>(zr) * (xr >= 0.f ? xr + 0.5f : sigmoid<FAST>(xr));
}

// Runs through tokens t0 .. t1 - 1 of four channels from state s, writing the output.
template <typename TI, typename TO>
__device__ __forceinline__ void run(const Scan& p, int t0, int t1, int c, float* s) {
  constexpr bool FAST = sizeof(TO) == 2;
  const TI *z = (const TI*)p.z + c, *x = (const TI*)p.x + c, *g = (const TI*)p.g + c;
  TO* out = (TO*)p.out + c;
  for (int tb = t0; tb < t1; tb += U) {
    float zv[U][V], xv[U][V], gv[U][V];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u < t1) {
        const int64_t at = (int64_t)(tb + u) * p.ld;
        ld4(z + at, zv[u]);
        ld4(x + at, xv[u]);
        ld4(g + at, gv[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u < t1) {
        float o[V];
#pragma unroll
        for (int i = 0; i < V; ++i) {
          float keep, add;
          step<FAST>(zv[u][i], xv[u][i], keep, add);
          s[i] = fmaf(keep, s[i], add);
          o[i] = s[i] * gv[u][i] * sigmoid<FAST>(gv[u][i]);
        }
        st4(out + (int64_t)(tb + u) * p.out_ld, o);
      }
    }
  }
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(128) gated_scan_kernel(const Scan p) {
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.y;
  if (c >= p.n) return;
  const int t0 = p.cu_q != nullptr ? p.cu_q[b] : b, t1 = p.cu_q != nullptr ? p.cu_q[b + 1] : b + 1;
  if (t0 >= t1) return;
  float* st = p.state + (int64_t)p.req[b] * p.state_row + c;
  float s[V] = {};
  if (p.first_pos[b] != 0) ld4(st, s);
  run<TI, TO>(p, t0, t1, c, s);
  st4(st, s);
}

template <typename TI, bool FAST>
__global__ void __launch_bounds__(128) chunk_sums_kernel(const Scan p, const Steps q) {
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, ch = blockIdx.y;
  if (c >= p.n) return;
  const int b = q.chunk_req[ch];
  if (q.cu_chunk[b] == ch) {
    float s[V] = {};
    if (p.first_pos[b] != 0) ld4(p.state + (int64_t)p.req[b] * p.state_row + c, s);
    st4(q.start + (int64_t)b * p.n + c, s);
  }
  if (q.cu_chunk[b + 1] - 1 == ch) return;  // nobody composes the last chunk
  const int t0 = q.tok0[ch], t1 = t0 + q.len[ch];
  const TI *z = (const TI*)p.z + c, *x = (const TI*)p.x + c;
  float a[V], s[V];
#pragma unroll
  for (int i = 0; i < V; ++i) a[i] = 1.f, s[i] = 0.f;
  for (int tb = t0; tb < t1; tb += U) {
    float zv[U][V], xv[U][V];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u < t1) {
        ld4(z + (int64_t)(tb + u) * p.ld, zv[u]);
        ld4(x + (int64_t)(tb + u) * p.ld, xv[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u < t1) {
#pragma unroll
        for (int i = 0; i < V; ++i) {
          float keep, add;
          step<FAST>(zv[u][i], xv[u][i], keep, add);
          a[i] *= keep;
          s[i] = fmaf(keep, s[i], add);
        }
      }
    }
  }
  st4(q.a + (int64_t)ch * p.n + c, a);
  st4(q.b + (int64_t)ch * p.n + c, s);
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(128) chunk_output_kernel(const Scan p, const Steps q) {
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, ch = blockIdx.y;
  if (c >= p.n) return;
  const int b = q.chunk_req[ch], c0 = q.cu_chunk[b];
  float s[V];
  ld4(q.start + (int64_t)b * p.n + c, s);
  for (int k = c0; k < ch; k += U) {
    float a[U][V], e[U][V];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (k + u < ch) {
        ld4(q.a + (int64_t)(k + u) * p.n + c, a[u]);
        ld4(q.b + (int64_t)(k + u) * p.n + c, e[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (k + u < ch) {
#pragma unroll
        for (int i = 0; i < V; ++i) s[i] = fmaf(a[u][i], s[i], e[u][i]);
      }
    }
  }
  run<TI, TO>(p, q.tok0[ch], q.tok0[ch] + q.len[ch], c, s);
  if (q.cu_chunk[b + 1] - 1 == ch) st4(p.state + (int64_t)p.req[b] * p.state_row + c, s);
}

bool ok(const Scan& p, int in_dt, int out_dt) {
  const uintptr_t in_mask = in_dt == 0 ? 15 : 7, out_mask = out_dt == 0 ? 15 : 7;
  return p.n > 0 && (p.n % V) == 0 && (p.ld % V) == 0 && (p.out_ld % V) == 0 && (p.state_row % V) == 0 &&
         (((uintptr_t)p.z | (uintptr_t)p.x | (uintptr_t)p.g) & in_mask) == 0 && ((uintptr_t)p.out & out_mask) == 0 &&
         ((uintptr_t)p.state & 15) == 0;
}

}  // namespace

// Number formats (in_dt of z, x, g; out_dt of out): 0 = fp32, 1 = bf16.  cu_q null: one token per request (row b).  first_pos[b]:
// position of the request's first token in this pass; 0 starts from a zero state.  n: channels, a multiple of 4.
LLB_EXPORT int llb_gated_scan(const void* z, const void* x, const void* g, int in_dt, int64_t ld, void* out, int out_dt,
                              int64_t out_ld, float* state, int64_t state_row, const int* req, const int* cu_q,
                              const int* first_pos, int B, int n, cudaStream_t st) {
  if (B <= 0) return LLB_OK;
  const Scan p{z, x, g, out, state, ld, out_ld, state_row, req, cu_q, first_pos, n};
  if (!ok(p, in_dt, out_dt) || B > 65535) return LLB_ERR_BAD_ARG;
  const dim3 grid(cdiv(n, 128 * V), B);
  if (in_dt == 1 && out_dt == 1)
    launch_pdl(gated_scan_kernel<bf16, bf16>, grid, dim3(128), 0, st, p);
  else if (in_dt == 0 && out_dt == 1)
    launch_pdl(gated_scan_kernel<float, bf16>, grid, dim3(128), 0, st, p);
  else if (in_dt == 0 && out_dt == 0)
    launch_pdl(gated_scan_kernel<float, float>, grid, dim3(128), 0, st, p);
  else
    return LLB_ERR_UNSUPPORTED;
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}

// tok0, len, chunk_req [n_chunks], cu_chunk [B + 1]; a, b: fp32 scratch [n_chunks, n], start: fp32 scratch [B, n].
LLB_EXPORT int llb_gated_chunks(const void* z, const void* x, const void* g, int in_dt, int64_t ld, void* out, int out_dt,
                                int64_t out_ld, float* state, int64_t state_row, const int* req, const int* first_pos,
                                const int* tok0, const int* len, const int* cu_chunk, const int* chunk_req, float* a, float* b,
                                float* start, int n_chunks, int n, cudaStream_t st) {
  if (n_chunks <= 0) return LLB_OK;
  const Scan p{z, x, g, out, state, ld, out_ld, state_row, req, nullptr, first_pos, n};
  const Steps q{tok0, len, cu_chunk, chunk_req, a, b, start};
  if (!ok(p, in_dt, out_dt) || n_chunks > 65535) return LLB_ERR_BAD_ARG;
  const dim3 grid(cdiv(n, 128 * V), n_chunks);
#define LLB_CHUNKS(TI, TO)                                                                          \
  launch_pdl(chunk_sums_kernel<TI, sizeof(TO) == 2>, grid, dim3(128), 0, st, p, q);                  \
  LLB_LAUNCH_CHECK();                                                                               \
  launch_pdl(chunk_output_kernel<TI, TO>, grid, dim3(128), 0, st, p, q)
  if (in_dt == 1 && out_dt == 1) {
    LLB_CHUNKS(bf16, bf16);
  } else if (in_dt == 0 && out_dt == 1) {
    LLB_CHUNKS(float, bf16);
  } else if (in_dt == 0 && out_dt == 0) {
    LLB_CHUNKS(float, float);
  } else {
    return LLB_ERR_UNSUPPORTED;
  }
#undef LLB_CHUNKS
  LLB_LAUNCH_CHECK();
  return LLB_OK;
}
