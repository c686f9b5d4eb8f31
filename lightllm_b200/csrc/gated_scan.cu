// Elementwise gated recurrences over fp32 states, one value per channel:
//
//   S_t = (1 - z_t) S_(t-1) + z_t c_t,   o_t = S_t * silu(g_t),   z = sigmoid(zr),   c = xr + 1/2 where xr >= 0, else sigmoid(xr)
//
// (minGRU: gate and candidate read the current token alone.)  zr, xr and g are columns of one projection, its biases already added.
//
//   gated_scan      token by token: decode steps, and passes of short portions.  A thread owns two channels of one request.
//   gated_chunks    longer prompts, a chunk of tokens at a time:
//     chunk_sums    every chunk as one step S -> a S + b: a = product of (1 - z), b = the state that starts from zero; the states at
//                   the start of the pass are copied aside, since the last kernel writes the new ones
//     chunk_output  composes the steps of the request's earlier chunks, then runs through the chunk's tokens again and writes o
#include "common.cuh"

using namespace llb;

namespace {

constexpr int V = 2;    // channels per thread
constexpr int U = 8;    // tokens in flight

// V channels as loaded
template <typename T>
struct Raw {};
template <>
struct Raw<float> {
  float2 r;
  __device__ __forceinline__ void load(const float* p) { r = *reinterpret_cast<const float2*>(p); }
  __device__ __forceinline__ float operator[](int i) const { return i == 0 ? r.x : r.y; }
};
template <>
struct Raw<bf16> {
  uint32_t r;
  __device__ __forceinline__ void load(const bf16* p) { r = *reinterpret_cast<const uint32_t*>(p); }
  __device__ __forceinline__ float operator[](int i) const { return __uint_as_float(i == 0 ? r << 16 : r & 0xffff0000u); }
};
__device__ __forceinline__ void ldv(const float* p, float* f) {
  const float2 a = *reinterpret_cast<const float2*>(p);
  f[0] = a.x; f[1] = a.y;
}
__device__ __forceinline__ void stv(float* p, const float* f) { *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]); }
__device__ __forceinline__ void stv(bf16* p, const float* f) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(f[0], f[1]); }
// sigmoid(v) and sigmoid(-v) = 1 - sigmoid(v), either without cancellation.  FAST: the bf16 path, where v is rounded to 8 bits
template <bool FAST>
__device__ __forceinline__ void sigmoids(float v, float& pos, float& neg) {
  const float e = FAST ? __expf(-fabsf(v)) : expf(-fabsf(v));
  const float big = FAST ? __fdividef(1.f, 1.f + e) : 1.f / (1.f + e);
  const float small = e * big;
  pos = v >= 0.f ? big : small;
  neg = v >= 0.f ? small : big;
}
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

template <bool FAST>
__device__ __forceinline__ void step(float zr, float xr, float& keep, float& add) {
  sigmoids<FAST>(zr, add, keep);
  const float c = sigmoid<FAST>(xr);
  add *= xr >= 0.f ? xr + 0.5f : c;
}

// U tokens of N matrices with row pitch ld, from row t on; rows past `last` repeat it
template <typename TI, int N>
struct Batch {
  Raw<TI> v[N][U];
  __device__ __forceinline__ void load(const TI* const* m, int64_t ld, int t, int last) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int64_t at = (int64_t)min(t + u, last) * ld;
#pragma unroll
      for (int k = 0; k < N; ++k) v[k][u].load(m[k] + at);
    }
  }
};

// Runs through tokens t0 .. t1 - 1 (at least one) of a thread's channels from state s, writing the output; the loads of the next
// batch are under way meanwhile.
template <typename TI, typename TO>
__device__ __forceinline__ void run(const Scan& p, int t0, int t1, int c, float* s) {
  constexpr bool FAST = sizeof(TO) == 2;
  const TI* const m[3] = {(const TI*)p.z + c, (const TI*)p.x + c, (const TI*)p.g + c};
  TO* out = (TO*)p.out + c;
  Batch<TI, 3> cur;
  cur.load(m, p.ld, t0, t1 - 1);
  for (int tb = t0; tb < t1; tb += U) {
    Batch<TI, 3> next = cur;
    if (tb + U < t1) next.load(m, p.ld, tb + U, t1 - 1);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u >= t1) break;
      float o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float keep, add;
        step<FAST>(cur.v[0][u][i], cur.v[1][u][i], keep, add);
        s[i] = fmaf(keep, s[i], add);
        const float g = cur.v[2][u][i];
        o[i] = s[i] * g * sigmoid<FAST>(g);
      }
      stv(out + (int64_t)(tb + u) * p.out_ld, o);
    }
    cur = next;
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
  if (p.first_pos[b] != 0) ldv(st, s);
  run<TI, TO>(p, t0, t1, c, s);
  stv(st, s);
}

template <typename TI, bool FAST>
__global__ void __launch_bounds__(128) chunk_sums_kernel(const Scan p, const Steps q) {
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, ch = blockIdx.y;
  if (c >= p.n) return;
  const int b = q.chunk_req[ch];
  if (q.cu_chunk[b] == ch) {
    float s[V] = {};
    if (p.first_pos[b] != 0) ldv(p.state + (int64_t)p.req[b] * p.state_row + c, s);
    stv(q.start + (int64_t)b * p.n + c, s);
  }
  if (q.cu_chunk[b + 1] - 1 == ch) return;  // nobody composes the last chunk
  const int t0 = q.tok0[ch], t1 = t0 + q.len[ch];
  const TI* const m[2] = {(const TI*)p.z + c, (const TI*)p.x + c};
  float a[V], s[V];
#pragma unroll
  for (int i = 0; i < V; ++i) a[i] = 1.f, s[i] = 0.f;
  Batch<TI, 2> cur;
  cur.load(m, p.ld, t0, t1 - 1);
  for (int tb = t0; tb < t1; tb += U) {
    Batch<TI, 2> next = cur;
    if (tb + U < t1) next.load(m, p.ld, tb + U, t1 - 1);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u >= t1) break;
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float keep, add;
        step<FAST>(cur.v[0][u][i], cur.v[1][u][i], keep, add);
        a[i] *= keep;
        s[i] = fmaf(keep, s[i], add);
      }
    }
    cur = next;
  }
  stv(q.a + (int64_t)ch * p.n + c, a);
  stv(q.b + (int64_t)ch * p.n + c, s);
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(128) chunk_output_kernel(const Scan p, const Steps q) {
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, ch = blockIdx.y;
  if (c >= p.n) return;
  const int b = q.chunk_req[ch], c0 = q.cu_chunk[b];
  float s[V];
  ldv(q.start + (int64_t)b * p.n + c, s);
  for (int k = c0; k < ch; k += U) {
    float a[U][V], e[U][V];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (k + u < ch) {
        ldv(q.a + (int64_t)(k + u) * p.n + c, a[u]);
        ldv(q.b + (int64_t)(k + u) * p.n + c, e[u]);
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
  if (q.cu_chunk[b + 1] - 1 == ch) stv(p.state + (int64_t)p.req[b] * p.state_row + c, s);
}

bool ok(const Scan& p, int in_dt, int out_dt) {
  const uintptr_t in_mask = in_dt == 0 ? 7 : 3, out_mask = out_dt == 0 ? 7 : 3;
  return p.n > 0 && (p.n % V) == 0 && (p.ld % V) == 0 && (p.out_ld % V) == 0 && (p.state_row % V) == 0 &&
         (((uintptr_t)p.z | (uintptr_t)p.x | (uintptr_t)p.g) & in_mask) == 0 && ((uintptr_t)p.out & out_mask) == 0 &&
         ((uintptr_t)p.state & 7) == 0;
}

}  // namespace

// Number formats (in_dt of z, x, g; out_dt of out): 0 = fp32, 1 = bf16.  cu_q null: one token per request (row b).  first_pos[b]:
// position of the request's first token in this pass; 0 starts from a zero state.  n: channels, an even number.
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
