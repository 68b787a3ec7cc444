// What happens to the 32-bit residual stream between two products, a row per block, in one pass over the row:
//
//   x[t, :] += u[t, :]      with u the result of a sublayer after
//     gate:  y * s * sigmoid(r)     a constant s per channel and a gate r per channel (columns of the product that
//                                   read the sublayer's input)
//     rms:   y / rms(y) * s         an RMS norm with a weight s (eps under the root)
//   or x[t, :] = v / rms(v) * s with v = a x[t, :] + y, a constant a (the norm of the whole sum)
//   and, from the updated row, optionally what the next sublayer reads:
//     copy:       x in the compute dtype
//     layer norm: (x - mean) / sqrt(mean((x - mean)^2) + eps2) * w2 (+ b2)
//     rms norm:   x / sqrt(mean(x^2) + eps2) * w2
//
// y is a float32 row, or (``picked``) the weighted sum of the rows of a token's chosen experts, added up in the
// order of their choice, or both together, the row behind a gate of one number (sigmoid of ``mix``).  Statistics, gates and sums are 32-bit.
//
// Beside it: a table's row per token that joins the stream behind a gate made from the stream itself
// (token_gate_kernel, token_gate_mul_kernel), and the soft cap of the logits.
#include <math.h>

#include "common.cuh"

namespace {

enum { FROM_GATE = 0, FROM_RMS = 1, FROM_SUM = 2 };
enum { POST_NONE = 0, POST_COPY = 1, POST_LAYER = 2, POST_RMS = 3 };

struct StreamArgs {
  float* x;                  // [T, d], updated in place
  void* out;                 // [T, d] of the compute dtype, or null
  const float* y;            // [T, d]; may be null with picked
  const float* picked;       // rows of d
  const int* row_of_pair;    // null: pair p lies at row p
  const float* pair_weight;  // [T, top]; null: 1
  const float* mix;          // y times sigmoid(mix[t * mix_stride]); null: y as it is
  const float* gate;         // rows of gate_stride
  const float* s;            // [d]
  const float* w2;           // [d]
  const float* b2;           // [d] or null
  long long gate_stride, mix_stride;
  int d, top, post;
  float factor;              // of x in a normed sum
  float eps, eps2;
};

__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }

// Sum over a block of whole warps, the same order in every thread; ``red`` holds 32 floats per use.
__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) total += red[w];
  return total;
}

__device__ __forceinline__ void store4(float* dst, const float (&v)[4]) { *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* dst, const float (&v)[4]) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 packed;
  packed.x = *reinterpret_cast<uint32_t*>(&lo);
  packed.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}
__device__ __forceinline__ void load4(const float* src, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(src);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}

// Rows in registers: NV pieces of four columns to a thread (piece p at column (p * blockDim.x + threadIdx.x) * 4).
template <typename O, int FROM, int NV>
__global__ void __launch_bounds__(256)
stream_update_vec_kernel(StreamArgs a) {
  __shared__ float red[4][32];
  pdl_trigger();
  const int t = blockIdx.x, d = a.d;
  const size_t at = (size_t)t * d;
  float s[NV][4], w2[NV][4];
#pragma unroll
  for (int p = 0; p < NV; ++p) {             // weights do not depend on the kernels before this one
    const int c = (p * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) { s[p][i] = 0.f; w2[p][i] = 0.f; }
    if (c < d) {
      load4(a.s + c, s[p]);
      if (a.post >= POST_LAYER) load4(a.w2 + c, w2[p]);
    }
  }
  pdl_wait();
  float v[NV][4], u[NV][4];
  const float share = a.mix ? sigmoidf(a.mix[(size_t)t * a.mix_stride]) : 1.f;
#pragma unroll
  for (int p = 0; p < NV; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) { v[p][i] = 0.f; u[p][i] = 0.f; }
    if (c >= d) continue;
    load4(a.x + at + c, v[p]);
    if (a.picked) {
      for (int k = 0; k < a.top; ++k) {
        const size_t pair = (size_t)t * a.top + k;
        const float w = a.pair_weight ? a.pair_weight[pair] : 1.f;
        float y[4];
        load4(a.picked + (size_t)(a.row_of_pair ? a.row_of_pair[pair] : pair) * d + c, y);
#pragma unroll
        for (int i = 0; i < 4; ++i) u[p][i] = fmaf(w, y[i], u[p][i]);
      }
    }
    if (a.y) {
      float y[4];
      load4(a.y + at + c, y);
#pragma unroll
      for (int i = 0; i < 4; ++i) u[p][i] = fmaf(share, y[i], u[p][i]);
    }
    if (FROM == FROM_GATE) {
      float r[4];
      load4(a.gate + (size_t)t * a.gate_stride + c, r);
#pragma unroll
      for (int i = 0; i < 4; ++i) v[p][i] = fmaf(u[p][i] * s[p][i], sigmoidf(r[i]), v[p][i]);
    }
  }
  if (FROM == FROM_RMS) {
    float q = 0.f;
#pragma unroll
    for (int p = 0; p < NV; ++p)
#pragma unroll
      for (int i = 0; i < 4; ++i) q = fmaf(u[p][i], u[p][i], q);
    const float inv = 1.0f / sqrtf(block_total(q, red[0]) / (float)d + a.eps);
#pragma unroll
    for (int p = 0; p < NV; ++p)
#pragma unroll
      for (int i = 0; i < 4; ++i) v[p][i] = fmaf(u[p][i] * inv, s[p][i], v[p][i]);
  }
  if (FROM == FROM_SUM) {
    float q = 0.f;
#pragma unroll
    for (int p = 0; p < NV; ++p)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[p][i] = fmaf(a.factor, v[p][i], u[p][i]);
        q = fmaf(v[p][i], v[p][i], q);
      }
    const float inv = 1.0f / sqrtf(block_total(q, red[0]) / (float)d + a.eps);
#pragma unroll
    for (int p = 0; p < NV; ++p)
#pragma unroll
      for (int i = 0; i < 4; ++i) v[p][i] = v[p][i] * inv * s[p][i];
  }
#pragma unroll
  for (int p = 0; p < NV; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
    if (c < d) store4(a.x + at + c, v[p]);
  }
  if (a.post == POST_NONE) return;
  O* out = reinterpret_cast<O*>(a.out) + at;
  float mean = 0.f, inv2 = 1.f;
  if (a.post == POST_LAYER) {
    float q = 0.f;
#pragma unroll
    for (int p = 0; p < NV; ++p) q += (v[p][0] + v[p][1]) + (v[p][2] + v[p][3]);      // dead pieces are zeros
    mean = block_total(q, red[1]) / (float)d;
  }
  if (a.post >= POST_LAYER) {
    float q = 0.f;
#pragma unroll
    for (int p = 0; p < NV; ++p) {
      if ((p * blockDim.x + threadIdx.x) * 4 >= d) continue;
#pragma unroll
      for (int i = 0; i < 4; ++i) { const float e = v[p][i] - mean; q = fmaf(e, e, q); }
    }
    inv2 = 1.0f / sqrtf(block_total(q, red[2]) / (float)d + a.eps2);
  }
#pragma unroll
  for (int p = 0; p < NV; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
    if (c >= d) continue;
    float o[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      o[i] = v[p][i];
      if (a.post >= POST_LAYER) o[i] = fmaf((v[p][i] - mean) * inv2, w2[p][i], a.b2 ? a.b2[c + i] : 0.f);
    }
    store4(out + c, o);
  }
}

// Any width: a thread reads back its own stores.
template <typename O, int FROM>
__global__ void __launch_bounds__(256)
stream_update_kernel(StreamArgs a) {
  __shared__ float red[4][32];
  pdl_trigger();
  const int t = blockIdx.x, d = a.d;
  const size_t at = (size_t)t * d;
  pdl_wait();
  const float share = a.mix ? sigmoidf(a.mix[(size_t)t * a.mix_stride]) : 1.f;
  auto value = [&](int c) {
    float u = 0.f;
    for (int k = 0; a.picked && k < a.top; ++k) {
      const size_t pair = (size_t)t * a.top + k;
      u = fmaf(a.pair_weight ? a.pair_weight[pair] : 1.f, a.picked[(size_t)(a.row_of_pair ? a.row_of_pair[pair] : pair) * d + c], u);
    }
    return a.y ? fmaf(share, a.y[at + c], u) : u;
  };
  float inv = 1.f;
  if (FROM == FROM_RMS) {
    float q = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) { const float u = value(c); q = fmaf(u, u, q); }
    inv = 1.0f / sqrtf(block_total(q, red[0]) / (float)d + a.eps);
  }
  if (FROM == FROM_SUM) {
    float q = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) {
      const float v = fmaf(a.factor, a.x[at + c], value(c));
      a.x[at + c] = v;
      q = fmaf(v, v, q);
    }
    inv = 1.0f / sqrtf(block_total(q, red[0]) / (float)d + a.eps);
  }
  float sum = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    if (FROM == FROM_SUM) {
      const float v = a.x[at + c] * inv * a.s[c];
      a.x[at + c] = v;
      sum += v;
      continue;
    }
    const float u = value(c);
    const float v = FROM == FROM_GATE ? fmaf(u * a.s[c], sigmoidf(a.gate[(size_t)t * a.gate_stride + c]), a.x[at + c])
                                      : fmaf(u * inv, a.s[c], a.x[at + c]);
    a.x[at + c] = v;
    sum += v;
  }
  if (a.post == POST_NONE) return;
  O* out = reinterpret_cast<O*>(a.out) + at;
  float mean = 0.f, inv2 = 1.f;
  if (a.post == POST_LAYER) mean = block_total(sum, red[1]) / (float)d;
  if (a.post >= POST_LAYER) {
    float q = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) { const float e = a.x[at + c] - mean; q = fmaf(e, e, q); }
    inv2 = 1.0f / sqrtf(block_total(q, red[2]) / (float)d + a.eps2);
  }
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float o = a.x[at + c];
    if (a.post >= POST_LAYER) o = fmaf((o - mean) * inv2, a.w2[c], a.b2 ? a.b2[c] : 0.f);
    out[c] = from_float<O>(o);
  }
}

// out[t, j] = gelu_tanh(sum_c w[j, c] x[t, c]) * table[tok[t], col0 + j]: a warp per (row, j), for a handful of rows.
template <typename W>
__global__ void __launch_bounds__(256)
token_gate_kernel(W* __restrict__ out, const float* __restrict__ x, const W* __restrict__ w, const W* __restrict__ table,
                  long long table_stride, int col0, const int* __restrict__ tok, int d, int n, int vec) {
  pdl_trigger();
  const int t = blockIdx.x, lane = threadIdx.x & 31, j = blockIdx.y * 8 + (threadIdx.x >> 5);
  pdl_wait();
  if (j >= n) return;
  const float* row = x + (size_t)t * d;
  const W* wr = w + (size_t)j * d;
  const float e = to_float<W>(table[(size_t)tok[t] * table_stride + col0 + j]);
  float s = 0.f;
  if (vec) {
#pragma unroll 8
    for (int c = lane * 4; c < d; c += 128) {
      const float4 a = *reinterpret_cast<const float4*>(row + c);
      float b[4];
      if (sizeof(W) == 2) {
        const uint2 p = *reinterpret_cast<const uint2*>(wr + c);
        b[0] = __uint_as_float(p.x << 16); b[1] = __uint_as_float(p.x & 0xffff0000u);      // a bfloat16 is the upper half of a float
        b[2] = __uint_as_float(p.y << 16); b[3] = __uint_as_float(p.y & 0xffff0000u);
      } else {
        load4(reinterpret_cast<const float*>(wr) + c, b);
      }
      s = fmaf(a.x, b[0], fmaf(a.y, b[1], fmaf(a.z, b[2], fmaf(a.w, b[3], s))));
    }
  } else {
    for (int c = lane; c < d; c += 32) s = fmaf(row[c], to_float<W>(wr[c]), s);
  }
  s = warp_sum(s);
  if (lane == 0) out[(size_t)t * n + j] = from_float<W>(apply_activation(s, AYK_ACT_GELU_TANH) * e);
}

// The same from a product already made: out[t, j] = gelu_tanh(z[t, j]) * table[tok[t], col0 + j].
template <typename W>
__global__ void __launch_bounds__(256)
token_gate_mul_kernel(W* __restrict__ out, const float* __restrict__ z, const W* __restrict__ table, long long table_stride, int col0,
                      const int* __restrict__ tok, int n, long long total) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / n), j = (int)(i - (long long)t * n);
    out[i] = from_float<W>(apply_activation(z[i], AYK_ACT_GELU_TANH) * to_float<W>(table[(size_t)tok[t] * table_stride + col0 + j]));
  }
}

__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

__global__ void __launch_bounds__(256) softcap_vec_kernel(float4* __restrict__ x, long long n4, float cap) {
  pdl_trigger();
  pdl_wait();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n4) return;
  float4 v = x[i];
  v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap);
  v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap);
  x[i] = v;
}

template <typename O, int FROM>
void launch_stream(const StreamArgs& a, int T, bool vec, cudaStream_t stream) {
  if (!vec) {
    ayk_launch(stream_update_kernel<O, FROM>, dim3(T), dim3(256), 0, stream, a);
    return;
  }
  const int pieces = a.d / 4;
  const int threads = pieces >= 256 ? 256 : (pieces + 31) / 32 * 32;
  const int nv = (pieces + threads - 1) / threads;
  if (nv <= 1) ayk_launch(stream_update_vec_kernel<O, FROM, 1>, dim3(T), dim3(threads), 0, stream, a);
  else if (nv <= 2) ayk_launch(stream_update_vec_kernel<O, FROM, 2>, dim3(T), dim3(threads), 0, stream, a);
  else ayk_launch(stream_update_vec_kernel<O, FROM, 4>, dim3(T), dim3(threads), 0, stream, a);
}

}  // namespace

// See the head of the file.  from: 0 gate, 1 rms, 2 the norm of the sum (factor x + y); post: 0 none, 1 copy, 2 layer
// norm, 3 rms norm.  picked: rows of d, top per token, pair p = t * top + k at row row_of_pair[p] (null: p) with weight
// pair_weight[p] (null: 1); y, alone or beside picked, times sigmoid(mix[t * mix_stride]) (null: 1).
AYK_EXPORT int ayk_stream_update(float* x, void* out, const float* y, const float* picked, const int* row_of_pair,
                                 const float* pair_weight, int top, const float* mix, long long mix_stride, float factor, const float* gate, long long gate_stride, const float* s,
                                 const float* w2, const float* b2, int T, int d, int from, int post, float eps, float eps2,
                                 int out_dtype, cudaStream_t stream) {
  if (T == 0 || d == 0) return 0;
  AYK_REQUIRE((y || picked) && (!picked || top >= 1) && (!mix || y), "ayk_stream_update: rows, the rows of chosen experts, or both");
  AYK_REQUIRE((from == FROM_GATE && gate) || from == FROM_RMS || from == FROM_SUM, "ayk_stream_update: unknown source %d", from);
  AYK_REQUIRE(post >= POST_NONE && post <= POST_RMS && (post == POST_NONE || out) && (post < POST_LAYER || w2),
              "ayk_stream_update: what follows (%d) needs its output and weight", post);
  AYK_REQUIRE(out_dtype == AYK_DTYPE_F32 || out_dtype == AYK_DTYPE_BF16, "ayk_stream_update: unknown dtype %d", out_dtype);
  const StreamArgs a{x, out, y, picked, row_of_pair, pair_weight, mix, gate, s, w2, b2, gate_stride, mix_stride, d, top, post, factor, eps, eps2};
  const bool vec = d % 4 == 0 && d <= 4096 && (!gate || gate_stride % 4 == 0) &&
                   (((uintptr_t)x | (uintptr_t)out | (uintptr_t)y | (uintptr_t)picked | (uintptr_t)gate | (uintptr_t)s | (uintptr_t)w2) & 15) == 0;
  if (out_dtype == AYK_DTYPE_BF16) {
    if (from == FROM_GATE) launch_stream<__nv_bfloat16, FROM_GATE>(a, T, vec, stream);
    else if (from == FROM_SUM) launch_stream<__nv_bfloat16, FROM_SUM>(a, T, vec, stream);
    else launch_stream<__nv_bfloat16, FROM_RMS>(a, T, vec, stream);
  } else {
    if (from == FROM_GATE) launch_stream<float, FROM_GATE>(a, T, vec, stream);
    else if (from == FROM_SUM) launch_stream<float, FROM_SUM>(a, T, vec, stream);
    else launch_stream<float, FROM_RMS>(a, T, vec, stream);
  }
  return ayk_check_launch("ayk_stream_update");
}

// out [T, n] (the tables' dtype) = gelu_tanh(x w^T) * table[tok, col0 ..]: from the float32 rows x [T, d] and w [n, d], or,
// with z (float32 [T, n]), from the product already made.
AYK_EXPORT int ayk_token_gate(void* out, const float* x, const void* w, const float* z, const void* table, long long table_stride,
                              int col0, const int* tok, int T, int d, int n, int dtype, cudaStream_t stream) {
  if (T == 0 || n == 0) return 0;
  AYK_REQUIRE(z || (x && w), "ayk_token_gate: rows and a matrix, or their product");
  AYK_REQUIRE(dtype == AYK_DTYPE_F32 || dtype == AYK_DTYPE_BF16, "ayk_token_gate: unknown dtype %d", dtype);
  if (z) {
    const long long total = (long long)T * n;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    if (dtype == AYK_DTYPE_F32)
      ayk_launch(token_gate_mul_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)out, z, (const float*)table, table_stride,
                 col0, tok, n, total);
    else
      ayk_launch(token_gate_mul_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)out, z,
                 (const __nv_bfloat16*)table, table_stride, col0, tok, n, total);
    return ayk_check_launch("ayk_token_gate");
  }
  const dim3 grid(T, (n + 7) / 8);
  AYK_REQUIRE(grid.y <= 65535, "ayk_token_gate: %d columns", n);
  const int vec = d % 4 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
  if (dtype == AYK_DTYPE_F32)
    ayk_launch(token_gate_kernel<float>, grid, dim3(256), 0, stream, (float*)out, x, (const float*)w, (const float*)table, table_stride,
               col0, tok, d, n, vec);
  else
    ayk_launch(token_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (__nv_bfloat16*)out, x, (const __nv_bfloat16*)w,
               (const __nv_bfloat16*)table, table_stride, col0, tok, d, n, vec);
  return ayk_check_launch("ayk_token_gate");
}

// x = cap * tanh(x / cap) over n float32 numbers, in place.
AYK_EXPORT int ayk_softcap(float* x, long long n, float cap, cudaStream_t stream) {
  if (n == 0) return 0;
  AYK_REQUIRE(cap > 0.f, "ayk_softcap: the cap must be positive");
  if (n % 4 == 0 && ((uintptr_t)x & 15) == 0 && n / 1024 < 0x7fffffff) {
    ayk_launch(softcap_vec_kernel, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, stream, (float4*)x, n / 4, cap);
    return ayk_check_launch("ayk_softcap");
  }
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  ayk_launch(softcap_kernel, dim3(blocks), dim3(256), 0, stream, x, n, cap);
  return ayk_check_launch("ayk_softcap");
}
