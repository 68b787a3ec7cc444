// From float32 projection rows to queries, cached keys and cached values: every head may be RMS-normed over its numbers
// (a weight for all query heads, one for all key heads); the first ``rot`` dimensions
// of every query and key head turn by the position (dimension i is paired with i + rot/2, or with its neighbour;
// frequencies from the caller, angles, cos and sin 32-bit, cos and sin times a gain), the rest pass; the values may be
// blended with another layer's values of the same token, v <- keep v + mix first.
//
// One block per row, or with few rows several that share the row's heads and values (grid y): the row's cos and sin in
// shared memory, a warp per head.
#include <math.h>

#include "vec.cuh"

namespace {

// VEC 4: head sizes, half of the rotated dimensions (NEIGHBOURS: all of them), row strides and the columns where keys,
// values and the other layer's values start are multiples of 4, all tensors 16-byte aligned.
template <typename C, int VEC, bool NEIGHBOURS>
__global__ void __launch_bounds__(256)
rotary_prepare_kernel(C* __restrict__ qout, C* __restrict__ kpages, C* __restrict__ vpages, const float* __restrict__ proj,
                      long long stride, const float* __restrict__ qw, const float* __restrict__ kw, float eps,
                      const float* __restrict__ freq, float gain, int rot, const float* __restrict__ first,
                      long long first_stride, float keep, float mix, const int* __restrict__ row_req,
                      const int* __restrict__ positions, const int* __restrict__ table, int table_stride, int page_size,
                      int H, int G, int D, int v_width, int writes) {
  extern __shared__ __align__(16) float turn[];          // cos [rot / 2], sin [rot / 2]
  pdl_trigger();
  const int t = blockIdx.x, half = rot / 2;
  const int p = positions[t];
  const int page = table[(size_t)row_req[t] * table_stride + p / page_size];
  float* cs = turn;
  float* sn = turn + half;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf((float)p * freq[i], &s, &c);
    cs[i] = c * gain;
    sn[i] = s * gain;
  }
  __syncthreads();
  pdl_wait();
  const float* row = proj + (size_t)t * stride;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  const bool files = writes && page > 0;
  const size_t cell = files ? (size_t)page * page_size + (p % page_size) : 0;
  for (int n = blockIdx.y * nwarp + warp; n < H + G; n += gridDim.y * nwarp) {
    const bool key = n >= H;
    if (key && !files) break;
    const float* src = row + (size_t)n * D;
    C* dst = key ? kpages + (cell * G + (n - H)) * D : qout + ((size_t)t * H + n) * D;
    const float* nw = key ? kw : qw;
    float inv = 1.f;
    if (nw) {
      float s = 0.f;
      for (int d = lane * VEC; d < D; d += 32 * VEC) {
        float v[VEC];
        load_n(src + d, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s = fmaf(v[i], v[i], s);
      }
      inv = 1.0f / sqrtf(warp_sum(s) / (float)D + eps);
    }
    auto load = [&](int d, float (&v)[VEC]) {
      load_n(src + d, v);
      if (!nw) return;
      float w[VEC];
      load_n(nw + d, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * w[i];
    };
    for (int d = lane * VEC; d < D; d += 32 * VEC) {
      float v[VEC];
      load(d, v);
      if (NEIGHBOURS && d < rot) {                         // a run of VEC numbers is whole pairs, or one number of a pair
        if (VEC == 1) {
          float o[VEC];
          load(d ^ 1, o);
          v[0] = fmaf(o[0], (d & 1) ? sn[d >> 1] : -sn[d >> 1], v[0] * cs[d >> 1]);
        } else {
#pragma unroll
          for (int i = 0; i + 1 < VEC; i += 2) {
            const float c = cs[(d + i) >> 1], s = sn[(d + i) >> 1], a = v[i], b = v[i + 1];
            v[i] = fmaf(b, -s, a * c);
            v[i + 1] = fmaf(a, s, b * c);
          }
        }
      } else if (d < rot) {                                // a run of VEC numbers lies in one half
        const bool upper = d >= half;
        float o[VEC];
        load(upper ? d - half : d + half, o);
        const int i0 = upper ? d - half : d;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float c = cs[i0 + i], s = upper ? sn[i0 + i] : -sn[i0 + i];
          v[i] = fmaf(o[i], s, v[i] * c);
        }
      }
      store_n(dst + d, v);
    }
  }
  if (!files) return;
  const float* vsrc = row + (size_t)(H + G) * D;
  const float* other = first ? first + (size_t)t * first_stride : nullptr;
  C* vdst = vpages + cell * (size_t)v_width;
  for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; i < v_width; i += gridDim.y * blockDim.x * VEC) {
    float v[VEC];
    load_n(vsrc + i, v);
    if (other) {
      float o[VEC];
      load_n(other + i, o);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = fmaf(mix, o[e], keep * v[e]);
    }
    store_n(vdst + i, v);
  }
}

}  // namespace

// proj [T, stride] float32 rows [q (H D) | k (G D) | v (v_width) | ...]; qout [T, H D]; key and value pages of G D and
// v_width numbers per token.  qw, kw [D] float32 or null: the heads' norms.  rot 0: nothing turns; neighbours: pairs
// (2i, 2i + 1), else (i, i + rot/2).  first: float32 rows of first_stride, v_width used, or null.
AYK_EXPORT int ayk_rotary_prepare(void* qout, void* kpages, void* vpages, const float* proj, long long stride, const float* qw,
                                  const float* kw, float eps, const float* freq, float gain, int neighbours, int rot, const float* first, long long first_stride, float keep, float mix, const int* row_req,
                                  const int* positions, const int* table, int table_stride, int page_size, int T, int H, int G,
                                  int D, int v_width, int writes, int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  AYK_REQUIRE(H >= 1 && G >= 1 && D >= 1 && rot >= 0 && rot % 2 == 0 && rot <= D, "ayk_rotary_prepare: %d + %d heads of %d, %d of them turning", H, G, D, rot);
  const size_t smem = (size_t)rot * sizeof(float);
  AYK_REQUIRE(smem <= 48 * 1024, "ayk_rotary_prepare: %d rotated dimensions", rot);
  AYK_REQUIRE(!qw == !kw, "ayk_rotary_prepare: query and key norms come together");
  const bool vec = D % 4 == 0 && rot % (neighbours ? 4 : 8) == 0 && stride % 4 == 0 && v_width % 4 == 0 && (!first || first_stride % 4 == 0) &&
                   (((uintptr_t)proj | (uintptr_t)qout | (uintptr_t)kpages | (uintptr_t)vpages | (uintptr_t)first | (uintptr_t)qw | (uintptr_t)kw) & 15) == 0;
  const int shares = T >= 64 ? 1 : ((H + G + 7) / 8 < 16 ? (H + G + 7) / 8 : 16);
#define AYK_RP(C, V)                                                                                                     \
  ayk_launch(neighbours ? rotary_prepare_kernel<C, V, true> : rotary_prepare_kernel<C, V, false>, dim3(T, shares), dim3(256), smem, stream, \
             (C*)qout, (C*)kpages, (C*)vpages, proj, stride, qw, kw, eps, freq, gain, rot, first, first_stride, keep, mix, row_req, \
             positions, table, table_stride, page_size, H, G, D, v_width, writes)
  if (dtype == AYK_DTYPE_F32) { if (vec) AYK_RP(float, 4); else AYK_RP(float, 1); }
  else if (dtype == AYK_DTYPE_BF16) { if (vec) AYK_RP(__nv_bfloat16, 4); else AYK_RP(__nv_bfloat16, 1); }
  else return ayk_fail("ayk_rotary_prepare: unknown dtype %d", dtype);
#undef AYK_RP
  return ayk_check_launch("ayk_rotary_prepare");
}
