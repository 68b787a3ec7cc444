// Linear attention with a constant decay per head (lightning attention): a matrix memory
//   S_t = lambda_h S_(t-1) + k_t v_t^T        [D x DV]
//   o_t = S_t^T q_t
// with no softmax and no other scale.  q, k and v are silu of projections.  S starts at zero, is kept in
// 32-bit, and lives in the request's state slot as [heads][D][DV] floats.  The heads' outputs of a token are
// then divided by the root mean square of all of them together, multiplied by a weight per channel and by
// sigmoid of a gate column (decay_finish_kernel).
//
// Powers of the decays come as a table [H][DECAY_CHUNK + 1] (powers[h][n] = lambda_h^n), made by the caller
// in double precision.
//
// Two forms.  decay_walk_kernel takes the tokens one by one from float32 projection rows
// [q (H D) | k (H D) | v (H DV) | ...] before their silu: single-token steps, and everything in the 32-bit
// engine.  decay_chunk_kernel takes 64 tokens at a time on the tensor cores (prompt portions in bfloat16)
// from bfloat16 rows [silu q | silu k | silu v].  Inside a chunk that starts from S_0,
//   o_t = lambda^(t+1) S_0^T q_t + sum_(s<=t) lambda^(t-s) (k_s . q_t) v_s          (t, s from 0)
//   S_L = lambda^L S_0 + sum_s lambda^(L-1-s) k_s v_s^T,
// no exponent is negative, so nothing overflows however strong the decay.  q, k and v are exact in bfloat16;
// whatever carries a decay or the state (S_0, the scores times their decay, the decayed values) enters its
// product as two bfloat16 parts, the rounding and the remainder, so that the products see 16 bits of them; sums
// are 32-bit and S itself stays in 32-bit registers.
//
// Long portions take the chunks side by side instead of one after the other, three launches: what every chunk adds
// to the memory, sum_s lambda^(L-1-s) k_s v_s^T, in float32 scratch (decay_chunk_sum_kernel); the walk over a
// request's chunks, which is now a sum per cell of S and leaves every chunk's S_0, in two bfloat16 parts, in the place of
// what the chunk added (decay_chunk_scan_kernel); and the outputs of every chunk from its S_0 (decay_chunk_out_kernel).  The
// arithmetic is the same.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int DECAY_CHUNK = 64;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// -------------------------------------------------------------------- walk --
// Block (32 value columns, head, request): lane = value column, the eight warps hold an eighth of S's rows
// each, in registers.  Per token every thread updates its rows and adds up q S over them; the partial sums meet
// in shared memory (two buffers in turn, one barrier per token).  q, k and v of up to 16 tokens at a time are
// brought in first.
constexpr int WWARPS = 8, WCOLS = 32, WTOK = 16;

template <int DP>          // rows of S per thread, at most
__global__ void __launch_bounds__(WWARPS * 32, DP <= 16 ? 4 : 1)
decay_walk_kernel(float* __restrict__ out, float* __restrict__ state, const float* __restrict__ proj, long long stride,
                  const float* __restrict__ powers, const int* __restrict__ req_q_start, const int* __restrict__ req_slot,
                  int H, int D, int DV, int settled) {
  extern __shared__ __align__(16) float sh[];
  float* qs = sh;                       // [WTOK][D]
  float* ks = qs + WTOK * D;            // [WTOK][D]
  float* vs = ks + WTOK * D;            // [WTOK][WCOLS]
  float* part = vs + WTOK * WCOLS;      // [2][WWARPS][WCOLS]
  pdl_trigger();
  const int c0 = blockIdx.x * WCOLS, h = blockIdx.y, r = blockIdx.z;
  const int first = req_q_start[r], n = req_q_start[r + 1] - first, slot = req_slot[r];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = c0 + lane;
  const bool col_ok = col < DV;
  const int per = (D + WWARPS - 1) / WWARPS, i0 = warp * per;
  const float lam = powers[h * (DECAY_CHUNK + 1) + 1];
  float* S = state + ((size_t)slot * H + h) * D * DV;
  // the state was left by an earlier step: it may be on its way while the kernel before this one still runs
  if (!settled) pdl_wait();
  float s[DP];
#pragma unroll
  for (int i = 0; i < DP; ++i) {
    const int row = i0 + i;
    s[i] = (i < per && row < D && col_ok) ? S[(size_t)row * DV + col] : 0.f;
  }
  if (settled) pdl_wait();
  const int qcol = h * D, kcol = H * D + h * D, vcol = 2 * H * D + h * DV;
  for (int t0 = 0; t0 < n; t0 += WTOK) {
    const int steps = min(WTOK, n - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < steps * D; i += blockDim.x) {
      const int tt = i / D, d = i - tt * D;
      const float* row = proj + (size_t)(first + t0 + tt) * stride;
      qs[i] = silu(row[qcol + d]);
      ks[i] = silu(row[kcol + d]);
    }
    for (int i = threadIdx.x; i < steps * WCOLS; i += blockDim.x) {
      const int tt = i / WCOLS, c = i - tt * WCOLS;
      vs[i] = c0 + c < DV ? silu(proj[(size_t)(first + t0 + tt) * stride + vcol + c0 + c]) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < steps; ++tt) {
      const float v = vs[tt * WCOLS + lane];
      const float* q = qs + tt * D + i0;
      const float* k = ks + tt * D + i0;
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DP; ++i) {
        if (i < per && i0 + i < D) {
          s[i] = fmaf(lam, s[i], k[i] * v);
          o = fmaf(q[i], s[i], o);
        }
      }
      float* mine = part + (tt & 1) * WWARPS * WCOLS;
      mine[warp * WCOLS + lane] = o;
      __syncthreads();
      if (warp == (tt & (WWARPS - 1)) && col_ok) {
        float total = 0.f;
#pragma unroll
        for (int w = 0; w < WWARPS; ++w) total += mine[w * WCOLS + lane];
        out[(size_t)(first + t0 + tt) * ((size_t)H * DV) + h * DV + col] = total;
      }
    }
  }
  if (n > 0) {
#pragma unroll
    for (int i = 0; i < DP; ++i) {
      const int row = i0 + i;
      if (i < per && row < D && col_ok) S[(size_t)row * DV + col] = s[i];
    }
  }
}

template <int DP>
int launch_walk(float* out, float* state, const float* proj, long long stride, const float* powers, const int* req_q_start,
                const int* req_slot, int R, int H, int D, int DV, int settled, cudaStream_t stream) {
  const size_t smem = ((size_t)2 * WTOK * D + WTOK * WCOLS + 2 * WWARPS * WCOLS) * sizeof(float);
  static AykPerDevice configured;
  if (smem > 48 * 1024 && !configured.here()) {
    cudaError_t err = cudaFuncSetAttribute(decay_walk_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (err != cudaSuccess) return ayk_fail("ayk_decay_walk: shared memory: %s", cudaGetErrorString(err));
    configured.here() = true;
  }
  ayk_launch(decay_walk_kernel<DP>, dim3((DV + WCOLS - 1) / WCOLS, H, R), dim3(WWARPS * 32), smem, stream, out, state, proj,
             stride, powers, req_q_start, req_slot, H, D, DV, settled);
  return ayk_check_launch("ayk_decay_walk");
}

// ------------------------------------------------------------------- chunk --
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async_16(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;                    // 0: nothing is read and the 16 bytes are zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}
// a and b as (rounding, remainder) pairs of bfloat16, packed for a fragment
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
  hi = *reinterpret_cast<uint32_t*>(&h);
  lo = *reinterpret_cast<uint32_t*>(&l);
}

constexpr int CWARPS = 4;
static_assert(CWARPS * 16 == DECAY_CHUNK, "a warp takes 16 tokens of a chunk");

__host__ __device__ inline size_t decay_chunk_bytes(int D, int COLS) {
  const int D16 = (D + 15) & ~15, LDK = D16 + 8, LDV = COLS + 8;
  return ((size_t)2 * 2 * DECAY_CHUNK * LDK           // q and k, two buffers
          + (size_t)2 * DECAY_CHUNK * LDV             // v, two buffers
          + (size_t)2 * DECAY_CHUNK * LDV             // decayed v, two parts
          + (size_t)2 * D16 * LDV) * sizeof(__nv_bfloat16)   // S_0, two parts
         + (DECAY_CHUNK + 4) * sizeof(float);
}

// Block (8 NT value columns, head, request), four warps.  Rows of S: tile i of 16 belongs to warp i % 4, MT tiles
// a warp, in the accumulators of the product that updates it; its two bfloat16 parts pass through shared
// memory once per chunk for the product with q.
template <int MT, int NT>
__global__ void __launch_bounds__(CWARPS * 32)
decay_chunk_kernel(float* __restrict__ out, float* __restrict__ state, const __nv_bfloat16* __restrict__ qkv, long long stride,
                   const float* __restrict__ powers, const int* __restrict__ req_q_start, const int* __restrict__ req_slot,
                   int H, int D, int DV, int vec, int settled) {
  constexpr int CT = DECAY_CHUNK, COLS = NT * 8, LDV = COLS + 8, THREADS = CWARPS * 32;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int D16 = (D + 15) & ~15, LDK = D16 + 8;
  __nv_bfloat16* Qb = reinterpret_cast<__nv_bfloat16*>(smem_raw);     // [2][CT][LDK]
  __nv_bfloat16* Kb = Qb + 2 * CT * LDK;                              // [2][CT][LDK]
  __nv_bfloat16* Vb = Kb + 2 * CT * LDK;                              // [2][CT][LDV]
  __nv_bfloat16* Vh = Vb + 2 * CT * LDV;                              // [CT][LDV]
  __nv_bfloat16* Vl = Vh + CT * LDV;
  __nv_bfloat16* Sh = Vl + CT * LDV;                                  // [D16][LDV]
  __nv_bfloat16* Sl = Sh + D16 * LDV;
  float* pw = reinterpret_cast<float*>(Sl + D16 * LDV);               // [CT + 1]
  pdl_trigger();
  const int c0 = blockIdx.x * COLS, h = blockIdx.y, r = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const int first = req_q_start[r], n = req_q_start[r + 1] - first, slot = req_slot[r];
  for (int i = tid; i <= CT; i += THREADS) pw[i] = powers[h * (CT + 1) + i];
  float* S = state + ((size_t)slot * H + h) * D * DV;
  if (!settled) pdl_wait();
  const int mtiles = D16 / 16;
  float sacc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int row = (warp + CWARPS * i) * 16 + gid + (c >> 1) * 8, col = c0 + j * 8 + tig * 2 + (c & 1);
        sacc[i][j][c] = (row < D && col < DV) ? S[(size_t)row * DV + col] : 0.f;
      }
  auto file_state = [&]() {              // S as two bfloat16 parts, for the next chunk's product with q
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int tile = warp + CWARPS * i;
      if (tile >= mtiles) break;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split_bf16(sacc[i][j][half * 2], sacc[i][j][half * 2 + 1], hi, lo);
          const int at = (tile * 16 + gid + half * 8) * LDV + j * 8 + tig * 2;
          *reinterpret_cast<uint32_t*>(Sh + at) = hi;
          *reinterpret_cast<uint32_t*>(Sl + at) = lo;
        }
    }
  };
  file_state();
  if (settled) pdl_wait();
  const int qcol = h * D, kcol = H * D + h * D, vcol = 2 * H * D + h * DV;
  // one chunk's rows into buffer b; tokens past the portion and the padding of a head are zeros
  auto fetch = [&](int t0, int b) {
    const int L = min(CT, n - t0);
    __nv_bfloat16* Qd = Qb + b * CT * LDK;
    __nv_bfloat16* Kd = Kb + b * CT * LDK;
    __nv_bfloat16* Vd = Vb + b * CT * LDV;
    if (vec) {                           // every head's row starts on a 16-byte boundary
      const int pieces = D16 / 8;
      for (int t = tid >> 3; t < CT; t += THREADS / 8) {
        const __nv_bfloat16* row = qkv + (size_t)(first + t0 + min(t, L - 1)) * stride;
        for (int p = tid & 7; p < pieces; p += 8) {
          const bool live = t < L && p * 8 < D;
          cp_async_16(Qd + t * LDK + p * 8, live ? row + qcol + p * 8 : qkv, live);
          cp_async_16(Kd + t * LDK + p * 8, live ? row + kcol + p * 8 : qkv, live);
        }
        if ((tid & 7) < NT) {
          const int p = tid & 7;
          const bool live = t < L && c0 + p * 8 < DV;
          cp_async_16(Vd + t * LDV + p * 8, live ? row + vcol + c0 + p * 8 : qkv, live);
        }
      }
    } else {
      const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
      for (int t = warp; t < CT; t += CWARPS) {
        const __nv_bfloat16* row = qkv + (size_t)(first + t0 + min(t, L - 1)) * stride;
        for (int d = lane; d < D16; d += 32) {
          const bool live = t < L && d < D;
          Qd[t * LDK + d] = live ? row[qcol + d] : zero;
          Kd[t * LDK + d] = live ? row[kcol + d] : zero;
        }
        for (int c = lane; c < COLS; c += 32) Vd[t * LDV + c] = (t < L && c0 + c < DV) ? row[vcol + c0 + c] : zero;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (n > 0) fetch(0, 0);
  const int ksteps = D16 / 16;
  int b = 0;
  for (int t0 = 0; t0 < n; t0 += CT, b ^= 1) {
    const int L = min(CT, n - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                     // this chunk's rows and S_0 are there; the last chunk's readers are through
    if (t0 + CT < n) fetch(t0 + CT, b ^ 1);
    const __nv_bfloat16* Qs = Qb + b * CT * LDK;
    const __nv_bfloat16* Ks = Kb + b * CT * LDK;
    const __nv_bfloat16* Vs = Vb + b * CT * LDV;
    for (int i = tid; i < CT * COLS / 2; i += THREADS) {           // the values as the chunk's end sees them
      const int t = i / (COLS / 2), c = (i - t * (COLS / 2)) * 2;
      const float w = t < L ? pw[L - 1 - t] : 0.f;
      const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(Vs + t * LDV + c);
      uint32_t hi, lo;
      split_bf16(w * __low2float(v), w * __high2float(v), hi, lo);
      *reinterpret_cast<uint32_t*>(Vh + t * LDV + c) = hi;
      *reinterpret_cast<uint32_t*>(Vl + t * LDV + c) = lo;
    }
    const int m0 = warp * 16;
    if (m0 < L) {
      float o[NT][4], sc[CT / 8][4];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[j][c] = 0.f;
#pragma unroll
      for (int j = 0; j < CT / 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) sc[j][c] = 0.f;
      const uint32_t q_addr = smem_addr(Qs + (m0 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + (lane >> 4) * 8);
      const uint32_t k_addr = smem_addr(Ks + ((lane >> 4) * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8);
      const int s_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8;
#pragma unroll 2
      for (int ks = 0; ks < ksteps; ++ks) {
        uint32_t qf[4];
        ldmatrix_x4(qf, q_addr + ks * 32);
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {                      // q S_0, both parts
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, smem_addr(Sh + s_at + ks * 16 * LDV + np * 16));
          ldmatrix_x4_trans(bl, smem_addr(Sl + s_at + ks * 16 * LDV + np * 16));
          mma_bf16(o[2 * np], qf, bh[0], bh[1]);
          mma_bf16(o[2 * np + 1], qf, bh[2], bh[3]);
          mma_bf16(o[2 * np], qf, bl[0], bl[1]);
          mma_bf16(o[2 * np + 1], qf, bl[2], bl[3]);
        }
#pragma unroll
        for (int kt = 0; kt < CT / 16; ++kt) {                     // q k^T with the keys up to this warp's tokens
          if (kt > warp) break;
          uint32_t bk[4];
          ldmatrix_x4(bk, k_addr + (uint32_t)(kt * 16 * LDK + ks * 16) * 2u);
          mma_bf16(sc[2 * kt], qf, bk[0], bk[1]);
          mma_bf16(sc[2 * kt + 1], qf, bk[2], bk[3]);
        }
      }
      const float w0 = pw[m0 + gid + 1], w1 = pw[m0 + gid + 9];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        o[j][0] *= w0; o[j][1] *= w0;
        o[j][2] *= w1; o[j][3] *= w1;
      }
#pragma unroll
      for (int kt = 0; kt < CT / 16; ++kt) {
        if (kt > warp) break;
        uint32_t ah[4], al[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int nt = 2 * kt + (i >> 1), half = i & 1;
          const int t = m0 + gid + half * 8, s = nt * 8 + tig * 2;
          const float a0 = s <= t ? sc[nt][half * 2] * pw[t - s] : 0.f;
          const float a1 = s + 1 <= t ? sc[nt][half * 2 + 1] * pw[t - s - 1] : 0.f;
          split_bf16(a0, a1, ah[i], al[i]);
        }
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t bv[4];
          ldmatrix_x4_trans(bv, smem_addr(Vs + s_at + kt * 16 * LDV + np * 16));
          mma_bf16(o[2 * np], ah, bv[0], bv[1]);
          mma_bf16(o[2 * np + 1], ah, bv[2], bv[3]);
          mma_bf16(o[2 * np], al, bv[0], bv[1]);
          mma_bf16(o[2 * np + 1], al, bv[2], bv[3]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = m0 + gid + half * 8;
        if (t >= L) continue;
        float* dst = out + (size_t)(first + t0 + t) * ((size_t)H * DV) + h * DV;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int col = c0 + j * 8 + tig * 2;
          if (col < DV) dst[col] = o[j][half * 2];
          if (col + 1 < DV) dst[col + 1] = o[j][half * 2 + 1];
        }
      }
    }
    __syncthreads();                     // the decayed values are there; S_0 has been read
    const float keep = pw[L];
    const int a_at = ((lane & 7) + (lane >> 4) * 8) * LDK + ((lane >> 3) & 1) * 8;
    const int v_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8;
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int tile = warp + CWARPS * i;
      if (tile >= mtiles) break;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) sacc[i][j][c] *= keep;
#pragma unroll
      for (int ks = 0; ks < CT / 16; ++ks) {
        if (ks * 16 >= L) break;
        uint32_t af[4];
        ldmatrix_x4_trans(af, smem_addr(Ks + ks * 16 * LDK + tile * 16 + a_at));
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, smem_addr(Vh + ks * 16 * LDV + np * 16 + v_at));
          ldmatrix_x4_trans(bl, smem_addr(Vl + ks * 16 * LDV + np * 16 + v_at));
          mma_bf16(sacc[i][2 * np], af, bh[0], bh[1]);
          mma_bf16(sacc[i][2 * np + 1], af, bh[2], bh[3]);
          mma_bf16(sacc[i][2 * np], af, bl[0], bl[1]);
          mma_bf16(sacc[i][2 * np + 1], af, bl[2], bl[3]);
        }
      }
    }
    if (t0 + CT < n) file_state();
  }
  if (n <= 0) return;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int row = (warp + CWARPS * i) * 16 + gid + (c >> 1) * 8, col = c0 + j * 8 + tig * 2 + (c & 1);
        if (row < D && col < DV) S[(size_t)row * DV + col] = sacc[i][j][c];
      }
}

template <int MT, int NT>
int launch_chunk(float* out, float* state, const __nv_bfloat16* qkv, long long stride, const float* powers, const int* req_q_start,
                 const int* req_slot, int R, int H, int D, int DV, int vec, int settled, cudaStream_t stream) {
  const size_t smem = decay_chunk_bytes(D, NT * 8);
  static AykPerDevice configured;
  if (smem > 48 * 1024 && !configured.here()) {
    cudaError_t err = cudaFuncSetAttribute(decay_chunk_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (err != cudaSuccess) return ayk_fail("ayk_decay_chunk: shared memory: %s", cudaGetErrorString(err));
    configured.here() = true;
  }
  ayk_launch(decay_chunk_kernel<MT, NT>, dim3((DV + NT * 8 - 1) / (NT * 8), H, R), dim3(CWARPS * 32), smem, stream, out, state, qkv,
             stride, powers, req_q_start, req_slot, H, D, DV, vec, settled);
  return ayk_check_launch("ayk_decay_chunk");
}

// ------------------------------------------------------- chunks side by side --
// which chunk of which request is global chunk number c?  (chunks are numbered request by request)
__device__ __forceinline__ bool find_chunk(const int* req_q_start, int R, int c, int& req, int& t0) {
  for (int r = 0; r < R; ++r) {
    const int chunks = (req_q_start[r + 1] - req_q_start[r] + DECAY_CHUNK - 1) / DECAY_CHUNK;
    if (c < chunks) { req = r; t0 = c * DECAY_CHUNK; return true; }
    c -= chunks;
  }
  return false;
}

// 64 rows of ``n`` numbers (n16 = n rounded up to 16, or the width of a slice) from ``src`` into shared rows of ld;
// rows from L on and columns from n on are zeros.  ``vec``: 16-byte pieces, copied asynchronously.
template <int THREADS>
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, long long stride, int n, int n16, int L,
                                           bool vec) {
  if (vec) {
    const int pieces = n16 / 8;
    for (int t = threadIdx.x >> 3; t < DECAY_CHUNK; t += THREADS / 8)
      for (int p = threadIdx.x & 7; p < pieces; p += 8) {
        const bool live = t < L && p * 8 < n;
        cp_async_16(dst + t * ld + p * 8, live ? src + (size_t)t * stride + p * 8 : src, live);
      }
  } else {
    for (int t = threadIdx.x >> 5; t < DECAY_CHUNK; t += THREADS / 32)
      for (int d = threadIdx.x & 31; d < n16; d += 32)
        dst[t * ld + d] = (t < L && d < n) ? src[(size_t)t * stride + d] : __float2bfloat16_rn(0.f);
  }
}

__host__ __device__ inline size_t decay_sum_bytes(int D, int COLS) {
  const int LDK = ((D + 15) & ~15) + 8, LDV = COLS + 8;
  return ((size_t)DECAY_CHUNK * LDK + (size_t)3 * DECAY_CHUNK * LDV) * sizeof(__nv_bfloat16) + (DECAY_CHUNK + 4) * sizeof(float);
}

// scratch [chunk][H][D][DV] = sum_s lambda^(L-1-s) k_s v_s^T.  Block (8 NT value columns, head, chunk), four warps.
template <int MT, int NT>
__global__ void __launch_bounds__(CWARPS * 32)
decay_chunk_sum_kernel(float* __restrict__ scratch, const __nv_bfloat16* __restrict__ qkv, long long stride,
                       const float* __restrict__ powers, const int* __restrict__ req_q_start, int R, int H, int D, int DV, int vec) {
  constexpr int CT = DECAY_CHUNK, COLS = NT * 8, LDV = COLS + 8, THREADS = CWARPS * 32;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int D16 = (D + 15) & ~15, LDK = D16 + 8;
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);     // [CT][LDK]
  __nv_bfloat16* Vs = Ks + CT * LDK;                                  // [CT][LDV]
  __nv_bfloat16* Vh = Vs + CT * LDV;
  __nv_bfloat16* Vl = Vh + CT * LDV;
  float* pw = reinterpret_cast<float*>(Vl + CT * LDV);
  pdl_trigger();
  const int c0 = blockIdx.x * COLS, h = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  int req = 0, t0 = 0;
  if (!find_chunk(req_q_start, R, blockIdx.z, req, t0)) return;
  const int first = req_q_start[req] + t0, L = min(CT, req_q_start[req + 1] - first);
  for (int i = tid; i <= CT; i += THREADS) pw[i] = powers[h * (CT + 1) + i];
  pdl_wait();
  const __nv_bfloat16* row0 = qkv + (size_t)first * stride;
  fetch_rows<THREADS>(Ks, LDK, row0 + H * D + h * D, stride, D, D16, L, vec);
  fetch_rows<THREADS>(Vs, LDV, row0 + 2 * H * D + h * DV + c0, stride, DV - c0, COLS, L, vec);
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  for (int i = tid; i < CT * COLS / 2; i += THREADS) {
    const int t = i / (COLS / 2), c = (i - t * (COLS / 2)) * 2;
    const float w = t < L ? pw[L - 1 - t] : 0.f;
    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(Vs + t * LDV + c);
    uint32_t hi, lo;
    split_bf16(w * __low2float(v), w * __high2float(v), hi, lo);
    *reinterpret_cast<uint32_t*>(Vh + t * LDV + c) = hi;
    *reinterpret_cast<uint32_t*>(Vl + t * LDV + c) = lo;
  }
  __syncthreads();
  const int a_at = ((lane & 7) + (lane >> 4) * 8) * LDK + ((lane >> 3) & 1) * 8;
  const int v_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8;
  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[i][j][c] = 0.f;
#pragma unroll
  for (int ks = 0; ks < CT / 16; ++ks) {
    if (ks * 16 >= L) break;
    uint32_t bh[NT / 2][4], bl[NT / 2][4];
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      ldmatrix_x4_trans(bh[np], smem_addr(Vh + ks * 16 * LDV + np * 16 + v_at));
      ldmatrix_x4_trans(bl[np], smem_addr(Vl + ks * 16 * LDV + np * 16 + v_at));
    }
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int tile = warp + CWARPS * i;
      if (tile * 16 >= D16) break;
      uint32_t af[4];
      ldmatrix_x4_trans(af, smem_addr(Ks + ks * 16 * LDK + tile * 16 + a_at));
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        mma_bf16(acc[i][2 * np], af, bh[np][0], bh[np][1]);
        mma_bf16(acc[i][2 * np + 1], af, bh[np][2], bh[np][3]);
        mma_bf16(acc[i][2 * np], af, bl[np][0], bl[np][1]);
        mma_bf16(acc[i][2 * np + 1], af, bl[np][2], bl[np][3]);
      }
    }
  }
  float* dst = scratch + ((size_t)blockIdx.z * H + h) * D * DV;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = (warp + CWARPS * i) * 16 + gid + half * 8, col = c0 + j * 8 + tig * 2;
        if (row >= D || col >= DV) continue;
        float* at = dst + (size_t)row * DV + col;
        if (DV % 2 == 0) {
          *reinterpret_cast<float2*>(at) = make_float2(acc[i][j][half * 2], acc[i][j][half * 2 + 1]);
        } else {
          at[0] = acc[i][j][half * 2];
          if (col + 1 < DV) at[1] = acc[i][j][half * 2 + 1];
        }
      }
}

// Per eight cells of S: the walk over a request's chunks.  Scratch gets every chunk's S_0 in the place of what the chunk
// added, as two bfloat16 parts (eight roundings, then eight remainders: the 32 bytes of the eight cells); the state the last S.
__global__ void __launch_bounds__(128)
decay_chunk_scan_kernel(float* __restrict__ scratch, float* __restrict__ state, const float* __restrict__ powers,
                        const int* __restrict__ req_q_start, const int* __restrict__ req_slot, int H, int cells) {
  constexpr int AHEAD = 8;
  pdl_trigger();
  const int i = (blockIdx.x * 128 + threadIdx.x) * 8, h = blockIdx.y, r = blockIdx.z;
  int chunk0 = 0;
  for (int q = 0; q < r; ++q) chunk0 += (req_q_start[q + 1] - req_q_start[q] + DECAY_CHUNK - 1) / DECAY_CHUNK;
  const int n = req_q_start[r + 1] - req_q_start[r], chunks = (n + DECAY_CHUNK - 1) / DECAY_CHUNK;
  const float whole = powers[h * (DECAY_CHUNK + 1) + DECAY_CHUNK];
  const float last = powers[h * (DECAY_CHUNK + 1) + (n - (chunks - 1) * DECAY_CHUNK)];
  pdl_wait();
  if (i >= cells) return;
  float4* S = reinterpret_cast<float4*>(state + ((size_t)req_slot[r] * H + h) * cells + i);
  float4 s0 = S[0], s1 = S[1];
  float* at = scratch + ((size_t)chunk0 * H + h) * cells + i;
  const size_t step = (size_t)H * cells;
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
    float4 add[AHEAD][2];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < chunks) {
        add[u][0] = *reinterpret_cast<const float4*>(at + u * step);
        add[u][1] = *reinterpret_cast<const float4*>(at + u * step + 4);
      }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      if (c0 + u >= chunks) break;
      uint4 hi, lo;
      split_bf16(s0.x, s0.y, hi.x, lo.x);
      split_bf16(s0.z, s0.w, hi.y, lo.y);
      split_bf16(s1.x, s1.y, hi.z, lo.z);
      split_bf16(s1.z, s1.w, hi.w, lo.w);
      *reinterpret_cast<uint4*>(at + u * step) = hi;
      *reinterpret_cast<uint4*>(at + u * step + 4) = lo;
      const float w = c0 + u == chunks - 1 ? last : whole;
      s0.x = fmaf(w, s0.x, add[u][0].x); s0.y = fmaf(w, s0.y, add[u][0].y);
      s0.z = fmaf(w, s0.z, add[u][0].z); s0.w = fmaf(w, s0.w, add[u][0].w);
      s1.x = fmaf(w, s1.x, add[u][1].x); s1.y = fmaf(w, s1.y, add[u][1].y);
      s1.z = fmaf(w, s1.z, add[u][1].z); s1.w = fmaf(w, s1.w, add[u][1].w);
    }
    at += AHEAD * step;
  }
  S[0] = s0;
  S[1] = s1;
}

__host__ __device__ inline size_t decay_out_bytes(int D, int COLS) {
  const int D16 = (D + 15) & ~15, LDK = D16 + 8, LDV = COLS + 8;
  return ((size_t)2 * DECAY_CHUNK * LDK + (size_t)DECAY_CHUNK * LDV + (size_t)2 * D16 * LDV) * sizeof(__nv_bfloat16) +
         (DECAY_CHUNK + 4) * sizeof(float);
}

// The outputs of one chunk from its S_0 (scratch).  Block (8 NT value columns, head, chunk), four warps of 16 tokens.
template <int NT>
__global__ void __launch_bounds__(CWARPS * 32)
decay_chunk_out_kernel(float* __restrict__ out, const float* __restrict__ scratch, const __nv_bfloat16* __restrict__ qkv,
                       long long stride, const float* __restrict__ powers, const int* __restrict__ req_q_start, int R, int H, int D,
                       int DV, int vec) {
  constexpr int CT = DECAY_CHUNK, COLS = NT * 8, LDV = COLS + 8, THREADS = CWARPS * 32;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int D16 = (D + 15) & ~15, LDK = D16 + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);     // [CT][LDK]
  __nv_bfloat16* Ks = Qs + CT * LDK;                                  // [CT][LDK]
  __nv_bfloat16* Vs = Ks + CT * LDK;                                  // [CT][LDV]
  __nv_bfloat16* Sh = Vs + CT * LDV;                                  // [D16][LDV]
  __nv_bfloat16* Sl = Sh + D16 * LDV;
  float* pw = reinterpret_cast<float*>(Sl + D16 * LDV);
  pdl_trigger();
  const int c0 = blockIdx.x * COLS, h = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  int req = 0, t0 = 0;
  if (!find_chunk(req_q_start, R, blockIdx.z, req, t0)) return;
  const int first = req_q_start[req] + t0, L = min(CT, req_q_start[req + 1] - first);
  for (int i = tid; i <= CT; i += THREADS) pw[i] = powers[h * (CT + 1) + i];
  pdl_wait();
  const __nv_bfloat16* row0 = qkv + (size_t)first * stride;
  fetch_rows<THREADS>(Qs, LDK, row0 + h * D, stride, D, D16, L, vec);
  fetch_rows<THREADS>(Ks, LDK, row0 + H * D + h * D, stride, D, D16, L, vec);
  fetch_rows<THREADS>(Vs, LDV, row0 + 2 * H * D + h * DV + c0, stride, DV - c0, COLS, L, vec);
  // S_0 as the scan left it: per eight cells 16 bytes of roundings and 16 of remainders
  const float* S = scratch + ((size_t)blockIdx.z * H + h) * D * DV + c0;
  for (int i = tid; i < D16 * NT; i += THREADS) {
    const int d = i / NT, c = (i - d * NT) * 8;
    const bool live = d < D && c0 + c < DV;
    const float* src = live ? S + (size_t)d * DV + c : scratch;
    cp_async_16(Sh + d * LDV + c, src, live);
    cp_async_16(Sl + d * LDV + c, live ? src + 4 : src, live);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int m0 = warp * 16;
  if (m0 >= L) return;
  float o[NT][4], sc[CT / 8][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[j][c] = 0.f;
#pragma unroll
  for (int j = 0; j < CT / 8; ++j)
#pragma unroll
    for (int c = 0; c < 4; ++c) sc[j][c] = 0.f;
  const uint32_t q_addr = smem_addr(Qs + (m0 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + (lane >> 4) * 8);
  const uint32_t k_addr = smem_addr(Ks + ((lane >> 4) * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8);
  const int s_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8;
  for (int ks = 0; ks < D16 / 16; ++ks) {
    uint32_t qf[4];
    ldmatrix_x4(qf, q_addr + ks * 32);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(bh, smem_addr(Sh + s_at + ks * 16 * LDV + np * 16));
      ldmatrix_x4_trans(bl, smem_addr(Sl + s_at + ks * 16 * LDV + np * 16));
      mma_bf16(o[2 * np], qf, bh[0], bh[1]);
      mma_bf16(o[2 * np + 1], qf, bh[2], bh[3]);
      mma_bf16(o[2 * np], qf, bl[0], bl[1]);
      mma_bf16(o[2 * np + 1], qf, bl[2], bl[3]);
    }
#pragma unroll
    for (int kt = 0; kt < CT / 16; ++kt) {
      if (kt > warp) break;
      uint32_t bk[4];
      ldmatrix_x4(bk, k_addr + (uint32_t)(kt * 16 * LDK + ks * 16) * 2u);
      mma_bf16(sc[2 * kt], qf, bk[0], bk[1]);
      mma_bf16(sc[2 * kt + 1], qf, bk[2], bk[3]);
    }
  }
  const float w0 = pw[m0 + gid + 1], w1 = pw[m0 + gid + 9];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    o[j][0] *= w0; o[j][1] *= w0;
    o[j][2] *= w1; o[j][3] *= w1;
  }
#pragma unroll
  for (int kt = 0; kt < CT / 16; ++kt) {
    if (kt > warp) break;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int nt = 2 * kt + (i >> 1), half = i & 1;
      const int t = m0 + gid + half * 8, s = nt * 8 + tig * 2;
      const float a0 = s <= t ? sc[nt][half * 2] * pw[t - s] : 0.f;
      const float a1 = s + 1 <= t ? sc[nt][half * 2 + 1] * pw[t - s - 1] : 0.f;
      split_bf16(a0, a1, ah[i], al[i]);
    }
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t bv[4];
      ldmatrix_x4_trans(bv, smem_addr(Vs + s_at + kt * 16 * LDV + np * 16));
      mma_bf16(o[2 * np], ah, bv[0], bv[1]);
      mma_bf16(o[2 * np + 1], ah, bv[2], bv[3]);
      mma_bf16(o[2 * np], al, bv[0], bv[1]);
      mma_bf16(o[2 * np + 1], al, bv[2], bv[3]);
    }
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = m0 + gid + half * 8;
    if (t >= L) continue;
    float* dst = out + (size_t)(first + t) * ((size_t)H * DV) + h * DV;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = c0 + j * 8 + tig * 2;
      if (DV % 2 == 0) {
        if (col < DV) *reinterpret_cast<float2*>(dst + col) = make_float2(o[j][half * 2], o[j][half * 2 + 1]);
      } else {
        if (col < DV) dst[col] = o[j][half * 2];
        if (col + 1 < DV) dst[col + 1] = o[j][half * 2 + 1];
      }
    }
  }
}

template <int MT, int NT>
int launch_side_by_side(float* out, float* state, float* scratch, const __nv_bfloat16* qkv, long long stride, const float* powers,
                        const int* req_q_start, const int* req_slot, int R, int chunks, int H, int D, int DV, int vec,
                        cudaStream_t stream) {
  const size_t sum_smem = decay_sum_bytes(D, NT * 8), out_smem = decay_out_bytes(D, NT * 8);
  static AykPerDevice configured;
  if (!configured.here()) {
    cudaError_t err = cudaFuncSetAttribute(decay_chunk_sum_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (err == cudaSuccess) err = cudaFuncSetAttribute(decay_chunk_out_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (err != cudaSuccess) return ayk_fail("ayk_decay_chunks: shared memory: %s", cudaGetErrorString(err));
    configured.here() = true;
  }
  const int slices = (DV + NT * 8 - 1) / (NT * 8), cells = D * DV;
  ayk_launch(decay_chunk_sum_kernel<MT, NT>, dim3(slices, H, chunks), dim3(CWARPS * 32), sum_smem, stream, scratch, qkv, stride, powers,
             req_q_start, R, H, D, DV, vec);
  ayk_launch(decay_chunk_scan_kernel, dim3((cells / 8 + 127) / 128, H, R), dim3(128), 0, stream, scratch, state, powers, req_q_start,
             req_slot, H, cells);
  ayk_launch(decay_chunk_out_kernel<NT>, dim3(slices, H, chunks), dim3(CWARPS * 32), out_smem, stream, out, (const float*)scratch, qkv,
             stride, powers, req_q_start, R, H, D, DV, vec);
  return ayk_check_launch("ayk_decay_chunks");
}

// ------------------------------------------------------------------ finish --
// out[t, :] = raw[t, :] / rms(raw[t, :]) * w * sigmoid(gate[t, :]) over a row of n numbers (all heads together).
template <typename C, int VEC>
__global__ void __launch_bounds__(256)
decay_finish_kernel(C* __restrict__ out, const float* __restrict__ raw, const float* __restrict__ gate, long long gate_stride,
                    const float* __restrict__ w, int n, float eps) {
  __shared__ float red[8];
  pdl_trigger();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  const float* src = raw + (size_t)t * n;
  const float* g = gate + (size_t)t * gate_stride;
  C* dst = out + (size_t)t * n;
  float s = 0.f;
  if (VEC == 4) {
    for (int i = threadIdx.x * 4; i < n; i += 1024) {
      const float4 v = *reinterpret_cast<const float4*>(src + i);
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    }
  } else {
    for (int i = threadIdx.x; i < n; i += 256) s = fmaf(src[i], src[i], s);
  }
  s = warp_sum(s);
  if (lane == 0) red[warp] = s;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) total += red[i];
  const float inv = 1.0f / sqrtf(total / (float)n + eps);
  if (VEC == 4) {
    for (int i = threadIdx.x * 4; i < n; i += 1024) {
      const float4 v = *reinterpret_cast<const float4*>(src + i), z = *reinterpret_cast<const float4*>(g + i);
      const float4 a = *reinterpret_cast<const float4*>(w + i);
      const float r[4] = {v.x * inv * a.x / (1.0f + expf(-z.x)), v.y * inv * a.y / (1.0f + expf(-z.y)),
                          v.z * inv * a.z / (1.0f + expf(-z.z)), v.w * inv * a.w / (1.0f + expf(-z.w))};
      if (sizeof(C) == 4) {
        *reinterpret_cast<float4*>(dst + i) = make_float4(r[0], r[1], r[2], r[3]);
      } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
        uint2 packed;
        packed.x = *reinterpret_cast<uint32_t*>(&lo);
        packed.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(dst + i) = packed;
      }
    }
  } else {
    for (int i = threadIdx.x; i < n; i += 256) dst[i] = from_float<C>(src[i] * inv * w[i] / (1.0f + expf(-g[i])));
  }
}

}  // namespace

AYK_EXPORT int ayk_decay_chunk_tokens() { return DECAY_CHUNK; }

// out [T, H * DV] float32 = S_t^T q_t, token by token; state [slots, H, D, DV] float32 is read at the start of a
// request's portion and written at its end.  proj: float32 rows of ``stride`` [q | k | v | ...] before their silu.
// settled: earlier steps' states are complete when the kernel is scheduled.
AYK_EXPORT int ayk_decay_walk(float* out, float* state, const float* proj, long long stride, const float* powers,
                              const int* req_q_start, const int* req_slot, int R, int H, int D, int DV, int settled,
                              cudaStream_t stream) {
  if (R == 0) return 0;
  AYK_REQUIRE(D >= 1 && D <= 1024 && DV >= 1, "ayk_decay_walk: heads of %d x %d (keys of at most 1024 numbers)", D, DV);
  AYK_REQUIRE(H <= 65535 && R <= 65535, "ayk_decay_walk: %d heads, %d requests", H, R);
  const int per = (D + WWARPS - 1) / WWARPS;
#define AYK_DW(DP) return launch_walk<DP>(out, state, proj, stride, powers, req_q_start, req_slot, R, H, D, DV, settled, stream)
  if (per <= 4) AYK_DW(4);
  if (per <= 8) AYK_DW(8);
  if (per <= 16) AYK_DW(16);
  if (per <= 32) AYK_DW(32);
  AYK_DW(128);
#undef AYK_DW
}

// Whether the chunked form takes heads of D numbers.
AYK_EXPORT int ayk_decay_chunk_takes(int D) { return D >= 1 && D <= 256 && decay_chunk_bytes(D, 32) <= 227 * 1024; }

// The same 64 tokens at a time from bfloat16 rows of ``stride`` [silu q | silu k | silu v].  cols: value columns per
// block, 16 or 32 (0: 32, or 16 where blocks of 32 would leave many multiprocessors without one).
AYK_EXPORT int ayk_decay_chunk(float* out, float* state, const void* qkv, long long stride, const float* powers,
                               const int* req_q_start, const int* req_slot, int R, int H, int D, int DV, int cols,
                               int settled, cudaStream_t stream) {
  if (R == 0) return 0;
  AYK_REQUIRE(ayk_decay_chunk_takes(D) && DV >= 1, "ayk_decay_chunk: heads of %d x %d (keys of at most 256 numbers)", D, DV);
  AYK_REQUIRE(H <= 65535 && R <= 65535, "ayk_decay_chunk: %d heads, %d requests", H, R);
  const bool narrow = cols ? cols == 16 : (long long)((DV + 31) / 32) * H * R * 4 < (long long)ayk_sm_count() * 3 && DV > 16;
  const int vec = D % 8 == 0 && DV % 8 == 0 && stride % 8 == 0 && ((uintptr_t)qkv & 15) == 0;
  const __nv_bfloat16* rows = (const __nv_bfloat16*)qkv;
  const int mt = ((D + 15) / 16 + CWARPS - 1) / CWARPS;
#define AYK_DC(M, N) return launch_chunk<M, N>(out, state, rows, stride, powers, req_q_start, req_slot, R, H, D, DV, vec, settled, stream)
  if (narrow) {
    if (mt <= 1) AYK_DC(1, 2);
    if (mt <= 2) AYK_DC(2, 2);
    AYK_DC(4, 2);
  }
  if (mt <= 1) AYK_DC(1, 4);
  if (mt <= 2) AYK_DC(2, 4);
  AYK_DC(4, 4);
#undef AYK_DC
}

// Whether the form that takes a portion's chunks side by side takes these heads.
AYK_EXPORT int ayk_decay_chunks_takes(int D, int DV) {
  return ayk_decay_chunk_takes(D) && DV % 8 == 0 && decay_out_bytes(D, 64) <= 227 * 1024;
}

// The same with all chunks of the R requests side by side (three launches).  chunks: at least as many as the requests'
// portions have (surplus blocks leave); every request brings at least one row.  scratch: float32 [chunks][H][D][DV].
AYK_EXPORT int ayk_decay_chunks(float* out, float* state, float* scratch, const void* qkv, long long stride, const float* powers,
                                const int* req_q_start, const int* req_slot, int R, int chunks, int H, int D, int DV,
                                cudaStream_t stream) {
  if (R == 0 || chunks == 0) return 0;
  AYK_REQUIRE(ayk_decay_chunks_takes(D, DV), "ayk_decay_chunks: heads of %d x %d", D, DV);
  AYK_REQUIRE(H <= 65535 && R <= 65535 && chunks <= 65535, "ayk_decay_chunks: %d heads, %d requests, %d chunks", H, R, chunks);
  const int vec = D % 8 == 0 && DV % 8 == 0 && stride % 8 == 0 && ((uintptr_t)qkv & 15) == 0;
  const __nv_bfloat16* rows = (const __nv_bfloat16*)qkv;
  const int mt = ((D + 15) / 16 + CWARPS - 1) / CWARPS;
#define AYK_DS(M, N) return launch_side_by_side<M, N>(out, state, scratch, rows, stride, powers, req_q_start, req_slot, R, chunks, H, D, DV, vec, stream)
  if (DV <= 32) {
    if (mt <= 1) AYK_DS(1, 4);
    if (mt <= 2) AYK_DS(2, 4);
    AYK_DS(4, 4);
  }
  if (mt <= 1) AYK_DS(1, 8);
  if (mt <= 2) AYK_DS(2, 8);
  AYK_DS(4, 8);
#undef AYK_DS
}

// out[t, :] = raw[t, :] / rms(raw[t, :]) * w * sigmoid(gate[t, :]), rows of n numbers; gate: float32 rows of gate_stride.
AYK_EXPORT int ayk_decay_finish(void* out, const float* raw, const float* gate, long long gate_stride, const float* w, int T,
                                int n, float eps, int out_dtype, cudaStream_t stream) {
  if (T == 0 || n == 0) return 0;
  const bool vec = n % 4 == 0 && gate_stride % 4 == 0 &&
                   (((uintptr_t)out | (uintptr_t)raw | (uintptr_t)gate | (uintptr_t)w) & 15) == 0;
#define AYK_DF(C, V) ayk_launch(decay_finish_kernel<C, V>, dim3(T), dim3(256), 0, stream, (C*)out, raw, gate, gate_stride, w, n, eps)
  if (out_dtype == AYK_DTYPE_F32) { if (vec) AYK_DF(float, 4); else AYK_DF(float, 1); }
  else if (out_dtype == AYK_DTYPE_BF16) { if (vec) AYK_DF(__nv_bfloat16, 4); else AYK_DF(__nv_bfloat16, 1); }
  else return ayk_fail("ayk_decay_finish: unknown dtype %d", out_dtype);
#undef AYK_DF
  return ayk_check_launch("ayk_decay_finish");
}
