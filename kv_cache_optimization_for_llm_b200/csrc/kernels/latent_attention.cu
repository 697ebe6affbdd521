// Attention whose keys and values are up-projections of a small latent per token: only the
// latent c (RMS-normed, `rank` wide) and one rotated key part shared by all heads (`rot` wide)
// are cached, as one row of Dc = rank + rot elements per token in the paged cache.
//
// The up-projections are moved to the query side: with k_h = U_h c the score q.k_h equals
// (U_h^T q).c, so every head attends with an "absorbed" query [U_h^T q_plain | q_rot] over the
// same cached rows, the weighted sum of the latents comes out [rank] wide per head and the
// value up-projection is applied to it afterwards.  The kernels:
//   latent_prep       per token: RMS norm of the query latent (where queries have one), RMS norm of the
//                     key/value latent, interleaved rotary encoding of the shared key part, cache write
//   head_gemm         a product per head, out[t, h, :] = W[h] . in[t, h, :]  (absorbs the queries,
//                     and up-projects the attended latents; with a gate its result is multiplied by
//                     the gate's sigmoid)
//   head_rows         for steps whose per-head products the library made: [heads, tokens, N] back to one
//                     row per token, with the same optional gate
//   latent_rows       for long runs of tokens, whose keys and values are worth making: the cached rows that the runs see,
//                     gathered into one matrix that a batched product turns into every head's [key | value] rows
//   latent_attention  causal softmax attention of all heads over the cached rows, optionally over a sliding
//                     window (position i sees j with i - j < window), optionally with a sink:
//                     the denominator also holds exp(sink_h), a key without a value
// Scores, softmax weights, sums and angles are float32.  Keys are walked in chunks of 32 by
// absolute position, so a token's result does not depend on how its request was cut into steps,
// on the rest of the batch or on where its pages lie.
#include "cluster.cuh"
#include "common.cuh"

#include <math_constants.h>

__device__ __forceinline__ void ldsm_x4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3,
                                               unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// ---------------------------------------------------------------- prep
// d_in [T, ld]: the query latent at column 0 (q_rank wide), the key/value latent at column
// kv_off (rank wide) followed by the shared key part (rot wide).
// cq[t] = rms(d_in[t, :q_rank]) * wq (q_rank 0: no query latent);  page row = [ rms(latent) * wkv | rotate(shared part) ].
// Rotation: pairs (2i, 2i + 1) for i < rdims / 2 turn by cos/sin[pos, i]; the rest passes.
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ d_in, int ld, int q_rank, int kv_off, int rank, int rot, int rdims,
                   const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len,
                   const int* __restrict__ positions, const int* __restrict__ token_req,
                   const int* __restrict__ block_table, int max_pages, int page_size, int num_pages,
                   T* __restrict__ cq, T* __restrict__ pages, int write, int* status) {
  __shared__ float part[8];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos = positions[t];
  const T* row = d_in + (size_t)t * ld;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) { const float x = to_f32(row[i]); sq += x * x; }
  for (int i = threadIdx.x; i < rank; i += blockDim.x) { const float x = to_f32(row[kv_off + i]); sk += x * x; }
  sq = warp_sum(sq); sk = warp_sum(sk);
  if (lane == 0) { part[warp] = sq; part[4 + warp] = sk; }
  __syncthreads();
  sq = part[0] + part[1] + part[2] + part[3];
  sk = part[4] + part[5] + part[6] + part[7];
  const float iq = 1.0f / sqrtf(sq / (float)q_rank + eps), ik = 1.0f / sqrtf(sk / (float)rank + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    cq[(size_t)t * q_rank + i] = from_f32<T>(to_f32(row[i]) * iq * wq[i]);
  if (!write) return;
  if (pos < 0 || (rdims > 0 && pos >= table_len)) {
    if (threadIdx.x == 0) atomicCAS(status, 0, KVB_STATUS_BAD_POSITION);
    return;
  }
  const int lp = pos / page_size;
  const int page = lp < max_pages ? block_table[(size_t)token_req[t] * max_pages + lp] : -1;
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicCAS(status, 0, KVB_STATUS_UNMAPPED_PAGE);
    return;
  }
  T* dst = pages + ((size_t)page * page_size + (pos % page_size)) * (rank + rot);
  for (int i = threadIdx.x; i < rank; i += blockDim.x) dst[i] = from_f32<T>(to_f32(row[kv_off + i]) * ik * wkv[i]);
  const int half = rdims >> 1;
  const T* kr = row + kv_off + rank;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
    const float u = to_f32(kr[2 * i]), v = to_f32(kr[2 * i + 1]);
    dst[rank + 2 * i] = from_f32<T>(u * c - v * s);
    dst[rank + 2 * i + 1] = from_f32<T>(v * c + u * s);
  }
  for (int i = rdims + threadIdx.x; i < rot; i += blockDim.x) dst[rank + i] = kr[i];
}

// The same for bfloat16 rows whose segments are multiples of 8 wide: a warp per token, 16-byte accesses, no barrier.
__device__ __forceinline__ float square_sum8(const uint4& u) {
  const unsigned w[4] = {u.x, u.y, u.z, u.w};
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float a = __uint_as_float(w[i] << 16), b = __uint_as_float(w[i] & 0xffff0000u);
    s = fmaf(a, a, s);
    s = fmaf(b, b, s);
  }
  return s;
}
__device__ __forceinline__ uint4 scaled8(const uint4& u, float f, const float* weight) {
  const unsigned w[4] = {u.x, u.y, u.z, u.w};
  const float4 lo = *reinterpret_cast<const float4*>(weight), hi = *reinterpret_cast<const float4*>(weight + 4);
  const float c[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
  unsigned r[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(__uint_as_float(w[i] << 16) * f * c[2 * i],
                                                   __uint_as_float(w[i] & 0xffff0000u) * f * c[2 * i + 1]);
    r[i] = *reinterpret_cast<const unsigned*>(&v);
  }
  return make_uint4(r[0], r[1], r[2], r[3]);
}

constexpr int kPrepWarps = 4;

__global__ void __launch_bounds__(kPrepWarps * 32)
latent_prep_bf16x8_kernel(const __nv_bfloat16* __restrict__ d_in, int ld, int q_rank, int kv_off, int rank, int rot, int rdims,
                          const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                          const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len,
                          const int* __restrict__ positions, const int* __restrict__ token_req,
                          const int* __restrict__ block_table, int max_pages, int page_size, int num_pages,
                          __nv_bfloat16* __restrict__ cq, __nv_bfloat16* __restrict__ pages, int write, int T_, int* status) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x * kPrepWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T_) return;
  const __nv_bfloat16* row = d_in + (size_t)t * ld;
  const uint4* q4 = reinterpret_cast<const uint4*>(row);
  const uint4* k4 = reinterpret_cast<const uint4*>(row + kv_off);
  const int nq = q_rank >> 3, nk = rank >> 3;
  const int pos = positions[t], req = token_req[t];
  float sq = 0.f, sk = 0.f;
  for (int i = lane; i < nq; i += 32) sq += square_sum8(q4[i]);
  if (write)
    for (int i = lane; i < nk; i += 32) sk += square_sum8(k4[i]);
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  const float iq = 1.0f / sqrtf(sq / (float)q_rank + eps), ik = 1.0f / sqrtf(sk / (float)rank + eps);
  uint4* cq4 = reinterpret_cast<uint4*>(cq + (size_t)t * q_rank);
  for (int i = lane; i < nq; i += 32) cq4[i] = scaled8(q4[i], iq, wq + 8 * i);
  if (!write) return;
  if (pos < 0 || (rdims > 0 && pos >= table_len)) {
    if (lane == 0) atomicCAS(status, 0, KVB_STATUS_BAD_POSITION);
    return;
  }
  const int lp = pos / page_size;
  const int page = lp < max_pages ? block_table[(size_t)req * max_pages + lp] : -1;
  if (page < 0 || page >= num_pages) {
    if (lane == 0) atomicCAS(status, 0, KVB_STATUS_UNMAPPED_PAGE);
    return;
  }
  __nv_bfloat16* dst = pages + ((size_t)page * page_size + (pos % page_size)) * (rank + rot);
  for (int i = lane; i < nk; i += 32) reinterpret_cast<uint4*>(dst)[i] = scaled8(k4[i], ik, wkv + 8 * i);
  const int half = rdims >> 1;
  const __nv_bfloat16* kr = row + kv_off + rank;
  for (int i = lane; i < half; i += 32) {
    const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
    const float u = __bfloat162float(kr[2 * i]), v = __bfloat162float(kr[2 * i + 1]);
    dst[rank + 2 * i] = __float2bfloat16_rn(u * c - v * s);
    dst[rank + 2 * i + 1] = __float2bfloat16_rn(v * c + u * s);
  }
  for (int i = rdims + lane; i < rot; i += 32) dst[rank + i] = kr[i];
}

KVB_EXPORT int kvb_latent_prep(const void* d_in, int ld, int q_rank, int kv_off, int rank, int rot, int rdims,
                               const float* wq, const float* wkv, float eps, const float* cos_t, const float* sin_t,
                               int table_len, const int* positions, const int* token_req, const int* block_table,
                               int max_pages, int page_size, int num_pages, void* cq, void* pages, int write,
                               int T_, int dtype, int* status, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (q_rank < 0 || rank < 1 || rot < 0 || rdims < 0 || (rdims & 1) || rdims > rot) return KVB_ERR_BAD_SIZE;
  const uintptr_t at = reinterpret_cast<uintptr_t>(d_in) | reinterpret_cast<uintptr_t>(cq) | reinterpret_cast<uintptr_t>(pages) |
                       reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wkv);
  if (dtype == KVB_BF16 && ((ld | q_rank | kv_off | rank | (rank + rot)) & 7) == 0 && (at & 15) == 0) {
    kvb_launch(latent_prep_bf16x8_kernel, dim3((T_ + kPrepWarps - 1) / kPrepWarps), dim3(kPrepWarps * 32), 0, stream,
               (const __nv_bfloat16*)d_in, ld, q_rank, kv_off, rank, rot, rdims, wq, wkv, eps, cos_t, sin_t, table_len, positions,
               token_req, block_table, max_pages, page_size, num_pages, (__nv_bfloat16*)cq, (__nv_bfloat16*)pages, write, T_, status);
    return kvb_launch_result();
  }
  KVB_DISPATCH_DTYPE(dtype, T, (kvb_launch(latent_prep_kernel<T>, dim3(T_), dim3(128), 0, stream, (const T*)d_in, ld,
                                            q_rank, kv_off, rank, rot, rdims, wq, wkv, eps, cos_t, sin_t, table_len,
                                            positions, token_req, block_table, max_pages, page_size, num_pages,
                                            (T*)cq, (T*)pages, write, status)));
  return kvb_launch_result();
}

// ---------------------------------------------------------------- a product per head
// out[t, h * hs_out + n] = sum_k in[t, h * hs_in + k] * W[h, n, k]   for n < N, k < K, h < H.
// Plain FMA in ascending k with float32 sums: an output does not depend on the number of rows.
constexpr int HG_BM = 64, HG_BN = 64, HG_BK = 16;

// With `gate` (row stride ld_gate, the layout of out): times sigmoid(gate[t, h * hs_out + n]).
template <typename T>
__global__ void __launch_bounds__(256)
head_gemm_kernel(const T* __restrict__ in, int ld_in, int hs_in, const T* __restrict__ W, T* __restrict__ out,
                 int ld_out, int hs_out, int M, int N, int K, const T* __restrict__ gate, int ld_gate) {
  __shared__ float As[HG_BK][HG_BM + 4];
  __shared__ float Ws[HG_BK][HG_BN + 4];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.z;
  const T* A = in + (size_t)h * hs_in;
  const T* Wh = W + (size_t)h * N * K;
  const int tid = threadIdx.x;
  const int m0 = blockIdx.y * HG_BM, n0 = blockIdx.x * HG_BN;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const int lrow = tid >> 2, lk = (tid & 3) * 4;
  for (int k0 = 0; k0 < K; k0 += HG_BK) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int k = k0 + lk + u;
      const int am = m0 + lrow, wn = n0 + lrow;
      As[lk + u][lrow] = (am < M && k < K) ? to_f32(A[(size_t)am * ld_in + k]) : 0.f;
      Ws[lk + u][lrow] = (wn < N && k < K) ? to_f32(Wh[(size_t)wn * K + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < HG_BK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = Ws[kk][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) {
        float v = acc[i][j];
        if (gate != nullptr) v *= 1.0f / (1.0f + expf(-to_f32(gate[(size_t)m * ld_gate + (size_t)h * hs_out + n])));
        out[(size_t)m * ld_out + (size_t)h * hs_out + n] = from_f32<T>(v);
      }
    }
  }
}

// The same product on mma.sync m16n8k16 for bfloat16 steps of few rows, which are bound by bringing the weights: a warp
// takes 8 rows n of W[h] and up to 16 MT rows m; lane (g, t) loads 16 bytes, the elements k0 + 8 t .. + 7, of row n0 + g of
// W and of rows g and g + 8 of every tile of the input, and hands elements 0 - 3 to one product and 4 - 7 to the next: the
// order of the k within a product is free as long as both operands have the same.  K a multiple of 8.
constexpr int HM_WARPS = 4;

template <int MT>
__global__ void __launch_bounds__(HM_WARPS * 32)
head_gemm_mma_kernel(const __nv_bfloat16* __restrict__ in, int ld_in, int hs_in, const __nv_bfloat16* __restrict__ W,
                     __nv_bfloat16* __restrict__ out, int ld_out, int hs_out, int M, int N, int K,
                     const __nv_bfloat16* __restrict__ gate, int ld_gate) {
  pdl_trigger();
  const int h = blockIdx.z, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n0 = (blockIdx.x * HM_WARPS + (threadIdx.x >> 5)) * 8, m0 = blockIdx.y * 16 * MT;
  if (n0 >= N) return;
  const __nv_bfloat16* w = W + ((size_t)h * N + min(n0 + g, N - 1)) * K + 8 * t;
  const __nv_bfloat16* a[2 * MT];
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) a[i] = in + (size_t)min(m0 + 8 * i + g, M - 1) * ld_in + (size_t)h * hs_in + 8 * t;
  float acc[MT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  // the weights do not depend on what runs before: the first pieces are on their way while the kernel waits
  constexpr int AHEAD = 4;
  uint4 b[AHEAD];
#pragma unroll
  for (int s = 0; s < AHEAD; ++s)
    b[s] = 32 * s + 8 * t < K ? *reinterpret_cast<const uint4*>(w + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
  pdl_wait();
  for (int k0 = 0; k0 < K; k0 += 32 * AHEAD) {
    uint4 next[AHEAD];
#pragma unroll
    for (int s = 0; s < AHEAD; ++s) {
      const int k = k0 + 32 * (AHEAD + s);
      next[s] = k + 8 * t < K ? *reinterpret_cast<const uint4*>(w + k) : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int s = 0; s < AHEAD; ++s) {
      const int k = k0 + 32 * s;
      if (k >= K) break;
      const bool in_row = k + 8 * t < K;
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const uint4 lo = in_row ? *reinterpret_cast<const uint4*>(a[2 * i] + k) : make_uint4(0u, 0u, 0u, 0u);
        const uint4 hi = in_row ? *reinterpret_cast<const uint4*>(a[2 * i + 1] + k) : make_uint4(0u, 0u, 0u, 0u);
        mma_bf16_16816(acc[i], lo.x, hi.x, lo.y, hi.y, b[s].x, b[s].y);
        mma_bf16_16816(acc[i], lo.z, hi.z, lo.w, hi.w, b[s].z, b[s].w);
      }
    }
#pragma unroll
    for (int s = 0; s < AHEAD; ++s) b[s] = next[s];
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int m = m0 + 16 * i + g + 8 * (e >> 1), n = n0 + 2 * t + (e & 1);
      if (m < M && n < N) {
        float v = acc[i][e];
        if (gate != nullptr) v *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)m * ld_gate + (size_t)h * hs_out + n])));
        out[(size_t)m * ld_out + (size_t)h * hs_out + n] = __float2bfloat16_rn(v);
      }
    }
}

KVB_EXPORT int kvb_head_gemm(const void* in, int ld_in, int hs_in, const void* W, void* out, int ld_out, int hs_out,
                             int M, int N, int K, int H, const void* gate, int ld_gate, int tensor_cores, int dtype,
                             cudaStream_t stream) {
  if (M <= 0 || N <= 0 || H <= 0) return 0;
  if (K <= 0 || H > 65535) return KVB_ERR_BAD_SIZE;
  dim3 grid((N + HG_BN - 1) / HG_BN, (M + HG_BM - 1) / HG_BM, H);
  if (grid.y > 65535) return KVB_ERR_BAD_SIZE;
  if (tensor_cores && dtype == KVB_BF16 && ((K | ld_in | hs_in) & 7) == 0 &&
      ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(W)) & 15) == 0) {
    using B = __nv_bfloat16;
    const int nb = (N + 8 * HM_WARPS - 1) / (8 * HM_WARPS);
#define KVB_HEAD_MMA(MT)                                                                                               \
    kvb_launch(head_gemm_mma_kernel<MT>, dim3(nb, (M + 16 * MT - 1) / (16 * MT), H), dim3(HM_WARPS * 32), 0, stream,   \
               (const B*)in, ld_in, hs_in, (const B*)W, (B*)out, ld_out, hs_out, M, N, K, (const B*)gate, ld_gate)
    if (M <= 16) KVB_HEAD_MMA(1);
    else if (M <= 32) KVB_HEAD_MMA(2);
    else KVB_HEAD_MMA(4);
#undef KVB_HEAD_MMA
    return kvb_launch_result();
  }
  KVB_DISPATCH_DTYPE(dtype, T, (kvb_launch(head_gemm_kernel<T>, grid, dim3(256), 0, stream, (const T*)in, ld_in, hs_in,
                                            (const T*)W, (T*)out, ld_out, hs_out, M, N, K, (const T*)gate, ld_gate)));
  return kvb_launch_result();
}

// in [H, T, N] dense (a batched product's result) -> out[t, h * N + n], times sigmoid(gate[t, h * N + n]) when there is a
// gate.  VEC elements per thread (N a multiple of VEC; 16-byte accesses with VEC 8).
template <int VEC>
__global__ void __launch_bounds__(256)
head_rows_kernel(const __nv_bfloat16* __restrict__ in, __nv_bfloat16* __restrict__ out, int ld_out,
                 const __nv_bfloat16* __restrict__ gate, int ld_gate, int T_, int H, int N, size_t total) {
  pdl_trigger();
  pdl_wait();
  const int per_head = N / VEC;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t th = idx / per_head;
    const int n = (int)(idx - th * per_head) * VEC;
    const size_t t = th / H;
    const int h = (int)(th - t * H);
    const __nv_bfloat16* src = in + ((size_t)h * T_ + t) * N + n;
    const __nv_bfloat16* g = gate != nullptr ? gate + t * ld_gate + (size_t)h * N + n : nullptr;
    __nv_bfloat16* dst = out + t * ld_out + (size_t)h * N + n;
    alignas(16) __nv_bfloat16 x[VEC];
    alignas(16) __nv_bfloat16 gv[VEC];
    if (VEC == 8) {
      *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(src);
      if (g != nullptr) *reinterpret_cast<uint4*>(gv) = *reinterpret_cast<const uint4*>(g);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) { x[i] = src[i]; if (g != nullptr) gv[i] = g[i]; }
    }
    if (g != nullptr) {
#pragma unroll
      for (int i = 0; i < VEC; ++i)
        x[i] = __float2bfloat16_rn(__bfloat162float(x[i]) / (1.0f + expf(-__bfloat162float(gv[i]))));
    }
    if (VEC == 8) {
      *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(x);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) dst[i] = x[i];
    }
  }
}

KVB_EXPORT int kvb_head_rows(const void* in, void* out, int ld_out, const void* gate, int ld_gate, int T_, int H, int N,
                             cudaStream_t stream) {
  if (T_ <= 0 || H <= 0) return 0;
  if (N < 1) return KVB_ERR_BAD_SIZE;
  const bool vec = N % 8 == 0 && ld_out % 8 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 &&
                   (gate == nullptr || (ld_gate % 8 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0));
  const size_t total = (size_t)T_ * H * (vec ? N / 8 : N);
  const size_t want = (total + 255) / 256;
  const int blocks = (int)(want < (size_t)kvb_sm_count() * 16 ? want : (size_t)kvb_sm_count() * 16);
  using B = __nv_bfloat16;
  if (vec)
    kvb_launch(head_rows_kernel<8>, dim3(blocks), dim3(256), 0, stream, (const B*)in, (B*)out, ld_out, (const B*)gate, ld_gate,
               T_, H, N, total);
  else
    kvb_launch(head_rows_kernel<1>, dim3(blocks), dim3(256), 0, stream, (const B*)in, (B*)out, ld_out, (const B*)gate, ld_gate,
               T_, H, N, total);
  return kvb_launch_result();
}

// ---------------------------------------------------------------- the rows that long runs see
// A block fills eight rows, one per warp, of a page of `rows_per_page` rows of out [n_pages * rows_per_page, rank]: info [n_pages, 4] int32 holds the
// request's row in the batch, the position of the page's first row, and the first position that the run sees; rows
// in front of that or behind the request's last token are zero.  16-byte pieces.
__global__ void __launch_bounds__(256)
latent_rows_kernel(const __nv_bfloat16* __restrict__ pages, const int* __restrict__ block_table, int max_pages, int page_size,
                   int num_pages, const int* __restrict__ ctx_len, const int4* __restrict__ info, int rows_per_page,
                   int vecs, __nv_bfloat16* __restrict__ out, int* status) {
  pdl_trigger();
  pdl_wait();
  const int4 page_info = info[blockIdx.x];
  const int req = page_info.x, first = page_info.y, lowest = page_info.z;
  const int end = ctx_len[req];
  const int* table = block_table + (size_t)req * max_pages;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.y * 8 + warp;
  if (r < rows_per_page) {
    const int pos = first + r;
    const uint4* src = nullptr;
    if (pos >= lowest && pos < end) {
      const int lp = pos / page_size;
      const int page = lp < max_pages ? table[lp] : -1;
      if (page < 0 || page >= num_pages) { if (lane == 0) atomicCAS(status, 0, KVB_STATUS_UNMAPPED_PAGE); }
      else src = reinterpret_cast<const uint4*>(pages) + ((size_t)page * page_size + pos % page_size) * vecs;
    }
    uint4* dst = reinterpret_cast<uint4*>(out) + ((size_t)blockIdx.x * rows_per_page + r) * vecs;
    for (int v = lane; v < vecs; v += 32) dst[v] = src != nullptr ? src[v] : make_uint4(0u, 0u, 0u, 0u);
  }
}

// bfloat16, rank a multiple of 8, cache rows of rank elements (nothing behind the latent).
KVB_EXPORT int kvb_latent_rows(const void* pages, const int* block_table, int max_pages, int page_size, int num_pages,
                               const int* ctx_len, const int* info, int n_pages, int rows_per_page, int rank, void* out,
                               int* status, cudaStream_t stream) {
  if (n_pages <= 0) return 0;
  if (rank < 8 || rank % 8 != 0 || rows_per_page < 1) return KVB_ERR_BAD_SIZE;
  if ((reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(info) | reinterpret_cast<uintptr_t>(out)) & 15)
    return KVB_ERR_ALIGN;
  kvb_launch(latent_rows_kernel, dim3(n_pages, (rows_per_page + 7) / 8), dim3(256), 0, stream, (const __nv_bfloat16*)pages, block_table, max_pages,
             page_size, num_pages, ctx_len, (const int4*)info, rows_per_page, rank / 8, (__nv_bfloat16*)out, status);
  return kvb_launch_result();
}

// ---------------------------------------------------------------- attention over the cached rows
// A block takes one query token and up to kLatWarps heads, one head per warp.  The block loads a
// chunk of 32 cached rows into shared memory once for all its heads; a lane scores one key
// (dot over Dc), the warp keeps a running maximum and sum that start from the sink
// (m = sink_h, l = 1: the sink counts once and has no value; without one m = -inf, l = 0), and lanes then own value dims.
constexpr int kLatWarps = 8;

template <typename T> struct Word;     // a 4-byte word of shared memory: 1 float or 2 bfloat16
template <> struct Word<float> {
  static constexpr int N = 1;
  static __device__ __forceinline__ float dot(const float* q, unsigned w) { return q[0] * __uint_as_float(w); }
};
template <> struct Word<__nv_bfloat16> {
  static constexpr int N = 2;
  static __device__ __forceinline__ float dot(const float* q, unsigned w) {
    return fmaf(q[1], __uint_as_float(w & 0xffff0000u), q[0] * __uint_as_float(w << 16));
  }
};

template <typename T, int NR>
__global__ void __launch_bounds__(kLatWarps * 32)
latent_attention_kernel(const T* __restrict__ q_abs, int ld_qa, int hs_qa,     // [T, H, rank] absorbed plain part
                        const T* __restrict__ q_raw, int ld_q, int hs_q,        // rotated part before rotation, rot wide
                        const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len, int rdims,
                        const T* __restrict__ pages, const int* __restrict__ block_table, int max_pages,
                        int page_size, int num_pages, const int* __restrict__ positions,
                        const int* __restrict__ token_req, const float* __restrict__ sink, float scale, int window,
                        T* __restrict__ out, int ld_out, int hs_out, int H, int rank, int rot, int* status) {
  extern __shared__ unsigned lat_smem[];
  constexpr int EW = Word<T>::N;
  const int Dc = rank + rot;
  const int words = Dc / EW;
  const int stride = words | 1;                       // odd: lanes reading one column of a chunk hit 32 banks
  float* q_s = reinterpret_cast<float*>(lat_smem);    // [kLatWarps][Dc]
  unsigned* k_s = lat_smem + kLatWarps * Dc;          // [32][stride]
  __shared__ long long row_of[32];                    // element offset of each key's row, -1: not readable

  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * kLatWarps + warp;
  const bool live = h < H;
  const int pos = positions[t];
  const int* table = block_table + (size_t)token_req[t] * max_pages;
  const bool bad_pos = rdims > 0 && (pos < 0 || pos >= table_len);
  if (bad_pos && threadIdx.x == 0) atomicCAS(status, 0, KVB_STATUS_BAD_POSITION);

  if (live) {
    float* q = q_s + warp * Dc;
    for (int i = lane; i < rank; i += 32) q[i] = to_f32(q_abs[(size_t)t * ld_qa + (size_t)h * hs_qa + i]);
    const T* qr = q_raw + (size_t)t * ld_q + (size_t)h * hs_q;
    const int half = rdims >> 1;
    for (int i = lane; i < half; i += 32) {
      float c = 1.f, s = 0.f;
      if (!bad_pos) { c = cos_t[(size_t)pos * half + i]; s = sin_t[(size_t)pos * half + i]; }
      const float u = to_f32(qr[2 * i]), v = to_f32(qr[2 * i + 1]);
      q[rank + 2 * i] = u * c - v * s;
      q[rank + 2 * i + 1] = v * c + u * s;
    }
    for (int i = rdims + lane; i < rot; i += 32) q[rank + i] = to_f32(qr[i]);
  }
  float m = sink == nullptr ? -CUDART_INF_F : (live ? sink[h] : 0.f), l = sink == nullptr ? 0.f : 1.f;
  float acc[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) acc[r] = 0.f;

  const int lowest = window > 0 ? max(0, pos - window + 1) : 0;     // the first key the token sees
  for (int c0 = lowest & ~31; c0 <= pos; c0 += 32) {
    const int n_keys = min(32, pos - c0 + 1);
    __syncthreads();                                  // the chunk before is used up (and q_s is written)
    if (threadIdx.x < 32) {
      long long off = -1;
      if (threadIdx.x < n_keys && c0 + (int)threadIdx.x >= lowest) {
        const int j = c0 + threadIdx.x;
        const int lp = j / page_size;
        const int page = lp < max_pages ? table[lp] : -1;
        if (page < 0 || page >= num_pages) atomicCAS(status, 0, KVB_STATUS_UNMAPPED_PAGE);
        else off = ((long long)page * page_size + (j % page_size)) * Dc;
      }
      row_of[threadIdx.x] = off;
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < n_keys * words; idx += blockDim.x) {
      const int j = idx / words, w = idx - j * words;
      const long long off = row_of[j];
      k_s[j * stride + w] = off >= 0 ? reinterpret_cast<const unsigned*>(pages + off)[w] : 0u;
    }
    __syncthreads();
    if (!live) continue;
    const float* q = q_s + warp * Dc;
    float s = -CUDART_INF_F;
    if (lane < n_keys && row_of[lane] >= 0) {
      const unsigned* kr = k_s + lane * stride;
      float dot = 0.f;
      for (int w = 0; w < words; ++w) dot += Word<T>::dot(q + w * EW, kr[w]);
      s = dot * scale;
    }
    const float m_new = fmaxf(m, warp_max(s));
    if (m_new == -CUDART_INF_F) continue;              // no readable key yet, and no sink
    const float corr = expf(m - m_new);
    const float p = s == -CUDART_INF_F ? 0.f : expf(s - m_new);
    l = l * corr + warp_sum(p);
#pragma unroll
    for (int r = 0; r < NR; ++r) acc[r] *= corr;
    const T* kt = reinterpret_cast<const T*>(k_s);
    for (int j = 0; j < n_keys; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const T* vr = kt + (size_t)j * stride * EW;
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = r * 32 + lane;
        if (i < rank) acc[r] = fmaf(pj, to_f32(vr[i]), acc[r]);
      }
    }
    m = m_new;
  }
  if (!live) return;
  T* o = out + (size_t)t * ld_out + (size_t)h * hs_out;
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int i = r * 32 + lane;
    if (i < rank) o[i] = from_f32<T>(l > 0.f ? acc[r] / l : 0.f);
  }
}

template <typename T, int NR>
static int launch_latent(const void* q_abs, int ld_qa, int hs_qa, const void* q_raw, int ld_q, int hs_q,
                         const float* cos_t, const float* sin_t, int table_len, int rdims, const void* pages,
                         const int* block_table, int max_pages, int page_size, int num_pages, const int* positions,
                         const int* token_req, const float* sink, float scale, int window, void* out, int ld_out,
                         int hs_out, int T_, int H, int rank, int rot, int* status, cudaStream_t stream) {
  const int Dc = rank + rot;
  const int words = Dc / Word<T>::N;
  const size_t smem = ((size_t)kLatWarps * Dc + 32 * (size_t)(words | 1)) * 4;
  if (smem > 200 * 1024) return KVB_ERR_BAD_SIZE;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  kvb_launch(latent_attention_kernel<T, NR>, dim3(T_, (H + kLatWarps - 1) / kLatWarps), dim3(kLatWarps * 32), smem,
             stream, (const T*)q_abs, ld_qa, hs_qa, (const T*)q_raw, ld_q, hs_q, cos_t, sin_t, table_len, rdims,
             (const T*)pages, block_table, max_pages, page_size, num_pages, positions, token_req, sink, scale, window,
             (T*)out, ld_out, hs_out, H, rank, rot, status);
  return kvb_launch_result();
}

// window 0: every key up to the token's own.  Refuses: rank > 512; in bfloat16 an odd rank + rot or a cache that is not 4-byte aligned.
KVB_EXPORT int kvb_latent_attention(const void* q_abs, int ld_qa, int hs_qa, const void* q_raw, int ld_q, int hs_q,
                                    const float* cos_t, const float* sin_t, int table_len, int rdims,
                                    const void* pages, const int* block_table, int max_pages, int page_size,
                                    int num_pages, const int* positions, const int* token_req, const float* sink,
                                    float scale, int window, void* out, int ld_out, int hs_out, int T_, int H, int rank,
                                    int rot, int dtype, int* status, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (window < 0) return KVB_ERR_BAD_SIZE;
  if (rank < 1 || rank > 512 || rot < 0 || H < 1 || (rdims & 1) || rdims > rot) return KVB_ERR_BAD_SIZE;
  if (dtype == KVB_BF16 && ((rank + rot) & 1)) return KVB_ERR_BAD_SIZE;
  if (reinterpret_cast<uintptr_t>(pages) & 3) return KVB_ERR_ALIGN;
#define KVB_LATENT(NR)                                                                                              \
  KVB_DISPATCH_DTYPE(dtype, T, return (launch_latent<T, NR>(q_abs, ld_qa, hs_qa, q_raw, ld_q, hs_q, cos_t, sin_t,  \
                                                            table_len, rdims, pages, block_table, max_pages,       \
                                                            page_size, num_pages, positions, token_req, sink,      \
                                                            scale, window, out, ld_out, hs_out, T_, H, rank, rot,  \
                                                            status, stream)))
  if (rank <= 64) { KVB_LATENT(2); }
  else if (rank <= 128) { KVB_LATENT(4); }
  else if (rank <= 256) { KVB_LATENT(8); }
  else { KVB_LATENT(16); }
#undef KVB_LATENT
  return KVB_ERR_BAD_DTYPE;
}

// ---------------------------------------------------------------- the same attention on tensor cores (bfloat16)
// A block takes a tile of up to 64 rows, a row being one (token, head) pair: consecutive tokens
// of one request, all heads (at most 64 of them; more heads take further blocks along y).  Keys
// come in chunks of 32 by absolute position.  Per chunk: S = Q K^T by mma.sync m16n8k16 (each of
// the eight warps 16 rows x 16 keys over all of Dc), the scores go through shared memory to a
// softmax step of four threads per row (running maximum and sum start at the sink, as above;
// keys behind a row's own position are masked), the weights come back as bfloat16 and
// O += P V runs on the same chunk in shared memory, whose first `rank` columns are the values
// (each warp 16 rows x half of the value columns, accumulators in registers).  A row's result
// depends on its own query and on the chunks only, not on what else shares its tile.
constexpr int TC_ROWS = 64, TC_KEYS = 32, TC_THREADS = 256, TC_SPAD = 33, TC_PPAD = 40;

// NT: tiles of 8 value columns per warp at most (a warp owns half of the value columns): rank <= 16 NT.
template <int NT>
__global__ void __launch_bounds__(TC_THREADS, 1)
latent_attention_tc_kernel(const __nv_bfloat16* __restrict__ q_abs, int ld_qa, int hs_qa,
                           const __nv_bfloat16* __restrict__ q_raw, int ld_q, int hs_q,
                           const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len, int rdims,
                           const __nv_bfloat16* __restrict__ pages, const int* __restrict__ block_table, int max_pages,
                           int page_size, int num_pages, const int* __restrict__ positions,
                           const int* __restrict__ q_start, const int* __restrict__ tiles, int tokens_per_tile,
                           const float* __restrict__ sink, float scale, int window, __nv_bfloat16* __restrict__ out,
                           int ld_out, int hs_out, int H, int rank, int rot, int* status) {
  extern __shared__ uint4 tc_smem4[];
  const int Dc = rank + rot, DcP = Dc + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(tc_smem4);              // [64][DcP]
  __nv_bfloat16* Ks0 = Qs + TC_ROWS * DcP;                                      // two buffers of [32][DcP]
  __nv_bfloat16* Ps = Ks0 + 2 * TC_KEYS * DcP;                                  // [64][TC_PPAD]
  float* Ss = reinterpret_cast<float*>(Ps + TC_ROWS * TC_PPAD);                 // [64][TC_SPAD]
  float* m_s = Ss + TC_ROWS * TC_SPAD;
  float* l_s = m_s + TC_ROWS;
  float* corr_s = l_s + TC_ROWS;
  int* pos_s = reinterpret_cast<int*>(corr_s + TC_ROWS);
  __shared__ int row_ok[2][TC_KEYS];              // per buffer: whether the key's row could be read

  pdl_trigger();
  pdl_wait();
  int req, first, ntok;
  if (tiles != nullptr) {
    req = tiles[4 * blockIdx.x]; first = tiles[4 * blockIdx.x + 1]; ntok = tiles[4 * blockIdx.x + 2];
  } else {
    req = blockIdx.x; first = q_start[req]; ntok = q_start[req + 1] - first;
  }
  ntok = min(ntok, tokens_per_tile);
  const int h0 = blockIdx.y * TC_ROWS;
  const int HB = min(TC_ROWS, H - h0);
  const int rows_used = ntok * HB;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int* table = block_table + (size_t)req * max_pages;
  const int half = rdims >> 1;

  // the tile's queries: absorbed plain part as it is, the rotated part turned here
  for (int r = warp; r < TC_ROWS; r += TC_THREADS / 32) {
    __nv_bfloat16* q = Qs + (size_t)r * DcP;
    if (r >= rows_used) {
      for (int i = lane; i < DcP; i += 32) q[i] = __float2bfloat16_rn(0.f);
      if (lane == 0) { pos_s[r] = -1; m_s[r] = 0.f; l_s[r] = 1.f; }
      continue;
    }
    const int tl = r / HB, hh = h0 + r - tl * HB;
    const int tr = first + tl;
    const int pos = positions[tr];
    const bool bad_pos = rdims > 0 && (pos < 0 || pos >= table_len);
    if (bad_pos && lane == 0) atomicCAS(status, 0, KVB_STATUS_BAD_POSITION);
    const __nv_bfloat16* qa = q_abs + (size_t)tr * ld_qa + (size_t)hh * hs_qa;
    for (int i = lane; i < rank; i += 32) q[i] = qa[i];
    const __nv_bfloat16* qr = q_raw + (size_t)tr * ld_q + (size_t)hh * hs_q;
    for (int i = lane; i < half; i += 32) {
      float c = 1.f, sn = 0.f;
      if (!bad_pos) { c = cos_t[(size_t)pos * half + i]; sn = sin_t[(size_t)pos * half + i]; }
      const float u = __bfloat162float(qr[2 * i]), v = __bfloat162float(qr[2 * i + 1]);
      q[rank + 2 * i] = __float2bfloat16_rn(u * c - v * sn);
      q[rank + 2 * i + 1] = __float2bfloat16_rn(v * c + u * sn);
    }
    for (int i = rdims + lane; i < rot; i += 32) q[rank + i] = qr[i];
    for (int i = Dc + lane; i < DcP; i += 32) q[i] = __float2bfloat16_rn(0.f);
    if (lane == 0) {
      pos_s[r] = pos;
      m_s[r] = sink == nullptr ? -CUDART_INF_F : sink[hh];
      l_s[r] = sink == nullptr ? 0.f : 1.f;
    }
  }
  const int max_pos = ntok > 0 ? positions[first + ntok - 1] : -1;
  // the first key that any row of the tile sees; the chunk it lies in is the first one walked
  const int lowest = window > 0 && ntok > 0 ? max(0, positions[first] - window + 1) : 0;
  const int c_first = lowest / TC_KEYS * TC_KEYS;

  const int g = lane >> 2, t4 = lane & 3;
  const int mrow = (warp & 3) * 16;
  const int nt_used = rank / 16;                 // tiles of 8 columns in this warp's half of the values
  const int ncol0 = (warp >> 2) * (rank / 2);
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }

  // A chunk's rows are requested (cp.async, 16 bytes a piece) one chunk ahead, into the other buffer.
  const int vecs = Dc >> 3;                        // 16-byte pieces per row
  auto request_chunk = [&](int c0, int buf) {
    __nv_bfloat16* Kb = Ks0 + (size_t)buf * TC_KEYS * DcP;
    for (int j = warp; j < TC_KEYS; j += TC_THREADS / 32) {
      const int key = c0 + j;
      long long off = -1;
      if (key <= max_pos && key >= lowest) {
        const int lp = key / page_size;
        const int page = lp < max_pages ? table[lp] : -1;
        if (page < 0 || page >= num_pages) { if (lane == 0) atomicCAS(status, 0, KVB_STATUS_UNMAPPED_PAGE); }
        else off = ((long long)page * page_size + (key % page_size)) * Dc;
      }
      if (lane == 0) row_ok[buf][j] = off >= 0;
      __nv_bfloat16* dst = Kb + (size_t)j * DcP;
      if (off >= 0) {
        const __nv_bfloat16* src = pages + off;
        for (int v = lane; v < vecs; v += 32) {
          const unsigned d = (unsigned)__cvta_generic_to_shared(dst + 8 * v);
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"(d), "l"(src + 8 * v) : "memory");
        }
      } else {
        for (int v = lane; v < vecs; v += 32) reinterpret_cast<uint4*>(dst)[v] = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (max_pos >= 0) request_chunk(c_first, 0);
  const bool row_group_live = mrow < rows_used;   // a warp whose 16 rows are all empty only keeps the barriers
  int it = 0;
  for (int c0 = c_first; c0 <= max_pos; c0 += TC_KEYS, ++it) {
    const int n_keys = min(TC_KEYS, max_pos - c0 + 1);
    const __nv_bfloat16* Ks = Ks0 + (size_t)(it & 1) * TC_KEYS * DcP;
    const int* ok = row_ok[it & 1];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has arrived; the chunk before is used up (first round: Qs and the row state are written)
    if (c0 + TC_KEYS <= max_pos) request_chunk(c0 + TC_KEYS, (it + 1) & 1);
    // ---- scores: this warp's 16 rows against 16 of the chunk's keys
    if (row_group_live) {
      const int kcol = (warp >> 2) * 16;
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const __nv_bfloat16* a_ptr = Qs + (size_t)(mrow + (lane & 15)) * DcP + (lane >> 4) * 8;
      const __nv_bfloat16* b_ptr = Ks + (size_t)(kcol + ((lane >> 4) << 3) + (lane & 7)) * DcP + ((lane >> 3) & 1) * 8;
      // two sets of sums, for the even and the odd steps along Dc: four chains of dependent products instead
      // of two, and the operands of a pair of steps are fetched together (the same order for every row)
      float u0[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f};
      int ks = 0;
      for (; ks + 32 <= Dc; ks += 32) {
        unsigned a0, a1, a2, a3, b0, b1, b2, b3, c0_, c1_, c2_, c3_, d0, d1, d2, d3;
        ldsm_x4(a0, a1, a2, a3, a_ptr + ks);
        ldsm_x4(b0, b1, b2, b3, b_ptr + ks);
        ldsm_x4(c0_, c1_, c2_, c3_, a_ptr + ks + 16);
        ldsm_x4(d0, d1, d2, d3, b_ptr + ks + 16);
        mma_bf16_16816(s0, a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(s1, a0, a1, a2, a3, b2, b3);
        mma_bf16_16816(u0, c0_, c1_, c2_, c3_, d0, d1);
        mma_bf16_16816(u1, c0_, c1_, c2_, c3_, d2, d3);
      }
      if (ks < Dc) {
        unsigned a0, a1, a2, a3, b0, b1, b2, b3;
        ldsm_x4(a0, a1, a2, a3, a_ptr + ks);
        ldsm_x4(b0, b1, b2, b3, b_ptr + ks);
        mma_bf16_16816(s0, a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(s1, a0, a1, a2, a3, b2, b3);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) { s0[e] += u0[e]; s1[e] += u1[e]; }
      float* srow = Ss + (size_t)(mrow + g) * TC_SPAD + kcol + 2 * t4;
      srow[0] = s0[0] * scale; srow[1] = s0[1] * scale; srow[8] = s1[0] * scale; srow[9] = s1[1] * scale;
      srow += 8 * TC_SPAD;
      srow[0] = s0[2] * scale; srow[1] = s0[3] * scale; srow[8] = s1[2] * scale; srow[9] = s1[3] * scale;
    }
    __syncthreads();
    // ---- softmax step: four threads per row, eight keys each
    {
      const int row = tid >> 2, k0 = (tid & 3) * 8;
      const int pos_r = pos_s[row];
      const int low_r = window > 0 ? pos_r - window + 1 : 0;
      float sv[8], mx = -CUDART_INF_F;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int kk = k0 + e;
        const bool valid = kk < n_keys && c0 + kk <= pos_r && c0 + kk >= low_r && ok[kk];
        sv[e] = valid ? Ss[(size_t)row * TC_SPAD + kk] : -CUDART_INF_F;
        mx = fmaxf(mx, sv[e]);
      }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_old = m_s[row];
      const float m_new = fmaxf(m_old, mx);
      float psum = 0.f;
      __nv_bfloat16* prow = Ps + (size_t)row * TC_PPAD + k0;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float p = sv[e] == -CUDART_INF_F ? 0.f : expf(sv[e] - m_new);
        psum += p;
        prow[e] = __float2bfloat16_rn(p);
      }
      psum += __shfl_xor_sync(0xffffffffu, psum, 1);
      psum += __shfl_xor_sync(0xffffffffu, psum, 2);
      if ((tid & 3) == 0) {
        const float corr = m_old == m_new ? 1.f : expf(m_old - m_new);     // also where neither a key nor a sink was met yet
        m_s[row] = m_new;
        l_s[row] = l_s[row] * corr + psum;
        corr_s[row] = corr;
      }
    }
    __syncthreads();
    // ---- O = O * corr + P V for this warp's 16 rows and its half of the value columns
    if (row_group_live) {
      const float c_lo = corr_s[mrow + g], c_hi = corr_s[mrow + g + 8];
#pragma unroll
      for (int n = 0; n < NT; ++n) { acc[n][0] *= c_lo; acc[n][1] *= c_lo; acc[n][2] *= c_hi; acc[n][3] *= c_hi; }
      const __nv_bfloat16* a_ptr = Ps + (size_t)(mrow + (lane & 15)) * TC_PPAD + (lane >> 4) * 8;
      const __nv_bfloat16* b_ptr = Ks + (size_t)(((lane >> 3) & 1) * 8 + (lane & 7)) * DcP + ncol0 + (lane >> 4) * 8;
#pragma unroll
      for (int ks = 0; ks < TC_KEYS; ks += 16) {
        unsigned a0, a1, a2, a3;
        ldsm_x4(a0, a1, a2, a3, a_ptr + ks);
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          if (2 * np < nt_used) {              // an odd last tile takes a neighbour along whose sums nobody reads
            unsigned b0, b1, b2, b3;
            ldsm_x4_trans(b0, b1, b2, b3, b_ptr + (size_t)ks * DcP + np * 16);
            mma_bf16_16816(acc[2 * np], a0, a1, a2, a3, b0, b1);
            mma_bf16_16816(acc[2 * np + 1], a0, a1, a2, a3, b2, b3);
          }
        }
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int hrow = 0; hrow < 2; ++hrow) {
    const int r = mrow + g + 8 * hrow;
    if (r >= rows_used) continue;
    const int tl = r / HB, hh = h0 + r - tl * HB;
    const float inv = l_s[r] > 0.f ? 1.0f / l_s[r] : 0.f;
    __nv_bfloat16* o = out + (size_t)(first + tl) * ld_out + (size_t)hh * hs_out + ncol0 + 2 * t4;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      if (n < nt_used) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(acc[n][2 * hrow] * inv, acc[n][2 * hrow + 1] * inv);
        *reinterpret_cast<__nv_bfloat162*>(o + n * 8) = v;
      }
    }
  }
}

// Rows of (token, head) pairs per tile: tokens per tile for a number of heads.
KVB_EXPORT int kvb_latent_attention_tc_tokens_per_tile(int H) { return H >= TC_ROWS ? 1 : TC_ROWS / H; }

// Whether the tensor-core form takes these sizes: rank and rank + rot multiples of 16, rank up to 512.
KVB_EXPORT int kvb_latent_attention_tc_supported(int rank, int rot) {
  return rank >= 16 && rank <= 512 && rank % 16 == 0 && (rank + rot) % 16 == 0 ? 1 : 0;
}

template <int NT>
static int launch_latent_tc(const void* q_abs, int ld_qa, int hs_qa, const void* q_raw, int ld_q, int hs_q,
                            const float* cos_t, const float* sin_t, int table_len, int rdims, const void* pages,
                            const int* block_table, int max_pages, int page_size, int num_pages, const int* positions,
                            const int* q_start, const int* tiles, int n_tiles, const float* sink, float scale, int window,
                            void* out, int ld_out, int hs_out, int H, int rank, int rot, int* status, cudaStream_t stream) {
  const int DcP = rank + rot + 8;
  const size_t smem = (size_t)(TC_ROWS + 2 * TC_KEYS) * DcP * 2 + (size_t)TC_ROWS * TC_PPAD * 2 +
                      (size_t)TC_ROWS * TC_SPAD * 4 + 4 * TC_ROWS * 4;
  if (smem > 220 * 1024) return KVB_ERR_BAD_SIZE;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_tc_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  using B = __nv_bfloat16;
  kvb_launch(latent_attention_tc_kernel<NT>, dim3(n_tiles, (H + TC_ROWS - 1) / TC_ROWS), dim3(TC_THREADS), smem, stream,
             (const B*)q_abs, ld_qa, hs_qa, (const B*)q_raw, ld_q, hs_q, cos_t, sin_t, table_len, rdims, (const B*)pages,
             block_table, max_pages, page_size, num_pages, positions, q_start, tiles,
             kvb_latent_attention_tc_tokens_per_tile(H), sink, scale, window, (B*)out, ld_out, hs_out, H, rank, rot, status);
  return kvb_launch_result();
}

// tiles: [n_tiles, 4] int32 rows (request row, first token row, tokens, 0) of at most
// kvb_latent_attention_tc_tokens_per_tile(H) tokens each, or null: one tile per request (n_tiles requests, each
// bringing at most that many tokens).  Everything 16-byte aligned: the cache, and rows of rank + rot elements.
KVB_EXPORT int kvb_latent_attention_tc(const void* q_abs, int ld_qa, int hs_qa, const void* q_raw, int ld_q, int hs_q,
                                       const float* cos_t, const float* sin_t, int table_len, int rdims,
                                       const void* pages, const int* block_table, int max_pages, int page_size,
                                       int num_pages, const int* positions, const int* q_start, const int* tiles,
                                       int n_tiles, const float* sink, float scale, int window, void* out, int ld_out,
                                       int hs_out, int H, int rank, int rot, int* status, cudaStream_t stream) {
  if (n_tiles <= 0) return 0;
  if (window < 0) return KVB_ERR_BAD_SIZE;
  if (!kvb_latent_attention_tc_supported(rank, rot) || H < 1 || (rdims & 1) || rdims > rot) return KVB_ERR_BAD_SIZE;
  if ((reinterpret_cast<uintptr_t>(pages) & 15) || (reinterpret_cast<uintptr_t>(out) & 3) || (ld_out & 1) || (hs_out & 1))
    return KVB_ERR_ALIGN;
#define KVB_LATENT_TC(NT)                                                                                            \
  return launch_latent_tc<NT>(q_abs, ld_qa, hs_qa, q_raw, ld_q, hs_q, cos_t, sin_t, table_len, rdims, pages,        \
                              block_table, max_pages, page_size, num_pages, positions, q_start, tiles, n_tiles, sink, \
                              scale, window, out, ld_out, hs_out, H, rank, rot, status, stream)
  if (rank <= 64) { KVB_LATENT_TC(4); }
  if (rank <= 128) { KVB_LATENT_TC(8); }
  if (rank <= 256) { KVB_LATENT_TC(16); }
  KVB_LATENT_TC(32);
#undef KVB_LATENT_TC
}

// ---------------------------------------------------------------- single tokens: a request's keys dealt over a cluster
// A step of single tokens has few rows per request (its heads) and many cached rows: a cluster of S blocks takes one
// request and up to 16 heads, block s the chunks of 64 keys s, s + S, ... (chunks by absolute position, the first one that
// the window reaches first).  Per chunk: S = Q K^T by mma.sync (each of the sixteen warps 16 heads x 8 keys over half of
// Dc), a softmax step of one head per warp (running maximum and sum), O += P V (each warp 16 heads x its pairs of
// 8 value columns).  A row is one bulk copy (cp.async.bulk) that counts its bytes on the buffer's barrier, requested one
// chunk ahead.  Then the blocks tell each other their maxima and sums, every block scales its sums and hands each other
// block the columns that one writes out; the sink joins there.
constexpr int LD_KEYS = 64, LD_WARPS = 16, LD_THREADS = LD_WARPS * 32, LD_SPAD = 68, LD_PPAD = 72;
constexpr unsigned LD_SPINS = 1u << 20;      // polls of a barrier before a block gives up

__device__ __forceinline__ bool ld_wait(unsigned long long* bar, unsigned parity) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(bar);
  for (unsigned i = 0; i < LD_SPINS; ++i) {
    unsigned ok;
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.b32 %0, 1, 0, p;\n\t}"
                 : "=r"(ok) : "r"(addr), "r"(parity) : "memory");
    if (ok) return true;
  }
  return false;
}

struct LatentDecodeArgs {
  const __nv_bfloat16* q_abs; int ld_qa, hs_qa;
  const __nv_bfloat16* q_raw; int ld_q, hs_q;
  const float* cos_t; const float* sin_t; int table_len, rdims;
  const __nv_bfloat16* pages; const int* block_table; int max_pages, page_size, page_shift, num_pages;      // page_shift: -1 where the size is no power of two
  const int* positions; const int* q_start;
  const float* sink; float scale; int window;
  __nv_bfloat16* out; int ld_out, hs_out, H, rank, rot;
  int* status;
};

// NP: pairs of 8 value columns per warp at most: rank <= 256 NP.
template <int NP>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(LatentDecodeArgs p) {
  extern __shared__ uint4 ld_smem4[];
  const int Dc = p.rank + p.rot, DcP = Dc + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(ld_smem4);              // [16][DcP]
  __nv_bfloat16* Ks0 = Qs + 16 * DcP;                                           // two buffers of [64][DcP]
  __nv_bfloat16* Ps = Ks0 + 2 * LD_KEYS * DcP;                                  // [16][LD_PPAD]
  float* Ss = reinterpret_cast<float*>(Ps + 16 * LD_PPAD);                      // [2][16][LD_SPAD]: the halves of Dc
  float* merged = reinterpret_cast<float*>(Ks0);                                // [S][own pairs][16][16], once the keys are done with
  __shared__ float m_s[16], l_s[16], corr_s[16];
  __shared__ float all_m[8 * 16], all_l[8 * 16];                                // of every block of the cluster
  __shared__ int row_ok[2][LD_KEYS];
  __shared__ __align__(8) unsigned long long full[2];                           // a buffer's rows have arrived
  const int S = gridDim.z, part = blockIdx.z;                                   // the cluster lies along z
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_trigger();
  if (tid < 2) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" :: "r"((unsigned)__cvta_generic_to_shared(full + tid)), "r"(LD_WARPS));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (S > 1) cluster_meet();                       // every block of the cluster runs before another writes into it
  else __syncthreads();
  pdl_wait();
  const int req = blockIdx.x, h0 = blockIdx.y * 16, HB = min(16, p.H - h0);
  const int tr = p.q_start[req], pos = p.positions[tr];
  const int* table = p.block_table + (size_t)req * p.max_pages;
  const int lowest = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int first = lowest / LD_KEYS + part, last = pos >= 0 ? pos / LD_KEYS : -1;      // this block's chunks: first, first + S, ...
  const int half = p.rdims >> 1;
  const unsigned row_bytes = (unsigned)Dc * 2u;

  // a warp brings four rows, a lane each
  auto request_chunk = [&](int c, int buf) {
    const int slot = warp * 4 + (lane & 3), key = c * LD_KEYS + slot;
    long long row = -1;
    if (lane < 4 && key >= lowest && key <= pos) {
      const int lp = p.page_shift >= 0 ? key >> p.page_shift : key / p.page_size;
      const int page = lp < p.max_pages ? table[lp] : -1;
      if (page < 0 || page >= p.num_pages) atomicCAS(p.status, 0, KVB_STATUS_UNMAPPED_PAGE);
      else row = (long long)page * p.page_size + (key - lp * p.page_size);
    }
    const unsigned here = __ballot_sync(0xffffffffu, row >= 0);
    __nv_bfloat16* Kb = Ks0 + (size_t)buf * LD_KEYS * DcP;
    const unsigned bar = (unsigned)__cvta_generic_to_shared(full + buf);
    if (lane < 4) row_ok[buf][slot] = row >= 0;
    if (lane == 0)
      asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" :: "r"(bar), "r"(__popc(here) * row_bytes) : "memory");
    __syncwarp();
    if (row >= 0)
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                   :: "r"((unsigned)__cvta_generic_to_shared(Kb + (size_t)slot * DcP)), "l"(p.pages + row * Dc), "r"(row_bytes), "r"(bar)
                   : "memory");
    if (here != 0xfu) {                            // keys that are not there: zeros (at the ends of the window only)
      for (int r = 0; r < 4; ++r)
        if (!((here >> r) & 1u))
          for (int v = lane; v < Dc / 8; v += 32) reinterpret_cast<uint4*>(Kb + (size_t)(warp * 4 + r) * DcP)[v] = make_uint4(0u, 0u, 0u, 0u);
    }
  };
  if (first <= last) request_chunk(first, 0);

  // the heads' queries: absorbed plain part as it is, the rotated part turned here; a row a warp
  const bool bad_pos = p.rdims > 0 && (pos < 0 || pos >= p.table_len);
  if (bad_pos && tid == 0) atomicCAS(p.status, 0, KVB_STATUS_BAD_POSITION);
  {
    __nv_bfloat16* q = Qs + (size_t)warp * DcP;
    if (warp >= HB) {
      for (int i = lane; i < DcP; i += 32) q[i] = __float2bfloat16_rn(0.f);
    } else {
      const __nv_bfloat16* qa = p.q_abs + (size_t)tr * p.ld_qa + (size_t)(h0 + warp) * p.hs_qa;
      for (int i = lane; i < p.rank / 8; i += 32) reinterpret_cast<uint4*>(q)[i] = reinterpret_cast<const uint4*>(qa)[i];
      const __nv_bfloat16* qr = p.q_raw + (size_t)tr * p.ld_q + (size_t)(h0 + warp) * p.hs_q;
      for (int i = lane; i < half; i += 32) {
        float c = 1.f, sn = 0.f;
        if (!bad_pos) { c = p.cos_t[(size_t)pos * half + i]; sn = p.sin_t[(size_t)pos * half + i]; }
        const float u = __bfloat162float(qr[2 * i]), v = __bfloat162float(qr[2 * i + 1]);
        q[p.rank + 2 * i] = __float2bfloat16_rn(u * c - v * sn);
        q[p.rank + 2 * i + 1] = __float2bfloat16_rn(v * c + u * sn);
      }
      for (int i = p.rdims + lane; i < p.rot; i += 32) q[p.rank + i] = qr[i];
    }
    if (lane == 0) { m_s[warp] = -CUDART_INF_F; l_s[warp] = 0.f; }
  }
  const int g = lane >> 2, t4 = lane & 3, n_pairs = p.rank / 16;
  const int steps = Dc / 16, k_from = (warp >> 3) ? (steps + 1) / 2 * 16 : 0, k_to = (warp >> 3) ? Dc : (steps + 1) / 2 * 16;
  float acc[NP][2][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][0][e] = acc[i][1][e] = 0.f;

  bool arrived = true;
  int it = 0;
  for (int c = first; c <= last; c += S, ++it) {
    const int buf = it & 1;
    const __nv_bfloat16* Ks = Ks0 + (size_t)buf * LD_KEYS * DcP;
    __syncthreads();                               // the chunk before is used up (first round: Qs and the row state are written)
    if (c + S <= last) request_chunk(c + S, buf ^ 1);
    arrived = ld_wait(full + buf, (unsigned)(it >> 1) & 1u) && arrived;
    {
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const __nv_bfloat16* a_ptr = Qs + (size_t)(lane & 15) * DcP + (lane >> 4) * 8;
      const __nv_bfloat16* b_row = Ks + (size_t)((warp & 7) * 8 + (lane & 7)) * DcP;
      int ks = k_from;
#pragma unroll 4
      for (; ks + 32 <= k_to; ks += 32) {
        unsigned a0, a1, a2, a3, e0, e1, e2, e3, b0, b1, b2, b3;
        ldsm_x4(a0, a1, a2, a3, a_ptr + ks);
        ldsm_x4(e0, e1, e2, e3, a_ptr + ks + 16);
        ldsm_x4(b0, b1, b2, b3, b_row + ks + (lane >> 3) * 8);
        mma_bf16_16816(s0, a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(s1, e0, e1, e2, e3, b2, b3);
      }
      if (ks < k_to) {
        unsigned a0, a1, a2, a3, b0, b1, b2, b3;
        ldsm_x4(a0, a1, a2, a3, a_ptr + ks);
        ldsm_x4(b0, b1, b2, b3, b_row + ks + ((lane >> 3) & 1) * 8);
        mma_bf16_16816(s0, a0, a1, a2, a3, b0, b1);
      }
      float* srow = Ss + ((warp >> 3) * 16 + g) * LD_SPAD + (warp & 7) * 8 + 2 * t4;
      *reinterpret_cast<float2*>(srow) = make_float2(s0[0] + s1[0], s0[1] + s1[1]);
      *reinterpret_cast<float2*>(srow + 8 * LD_SPAD) = make_float2(s0[2] + s1[2], s0[3] + s1[3]);
    }
    __syncthreads();
    {
      const float* s = Ss + warp * LD_SPAD + lane;
      const float a = row_ok[buf][lane] ? (s[0] + s[16 * LD_SPAD]) * p.scale : -CUDART_INF_F;
      const float b = row_ok[buf][lane + 32] ? (s[32] + s[16 * LD_SPAD + 32]) * p.scale : -CUDART_INF_F;
      const float m_old = m_s[warp], m_new = fmaxf(m_old, warp_max(fmaxf(a, b)));
      const float pa = a == -CUDART_INF_F ? 0.f : expf(a - m_new), pb = b == -CUDART_INF_F ? 0.f : expf(b - m_new);
      Ps[warp * LD_PPAD + lane] = __float2bfloat16_rn(pa);
      Ps[warp * LD_PPAD + lane + 32] = __float2bfloat16_rn(pb);
      const float sum = warp_sum(pa + pb);
      if (lane == 0) {
        const float corr = m_old == m_new ? 1.f : expf(m_old - m_new);
        m_s[warp] = m_new;
        l_s[warp] = l_s[warp] * corr + sum;
        corr_s[warp] = corr;
      }
    }
    __syncthreads();
    const float c_lo = corr_s[g], c_hi = corr_s[g + 8];
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        acc[i][u][0] *= c_lo; acc[i][u][1] *= c_lo; acc[i][u][2] *= c_hi; acc[i][u][3] *= c_hi;
      }
#pragma unroll
    for (int kk = 0; kk < LD_KEYS; kk += 16) {
      unsigned a0, a1, a2, a3;
      ldsm_x4(a0, a1, a2, a3, Ps + (size_t)(lane & 15) * LD_PPAD + (lane >> 4) * 8 + kk);
      const __nv_bfloat16* b_row = Ks + (size_t)(kk + ((lane >> 3) & 1) * 8 + (lane & 7)) * DcP + (lane >> 4) * 8;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int pair = warp + LD_WARPS * i;
        if (pair < n_pairs) {
          unsigned b0, b1, b2, b3;
          ldsm_x4_trans(b0, b1, b2, b3, b_row + pair * 16);
          mma_bf16_16816(acc[i][0], a0, a1, a2, a3, b0, b1);
          mma_bf16_16816(acc[i][1], a0, a1, a2, a3, b2, b3);
        }
      }
    }
  }
  if (!arrived) {                                  // copies that may still run must not meet the block's end
    if (lane == 0) atomicCAS(p.status, 0, KVB_STATUS_WAIT_TIMEOUT);
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);
  }
  __syncthreads();
  // ---- the blocks' maxima and sums
  if (S > 1) {
    if (tid < 16 * S) {
      const int to = tid >> 4, r = tid & 15;
      store_in_block(all_m + part * 16 + r, to, m_s[r]);
      store_in_block(all_l + part * 16 + r, to, l_s[r]);
    }
    cluster_meet();                                // and every block is done with its keys
  } else {
    if (tid < 16) { all_m[tid] = m_s[tid]; all_l[tid] = l_s[tid]; }
    __syncthreads();
  }
  float f[2];                                      // what this block's sums of heads g and g + 8 are multiplied by
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int r = g + 8 * u;
    const float sink = p.sink != nullptr && r < HB ? p.sink[h0 + r] : -CUDART_INF_F;
    float m = sink;
    for (int s = 0; s < S; ++s) m = fmaxf(m, all_m[s * 16 + r]);
    float l = 0.f;
    if (m != -CUDART_INF_F) {
      l = sink == -CUDART_INF_F ? 0.f : expf(sink - m);
      for (int s = 0; s < S; ++s)
        if (all_m[s * 16 + r] != -CUDART_INF_F) l += all_l[s * 16 + r] * expf(all_m[s * 16 + r] - m);
    }
    const float own = all_m[part * 16 + r];
    f[u] = own != -CUDART_INF_F && l > 0.f ? expf(own - m) / l : 0.f;
  }
  __nv_bfloat16* out = p.out + (size_t)tr * p.ld_out + (size_t)h0 * p.hs_out;
  if (S == 1) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int pair = warp + LD_WARPS * i;
      if (pair >= n_pairs) continue;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int hi = 0; hi < 2; ++hi) {
          const int r = g + 8 * hi;
          if (r < HB)
            *reinterpret_cast<__nv_bfloat162*>(out + (size_t)r * p.hs_out + pair * 16 + u * 8 + 2 * t4) =
                __floats2bfloat162_rn(acc[i][u][2 * hi] * f[hi], acc[i][u][2 * hi + 1] * f[hi]);
        }
    }
    return;
  }
  // ---- pair q of the columns is written out by block q mod S: everybody hands it the (scaled) sums
  const int own_pairs = (n_pairs + S - 1) / S;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int pair = warp + LD_WARPS * i;
    if (pair >= n_pairs) continue;
    float* to = merged + ((size_t)part * own_pairs + pair / S) * 256 + g * 16 + 2 * t4;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      store2_in_block(to + u * 8, pair % S, acc[i][u][0] * f[0], acc[i][u][1] * f[0]);
      store2_in_block(to + 128 + u * 8, pair % S, acc[i][u][2] * f[1], acc[i][u][3] * f[1]);
    }
  }
  cluster_meet();                                  // the last time anything is written into another block
  for (int i = tid; i < own_pairs * 128; i += LD_THREADS) {
    const int lp = i >> 7, r = (i >> 3) & 15, col = (i & 7) * 2, pair = lp * S + part;
    if (pair >= n_pairs || r >= HB) continue;
    float a = 0.f, b = 0.f;
    for (int s = 0; s < S; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(merged + ((size_t)s * own_pairs + lp) * 256 + r * 16 + col);
      a += v.x;
      b += v.y;
    }
    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)r * p.hs_out + pair * 16 + col) = __floats2bfloat162_rn(a, b);
  }
}

static size_t latent_decode_smem(int Dc) {
  return (size_t)(16 + 2 * LD_KEYS) * (Dc + 8) * 2 + 16 * LD_PPAD * 2 + 32 * LD_SPAD * 4;
}

// Whether the form for single tokens takes these sizes: those of the tensor-core form whose chunks fit shared memory.
KVB_EXPORT int kvb_latent_decode_supported(int rank, int rot) {
  return kvb_latent_attention_tc_supported(rank, rot) && latent_decode_smem(rank + rot) <= 220 * 1024 ? 1 : 0;
}

// n_reqs requests, each with one token: row q_start[r] of the queries, the positions and the result.  max_keys: the most keys
// that one of them may see (what the launch is sized by; any number is right).  The rest as for kvb_latent_attention_tc.
KVB_EXPORT int kvb_latent_decode(const void* q_abs, int ld_qa, int hs_qa, const void* q_raw, int ld_q, int hs_q,
                                 const float* cos_t, const float* sin_t, int table_len, int rdims, const void* pages,
                                 const int* block_table, int max_pages, int page_size, int num_pages, const int* positions,
                                 const int* q_start, int n_reqs, int max_keys, const float* sink, float scale, int window,
                                 void* out, int ld_out, int hs_out, int H, int rank, int rot, int* status,
                                 cudaStream_t stream) {
  if (n_reqs <= 0) return 0;
  if (!kvb_latent_decode_supported(rank, rot) || H < 1 || (rdims & 1) || rdims > rot || window < 0 || (H + 15) / 16 > 65535)
    return KVB_ERR_BAD_SIZE;
  if (((reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(q_abs)) & 15) || ((ld_qa | hs_qa) & 7) ||
      (reinterpret_cast<uintptr_t>(out) & 3) || (ld_out & 1) || (hs_out & 1))
    return KVB_ERR_ALIGN;
  using B = __nv_bfloat16;
  int page_shift = 0;
  while ((1 << page_shift) < page_size) ++page_shift;
  if ((1 << page_shift) != page_size) page_shift = -1;
  const LatentDecodeArgs a{(const B*)q_abs, ld_qa, hs_qa, (const B*)q_raw, ld_q, hs_q, cos_t, sin_t, table_len, rdims,
                           (const B*)pages, block_table, max_pages, page_size, page_shift, num_pages, positions, q_start, sink, scale,
                           window, (B*)out, ld_out, hs_out, H, rank, rot, status};
  const size_t smem = latent_decode_smem(rank + rot);
  const int tiles = (H + 15) / 16, chunks = (max_keys + LD_KEYS - 1) / LD_KEYS;
  int S = 1;                          // blocks per request: as many as find an SM of their own and a chunk to take
  while (S < 8 && n_reqs * tiles * 2 * S <= kvb_sm_count() && 2 * S <= chunks) S *= 2;
  const dim3 grid(n_reqs, tiles, S);
#define KVB_LATENT_DECODE(NP)                                                                                           \
  do {                                                                                                                  \
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e != cudaSuccess) return (int)e;                                                                                \
    if (S > 1) e = kvb_launch_cluster(latent_decode_kernel<NP>, grid, dim3(LD_THREADS), dim3(1, 1, S), smem, stream, a); \
    else e = kvb_launch(latent_decode_kernel<NP>, grid, dim3(LD_THREADS), smem, stream, a);                             \
    return e != cudaSuccess ? (int)e : kvb_launch_result();                                                             \
  } while (0)
  if (rank <= 256) KVB_LATENT_DECODE(1);
  KVB_LATENT_DECODE(2);
#undef KVB_LATENT_DECODE
}
