// A layer's own input from each token: a row of a table (the layer's slice of the token's row), gated by the
// residual stream, brought to the model's width, normed and added to the stream:
//   y = W_p (gelu_tanh(W_g x) * e),   x <- x + y / sqrt(mean(y^2) + eps) * w
//
//   * token_gate_kernel: for steps whose two products are made by the step's matrix product kernels: the middle,
//     a[t, j] = gelu_tanh(p[t, j]) * table[token, first + j].
//   * token_input_step_kernel: for steps of few tokens: all of it in one launch, the norm and the addition of the
//     branch that is still pending in front of it included.
#include "cluster.cuh"
#include "common.cuh"

__device__ __forceinline__ float gelu_tanh(float z) {
  const float c = 0.7978845608028654f;   // sqrt(2 / pi)
  return 0.5f * z * (1.0f + tanhf(c * (z + 0.044715f * z * z * z)));
}

// The token's id: ids[t], or, below zero, the one that the sampling kernel of the step before left in row -(id + 1).
// -1 where neither names a row of the table.
__device__ __forceinline__ int token_of(const int* ids, const int* sampled, int n_sampled, int t, int V) {
  int id = ids[t];
  if (id < 0 && sampled != nullptr && -(id + 1) < n_sampled) id = sampled[-(id + 1)];
  return id < 0 || id >= V ? -1 : id;
}

template <typename T>
__global__ void __launch_bounds__(256)
token_gate_kernel(const T* __restrict__ p, int ld_p, const T* __restrict__ table, int ld_table, int first, int V,
                  const int* __restrict__ ids, const int* __restrict__ sampled, int n_sampled, T* __restrict__ out, int n,
                  int ld_out, size_t total, int* status) {
  pdl_trigger();
  pdl_wait();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(idx / ld_out), j = (int)(idx - (size_t)t * ld_out);
    float a = 0.f;
    if (j < n) {
      const int id = token_of(ids, sampled, n_sampled, t, V);
      if (id < 0) atomicCAS(status, 0, KVB_STATUS_BAD_TOKEN);
      else a = gelu_tanh(to_f32(p[(size_t)t * ld_p + j])) * to_f32(table[(size_t)id * ld_table + first + j]);
    }
    out[idx] = from_f32<T>(a);
  }
}

// p [T, >= n] with row stride ld_p; table [V, ld_table], of which columns first .. first + n - 1 are read;
// out [T, ld_out] dense, the columns behind n zero.
KVB_EXPORT int kvb_token_gate(const void* p, int ld_p, const void* table, int ld_table, int first, int V, const int* ids,
                              const int* sampled, int n_sampled, void* out, int T_, int n, int ld_out, int dtype,
                              int* status, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (n < 1 || ld_out < n || first < 0 || first + n > ld_table || ld_p < n) return KVB_ERR_BAD_SIZE;
  const size_t total = (size_t)T_ * ld_out;
  const size_t want = (total + 255) / 256;
  const int blocks = (int)(want < (size_t)kvb_sm_count() * 16 ? want : (size_t)kvb_sm_count() * 16);
  KVB_DISPATCH_DTYPE(dtype, T, (kvb_launch(token_gate_kernel<T>, dim3(blocks), dim3(256), 0, stream, (const T*)p, ld_p,
                                            (const T*)table, ld_table, first, V, ids, sampled, n_sampled, (T*)out, n,
                                            ld_out, total, status)));
  return kvb_launch_result();
}

// ---------------------------------------------------------------- the whole branch in one launch
// A cluster of kStepBlocks blocks takes NT tokens.  Block r owns columns [c0, c1) of the stream, for the rows of x, for
// the columns of W_g and for the rows of W_p alike, so the stream itself never leaves its block; what crosses the
// cluster (written into every block's shared memory, then one hardware barrier) is three sets of partial sums: the
// squares of the pending branch output, the products W_g x, and the squares of y.  A step of few tokens is bound by
// bringing the weights, which are read once per cluster; their lines are requested into L2 before the kernel waits for
// its predecessor.  This form, for float32, does both products with plain FMAs.
// Every sum is taken in an order that depends on the sizes only.
constexpr int kStepBlocks = 8, kStepThreads = 256, kStepWarps = kStepThreads / 32;

template <typename T> struct Piece;      // 16 bytes of a row
template <> struct Piece<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void open(const uint4& u, float* f) {
    f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
  }
};
template <> struct Piece<__nv_bfloat16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void open(const uint4& u, float* f) {
    const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
  }
};

// acc[n] = row . v[n] for NT vectors of shared memory (stride ldv): the `lanes` lanes of a group share the row, each its
// pieces of 16 bytes; the group's sums are added across it, so that all of its lanes hold them.
template <typename T, int NT>
__device__ __forceinline__ void group_dots(const T* row, const float* v, int ldv, int n_cols, int lane, int lanes, bool live,
                                           float (&acc)[NT]) {
  constexpr int N = Piece<T>::N;
#pragma unroll
  for (int n = 0; n < NT; ++n) acc[n] = 0.f;
  if (live) {
#pragma unroll 4
    for (int c = lane * N; c < n_cols; c += lanes * N) {
      float w[N];
      Piece<T>::open(*reinterpret_cast<const uint4*>(row + c), w);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float* x = v + n * ldv + c;
#pragma unroll
        for (int i = 0; i < N; i += 4) {
          const float4 f = *reinterpret_cast<const float4*>(x + i);
          acc[n] = fmaf(w[i], f.x, acc[n]);
          acc[n] = fmaf(w[i + 1], f.y, acc[n]);
          acc[n] = fmaf(w[i + 2], f.z, acc[n]);
          acc[n] = fmaf(w[i + 3], f.w, acc[n]);
        }
      }
    }
  }
  for (int o = lanes >> 1; o > 0; o >>= 1)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[n] += __shfl_xor_sync(0xffffffffu, acc[n], o);
}

// The sum of v[n] over the block for NT values at once, into every block's `slots` [kStepBlocks][NT] at this block's place.
template <int NT>
__device__ __forceinline__ void share_sums(const float (&v)[NT], float* part, float* slots, int rank) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const float s = warp_sum(v[n]);
    if (lane == 0) part[warp * NT + n] = s;
  }
  __syncthreads();
  if (threadIdx.x < NT * kStepBlocks) {
    const int n = threadIdx.x % NT, to = threadIdx.x / NT;
    float s = 0.f;
    for (int w = 0; w < kStepWarps; ++w) s += part[w * NT + n];
    store_in_block(slots + rank * NT + n, to, s);
  }
}

// delta null: nothing is pending; post_w null: delta joins as it is, else x = resid + delta / rms(delta) * post_w.
template <typename T, int NT>
__global__ void __launch_bounds__(kStepThreads)
token_input_step_kernel(float* __restrict__ resid, const T* __restrict__ delta, const float* __restrict__ post_w, float post_eps,
                        const T* __restrict__ w_gate, const T* __restrict__ w_proj, const float* __restrict__ norm_w,
                        float eps, const T* __restrict__ table, int ld_table, int first, int V, const int* __restrict__ ids,
                        const int* __restrict__ sampled, int n_sampled, T* __restrict__ out, int T_, int W, int dim, int dim_p,
                        int slice, int* status) {
  extern __shared__ float4 step_smem[];
  float* xs = reinterpret_cast<float*>(step_smem);      // [NT][slice] the stream, as the product reads it
  float* act = xs + NT * slice;                         // [NT][dim_p]
  float* sums = act + NT * dim_p;                       // [kStepBlocks][NT][dim] every block's share of W_g x
  float* ys = sums + kStepBlocks * NT * dim;            // [NT][slice]
  float* rs = ys + NT * slice;                          // [NT][slice] the float32 stream
  __shared__ float part[kStepWarps * NT];
  __shared__ float sq_pending[kStepBlocks * NT], sq_y[kStepBlocks * NT];
  __shared__ int token[NT];
  constexpr int N = Piece<T>::N;
  pdl_trigger();
  const int rank = blockIdx.x % kStepBlocks, t0 = blockIdx.x / kStepBlocks * NT;      // the cluster is kStepBlocks neighbours along x
  const int tid = threadIdx.x;
  const int n_tok = min(NT, T_ - t0);
  const int c0 = min(W, rank * slice), c1 = min(W, c0 + slice), nc = c1 - c0;
  if (t0 == 0) {       // the weights do not depend on what runs before: the first cluster asks for their lines
    constexpr int line = 128 / (int)sizeof(T);
    for (int i = tid; i < dim * ((nc + line - 1) / line); i += kStepThreads) {
      const int per = (nc + line - 1) / line, j = i / per;
      asm volatile("prefetch.global.L2 [%0];" ::"l"(w_gate + (size_t)j * W + c0 + (i - j * per) * line));
    }
    for (int i = tid * line; i < nc * dim_p; i += kStepThreads * line)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(w_proj + (size_t)c0 * dim_p + i));
  }
  cluster_meet();                                         // every block of the cluster runs before another writes into it
  pdl_wait();
  // ---- the stream, brought up to date
  float v[NT];
  if (delta != nullptr && post_w != nullptr) {
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      v[n] = 0.f;
      if (n < n_tok)
        for (int i = tid; i < nc; i += kStepThreads) {
          const float d = to_f32(delta[(size_t)(t0 + n) * W + c0 + i]);
          v[n] = fmaf(d, d, v[n]);
        }
    }
    share_sums<NT>(v, part, sq_pending, rank);
  }
  if (tid < NT) {
    int id = -1;
    if (tid < n_tok) {
      id = token_of(ids, sampled, n_sampled, t0 + tid, V);
      if (id < 0 && rank == 0) atomicCAS(status, 0, KVB_STATUS_BAD_TOKEN);
    }
    token[tid] = id;
  }
  cluster_meet();
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    float f = 1.f;
    if (delta != nullptr && post_w != nullptr) {
      float s = 0.f;
      for (int b = 0; b < kStepBlocks; ++b) s += sq_pending[b * NT + n];
      f = 1.0f / sqrtf(s / (float)W + post_eps);
    }
    for (int i = tid; i < slice; i += kStepThreads) {
      float x = 0.f;
      if (n < n_tok && i < nc) {
        const size_t at = (size_t)(t0 + n) * W + c0 + i;
        x = resid[at];
        if (delta != nullptr) x += to_f32(delta[at]) * f * (post_w != nullptr ? post_w[c0 + i] : 1.f);
      }
      rs[n * slice + i] = x;
      xs[n * slice + i] = to_f32(from_f32<T>(x));
    }
  }
  __syncthreads();
  // ---- this block's columns of W_g x, for all of its rows, to every block of the cluster
  {
    constexpr int lanes = 8, groups = kStepThreads / lanes;
    const int lane = tid % lanes, group = tid / lanes;
    for (int j0 = 0; j0 < dim; j0 += groups) {
      const int j = j0 + group;
      float acc[NT];
      group_dots<T, NT>(w_gate + (size_t)j * W + c0, xs, slice, nc, lane, lanes, j < dim, acc);
      if (j < dim)
#pragma unroll
        for (int n = 0; n < NT; ++n) store_in_block(sums + (rank * NT + n) * dim + j, lane, acc[n]);   // lane l feeds block l
    }
  }
  cluster_meet();
  for (int i = tid; i < NT * dim_p; i += kStepThreads) {
    const int n = i / dim_p, j = i - n * dim_p;
    float a = 0.f;
    if (j < dim && n < n_tok && token[n] >= 0) {
      float z = 0.f;
      for (int b = 0; b < kStepBlocks; ++b) z += sums[(b * NT + n) * dim + j];
      a = gelu_tanh(to_f32(from_f32<T>(z))) * to_f32(table[(size_t)token[n] * ld_table + first + j]);
      a = to_f32(from_f32<T>(a));
    }
    act[i] = a;
  }
  __syncthreads();
  // ---- this block's rows of y = W_p a
  {
    int lanes = 1;
    while (lanes < 8 && lanes * N < dim_p) lanes <<= 1;
    const int groups = kStepThreads / lanes, lane = tid % lanes, group = tid / lanes;
    for (int r0 = 0; r0 < nc; r0 += groups) {
      const int r = r0 + group;
      float acc[NT];
      group_dots<T, NT>(w_proj + (size_t)(c0 + r) * dim_p, act, dim_p, dim_p, lane, lanes, r < nc, acc);
      if (r < nc && lane == 0)
#pragma unroll
        for (int n = 0; n < NT; ++n) ys[n * slice + r] = acc[n];
    }
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    v[n] = 0.f;
    for (int i = tid; i < nc; i += kStepThreads) v[n] = fmaf(ys[n * slice + i], ys[n * slice + i], v[n]);
  }
  share_sums<NT>(v, part, sq_y, rank);
  cluster_meet();                                         // the last time anything is written into another block
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    if (n >= n_tok) break;
    float s = 0.f;
    for (int b = 0; b < kStepBlocks; ++b) s += sq_y[b * NT + n];
    const float f = 1.0f / sqrtf(s / (float)W + eps);
    for (int i = tid; i < nc; i += kStepThreads) {
      const size_t at = (size_t)(t0 + n) * W + c0 + i;
      const float x = rs[n * slice + i] + ys[n * slice + i] * f * norm_w[c0 + i];
      resid[at] = x;
      out[at] = from_f32<T>(x);
    }
  }
}

// ---------------------------------------------------------------- the same in bfloat16 on mma.sync
// A cluster takes 8 tokens, the upper half of the products' 16 rows staying empty.  A lane (g, t) loads 16 bytes of a row of
// weights, columns k0 + 8 t .. + 7, and the same columns of token g, and hands elements 0 - 3 to one m16n8k16 product
// and 4 - 7 to the next: the order of the columns within a product is free as long as both operands have the same.
// W_g x: warps take (tile of 8 rows, part of the block's columns) in turn; every part's sums go to every block.
// STAGED: the block's share of both matrices fits shared memory and is brought there before the kernel waits for its
// predecessor, so that nothing behind the wait but the rows themselves comes from further away.
constexpr int kStepTokens = 8;

__device__ __forceinline__ void mma_tokens(float (&c)[4], const uint4& a, const uint4& b) {
  const unsigned z = 0u;
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a.x), "r"(z), "r"(a.y), "r"(z), "r"(b.x), "r"(b.y));
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a.z), "r"(z), "r"(a.w), "r"(z), "r"(b.z), "r"(b.w));
}
// row . x over n_cols columns for 8 rows of weights (this lane's: `row`, valid when live) and 8 tokens (`x`: this lane's
// token's columns in shared memory): c[0], c[1] of lane (g, t) are token g's sums for rows 2 t and 2 t + 1.
__device__ __forceinline__ void tile_dots(const __nv_bfloat16* row, bool live, const __nv_bfloat16* x, int n_cols, int t, float (&c)[4]) {
  c[0] = c[1] = c[2] = c[3] = 0.f;
#pragma unroll 8
  for (int k = 0; k < n_cols; k += 32) {
    uint4 a = make_uint4(0u, 0u, 0u, 0u), b = a;
    if (k + 8 * t < n_cols) {
      a = *reinterpret_cast<const uint4*>(x + k + 8 * t);
      if (live) b = *reinterpret_cast<const uint4*>(row + k + 8 * t);
    }
    mma_tokens(c, a, b);
  }
}

// parts: into how many parts of `part_cols` columns (a multiple of 32) a block's columns are dealt for W_g x; dim_s: dim rounded up to
// a multiple of 8.
constexpr int kStepPad = 32;      // elements behind a row of shared memory: two rows of a product's operand, side by side, in different banks

template <bool STAGED>
__global__ void __launch_bounds__(kStepThreads)
token_input_step_mma_kernel(float* __restrict__ resid, const __nv_bfloat16* __restrict__ delta, const float* __restrict__ post_w,
                            float post_eps, const __nv_bfloat16* __restrict__ w_gate, const __nv_bfloat16* __restrict__ w_proj,
                            const float* __restrict__ norm_w, float eps, const __nv_bfloat16* __restrict__ table, int ld_table,
                            int first, int V, const int* __restrict__ ids, const int* __restrict__ sampled, int n_sampled,
                            __nv_bfloat16* __restrict__ out, int T_, int W, int dim, int dim_p, int slice, int parts,
                            int part_cols, int* status) {
  constexpr int NT = kStepTokens;
  extern __shared__ uint4 step_mma_smem[];
  const int xs_ld = slice + kStepPad, act_ld = dim_p + kStepPad, dim_s = (dim + 7) / 8 * 8;
  __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(step_mma_smem);      // [NT][xs_ld] the stream, as the product reads it
  __nv_bfloat16* act = xs + NT * xs_ld;                                      // [NT][act_ld]
  float* rs = reinterpret_cast<float*>(act + NT * act_ld);                   // [NT][slice] the float32 stream
  float* sums = rs + NT * slice;                                             // [kStepBlocks * parts][NT][dim_s] shares of W_g x
  float* ys = sums;                                                          // [NT][slice], once those are used up
  const int shares = kStepBlocks * parts * NT * dim_s;
  __nv_bfloat16* wg_s = reinterpret_cast<__nv_bfloat16*>(sums + max(shares, NT * slice));      // STAGED: [dim][xs_ld]
  __nv_bfloat16* wp_s = wg_s + dim * xs_ld;                                  // STAGED: [slice][act_ld]
  __shared__ float part_sq[kStepWarps * NT];
  __shared__ float sq_pending[kStepBlocks * NT], sq_y[kStepBlocks * NT];
  __shared__ int token[NT];
  pdl_trigger();
  const int rank = blockIdx.x % kStepBlocks, t0 = blockIdx.x / kStepBlocks * NT;      // the cluster is kStepBlocks neighbours along x
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int n_tok = min(NT, T_ - t0);
  const int c0 = min(W, rank * slice), c1 = min(W, c0 + slice), nc = c1 - c0;
  // the weights do not depend on what runs before
  if (STAGED) {
    const int per = nc / 8, per_p = dim_p / 8;
    auto bring = [](__nv_bfloat16* dst, const __nv_bfloat16* src) {
      const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"(d), "l"(src) : "memory");
    };
    for (int i = tid; i < dim * per; i += kStepThreads) {
      const int j = i / per, k = (i - j * per) * 8;
      bring(wg_s + (size_t)j * xs_ld + k, w_gate + (size_t)j * W + c0 + k);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < nc * per_p; i += kStepThreads) {
      const int r = i / per_p, k = (i - r * per_p) * 8;
      bring(wp_s + (size_t)r * act_ld + k, w_proj + (size_t)(c0 + r) * dim_p + k);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  } else if (t0 == 0) {       // the first cluster asks for their lines
    const int per = (nc + 63) / 64;
    for (int i = tid; i < dim * per; i += kStepThreads) {
      const int j = i / per;
      asm volatile("prefetch.global.L2 [%0];" ::"l"(w_gate + (size_t)j * W + c0 + (i - j * per) * 64));
    }
    for (int i = tid * 64; i < nc * dim_p; i += kStepThreads * 64)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(w_proj + (size_t)c0 * dim_p + i));
  }
  cluster_meet();                                         // every block of the cluster runs before another writes into it
  pdl_wait();
  // ---- the stream, brought up to date; a warp takes a token
  const bool live_tok = warp < n_tok;
  const size_t row_at = (size_t)(t0 + (live_tok ? warp : 0)) * W + c0;
  const bool normed = delta != nullptr && post_w != nullptr;
  // the rows of the table the tokens name, and the stream: asked for before anything is waited for
  int id_w = -1;
  if (live_tok) {
    id_w = token_of(ids, sampled, n_sampled, t0 + warp, V);
    if (id_w < 0 && rank == 0 && lane == 0) atomicCAS(status, 0, KVB_STATUS_BAD_TOKEN);
    for (int i = lane * 64; i < dim + 64; i += 2048)
      if (id_w >= 0) asm volatile("prefetch.global.L2 [%0];" ::"l"(table + (size_t)id_w * ld_table + first + min(i, dim - 1)));
    for (int i = lane * 32; i < nc; i += 1024) asm volatile("prefetch.global.L2 [%0];" ::"l"(resid + row_at + i));
  }
  if (lane == 0) token[warp] = id_w;
  if (normed) {
    float sq = 0.f;
    if (live_tok)
      for (int i = lane * 8; i < nc; i += 256) {
        float d[8];
        Piece<__nv_bfloat16>::open(*reinterpret_cast<const uint4*>(delta + row_at + i), d);
#pragma unroll
        for (int e = 0; e < 8; ++e) sq = fmaf(d[e], d[e], sq);
      }
    sq = warp_sum(sq);
    if (lane < kStepBlocks) store_in_block(sq_pending + rank * NT + warp, lane, sq);
  }
  if (normed) cluster_meet();
  else __syncthreads();
  {
    float f = 1.f;
    if (normed) {
      float s = 0.f;
#pragma unroll
      for (int b = 0; b < kStepBlocks; ++b) s += sq_pending[b * NT + warp];
      f = 1.0f / sqrtf(s / (float)W + post_eps);
    }
    for (int i = lane * 8; i < slice; i += 256) {
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (live_tok && i < nc) {
        const float4 lo = *reinterpret_cast<const float4*>(resid + row_at + i), hi = *reinterpret_cast<const float4*>(resid + row_at + i + 4);
        x[0] = lo.x; x[1] = lo.y; x[2] = lo.z; x[3] = lo.w; x[4] = hi.x; x[5] = hi.y; x[6] = hi.z; x[7] = hi.w;
        if (delta != nullptr) {
          float d[8];
          Piece<__nv_bfloat16>::open(*reinterpret_cast<const uint4*>(delta + row_at + i), d);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] += d[e] * f * (normed ? post_w[c0 + i + e] : 1.f);
        }
      }
      *reinterpret_cast<float4*>(rs + warp * slice + i) = make_float4(x[0], x[1], x[2], x[3]);
      *reinterpret_cast<float4*>(rs + warp * slice + i + 4) = make_float4(x[4], x[5], x[6], x[7]);
      __nv_bfloat162 h[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
      *reinterpret_cast<uint4*>(xs + warp * xs_ld + i) = *reinterpret_cast<const uint4*>(h);
    }
  }
  if (STAGED) asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  // ---- this block's columns of W_g x, for all of its rows, to every block of the cluster
  const int tiles = dim_s / 8;
  for (int u = warp; u < tiles * parts; u += kStepWarps) {
    const int tile = u % tiles, part = u / tiles, k0 = part * part_cols;
    const int j = tile * 8 + g;
    float c[4];
    const __nv_bfloat16* w_row = STAGED ? wg_s + (size_t)min(j, dim - 1) * xs_ld + k0 : w_gate + (size_t)j * W + c0 + k0;
    tile_dots(w_row, j < dim, xs + g * xs_ld + k0, max(0, min(part_cols, nc - k0)), t, c);
    if (g < n_tok) {
      float* to = sums + ((size_t)(rank * parts + part) * NT + g) * dim_s + tile * 8 + 2 * t;
#pragma unroll
      for (int b = 0; b < kStepBlocks; ++b) store2_in_block(to, b, c[0], c[1]);
    }
  }
  cluster_meet();
  for (int i = tid; i < NT * act_ld; i += kStepThreads) {
    const int n = i / act_ld, j = i - n * act_ld;
    float a = 0.f;
    if (j < dim && n < n_tok && token[n] >= 0) {
      float z = 0.f;
      for (int b = 0; b < kStepBlocks * parts; ++b) z += sums[((size_t)b * NT + n) * dim_s + j];
      a = gelu_tanh(__bfloat162float(__float2bfloat16_rn(z))) * __bfloat162float(table[(size_t)token[n] * ld_table + first + j]);
    }
    act[i] = __float2bfloat16_rn(a);
  }
  if (STAGED) asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();                                        // the shares are used up: their room is y's from here on
  // ---- this block's rows of y = W_p a
  float sq = 0.f;                                         // of token g, over this lane's rows
  for (int r0 = warp * 8; r0 < nc; r0 += kStepWarps * 8) {
    float c[4];
    tile_dots(STAGED ? wp_s + (size_t)(r0 + g) * act_ld : w_proj + (size_t)(c0 + r0 + g) * dim_p, true, act + g * act_ld, dim_p, t, c);     // nc is a multiple of 8
    ys[g * slice + r0 + 2 * t] = c[0];
    ys[g * slice + r0 + 2 * t + 1] = c[1];
    sq = fmaf(c[0], c[0], fmaf(c[1], c[1], sq));
  }
  sq += __shfl_xor_sync(0xffffffffu, sq, 1);
  sq += __shfl_xor_sync(0xffffffffu, sq, 2);
  if (t == 0) part_sq[warp * NT + g] = sq;
  __syncthreads();
  if (tid < NT * kStepBlocks) {
    const int n = tid % NT, to = tid / NT;
    float s = 0.f;
    for (int w = 0; w < kStepWarps; ++w) s += part_sq[w * NT + n];
    store_in_block(sq_y + rank * NT + n, to, s);
  }
  cluster_meet();                                         // the last time anything is written into another block
  if (!live_tok) return;
  float s = 0.f;
#pragma unroll
  for (int b = 0; b < kStepBlocks; ++b) s += sq_y[b * NT + warp];
  const float f = 1.0f / sqrtf(s / (float)W + eps);
  for (int i = lane * 4; i < nc; i += 128) {
    const float4 x = *reinterpret_cast<const float4*>(rs + warp * slice + i), y = *reinterpret_cast<const float4*>(ys + warp * slice + i);
    const float4 w = *reinterpret_cast<const float4*>(norm_w + c0 + i);
    const float4 v = make_float4(x.x + y.x * f * w.x, x.y + y.y * f * w.y, x.z + y.z * f * w.z, x.w + y.w * f * w.w);
    *reinterpret_cast<float4*>(resid + row_at + i) = v;
    __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    *reinterpret_cast<uint2*>(out + row_at + i) = *reinterpret_cast<const uint2*>(h);
  }
}

// How a block's columns are dealt over warps that would be idle otherwise.
static void step_parts(int slice, int dim, int* parts, int* part_cols) {
  const int tiles = (dim + 7) / 8, chunks = (slice + 31) / 32;
  int n = tiles >= kStepWarps ? 1 : kStepWarps / tiles;
  if (n > chunks) n = chunks;
  *part_cols = (chunks + n - 1) / n * 32;
  *parts = (slice + *part_cols - 1) / *part_cols;
}

static size_t step_mma_smem_bytes(int slice, int dim, int dim_p, bool staged) {
  int parts, cols;
  step_parts(slice, dim, &parts, &cols);
  const size_t shares = (size_t)kStepBlocks * parts * kStepTokens * ((dim + 7) / 8 * 8), y = (size_t)kStepTokens * slice;
  const size_t weights = staged ? (size_t)dim * (slice + kStepPad) + (size_t)slice * (dim_p + kStepPad) : 0;
  return (size_t)kStepTokens * (slice + dim_p + 2 * kStepPad) * 2 + (size_t)kStepTokens * slice * 4 + (shares > y ? shares : y) * 4 +
         weights * 2;
}

template <typename T, int NT>
static int launch_step(float* resid, const void* delta, const float* post_w, float post_eps, const void* w_gate,
                       const void* w_proj, const float* norm_w, float eps, const void* table, int ld_table, int first, int V,
                       const int* ids, const int* sampled, int n_sampled, void* out, int T_, int W, int dim, int dim_p,
                       int slice, size_t smem, int* status, cudaStream_t stream) {
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(token_input_step_kernel<T, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const cudaError_t e = kvb_launch_cluster(
      token_input_step_kernel<T, NT>, dim3((T_ + NT - 1) / NT * kStepBlocks), dim3(kStepThreads), dim3(kStepBlocks), smem, stream, resid,
      (const T*)delta, post_w, post_eps, (const T*)w_gate, (const T*)w_proj, norm_w, eps, (const T*)table, ld_table, first, V, ids,
      sampled, n_sampled, (T*)out, T_, W, dim, dim_p, slice, status);
  return e != cudaSuccess ? (int)e : kvb_launch_result();
}

static size_t step_smem_bytes(int nt, int slice, int dim, int dim_p) {
  return sizeof(float) * ((size_t)3 * nt * slice + (size_t)nt * dim_p + (size_t)kStepBlocks * nt * dim);
}

// Tokens that a cluster takes in a step of T_ tokens: one while the clusters do not fill the GPU, then more.
static int step_tokens(int T_) { return T_ <= 16 ? 1 : (T_ <= 32 ? 2 : 4); }

// Whether one launch can do the branch for steps of up to T_ tokens: W a multiple of 8, the shared memory at hand.
KVB_EXPORT int kvb_token_input_step_supported(int T_, int W, int dim, int dim_p, int dtype) {
  if (W < 8 || W % 8 != 0 || dim < 1 || dim_p < dim || dim_p % 8 != 0) return 0;
  const int slice = (W / 8 + kStepBlocks - 1) / kStepBlocks * 8;
  const size_t smem = dtype == KVB_BF16 ? step_mma_smem_bytes(slice, dim, dim_p, false) : step_smem_bytes(step_tokens(T_), slice, dim, dim_p);
  return smem <= 200 * 1024 ? 1 : 0;
}

// resid [T, W] float32, in place; delta [T, W] or null, post_w null or the weight of the RMS norm it passes first;
// w_gate [dim, W], w_proj [W, dim_p] (columns behind dim zero), norm_w [W]; table [V, ld_table], columns first ..
// first + dim - 1; out [T, W]: the new stream in the activations' type.  Everything dense, rows 16-byte aligned.
KVB_EXPORT int kvb_token_input_step(float* resid, const void* delta, const float* post_w, float post_eps, const void* w_gate,
                                    const void* w_proj, const float* norm_w, float eps, const void* table, int ld_table,
                                    int first, int V, const int* ids, const int* sampled, int n_sampled, void* out, int T_,
                                    int W, int dim, int dim_p, int dtype, int* status, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (!kvb_token_input_step_supported(T_, W, dim, dim_p, dtype) || first < 0 || first + dim > ld_table) return KVB_ERR_BAD_SIZE;
  if ((reinterpret_cast<uintptr_t>(resid) | reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(w_gate) |
       reinterpret_cast<uintptr_t>(w_proj) | reinterpret_cast<uintptr_t>(norm_w) | reinterpret_cast<uintptr_t>(out)) & 15)
    return KVB_ERR_ALIGN;
  const int slice = (W / 8 + kStepBlocks - 1) / kStepBlocks * 8;
  if (dtype == KVB_BF16) {
    using B = __nv_bfloat16;
    const bool staged = step_mma_smem_bytes(slice, dim, dim_p, true) <= 220 * 1024;
    const size_t smem = step_mma_smem_bytes(slice, dim, dim_p, staged);
    auto kernel = staged ? token_input_step_mma_kernel<true> : token_input_step_mma_kernel<false>;
    int parts, cols;
    step_parts(slice, dim, &parts, &cols);
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    e = kvb_launch_cluster(kernel, dim3((T_ + kStepTokens - 1) / kStepTokens * kStepBlocks), dim3(kStepThreads),
                           dim3(kStepBlocks), smem, stream, resid, (const B*)delta, post_w, post_eps, (const B*)w_gate,
                           (const B*)w_proj, norm_w, eps, (const B*)table, ld_table, first, V, ids, sampled, n_sampled, (B*)out, T_,
                           W, dim, dim_p, slice, parts, cols, status);
    return e != cudaSuccess ? (int)e : kvb_launch_result();
  }
  if (dtype != KVB_F32) return KVB_ERR_BAD_DTYPE;
  const int nt = step_tokens(T_);
  const size_t smem = step_smem_bytes(nt, slice, dim, dim_p);
#define KVB_STEP(NT)                                                                                                     \
  return launch_step<float, NT>(resid, delta, post_w, post_eps, w_gate, w_proj, norm_w, eps, table, ld_table, first, V, ids, \
                                sampled, n_sampled, out, T_, W, dim, dim_p, slice, smem, status, stream)
  if (nt == 1) KVB_STEP(1);
  if (nt == 2) KVB_STEP(2);
  KVB_STEP(4);
#undef KVB_STEP
}
