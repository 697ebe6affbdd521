// A layer's own input from each token: a row of a table (the layer's slice of the token's row), gated by the
// residual stream, brought to the model's width, normed and added to the stream:
//   y = W_p (gelu_tanh(W_g x) * e),   x <- x + y / sqrt(mean(y^2) + eps) * w
//
//   * token_gate_kernel: for steps whose two products are made by the step's matrix product kernels: the middle,
//     a[t, j] = gelu_tanh(p[t, j]) * table[token, first + j].
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
