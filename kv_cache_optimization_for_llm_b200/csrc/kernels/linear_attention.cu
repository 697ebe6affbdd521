// Linear attention whose memory decays per head and key channel and takes in what the decay makes room for.
//
// Per head, with raw projections zq, zf of N channels and v of Dv:
//     q = silu(zq),   f = l + (1 - l) sigmoid(zf + b)          l, b: learned, per head and channel
//     S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T                 S is N x Dv
//     o_t = S_t^T q_t / rms(S_t^T q_t) * weight                 the norm over the head's Dv values, weight shared by heads
// Decays, the activations of the projections, the memory and the norm are float32 in both precisions.  A request that
// starts at position 0 starts from a zero memory whatever its slot holds.  Sums run in an order fixed by the sizes alone.
//
// A block owns `cols` value columns of one (request, head); four lanes share a column, lane l holding memory rows
// l, l + 4, ... in registers for the whole run (where N is a multiple of 4, VEC, rows 16 j + 4 l .. + 3, so that one
// shared-memory load brings four rows).  The run is walked in pieces of 32 tokens whose f, q and v the block first brings
// into shared memory as float32.  A step's update is S <- x + f (S - x).  Where the block owns all of a head's columns (up to
// 128, with N up to 128) the read-outs of a piece meet in shared memory and leave normed; otherwise they go to a
// float32 scratch and head_norm_kernel follows.
//
// A long run is cut into chunks of `chunk` tokens that are walked side by side, in three launches:
//   LA_LOCAL   every chunk but a run's last, from a zero memory: what it ends with, and per channel the product of its decays
//   la_carry   per memory element, along the run's chunks in order: what each chunk begins with
//   LA_FINAL   every chunk from what it begins with, writing read-outs; the run's last chunk leaves the memory in the slot
// Request row r's chunk that begins at token row t keeps its matrices in row (r - row_off) + t / chunk of `local` and of
// `carry`.  A run of one chunk reads and writes its slot directly.
#include "common.cuh"

struct LinearArgs {
  const void* p; int ld, q_off, f_off, v_off;     // [T, ld] compute type: zq, zf (H * N each) and v (H * Dv)
  const float* f_bias; const float* lower;        // [H * N]
  const float* weight; float eps;                 // [Dv]
  float* state; long long slot_stride;            // slot 0's [H][Dv][N]
  float* y;                                       // [T, H * Dv] float32 read-outs (only where the norm is a launch of its own)
  void* out;                                      // [T, H * Dv] compute type
  const int* q_start; const int* req_start; const int* slots;
  int H, N, Dv, cols;
  int chunk, row_off;                             // chunk > 0: runs are cut; requests below row_off are single chunks
  float* local; float* carry; float* decay;       // chunked: [rows][H][Dv][N] twice and [rows][H][N]
};

constexpr int kLaPiece = 32;
enum { LA_WHOLE = 0, LA_LOCAL = 1, LA_FINAL = 2 };

__device__ __forceinline__ float la_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ float4 la_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 la_load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}

// NORM: the block owns all of its head's columns and norms the read-outs.  v4: the values may be loaded four at a time.
template <typename T, int NPT, int MODE, bool VEC, bool NORM>
__global__ void __launch_bounds__(NORM ? 512 : 256) linear_scan_kernel(LinearArgs a, int v4) {
  extern __shared__ __align__(16) float lsm[];
  const int N = a.N, cols = a.cols;
  float* Fs = lsm;                          // [piece][N] decays
  float* Qs = Fs + kLaPiece * N;            // [piece][N]                  (LA_LOCAL: [N], the product of the decays)
  float* xs = Qs + kLaPiece * N;            // [piece][cols] values
  float* ys = xs + kLaPiece * cols;         // [piece][cols] read-outs     (NORM)
  pdl_trigger();
  pdl_wait();
  const int splits = (a.Dv + cols - 1) / cols;
  const int h = blockIdx.x / splits, col0 = (blockIdx.x % splits) * cols;
  const int r = blockIdx.y;
  const int inner = a.H * a.Dv;
  const int my_cols = min(cols, a.Dv - col0);
  const int tid = threadIdx.x, l = tid & 3;
  const int pcol = tid >> 2;
  const bool owner = pcol < my_cols;
  const int pc = owner ? pcol : 0;
  int t0 = a.q_start[r], t1 = a.q_start[r + 1];
  const size_t at = ((size_t)h * a.Dv + col0 + pc) * N;          // this thread's column within a set of matrices
  float* st = a.state + (size_t)a.slots[r] * a.slot_stride + at;
  const float* from = a.req_start[r] > 0 ? st : nullptr;         // where the memory comes from, null for zeros
  float* to = st;                                                // where it goes, null for nowhere
  size_t row = 0;
  if (MODE != LA_WHOLE) {
    const int mine = t0 + (int)blockIdx.z * a.chunk;
    const bool single = t0 + a.chunk >= t1;                      // a run of one chunk
    if (MODE == LA_LOCAL ? mine + a.chunk >= t1 : (mine >= t1 && blockIdx.z > 0)) return;
    row = (size_t)(r - a.row_off) + mine / a.chunk;
    const size_t mat = row * (size_t)inner * N + at;
    if (MODE == LA_LOCAL) { from = nullptr; to = a.local + mat; }
    else if (!single) { from = a.carry + mat; to = mine + a.chunk >= t1 ? st : nullptr; }
    t0 = mine;
    t1 = min(t1, mine + a.chunk);
  }
  float S[NPT];
  if (VEC) {
#pragma unroll
    for (int j = 0; j < NPT / 4; ++j) {
      const int n = 16 * j + 4 * l;
      const float4 s4 = (from && owner && n < N) ? *reinterpret_cast<const float4*>(from + n) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[4 * j] = s4.x; S[4 * j + 1] = s4.y; S[4 * j + 2] = s4.z; S[4 * j + 3] = s4.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[i] = (from && owner && l + 4 * i < N) ? from[l + 4 * i] : 0.f;
  }
  const T* rows = static_cast<const T*>(a.p);
  const float* bias = a.f_bias + (size_t)h * N;
  const float* low = a.lower + (size_t)h * N;
  if (MODE == LA_LOCAL)
    for (int n = tid; n < N; n += blockDim.x) Qs[n] = 1.f;
  for (int c0 = t0; c0 < t1; c0 += kLaPiece) {
    const int nt = min(kLaPiece, t1 - c0);
    __syncthreads();
    if (VEC) {
      const int n4 = N >> 2;
      for (int idx = tid; idx < nt * n4; idx += blockDim.x) {
        const int tk = idx / n4, n = (idx - tk * n4) * 4;
        const T* src = rows + (size_t)(c0 + tk) * a.ld + (size_t)h * N + n;
        const float4 z = la_load4(src + a.f_off);
        const float4 b = la_load4(bias + n), lo = la_load4(low + n);
        float4 f;
        f.x = lo.x + (1.f - lo.x) * la_sigmoid(z.x + b.x);
        f.y = lo.y + (1.f - lo.y) * la_sigmoid(z.y + b.y);
        f.z = lo.z + (1.f - lo.z) * la_sigmoid(z.z + b.z);
        f.w = lo.w + (1.f - lo.w) * la_sigmoid(z.w + b.w);
        *reinterpret_cast<float4*>(Fs + tk * N + n) = f;
        if (MODE != LA_LOCAL) {
          float4 q = la_load4(src + a.q_off);
          q.x *= la_sigmoid(q.x); q.y *= la_sigmoid(q.y); q.z *= la_sigmoid(q.z); q.w *= la_sigmoid(q.w);
          *reinterpret_cast<float4*>(Qs + tk * N + n) = q;
        }
      }
    } else {
      for (int idx = tid; idx < nt * N; idx += blockDim.x) {
        const int tk = idx / N, n = idx - tk * N;
        const T* src = rows + (size_t)(c0 + tk) * a.ld + (size_t)h * N + n;
        Fs[idx] = low[n] + (1.f - low[n]) * la_sigmoid(to_f32(src[a.f_off]) + bias[n]);
        if (MODE != LA_LOCAL) {
          const float q = to_f32(src[a.q_off]);
          Qs[idx] = q * la_sigmoid(q);
        }
      }
    }
    if (v4) {
      const int c4 = my_cols >> 2;
      for (int idx = tid; idx < nt * c4; idx += blockDim.x) {
        const int tk = idx / c4, q = (idx - tk * c4) * 4;
        *reinterpret_cast<float4*>(xs + tk * cols + q) =
            la_load4(rows + (size_t)(c0 + tk) * a.ld + a.v_off + (size_t)h * a.Dv + col0 + q);
      }
    } else {
      for (int idx = tid; idx < nt * my_cols; idx += blockDim.x) {
        const int tk = idx / my_cols, q = idx - tk * my_cols;
        xs[tk * cols + q] = to_f32(rows[(size_t)(c0 + tk) * a.ld + a.v_off + (size_t)h * a.Dv + col0 + q]);
      }
    }
    __syncthreads();
    if (MODE == LA_LOCAL && col0 == 0) {
      for (int n = tid; n < N; n += blockDim.x) {
        float d = Qs[n];
        for (int tk = 0; tk < nt; ++tk) d *= Fs[tk * N + n];
        Qs[n] = d;
      }
    }
    for (int tk = 0; tk < nt; ++tk) {
      const float xv = xs[tk * cols + pc];
      const float* Ft = Fs + tk * N;
      const float* Qt = Qs + tk * N;
      float acc = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
      if (VEC) {
#pragma unroll
        for (int j = 0; j < NPT / 4; ++j) {
          const int n = 16 * j + 4 * l;
          if (n < N) {
            const float4 f = *reinterpret_cast<const float4*>(Ft + n);
            S[4 * j + 0] = fmaf(f.x, S[4 * j + 0] - xv, xv);
            S[4 * j + 1] = fmaf(f.y, S[4 * j + 1] - xv, xv);
            S[4 * j + 2] = fmaf(f.z, S[4 * j + 2] - xv, xv);
            S[4 * j + 3] = fmaf(f.w, S[4 * j + 3] - xv, xv);
            if (MODE != LA_LOCAL) {
              const float4 q = *reinterpret_cast<const float4*>(Qt + n);
              acc = fmaf(S[4 * j + 0], q.x, acc);
              a1 = fmaf(S[4 * j + 1], q.y, a1);
              a2 = fmaf(S[4 * j + 2], q.z, a2);
              a3 = fmaf(S[4 * j + 3], q.w, a3);
            }
          }
        }
        acc = (acc + a1) + (a2 + a3);
      } else {
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
          const int n = l + 4 * i;
          if (n < N) {
            S[i] = fmaf(Ft[n], S[i] - xv, xv);
            if (MODE != LA_LOCAL) acc = fmaf(S[i], Qt[n], acc);
          }
        }
      }
      if (MODE == LA_LOCAL) continue;
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      if (owner && l == 0) {
        if (NORM) ys[tk * cols + pc] = acc;
        else a.y[(size_t)(c0 + tk) * inner + (size_t)h * a.Dv + col0 + pc] = acc;
      }
    }
    if (NORM && MODE != LA_LOCAL) {
      __syncthreads();
      const int lane = tid & 31;
      T* out = static_cast<T*>(a.out);
      for (int tk = tid >> 5; tk < nt; tk += blockDim.x >> 5) {
        const float* y = ys + tk * cols;
        float ss = 0.f;
        for (int i = lane; i < a.Dv; i += 32) ss = fmaf(y[i], y[i], ss);
        const float g = 1.0f / sqrtf(warp_sum(ss) / (float)a.Dv + a.eps);
        T* o = out + (size_t)(c0 + tk) * inner + (size_t)h * a.Dv;
        for (int i = lane; i < a.Dv; i += 32) o[i] = from_f32<T>(y[i] * g * a.weight[i]);
      }
    }
  }
  if (owner && to) {
    if (VEC) {
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        const int n = 16 * j + 4 * l;
        if (n < N) *reinterpret_cast<float4*>(to + n) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < NPT; ++i)
        if (l + 4 * i < N) to[l + 4 * i] = S[i];
    }
  }
  if (MODE == LA_LOCAL && col0 == 0)
    for (int n = tid; n < N; n += blockDim.x) a.decay[(row * a.H + h) * N + n] = Qs[n];    // each thread reads what it wrote
}

// One thread per element of a request's matrices walks the run's chunks in order and writes what each begins with.
// Runs of one chunk are left alone.  The loads (four chunks' at a time) depend on no store.
__global__ void __launch_bounds__(256) linear_carry_kernel(LinearArgs a) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.y;
  const size_t per = (size_t)a.H * a.Dv * a.N;
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= per) return;
  const int t0 = a.q_start[r], t1 = a.q_start[r + 1];
  if (t0 + a.chunk >= t1) return;
  const unsigned col = (unsigned)e / (unsigned)a.N, n = (unsigned)e - col * (unsigned)a.N;
  const unsigned hn = col / (unsigned)a.Dv * (unsigned)a.N + n;
  const size_t per_decay = (size_t)a.H * a.N;
  const float* __restrict__ local = a.local;
  const float* __restrict__ decay = a.decay;
  float* __restrict__ carry = a.carry;
  float S = a.req_start[r] > 0 ? a.state[(size_t)a.slots[r] * a.slot_stride + e] : 0.f;
  const int nck = (t1 - t0 + a.chunk - 1) / a.chunk;
  const size_t row0 = (size_t)(r - a.row_off) + t0 / a.chunk;      // rows of one run follow one another
  int k = 0;
  for (; k + 4 < nck; k += 4) {
    float lo[4], de[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      lo[x] = local[(row0 + k + x) * per + e];
      de[x] = decay[(row0 + k + x) * per_decay + hn];
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      carry[(row0 + k + x) * per + e] = S;
      S = fmaf(de[x], S, lo[x]);
    }
  }
  for (; k < nck; ++k) {
    carry[(row0 + k) * per + e] = S;
    if (k + 1 < nck) S = fmaf(decay[(row0 + k) * per_decay + hn], S, local[(row0 + k) * per + e]);
  }
}

// y [T, H * Dv] float32 -> out[t, h, :] = y / sqrt(mean over the head of y^2 + eps) * weight.  A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
linear_head_norm_kernel(const float* __restrict__ y, const float* __restrict__ weight, T* __restrict__ out, long long units,
                        int Dv, float eps) {
  pdl_trigger();
  pdl_wait();
  const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31;
  const float* row = y + unit * Dv;
  float ss = 0.f;
  for (int i = lane; i < Dv; i += 32) ss = fmaf(row[i], row[i], ss);
  const float g = 1.0f / sqrtf(warp_sum(ss) / (float)Dv + eps);
  for (int i = lane; i < Dv; i += 32) out[unit * Dv + i] = from_f32<T>(row[i] * g * weight[i]);
}

// Whether the scan norms its read-outs itself (else it needs the float32 scratch y).
KVB_EXPORT int kvb_linear_scan_norms(int N, int Dv) { return N <= 128 && Dv <= 128 ? 1 : 0; }

template <typename T, int MODE, bool VEC>
static int launch_linear(const LinearArgs& a, dim3 grid, int threads, size_t smem, bool norm, int v4, cudaStream_t stream) {
  const int npt = (a.N + 3) / 4;
#define KVB_LA(NPT, NORM)                                                                                             \
  {                                                                                                                   \
    if (smem > 48 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(linear_scan_kernel<T, NPT, MODE, VEC, NORM>,                               \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                   \
      if (e != cudaSuccess) return (int)e;                                                                            \
    }                                                                                                                 \
    kvb_launch(linear_scan_kernel<T, NPT, MODE, VEC, NORM>, grid, dim3(threads), smem, stream, a, v4);                \
    return kvb_launch_result();                                                                                       \
  }
  if (norm) {
    if (npt <= 8) KVB_LA(8, true)
    if (npt <= 16) KVB_LA(16, true)
    KVB_LA(32, true)
  }
  if (npt <= 16) KVB_LA(16, false)
  if (npt <= 32) KVB_LA(32, false)
  KVB_LA(64, false)
#undef KVB_LA
}

template <typename T>
static int linear_scan_any(LinearArgs a, int R, int max_run, cudaStream_t stream) {
  const bool norm = kvb_linear_scan_norms(a.N, a.Dv) != 0;
  if (!norm && a.y == nullptr) return KVB_ERR_BAD_SIZE;
  const bool vec = a.N % 4 == 0 && a.ld % 4 == 0 && a.q_off % 4 == 0 && a.f_off % 4 == 0 && a.slot_stride % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.state) |
                     reinterpret_cast<uintptr_t>(a.f_bias) | reinterpret_cast<uintptr_t>(a.lower) |
                     reinterpret_cast<uintptr_t>(a.local) | reinterpret_cast<uintptr_t>(a.carry)) & 15) == 0;
  a.cols = norm ? a.Dv : (a.Dv < 64 ? a.Dv : 64);
  const int v4 = a.Dv % 4 == 0 && a.cols % 4 == 0 && a.ld % 4 == 0 && a.v_off % 4 == 0 &&
                 (kLaPiece * a.N) % 4 == 0 && (reinterpret_cast<uintptr_t>(a.p) & 15) == 0;
  const int splits = (a.Dv + a.cols - 1) / a.cols;
  const int threads = (a.cols * 4 + 31) / 32 * 32;
  const size_t smem = (size_t)kLaPiece * (2 * a.N + a.cols * (norm ? 2 : 1)) * sizeof(float);
  unsigned nck = 1;
  if (a.chunk > 0) {
    if (!a.local || !a.carry || !a.decay || max_run < 1 || a.chunk % kLaPiece) return KVB_ERR_BAD_SIZE;
    if ((long long)a.H * a.Dv * a.N > 0x7fffffffLL) return KVB_ERR_BAD_SIZE;
    nck = (unsigned)((max_run + a.chunk - 1) / a.chunk);
    if (nck > 65535) return KVB_ERR_BAD_SIZE;
  }
  const dim3 grid(a.H * splits, R, nck);
#define KVB_LA_MODE(MODE)                                                                                            \
  (vec ? launch_linear<T, MODE, true>(a, grid, threads, smem, norm, v4, stream)                                      \
       : launch_linear<T, MODE, false>(a, grid, threads, smem, norm, v4, stream))
  int rc;
  if (a.chunk > 0) {
    if ((rc = KVB_LA_MODE(LA_LOCAL)) != 0) return rc;
    const size_t per = (size_t)a.H * a.Dv * a.N;
    kvb_launch(linear_carry_kernel, dim3((unsigned)((per + 255) / 256), R), dim3(256), 0, stream, a);
    rc = KVB_LA_MODE(LA_FINAL);
  } else {
    rc = KVB_LA_MODE(LA_WHOLE);
  }
#undef KVB_LA_MODE
  return rc;
}

// max_run: the step's longest run (chunked launches only: the grid's third extent).  T_: tokens of the step.
// Refuses: N above 256, more than 65535 requests; a chunk that is no multiple of 32 tokens.
KVB_EXPORT int kvb_linear_scan(const LinearArgs* args, int T_, int R, int max_run, int dtype, cudaStream_t stream) {
  const LinearArgs a = *args;
  if (R <= 0 || T_ <= 0) return 0;
  if (a.H < 1 || a.N < 1 || a.N > 256 || a.Dv < 1 || R > 65535) return KVB_ERR_BAD_SIZE;
  int rc;
  KVB_DISPATCH_DTYPE(dtype, T, rc = linear_scan_any<T>(a, R, max_run, stream));
  if (rc != 0 || kvb_linear_scan_norms(a.N, a.Dv)) return rc;
  const long long units = (long long)T_ * a.H;
  KVB_DISPATCH_DTYPE(dtype, T, (kvb_launch(linear_head_norm_kernel<T>, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, stream,
                                            a.y, a.weight, (T*)a.out, units, a.Dv, a.eps)));
  return kvb_launch_result();
}
