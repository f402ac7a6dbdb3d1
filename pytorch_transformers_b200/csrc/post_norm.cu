// Blocks whose norm comes after the sum, on a float32 residual stream:
//     out = norm(alpha * x + y) * gain,      norm(v) = v / sqrt(mean(v^2) + eps),
// with y one of
//   * a branch's result (float32 or bfloat16 rows);
//   * two branches' results (float32 rows), each normed on its own: mult * (norm(a) * gain_a + norm(b) * gain_b);
//   * the chosen experts' rows of a routed feed-forward, weighed and summed here (float32, in the order of the choice);
// and the sum of a normed branch, out = x + norm(y) * gain. Each also writes the new stream rounded to the model dtype for
// the sublayers that read it. Then the gate of a per-token input: gelu_tanh(z) * the token's row of a table.
// A block per token; the row sits in shared memory as float32; V neighbouring entries a thread at a time.
#include "common.cuh"

namespace {

enum { PN_BRANCH = 0, PN_PAIR = 1, PN_EXPERTS = 2, PN_ADD = 3 };

struct PostNormArgs {
  const float* x;
  const void* y;               // PN_BRANCH, PN_ADD: rows of TA; PN_PAIR: the first branch, float32; PN_EXPERTS: float32 [pairs, width]
  const float* y2;             // PN_PAIR: the second branch
  const float* gain_a;
  const float* gain_b;
  const float* gates;          // PN_EXPERTS: [tokens, top]
  const int* row_of_pair;      // PN_EXPERTS: [tokens * top]
  const float* gain;
  float* out;
  void* copy;                  // the new stream in TO, or null
  int width, top;
  float alpha, mult, eps, eps_branch;
};

template <int V> __device__ __forceinline__ void get(const float* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    f[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void get(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
  } else {
    f[0] = __bfloat162float(*p);
  }
}
template <int V> __device__ __forceinline__ void put(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int V> __device__ __forceinline__ void put(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(f[0]);
  }
}

template <typename TA, typename TO, int KIND, int V>
__global__ void post_norm_kernel(PostNormArgs p) {
  extern __shared__ __align__(16) float row[];     // PN_PAIR: two rows
  __shared__ float scratch[32];
  const size_t t = blockIdx.x, base = t * p.width;
  const int step = blockDim.x * V, first = threadIdx.x * V, width = p.width;
  float ra = 0.f, rb = 0.f;
  if constexpr (KIND == PN_PAIR || KIND == PN_ADD) {
    float qa = 0.f, qb = 0.f;
    for (int i = first; i < width; i += step) {
      float a[V];
      if constexpr (KIND == PN_PAIR) get<V>(static_cast<const float*>(p.y) + base + i, a);
      else get<V>(static_cast<const TA*>(p.y) + base + i, a);
      put<V>(row + i, a);
#pragma unroll
      for (int e = 0; e < V; ++e) qa = fmaf(a[e], a[e], qa);
      if constexpr (KIND == PN_PAIR) {
        float b[V];
        get<V>(p.y2 + base + i, b);
        put<V>(row + width + i, b);
#pragma unroll
        for (int e = 0; e < V; ++e) qb = fmaf(b[e], b[e], qb);
      }
    }
    ra = 1.0f / sqrtf(block_sum(qa, scratch) / float(width) + p.eps_branch);
    if constexpr (KIND == PN_PAIR) rb = 1.0f / sqrtf(block_sum(qb, scratch) / float(width) + p.eps_branch);
  }
  float q = 0.f;
  for (int i = first; i < width; i += step) {
    float x[V], y[V];
    get<V>(p.x + base + i, x);
    if constexpr (KIND == PN_BRANCH) {
      get<V>(static_cast<const TA*>(p.y) + base + i, y);
    } else if constexpr (KIND == PN_EXPERTS) {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
      for (int k = 0; k < p.top; ++k) {
        const int r = p.row_of_pair[t * p.top + k];
        const float g = p.gates[t * p.top + k];
        float v[V];
        get<V>(static_cast<const float*>(p.y) + size_t(r) * width + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(g, v[e], y[e]);
      }
    } else if constexpr (KIND == PN_PAIR) {
      float a[V], b[V], ga[V], gb[V];
      get<V>(row + i, a);
      get<V>(row + width + i, b);
      get<V>(p.gain_a + i, ga);
      get<V>(p.gain_b + i, gb);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = p.mult * (a[e] * ra * ga[e] + b[e] * rb * gb[e]);
    } else {
      float a[V], g[V];
      get<V>(row + i, a);
      get<V>(p.gain + i, g);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = a[e] * ra * g[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      x[e] = fmaf(p.alpha, x[e], y[e]);
      q = fmaf(x[e], x[e], q);
    }
    if constexpr (KIND == PN_ADD) {
      put<V>(p.out + base + i, x);
      if (p.copy) put<V>(static_cast<TO*>(p.copy) + base + i, x);
    } else {
      put<V>(row + i, x);       // an entry is read and written by one thread only
    }
  }
  if constexpr (KIND == PN_ADD) return;
  const float rstd = 1.0f / sqrtf(block_sum(q, scratch) / float(width) + p.eps);
  for (int i = first; i < width; i += step) {
    float v[V], g[V];
    get<V>(row + i, v);
    get<V>(p.gain + i, g);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = v[e] * rstd * g[e];
    put<V>(p.out + base + i, v);
    if (p.copy) put<V>(static_cast<TO*>(p.copy) + base + i, v);
  }
}

template <typename TA, typename TO, int KIND, int V>
int launch_post_norm_v(const PostNormArgs& p, int n, cudaStream_t stream) {
  const size_t smem = size_t(p.width) * sizeof(float) * (KIND == PN_PAIR ? 2 : 1);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (cudaFuncSetAttribute(post_norm_kernel<TA, TO, KIND, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess)
      return PTB_ERR_LAUNCH;
    configured = smem;
  }
  const int units = (p.width + V - 1) / V;
  const int threads = units >= 512 ? 512 : (units >= 256 ? 256 : (units >= 128 ? 128 : 64));
  post_norm_kernel<TA, TO, KIND, V><<<n, threads, smem, stream>>>(p);
  return launch_status();
}

template <typename TA, int KIND>
int launch_post_norm(const PostNormArgs& p, int copy_dtype, int n, cudaStream_t stream) {
  const size_t a_word = 4 * sizeof(TA);
  const bool vec = p.width % 4 == 0 && aligned16(p.x) && aligned16(p.out) && aligned16(p.gain) &&
                   reinterpret_cast<uintptr_t>(p.y) % a_word == 0 && (p.y2 == nullptr || aligned16(p.y2)) &&
                   (p.gain_a == nullptr || (aligned16(p.gain_a) && aligned16(p.gain_b))) &&
                   reinterpret_cast<uintptr_t>(p.copy) % (copy_dtype == PTB_BF16 ? 8 : 16) == 0;
  if (copy_dtype == PTB_BF16)
    return vec ? launch_post_norm_v<TA, __nv_bfloat16, KIND, 4>(p, n, stream) : launch_post_norm_v<TA, __nv_bfloat16, KIND, 1>(p, n, stream);
  return vec ? launch_post_norm_v<TA, float, KIND, 4>(p, n, stream) : launch_post_norm_v<TA, float, KIND, 1>(p, n, stream);
}

// out[t][j] = gelu_tanh(z[t][j]) * table[ids[t]][first + j] for j < dim, 0 for j from dim to out_width. An id outside the
// table is clamped and bit 0 of *status is raised.
template <typename TZ, typename T>
__global__ void token_gate_kernel(const TZ* __restrict__ z, int z_width, const int* __restrict__ ids, const T* __restrict__ table,
                                  int rows, int table_width, int first, T* __restrict__ out, int out_width, int dim, int n,
                                  int* __restrict__ status) {
  const long long at = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (at >= (long long)n * out_width) return;
  const int t = int(at / out_width), j = int(at % out_width);
  float v = 0.f;
  if (j < dim) {
    int id = ids[t];
    if (id < 0 || id >= rows) {
      if (status) atomicOr(status, 1);
      id = min(max(id, 0), rows - 1);
    }
    v = apply_activation(to_f(z[size_t(t) * z_width + j]), PTB_ACT_GELU_TANH) * to_f(table[size_t(id) * table_width + first + j]);
  }
  out[at] = from_f<T>(v);
}

__global__ void round_rows_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ y, size_t total) {
  const size_t stride = size_t(gridDim.x) * blockDim.x;
  for (size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) y[i] = __float2bfloat16_rn(x[i]);
}

}  // namespace

// kind 0: y of y_dtype; 1: y and y2 float32 with gain_a, gain_b; 2: y float32 expert rows with gates and row_of_pair;
// 3: out = x + norm(y) * gain (alpha is one, eps_branch the norm's eps). copy: null or [n, width] of copy_dtype.
PTB_API int ptb_post_norm(int kind, const float* x, int y_dtype, const void* y, const float* y2, const float* gain_a,
                          const float* gain_b, const float* gates, const int* row_of_pair, int top, const float* gain, float* out,
                          int copy_dtype, void* copy, int n, int width, float alpha, float mult, float eps, float eps_branch,
                          cudaStream_t stream) {
  if (n <= 0) return PTB_OK;
  if (width <= 0 || size_t(width) * 8 > 200 * 1024 || kind < 0 || kind > 3) return PTB_ERR_SIZE;
  if ((kind == PN_PAIR && (y2 == nullptr || gain_a == nullptr || gain_b == nullptr || y_dtype != PTB_F32)) ||
      (kind == PN_EXPERTS && (gates == nullptr || row_of_pair == nullptr || top <= 0 || y_dtype != PTB_F32)))
    return PTB_ERR_SIZE;
  if ((y_dtype != PTB_F32 && y_dtype != PTB_BF16) || (copy != nullptr && copy_dtype != PTB_F32 && copy_dtype != PTB_BF16))
    return PTB_ERR_DTYPE;
  const PostNormArgs p{x, y, y2, gain_a, gain_b, gates, row_of_pair, gain, out, copy, width, top, alpha, mult, eps, eps_branch};
  const int cd = copy == nullptr ? PTB_F32 : copy_dtype;
  if (kind == PN_PAIR) return launch_post_norm<float, PN_PAIR>(p, cd, n, stream);
  if (kind == PN_EXPERTS) return launch_post_norm<float, PN_EXPERTS>(p, cd, n, stream);
  if (kind == PN_ADD)
    return y_dtype == PTB_F32 ? launch_post_norm<float, PN_ADD>(p, cd, n, stream) : launch_post_norm<__nv_bfloat16, PN_ADD>(p, cd, n, stream);
  return y_dtype == PTB_F32 ? launch_post_norm<float, PN_BRANCH>(p, cd, n, stream)
                            : launch_post_norm<__nv_bfloat16, PN_BRANCH>(p, cd, n, stream);
}

// z: [n, z_width] float32 or of `dtype`; table and out of `dtype`; out [n, out_width].
PTB_API int ptb_token_gate(int z_dtype, const void* z, int z_width, const int* ids, int dtype, const void* table, int rows,
                           int table_width, int first, void* out, int out_width, int dim, int n, int* status,
                           cudaStream_t stream) {
  if (n <= 0) return PTB_OK;
  if (dim <= 0 || out_width < dim || z_width < dim || rows <= 0 || first < 0 || first + dim > table_width) return PTB_ERR_SIZE;
  const unsigned blocks = unsigned(((long long)n * out_width + 255) / 256);
  if (z_dtype != PTB_F32) return PTB_ERR_DTYPE;
  if (dtype == PTB_F32)
    token_gate_kernel<float, float><<<blocks, 256, 0, stream>>>((const float*)z, z_width, ids, (const float*)table, rows, table_width,
                                                                first, (float*)out, out_width, dim, n, status);
  else if (dtype == PTB_BF16)
    token_gate_kernel<float, __nv_bfloat16><<<blocks, 256, 0, stream>>>((const float*)z, z_width, ids, (const __nv_bfloat16*)table,
                                                                        rows, table_width, first, (__nv_bfloat16*)out, out_width, dim,
                                                                        n, status);
  else
    return PTB_ERR_DTYPE;
  return launch_status();
}

// float32 values rounded to bfloat16
PTB_API int ptb_round_rows(const float* x, void* y, long long total, cudaStream_t stream) {
  if (total <= 0) return PTB_OK;
  const size_t want = (size_t(total) + 255) / 256, most = size_t(sm_count()) * 16;
  round_rows_kernel<<<int(want < most ? want : most), 256, 0, stream>>>(x, (__nv_bfloat16*)y, size_t(total));
  return launch_status();
}
