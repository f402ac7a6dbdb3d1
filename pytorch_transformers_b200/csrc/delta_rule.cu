// The gated delta rule: a key-value state that fades and is corrected towards the values at the keys it is asked for.
//
// Per head, with q_t, k_t [dim] unit vectors (q also times dim^-1/2), v_t [v_dim], l_t the logarithms of the decays (one
// per head, or one per key channel) and beta_t in (0, 1):
//     S <- diag(exp(l_t)) S,   u = beta_t (v_t - S^T k_t),   S <- S + k_t u^T,   o_t = S^T q_t,      S = 0 before the first token.
// q, k and v come from projections through a short causal convolution per channel and silu; several heads may share one
// query/key head (head h reads h / (heads / kv_heads)).
//
// A sequence's state in the cache's state area (float32): the convolution's last taps - 1 inputs, [taps - 1][channels]
// with channels = q's, k's, v's side by side, then S, laid out [heads][v_dim][dim] so that a column of S is contiguous.
//
// Three kernels: one that forms what enters the recurrence (convolution, silu, the heads' norms, decays, beta), one that
// keeps the convolution's last inputs after a step of several tokens, and one that walks tokens in order with S in
// registers. Prompts in bfloat16 with keys and values of 64 or 128 entries run in chunks instead (csrc/delta_rule_mma.cu).
#include "common.cuh"

namespace {

constexpr int MAX_TAPS = 64;
constexpr int PREP_WARPS = 8;
constexpr int PREP_RUN = 8;           // tokens of a warp in steps of many tokens
constexpr int FAST_TAPS = 4;          // the filter length whose inputs are held in registers
constexpr float UNIT_EPS = 1e-6f;     // inside the root of the unit vectors' norm

__device__ __forceinline__ float silu_of(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// V neighbouring values as floats
template <int V> struct Vals { float f[V]; };
template <int V> __device__ __forceinline__ Vals<V> load_vals(const float* p) {
  Vals<V> r;
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    r.f[0] = x.x; r.f[1] = x.y; r.f[2] = x.z; r.f[3] = x.w;
  } else {
    r.f[0] = *p;
  }
  return r;
}
template <int V> __device__ __forceinline__ Vals<V> load_vals(const __nv_bfloat16* p) {
  Vals<V> r;
  if constexpr (V == 4) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    r.f[0] = __uint_as_float(x.x << 16); r.f[1] = __uint_as_float(x.x & 0xffff0000u);
    r.f[2] = __uint_as_float(x.y << 16); r.f[3] = __uint_as_float(x.y & 0xffff0000u);
  } else {
    r.f[0] = __bfloat162float(*p);
  }
  return r;
}
template <int V> __device__ __forceinline__ void store_vals(float* p, const Vals<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.f[0], r.f[1], r.f[2], r.f[3]);
  else *p = r.f[0];
}
template <int V> __device__ __forceinline__ void store_vals(__nv_bfloat16* p, const Vals<V>& r) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(r.f[0], r.f[1]), b = __floats2bfloat162_rn(r.f[2], r.f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(r.f[0]);
  }
}

struct DeltaSizes {
  int heads, kv_heads, dim, v_dim, taps;
  __host__ __device__ int qk() const { return kv_heads * dim; }
  __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * v_dim; }
};

// A warp per (run of RUN tokens, unit). Units: the 2 kv_heads query and key heads (convolution, silu, inverse norm), the
// values in stretches of 128 channels (convolution, silu), the decays' logarithms per channel in stretches of 128
// (DECAY_CHANNEL), and one unit with beta and the decays' logarithms per head.
//   proj row t: [q | k | v] then, at b_off and a_off, the projections of beta and of the decay per head; z (float32 rows
//   z_stride apart): the decay's projection per channel.
//   act [tokens][channels] (T): the activated convolutions, rounded to T; inv [tokens][2 kv_heads]: what a query and a key
//   head is multiplied by to be a unit vector (queries: also dim^-1/2); logd [tokens][heads * dim or heads]; beta [tokens][heads].
// With `single` (one new token a sequence) the convolution's kept inputs are moved on here, each by the thread that read it.
//
// RUN > 1 (steps of many tokens): a warp's RUN neighbouring tokens of one sequence under a filter of FAST_TAPS taps have all
// their inputs loaded before the first is used, each once; runs that span sequences, other taps and wide heads go token by
// token. The sums are formed in the same order either way.
template <typename T, int V, int RUN>
__global__ void __launch_bounds__(32 * PREP_WARPS)
delta_prepare_kernel(const T* __restrict__ proj, int stride, const float* __restrict__ conv_w, float* __restrict__ state,
                     int state_stride, const int* __restrict__ slots, StepBatch sb, T* __restrict__ act,
                     float* __restrict__ inv, int b_off, int a_off, const float* __restrict__ z, int z_stride,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ logd,
                     float* __restrict__ beta, DeltaSizes sz, int single, float q_scale) {
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int C = sz.channels(), qk = sz.qk(), hv = sz.heads * sz.v_dim, hd = sz.heads * sz.dim, keep = sz.taps - 1;
  const int n_heads = 2 * sz.kv_heads, n_v = (hv + 127) / 128, n_d = z ? (hd + 127) / 128 : 0;
  const int unit = blockIdx.y * PREP_WARPS + warp;
  if (unit > n_heads + n_v + n_d) return;
  const int t0 = blockIdx.x * RUN, t1 = min(t0 + RUN, sb.n_tokens);
  if (z != nullptr && unit >= n_heads + n_v && unit < n_heads + n_v + n_d) {
    const int c0 = (unit - n_heads - n_v) * 128;
    if (V == 4 && (z_stride & 3) == 0) {       // four channels of one head a lane (the host checks: dim a multiple of 4)
      const int c = c0 + lane * 4;
      if (c >= hd) return;
      const float a = -expf(a_log[c / sz.dim]);
      const Vals<V> bias = load_vals<V>(dt_bias + c);
#pragma unroll 4
      for (int t = t0; t < t1; ++t) {
        Vals<V> x = load_vals<V>(z + size_t(t) * z_stride + c);
#pragma unroll
        for (int e = 0; e < V; ++e) x.f[e] = a * softplus_of(x.f[e] + bias.f[e]);
        store_vals<V>(logd + size_t(t) * hd + c, x);
      }
      return;
    }
    for (int u = 0; u < 4; ++u) {
      const int c = c0 + u * 32 + lane;
      if (c >= hd) return;
      const float a = -expf(a_log[c / sz.dim]);
      for (int t = t0; t < t1; ++t) logd[size_t(t) * hd + c] = a * softplus_of(z[size_t(t) * z_stride + c] + dt_bias[c]);
    }
    return;
  }
  if constexpr (RUN > 1) {
    constexpr int KEEP = FAST_TAPS - 1;
    const bool norm = unit < n_heads;
    const int c0 = norm ? unit * sz.dim : 2 * qk + (unit - n_heads) * 128, n = norm ? sz.dim : min(128, C - c0);
    const int seq = sb.tok_seq[t0];
    if (unit < n_heads + n_v && sz.taps == FAST_TAPS && n <= 32 * V && t1 == t0 + RUN && sb.tok_seq[t1 - 1] == seq) {
      const int i0 = t0 - sb.seq_start[seq], c = c0 + lane * V;
      const bool on = lane * V < n;
      Vals<V> x[KEEP + RUN], w[FAST_TAPS];
      if (on) {
        const float* st = state + size_t(slots[seq]) * state_stride + c;
#pragma unroll
        for (int r = 0; r < KEEP + RUN; ++r) {
          const int li = i0 + r - KEEP;
          x[r] = li >= 0 ? load_vals<V>(proj + size_t(t0 + r - KEEP) * stride + c) : load_vals<V>(st + size_t(KEEP + li) * C);
        }
#pragma unroll
        for (int tap = 0; tap < FAST_TAPS; ++tap) w[tap] = load_vals<V>(conv_w + size_t(tap) * C + c);
      }
#pragma unroll
      for (int r = 0; r < RUN; ++r) {
        float ss = 0.f;
        if (on) {
          Vals<V> y;
#pragma unroll
          for (int e = 0; e < V; ++e) {
            float v = 0.f;
#pragma unroll
            for (int tap = 0; tap < FAST_TAPS; ++tap) v = fmaf(w[tap].f[e], x[r + tap].f[e], v);
            y.f[e] = to_f(from_f<T>(silu_of(v)));
            ss = fmaf(y.f[e], y.f[e], ss);
          }
          store_vals<V>(act + size_t(t0 + r) * C + c, y);
        }
        if (norm) {
          const float q = 1.0f / sqrtf(warp_sum(ss) + UNIT_EPS);
          if (lane == 0) inv[size_t(t0 + r) * n_heads + unit] = unit < sz.kv_heads ? q * q_scale : q;
        }
      }
      return;
    }
  }
  for (int t = t0; t < t1; ++t) {
    if (unit < n_heads + n_v) {
      const int seq = sb.tok_seq[t], i = t - sb.seq_start[seq];
      float* st = keep > 0 ? state + size_t(slots[seq]) * state_stride : nullptr;
      const bool norm = unit < n_heads;
      const int c0 = norm ? unit * sz.dim : 2 * qk + (unit - n_heads) * 128;
      const int n = norm ? sz.dim : min(128, C - c0);
      float ss = 0.f;
      for (int j = lane * V; j < n; j += 32 * V) {
        const int c = c0 + j;
        Vals<V> y;
#pragma unroll
        for (int e = 0; e < V; ++e) y.f[e] = 0.f;
#pragma unroll 4
        for (int tap = 0; tap < sz.taps; ++tap) {
          const int li = i - (keep - tap);            // place among the sequence's new tokens; before them: the kept inputs
          const Vals<V> x = li >= 0 ? load_vals<V>(proj + size_t(t - (keep - tap)) * stride + c)
                                    : load_vals<V>(st + size_t(keep + li) * C + c);
          const Vals<V> w = load_vals<V>(conv_w + size_t(tap) * C + c);
#pragma unroll
          for (int e = 0; e < V; ++e) y.f[e] = fmaf(w.f[e], x.f[e], y.f[e]);
        }
        if (single && keep > 0) {
          for (int r = 0; r + 1 < keep; ++r) store_vals<V>(st + size_t(r) * C + c, load_vals<V>(st + size_t(r + 1) * C + c));
          store_vals<V>(st + size_t(keep - 1) * C + c, load_vals<V>(proj + size_t(t) * stride + c));
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
          y.f[e] = to_f(from_f<T>(silu_of(y.f[e])));
          ss = fmaf(y.f[e], y.f[e], ss);
        }
        store_vals<V>(act + size_t(t) * C + c, y);
      }
      if (norm) {
        const float r = 1.0f / sqrtf(warp_sum(ss) + UNIT_EPS);
        if (lane == 0) inv[size_t(t) * n_heads + unit] = unit < sz.kv_heads ? r * q_scale : r;
      }
    } else {
      for (int h = lane; h < sz.heads; h += 32) {
        beta[size_t(t) * sz.heads + h] = 1.f / (1.f + expf(-to_f(proj[size_t(t) * stride + b_off + h])));
        if (z == nullptr)
          logd[size_t(t) * sz.heads + h] =
              -expf(a_log[h]) * softplus_of(to_f(proj[size_t(t) * stride + a_off + h]) + dt_bias[h]);
      }
    }
  }
}

// The convolution's last taps - 1 inputs after a step: a thread per (sequence, channel), rows in ascending order (a row
// is read before it is written: what moves into row r comes from a row further on, or from the step's projections).
template <typename T>
__global__ void delta_keep_kernel(const T* __restrict__ proj, int stride, float* __restrict__ state, int state_stride,
                                  const int* __restrict__ slots, StepBatch sb, int channels, int keep) {
  const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int start = sb.seq_start[seq], n = sb.seq_new[seq];
  if (n <= 0) return;
  float* st = state + size_t(slots[seq]) * state_stride + c;
  for (int r = 0; r < keep; ++r) {
    const int li = n - keep + r;
    st[size_t(r) * channels] = li >= 0 ? to_f(proj[size_t(start + li) * stride + c]) : st[size_t(keep + li) * channels];
  }
}

// four sums over a warp's lanes: lane l gets the total of value l / 8 (a fixed order whatever else runs)
__device__ __forceinline__ float reduce4(const float (&v)[4], int lane) {
  const unsigned full = 0xffffffffu;
  const bool up = lane & 16, up8 = lane & 8;
  const float a = (up ? v[2] : v[0]) + __shfl_xor_sync(full, up ? v[0] : v[2], 16);
  const float b = (up ? v[3] : v[1]) + __shfl_xor_sync(full, up ? v[1] : v[3], 16);
  float s = (up8 ? b : a) + __shfl_xor_sync(full, up8 ? a : b, 8);
  s += __shfl_xor_sync(full, s, 4);
  s += __shfl_xor_sync(full, s, 2);
  s += __shfl_xor_sync(full, s, 1);
  return s;
}

// A warp owns four columns of S, lane l the rows l, l + 32, ...; the tokens of a sequence in order, the next token's
// values on their way while one is computed. Warps share nothing. grid (sequences, heads, column groups).
constexpr int WALK_WARPS = 4, WALK_COLS = 4;
template <typename T, int R, bool PER_HEAD>
__global__ void __launch_bounds__(32 * WALK_WARPS)
delta_walk_kernel(const T* __restrict__ act, const float* __restrict__ inv, const float* __restrict__ logd,
                  const float* __restrict__ beta, float* __restrict__ state, int state_stride, const int* __restrict__ slots,
                  StepBatch sb, float* __restrict__ out, DeltaSizes sz) {
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int seq = blockIdx.x, h = blockIdx.y, j0 = (blockIdx.z * WALK_WARPS + warp) * WALK_COLS;
  if (j0 >= sz.v_dim) return;
  const int dim = sz.dim, v_dim = sz.v_dim, C = sz.channels(), qk = sz.qk(), G = sz.kv_heads, g = h / (sz.heads / G);
  const int start = sb.seq_start[seq], n = sb.seq_new[seq];
  float* st = state + size_t(slots[seq]) * state_stride + size_t(sz.taps - 1) * C + (size_t(h) * v_dim + j0) * dim;
  float S[WALK_COLS][R];
#pragma unroll
  for (int c = 0; c < WALK_COLS; ++c)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = lane + 32 * r;
      S[c][r] = (j0 + c < v_dim && d < dim) ? st[size_t(c) * dim + d] : 0.f;
    }
  const int col = lane / 8;                    // the column whose sums this lane gets
  const bool col_on = j0 + col < v_dim;
  constexpr int L = PER_HEAD ? 1 : R;
  T qn[R], kn[R], vn;
  float ln[L], bn, rqn, rkn;
  auto fetch = [&](int t) {
    const T* row = act + size_t(t) * C;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = min(lane + 32 * r, dim - 1);      // a row past the end reads the last one and is multiplied by a zero state
      qn[r] = row[g * dim + d];
      kn[r] = row[qk + g * dim + d];
      if constexpr (!PER_HEAD) ln[r] = logd[(size_t(t) * sz.heads + h) * dim + d];
    }
    if constexpr (PER_HEAD) ln[0] = logd[size_t(t) * sz.heads + h];
    vn = row[2 * qk + h * v_dim + min(j0 + col, v_dim - 1)];
    bn = beta[size_t(t) * sz.heads + h];
    rqn = inv[size_t(t) * 2 * G + g];
    rkn = inv[size_t(t) * 2 * G + G + g];
  };
  if (n > 0) fetch(start);
  for (int i = 0; i < n; ++i) {
    float q[R], k[R], e[L];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const bool on = lane + 32 * r < dim;
      q[r] = on ? to_f(qn[r]) * rqn : 0.f;
      k[r] = on ? to_f(kn[r]) * rkn : 0.f;
    }
#pragma unroll
    for (int r = 0; r < L; ++r) e[r] = expm1f(ln[r]);
    const float v = to_f(vn), b = bn;
    if (i + 1 < n) fetch(start + i + 1);
    float sums[WALK_COLS];
#pragma unroll
    for (int c = 0; c < WALK_COLS; ++c) {
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        S[c][r] = fmaf(e[PER_HEAD ? 0 : r], S[c][r], S[c][r]);
        s = fmaf(k[r], S[c][r], s);
      }
      sums[c] = s;
    }
    const float mine = b * (v - reduce4(sums, lane));
    float o[WALK_COLS];
#pragma unroll
    for (int c = 0; c < WALK_COLS; ++c) {
      const float u = __shfl_sync(0xffffffffu, mine, c * 8);
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        S[c][r] = fmaf(k[r], u, S[c][r]);
        s = fmaf(q[r], S[c][r], s);
      }
      o[c] = s;
    }
    const float total = reduce4(o, lane);
    if ((lane & 7) == 0 && col_on) out[(size_t(start + i) * sz.heads + h) * v_dim + j0 + col] = total;
  }
#pragma unroll
  for (int c = 0; c < WALK_COLS; ++c)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = lane + 32 * r;
      if (j0 + c < v_dim && d < dim) st[size_t(c) * dim + d] = S[c][r];
    }
}

template <typename T>
int launch_delta_walk(const void* act, const float* inv, const float* logd, const float* beta, float* state, int state_stride,
                      const int* slots, const StepBatch& sb, float* out, const DeltaSizes& sz, int per_head,
                      cudaStream_t stream) {
  const int cols = WALK_WARPS * WALK_COLS;
  const dim3 grid(sb.n_seqs, sz.heads, (sz.v_dim + cols - 1) / cols);
#define PTB_WALK(R)                                                                                                       \
  do {                                                                                                                    \
    if (per_head)                                                                                                         \
      delta_walk_kernel<T, R, true><<<grid, 32 * WALK_WARPS, 0, stream>>>((const T*)act, inv, logd, beta, state,          \
                                                                          state_stride, slots, sb, out, sz);              \
    else                                                                                                                  \
      delta_walk_kernel<T, R, false><<<grid, 32 * WALK_WARPS, 0, stream>>>((const T*)act, inv, logd, beta, state,         \
                                                                           state_stride, slots, sb, out, sz);             \
  } while (0)
  if (sz.dim <= 32) PTB_WALK(1);
  else if (sz.dim <= 64) PTB_WALK(2);
  else if (sz.dim <= 128) PTB_WALK(4);
  else PTB_WALK(8);
#undef PTB_WALK
  return launch_status();
}

bool sizes_ok(const DeltaSizes& sz) {
  return sz.heads > 0 && sz.kv_heads > 0 && sz.heads % sz.kv_heads == 0 && sz.heads <= 65535 && sz.dim > 0 && sz.dim <= 256 &&
         sz.v_dim > 0 && sz.taps >= 1 && sz.taps <= MAX_TAPS;
}

}  // namespace

PTB_API int ptb_delta_max_dim() { return 256; }
PTB_API int ptb_delta_max_taps() { return MAX_TAPS; }

// What enters the recurrence (delta_prepare_kernel says what each array holds), and the convolution's kept inputs moved
// on. z null: one decay per head, whose projection lies in proj at a_off. conv_w float32 [taps][channels].
PTB_API int ptb_delta_prepare(int dtype, const void* proj, int stride, const float* conv_w, float* state, int state_stride,
                              const int* slots, const StepBatch* sb, void* act, float* inv, int b_off, int a_off,
                              const float* z, int z_stride, const float* a_log, const float* dt_bias, float* logd, float* beta,
                              int heads, int kv_heads, int dim, int v_dim, int taps, float q_scale, int single,
                              cudaStream_t stream) {
  if (sb->n_tokens <= 0 || sb->n_seqs <= 0) return PTB_OK;
  const DeltaSizes sz{heads, kv_heads, dim, v_dim, taps};
  if (!sizes_ok(sz) || stride < sz.channels() || b_off < 0 || b_off + heads > stride || sb->n_seqs > 65535 ||
      (z == nullptr && (a_off < 0 || a_off + heads > stride)) || (z != nullptr && z_stride < heads * dim))
    return PTB_ERR_SIZE;
  if (dtype != PTB_F32 && dtype != PTB_BF16) return PTB_ERR_DTYPE;
  const int hv = heads * v_dim, units = 2 * kv_heads + (hv + 127) / 128 + (z ? (heads * dim + 127) / 128 : 0) + 1;
  const int run = sb->n_tokens >= 4 * sm_count() ? PREP_RUN : 1;
  const dim3 grid((sb->n_tokens + run - 1) / run, (units + PREP_WARPS - 1) / PREP_WARPS);
  if (grid.y > 65535) return PTB_ERR_SIZE;
  const size_t word = dtype == PTB_F32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && hv % 4 == 0 && stride % 4 == 0 && state_stride % 4 == 0 &&
                   reinterpret_cast<uintptr_t>(proj) % word == 0 && reinterpret_cast<uintptr_t>(act) % word == 0 &&
                   aligned16(conv_w) && (taps == 1 || aligned16(state)) &&
                   (z == nullptr || (aligned16(z) && aligned16(dt_bias)));
#define PTB_PREP2(TT, VV, RR)                                                                                                  \
  delta_prepare_kernel<TT, VV, RR><<<grid, 32 * PREP_WARPS, 0, stream>>>((const TT*)proj, stride, conv_w, state, state_stride, \
                                                                         slots, *sb, (TT*)act, inv, b_off, a_off, z, z_stride,  \
                                                                         a_log, dt_bias, logd, beta, sz, single, q_scale)
#define PTB_PREP(TT)                                        \
  do {                                                      \
    if (vec && run > 1) PTB_PREP2(TT, 4, PREP_RUN);         \
    else if (vec) PTB_PREP2(TT, 4, 1);                      \
    else if (run > 1) PTB_PREP2(TT, 1, PREP_RUN);           \
    else PTB_PREP2(TT, 1, 1);                               \
  } while (0)
  if (dtype == PTB_F32) PTB_PREP(float);
  else PTB_PREP(__nv_bfloat16);
#undef PTB_PREP2
#undef PTB_PREP
  if (launch_status() != PTB_OK) return PTB_ERR_LAUNCH;
  if (single || taps == 1) return PTB_OK;
  const dim3 kgrid((sz.channels() + 255) / 256, sb->n_seqs);
  if (dtype == PTB_F32)
    delta_keep_kernel<float><<<kgrid, 256, 0, stream>>>((const float*)proj, stride, state, state_stride, slots, *sb,
                                                        sz.channels(), taps - 1);
  else
    delta_keep_kernel<__nv_bfloat16><<<kgrid, 256, 0, stream>>>((const __nv_bfloat16*)proj, stride, state, state_stride, slots,
                                                                *sb, sz.channels(), taps - 1);
  return launch_status();
}

// The step's tokens, every sequence walked in order from and to its state; act, inv, logd, beta as ptb_delta_prepare
// leaves them; out float32 [tokens, heads * v_dim].
PTB_API int ptb_delta_walk(int dtype, const void* act, const float* inv, const float* logd, const float* beta, float* state,
                           int state_stride, const int* slots, const StepBatch* sb, float* out, int heads, int kv_heads, int dim,
                           int v_dim, int taps, int per_head, cudaStream_t stream) {
  if (sb->n_tokens <= 0 || sb->n_seqs <= 0) return PTB_OK;
  const DeltaSizes sz{heads, kv_heads, dim, v_dim, taps};
  if (!sizes_ok(sz) || state_stride < (taps - 1) * sz.channels() + heads * dim * v_dim ||
      (v_dim + WALK_WARPS * WALK_COLS - 1) / (WALK_WARPS * WALK_COLS) > 65535)
    return PTB_ERR_SIZE;
  if (dtype == PTB_F32)
    return launch_delta_walk<float>(act, inv, logd, beta, state, state_stride, slots, *sb, out, sz, per_head, stream);
  if (dtype == PTB_BF16)
    return launch_delta_walk<__nv_bfloat16>(act, inv, logd, beta, state, state_stride, slots, *sb, out, sz, per_head, stream);
  return PTB_ERR_DTYPE;
}
