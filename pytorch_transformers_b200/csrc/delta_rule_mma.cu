// The gated delta rule in chunks of 64 tokens on the tensor cores (bfloat16 projections, mma.m16n8k16 with float32 sums).
//
// Inside a chunk of n <= 64 tokens let c_t be the sum of the decays' logarithms up to and including token t (a vector over
// key channels), S_0 the state before the chunk, and
//     L[t][s] = beta_t sum_d k_t[d] k_s[d] exp(c_t[d] - c_s[d])   for s < t,      P[t][s] = sum_d q_t[d] k_s[d] exp(c_t[d] - c_s[d])   for s <= t.
// The corrections u_t of the chunk's tokens solve (I + L) U = diag(beta) (V - Kc S_0) with Kc_t = k_t exp(c_t). With
// T = (I + L)^-1 diag(beta), W = T Kc and U_0 = T V (so U = U_0 - W S_0), Qc_t = q_t exp(c_t) and Kd_s = k_s exp(c_n - c_s):
//     S_n = diag(exp(c_n)) S_0 + B + M S_0,     B = Kd^T U_0,   M = -Kd^T W,
//     O   = O_0 + Q S_0,                        O_0 = P U_0,    Q = Qc - P W.
// Pass 1 (parallel over chunks and heads) forms M, Q, B, O_0 and exp(c_n); pass 2 walks a sequence's chunks in order with
// the state's float32 values in registers, one product [M; Q] S_0 a chunk, and writes the outputs.
//
// No factor can grow: inside a sub-block of 16 tokens sums of logarithms start at the sub-block, the exponent between two
// sub-blocks is the rest of the earlier one, the whole ones between and the beginning of the later one, and inside a
// sub-block the exponent of every pair of tokens is formed by itself. Float32 operands (the state, decayed keys and
// queries, T, P, W, U_0) enter the products split in two bfloat16 terms, hi hi + hi lo + lo hi; projections are bfloat16 as
// they are, their unit norms factors of the results.
#include "chunk_mma.cuh"

namespace {

constexpr float LOG2E_F = 1.4426950408889634f;

// hi and lo terms of two neighbouring values of a row of a swizzled [rows][D] tile
template <int D>
__device__ __forceinline__ void put_split(unsigned char* hi_tile, unsigned char* lo_tile, int row, int col, float x, float y) {
  uint32_t hi, lo;
  split_pack(x, y, hi, lo);
  const uint32_t off = swz<D>(row, col >> 3) + (col & 7) * 2;
  *reinterpret_cast<uint32_t*>(hi_tile + off) = hi;
  *reinterpret_cast<uint32_t*>(lo_tile + off) = lo;
}

template <int DK, int DV, bool PER_HEAD>
struct LocalSmem {
  static constexpr int KP = DK + 8, CP = PER_HEAD ? 1 : DK + 8, TP = CH + 1;
  static constexpr int cb = 0;                                   // [CH][CP] float: sums of logarithms from the sub-block's start
  static constexpr int tot = cb + (CH * CP * 4 + 127) / 128 * 128;   // [4][DK] float: the sub-blocks' totals
  static constexpr int q = tot + (PER_HEAD ? 128 : 4 * DK * 4);  // [CH][KP] bfloat16
  static constexpr int k = q + CH * KP * 2;
  static constexpr int v = k + CH * KP * 2;                      // [CH][DV] swizzled: values, then U_0's hi
  static constexpr int a = v + CH * DV * 2;                      // [CH][TP] float: L, then T diag(beta) hi and lo [CH][CH]
  static constexpr int p = a + CH * TP * 4;                      // P hi and lo [CH][CH]
  static constexpr int t = p + 2 * CH * CH * 2;                  // [CH][TP] float: (I + L)^-1
  static constexpr int x = t + CH * TP * 4;                      // [3][16][16] float
  static constexpr int kw = x + 3 * 256 * 4;                     // Kc hi and lo [CH][DK], then W
  static constexpr int ulo = kw + 2 * CH * DK * 2;               // [CH][DV]: U_0's lo
  static constexpr int kd = ulo + CH * DV * 2;                   // Kd hi and lo [CH][DK]
  static constexpr int small = kd + 2 * CH * DK * 2;             // rq, rk, beta [CH] float each
  static constexpr int bytes = small + 3 * CH * 4;
};

// One block = one chunk x one head; DK / 8 warps.
// mq [chunk][head][DK / 16 + 4 row tiles][DK / 16][hi, lo][32 lanes] 16-byte words: M's rows, then Q's, as mma A fragments.
// bo [chunk][head][DK / 16 + 4 row tiles][DV / 8][32 lanes] float4: B's rows, then O_0's, as mma C fragments.
// dec [chunk][head][DK]: exp(c_n).
template <int DK, int DV, bool PER_HEAD>
__global__ void __launch_bounds__(DK * 4)
delta_chunk_local_kernel(const __nv_bfloat16* __restrict__ act, const float* __restrict__ inv, const float* __restrict__ logd,
                         const float* __restrict__ beta, StepBatch sb, const int* __restrict__ chunk_seq,
                         const int* __restrict__ chunk_q0, uint4* __restrict__ mq, float4* __restrict__ bo,
                         float* __restrict__ dec, int heads, int kv_heads) {
  using L = LocalSmem<DK, DV, PER_HEAD>;
  extern __shared__ __align__(128) unsigned char sm[];
  constexpr int NW = DK / 8, NT = NW * 32, KP = L::KP, CP = L::CP, TP = L::TP, MT = DK / 16 + 4;
  float* cb = reinterpret_cast<float*>(sm + L::cb);
  float* tot = reinterpret_cast<float*>(sm + L::tot);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(sm + L::q);
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(sm + L::k);
  float* As = reinterpret_cast<float*>(sm + L::a);
  float* Ts = reinterpret_cast<float*>(sm + L::t);
  float* Xs = reinterpret_cast<float*>(sm + L::x);
  unsigned char *p_hi = sm + L::p, *p_lo = p_hi + CH * CH * 2, *t_hi = sm + L::a, *t_lo = t_hi + CH * CH * 2;
  unsigned char *w_hi = sm + L::kw, *w_lo = w_hi + CH * DK * 2, *u_hi = sm + L::v, *u_lo = sm + L::ulo;
  unsigned char *kd_hi = sm + L::kd, *kd_lo = kd_hi + CH * DK * 2;
  float *rq = reinterpret_cast<float*>(sm + L::small), *rk = rq + CH, *bt = rk + CH;
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g4 = lane >> 2, t4 = lane & 3, m = lane >> 3;
  const int seq = chunk_seq[c], q0 = chunk_q0[c];
  const int start = sb.seq_start[seq] + q0, n = min(CH, sb.seq_new[seq] - q0);
  const int g = h / (heads / kv_heads), C = 2 * kv_heads * DK + heads * DV;

  // ---- the chunk's rows (tokens from n on: zeros, beta 0)
  {
    StagedWords<DK, NT> qw, kw;
    StagedWords<DV, NT> vw;
    const __nv_bfloat16* row0 = act + size_t(start) * C;
    qw.load(row0 + g * DK, C, n, tid);
    kw.load(row0 + kv_heads * DK + g * DK, C, n, tid);
    vw.load(row0 + 2 * kv_heads * DK + h * DV, C, n, tid);
    if constexpr (!PER_HEAD) {
      constexpr int QUADS = DK / 4, PER = CH * QUADS / NT;
#pragma unroll
      for (int u = 0; u < PER; ++u) {
        const int i = tid + u * NT, row = i / QUADS, d = i % QUADS * 4;
        float4 l = make_float4(0.f, 0.f, 0.f, 0.f);
        if (row < n) l = *reinterpret_cast<const float4*>(logd + (size_t(start + row) * heads + h) * DK + d);
        *reinterpret_cast<float4*>(cb + row * CP + d) = make_float4(l.x * LOG2E_F, l.y * LOG2E_F, l.z * LOG2E_F, l.w * LOG2E_F);
      }
    } else {
      if (tid < CH) cb[tid] = tid < n ? logd[size_t(start + tid) * heads + h] * LOG2E_F : 0.f;
    }
    if (tid < CH) {
      const bool on = tid < n;
      rq[tid] = on ? inv[size_t(start + tid) * 2 * kv_heads + g] : 0.f;
      rk[tid] = on ? inv[size_t(start + tid) * 2 * kv_heads + kv_heads + g] : 0.f;
      bt[tid] = on ? beta[size_t(start + tid) * heads + h] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < qw.PER; ++u) {
      const int i = tid + u * NT, row = i / (DK / 8), cc = i % (DK / 8);
      *reinterpret_cast<uint4*>(qs + row * KP + cc * 8) = qw.w[u];
      *reinterpret_cast<uint4*>(ks + row * KP + cc * 8) = kw.w[u];
    }
    vw.store(u_hi, 0, tid);
    for (int i = tid; i < 2 * CH * CH * 2 / 16; i += NT) reinterpret_cast<uint4*>(p_hi)[i] = make_uint4(0, 0, 0, 0);
  }
  __syncthreads();

  // ---- sums of logarithms from each sub-block's start
  if constexpr (PER_HEAD) {
    if (tid < 4) {
      float s = 0.f;
      for (int i = 0; i < 16; ++i) cb[tid * 16 + i] = s += cb[tid * 16 + i];
      tot[tid] = s;
    }
  } else {
    for (int i = tid; i < 4 * DK; i += NT) {
      const int b = i / DK, d = i % DK;
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < 16; ++r) cb[(b * 16 + r) * CP + d] = s += cb[(b * 16 + r) * CP + d];
      tot[b * DK + d] = s;
    }
  }
  __syncthreads();
  auto cb_at = [&](int row, int d) { return PER_HEAD ? cb[row] : cb[row * CP + d]; };
  auto tot_at = [&](int b, int d) { return PER_HEAD ? tot[b] : tot[b * DK + d]; };
  // exponents (base 2): from the chunk's start to the token, and from the token to the chunk's end
  auto from_start = [&](int row, int d) {
    float s = 0.f;
    for (int b = 0; b < row / 16; ++b) s += tot_at(b, d);
    return s + cb_at(row, d);
  };
  auto to_end = [&](int row, int d) {
    float s = tot_at(row / 16, d) - cb_at(row, d);
    for (int b = row / 16 + 1; b < 4; ++b) s += tot_at(b, d);
    return s;
  };

  // ---- L and P between sub-blocks, a warp per (later, earlier, L or P); with one decay per head also inside them
  constexpr int PAIRS = PER_HEAD ? 10 : 6;
  for (int task = warp; task < 2 * PAIRS; task += NW) {
    const int pair = task >> 1;
    const bool is_p = task & 1;
    int i, j;
    if (PER_HEAD) {     // (0,0) (1,0) (1,1) (2,0) ...
      i = pair < 1 ? 0 : (pair < 3 ? 1 : (pair < 6 ? 2 : 3));
      j = pair - i * (i + 1) / 2;
    } else {            // (1,0) (2,0) (2,1) (3,0) ...
      i = pair < 1 ? 1 : (pair < 3 ? 2 : 3);
      j = pair - i * (i - 1) / 2;
    }
    const __nv_bfloat16* left = is_p ? qs : ks;
    float acc[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int row = i * 16 + g4 + (f & 1) * 8, d = kk * 16 + t4 * 2 + (f >> 1) * 8;
        const uint32_t w = *reinterpret_cast<const uint32_t*>(left + row * KP + d);
        if constexpr (PER_HEAD) {
          ah[f] = w;
        } else {
          const float2 e = *reinterpret_cast<const float2*>(cb + row * CP + d);
          split_pack(__uint_as_float(w << 16) * fast_exp2(e.x), __uint_as_float(w & 0xffff0000u) * fast_exp2(e.y), ah[f], al[f]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int f = 0; f < 2; ++f) {
          const int row = j * 16 + nt * 8 + g4, d = kk * 16 + t4 * 2 + f * 8;
          const uint32_t w = *reinterpret_cast<const uint32_t*>(ks + row * KP + d);
          if constexpr (PER_HEAD) {
            bh[f] = w;
          } else {
            const float2 e = *reinterpret_cast<const float2*>(cb + row * CP + d);
            float2 r = *reinterpret_cast<const float2*>(tot + j * DK + d);
            r.x -= e.x;
            r.y -= e.y;
            for (int b = j + 1; b < i; ++b) {
              const float2 o = *reinterpret_cast<const float2*>(tot + b * DK + d);
              r.x += o.x;
              r.y += o.y;
            }
            split_pack(__uint_as_float(w << 16) * fast_exp2(r.x), __uint_as_float(w & 0xffff0000u) * fast_exp2(r.y), bh[f], bl[f]);
          }
        }
        mma_bf16(acc[nt], ah, bh[0], bh[1]);
        if constexpr (!PER_HEAD) {
          mma_bf16(acc[nt], ah, bl[0], bl[1]);
          mma_bf16(acc[nt], al, bh[0], bh[1]);
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = i * 16 + g4 + half * 8, col = j * 16 + nt * 8 + t4 * 2;
        float v[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float f = rk[col + e] * (is_p ? rq[row] : rk[row] * bt[row]);
          if constexpr (PER_HEAD) {
            float x = i == j ? cb[row] - cb[col + e] : tot[j] - cb[col + e] + cb[row];
            for (int b = j + 1; b < i; ++b) x += tot[b];
            f = col + e <= row ? f * fast_exp2(x) : 0.f;       // what comes later takes no part
          }
          v[e] = acc[nt][half * 2 + e] * f;
        }
        if (is_p) {
          put_split<CH>(p_hi, p_lo, row, col, v[0], v[1]);
        } else {
          As[row * TP + col] = v[0];
          As[row * TP + col + 1] = v[1];
        }
      }
  }
  if constexpr (!PER_HEAD) {
    // ---- inside a sub-block: every pair of tokens with exponents of its own, four lanes along the channels
    const int sub = tid & 3;
    for (int task = tid >> 2; task < 4 * 136; task += NT / 4) {
      const int b = task / 136, pr = task % 136, ra = pr / 17, rb = pr % 17;
      const int r = rb <= ra ? ra : 15 - ra, s = rb <= ra ? rb : rb - ra - 1;     // s <= r
      const int row = b * 16 + r, col = b * 16 + s;
      float a = 0.f, p = 0.f;
#pragma unroll 4
      for (int d = sub * 4; d < DK; d += 16) {
        const float4 ct = *reinterpret_cast<const float4*>(cb + row * CP + d);
        const float4 cs = *reinterpret_cast<const float4*>(cb + col * CP + d);
        const uint2 kt = *reinterpret_cast<const uint2*>(ks + row * KP + d);
        const uint2 k2 = *reinterpret_cast<const uint2*>(ks + col * KP + d);
        const uint2 qt = *reinterpret_cast<const uint2*>(qs + row * KP + d);
        const float e0 = __uint_as_float(k2.x << 16) * fast_exp2(ct.x - cs.x), e1 = __uint_as_float(k2.x & 0xffff0000u) * fast_exp2(ct.y - cs.y);
        const float e2 = __uint_as_float(k2.y << 16) * fast_exp2(ct.z - cs.z), e3 = __uint_as_float(k2.y & 0xffff0000u) * fast_exp2(ct.w - cs.w);
        a = fmaf(__uint_as_float(kt.x << 16), e0, a);
        a = fmaf(__uint_as_float(kt.x & 0xffff0000u), e1, a);
        a = fmaf(__uint_as_float(kt.y << 16), e2, a);
        a = fmaf(__uint_as_float(kt.y & 0xffff0000u), e3, a);
        p = fmaf(__uint_as_float(qt.x << 16), e0, p);
        p = fmaf(__uint_as_float(qt.x & 0xffff0000u), e1, p);
        p = fmaf(__uint_as_float(qt.y << 16), e2, p);
        p = fmaf(__uint_as_float(qt.y & 0xffff0000u), e3, p);
      }
      // 4 * 136 tasks are whole warps of 8 tasks: all lanes of a warp are here together
      a += __shfl_xor_sync(0xffffffffu, a, 1);
      p += __shfl_xor_sync(0xffffffffu, p, 1);
      a += __shfl_xor_sync(0xffffffffu, a, 2);
      p += __shfl_xor_sync(0xffffffffu, p, 2);
      if (sub == 0) {
        As[row * TP + col] = a * rk[col] * rk[row] * bt[row];      // the diagonal is not read
        const float v = p * rk[col] * rq[row];
        const __nv_bfloat16 hi = __float2bfloat16_rn(v), lo = __float2bfloat16_rn(v - __bfloat162float(hi));
        const uint32_t off = swz<CH>(row, col >> 3) + (col & 7) * 2;
        *reinterpret_cast<__nv_bfloat16*>(p_hi + off) = hi;
        *reinterpret_cast<__nv_bfloat16*>(p_lo + off) = lo;
      }
    }
  }
  __syncthreads();

  // ---- (I + L)^-1 by sub-blocks: the four on the diagonal by substitution, a thread per column
  if (tid < 64) {
    const int b = tid / 16, cc = tid % 16;
    const float* Lb = As + b * 16 * TP + b * 16;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float s = r == cc ? 1.f : 0.f;
#pragma unroll
      for (int i = 0; i < r; ++i) s = fmaf(-Lb[r * TP + i], x[i], s);
      x[r] = s;
      Ts[(b * 16 + r) * TP + b * 16 + cc] = s;
    }
  }
  // decayed keys meanwhile: both as they stand at the token and as they reach the chunk's end
  for (int i = tid; i < CH * (DK / 8); i += NT) {
    const int row = i / (DK / 8), cc = i % (DK / 8);
    float f[8];
    unpack_bf16x8(*reinterpret_cast<const uint4*>(ks + row * KP + cc * 8), f);
    uint4 hi, lo, hi2, lo2;
    uint32_t *H = &hi.x, *Lo = &lo.x, *H2 = &hi2.x, *Lo2 = &lo2.x;
    const float r = rk[row];
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const int d = cc * 8 + e;
      const float x = f[e] * r, y = f[e + 1] * r;
      split_pack(x * fast_exp2(from_start(row, d)), y * fast_exp2(from_start(row, d + 1)), H[e / 2], Lo[e / 2]);
      split_pack(x * fast_exp2(to_end(row, d)), y * fast_exp2(to_end(row, d + 1)), H2[e / 2], Lo2[e / 2]);
    }
    const uint32_t off = swz<DK>(row, cc);
    *reinterpret_cast<uint4*>(w_hi + off) = hi;
    *reinterpret_cast<uint4*>(w_lo + off) = lo;
    *reinterpret_cast<uint4*>(kd_hi + off) = hi2;
    *reinterpret_cast<uint4*>(kd_lo + off) = lo2;
  }
  for (int d = tid; d < DK; d += NT)
    dec[(size_t(c) * heads + h) * DK + d] = fast_exp2(tot_at(0, d) + tot_at(1, d) + tot_at(2, d) + tot_at(3, d));
  __syncthreads();
  // ... and the others: T_ij = -T_ii sum_k L_ik T_kj, one distance from the diagonal after the other
#pragma unroll 1
  for (int lev = 1; lev < 4; ++lev) {
    for (int e = tid; e < (4 - lev) * 256; e += NT) {
      const int i = e / 256 + lev, j = i - lev, r = e % 256 / 16, cc = e % 16;
      float s = 0.f;
      for (int x = j * 16; x < i * 16; ++x) s = fmaf(As[(i * 16 + r) * TP + x], Ts[x * TP + j * 16 + cc], s);
      Xs[e] = s;
    }
    __syncthreads();
    for (int e = tid; e < (4 - lev) * 256; e += NT) {
      const int i = e / 256 + lev, j = i - lev, r = e % 256 / 16, cc = e % 16;
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < 16; ++x) s = fmaf(-Ts[(i * 16 + r) * TP + i * 16 + x], Xs[(e / 256) * 256 + x * 16 + cc], s);
      Ts[(i * 16 + r) * TP + j * 16 + cc] = s;
    }
    __syncthreads();
  }
  for (int i = tid; i < CH * (CH / 8); i += NT) {      // T diag(beta), over L
    const int row = i / (CH / 8), cc = i % (CH / 8);
    uint4 hi, lo;
    uint32_t *H = &hi.x, *Lo = &lo.x;
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const int s = cc * 8 + e;
      split_pack(s <= row ? Ts[row * TP + s] * bt[s] : 0.f, s + 1 <= row ? Ts[row * TP + s + 1] * bt[s + 1] : 0.f, H[e / 2], Lo[e / 2]);
    }
    *reinterpret_cast<uint4*>(t_hi + swz<CH>(row, cc)) = hi;
    *reinterpret_cast<uint4*>(t_lo + swz<CH>(row, cc)) = lo;
  }
  __syncthreads();

  // ---- W = T Kc and U_0 = T V: row tile mi, a stretch of columns; sub-blocks after the row tile's are zero
  constexpr int GROUPS = NW / 4, WN = DK / GROUPS / 8, UN = DV / GROUPS / 8;     // column tiles of a warp
  const int mi = warp & 3, ng = warp >> 2;
  const uint32_t th = smem_u32(t_hi), tl = smem_u32(t_lo), wh = smem_u32(w_hi), wl = smem_u32(w_lo), uh = smem_u32(u_hi), ul = smem_u32(u_lo);
  float wa[WN][4] = {}, ua[UN][4] = {};
  for (int kk = 0; kk <= mi; ++kk) {
    uint32_t ah[4], al[4];
    const uint32_t off = swz<CH>(mi * 16 + (lane & 15), kk * 2 + (lane >> 4));
    ldmatrix_x4(ah[0], ah[1], ah[2], ah[3], th + off);
    ldmatrix_x4(al[0], al[1], al[2], al[3], tl + off);
#pragma unroll
    for (int j = 0; j < WN; j += 2) {
      uint32_t b[4], bl[4];
      const uint32_t bo_ = swz<DK>(kk * 16 + (m & 1) * 8 + (lane & 7), ng * WN + j + (m >> 1));
      ldmatrix_x4_trans(b[0], b[1], b[2], b[3], wh + bo_);
      ldmatrix_x4_trans(bl[0], bl[1], bl[2], bl[3], wl + bo_);
      mma_bf16(wa[j], ah, b[0], b[1]);
      mma_bf16(wa[j + 1], ah, b[2], b[3]);
      mma_bf16(wa[j], ah, bl[0], bl[1]);
      mma_bf16(wa[j + 1], ah, bl[2], bl[3]);
      mma_bf16(wa[j], al, b[0], b[1]);
      mma_bf16(wa[j + 1], al, b[2], b[3]);
    }
#pragma unroll
    for (int j = 0; j < UN; j += 2) {
      uint32_t b[4];
      ldmatrix_x4_trans(b[0], b[1], b[2], b[3], uh + swz<DV>(kk * 16 + (m & 1) * 8 + (lane & 7), ng * UN + j + (m >> 1)));
      mma_bf16(ua[j], ah, b[0], b[1]);
      mma_bf16(ua[j + 1], ah, b[2], b[3]);
      mma_bf16(ua[j], al, b[0], b[1]);
      mma_bf16(ua[j + 1], al, b[2], b[3]);
    }
  }
  __syncthreads();      // Kc and V have been read by everybody: W and U_0 take their places
#pragma unroll
  for (int j = 0; j < WN; ++j) {
    const int col = (ng * WN + j) * 8 + t4 * 2;
    put_split<DK>(w_hi, w_lo, mi * 16 + g4, col, wa[j][0], wa[j][1]);
    put_split<DK>(w_hi, w_lo, mi * 16 + g4 + 8, col, wa[j][2], wa[j][3]);
  }
#pragma unroll
  for (int j = 0; j < UN; ++j) {
    const int col = (ng * UN + j) * 8 + t4 * 2;
    put_split<DV>(u_hi, u_lo, mi * 16 + g4, col, ua[j][0], ua[j][1]);
    put_split<DV>(u_hi, u_lo, mi * 16 + g4 + 8, col, ua[j][2], ua[j][3]);
  }
  __syncthreads();

  uint4* mq_c = mq + (size_t(c) * heads + h) * MT * (DK / 16) * 2 * 32;
  float4* bo_c = bo + (size_t(c) * heads + h) * MT * (DV / 8) * 32;
  // ---- Q = Qc - P W and O_0 = P U_0
  {
    const uint32_t ph = smem_u32(p_hi), pl = smem_u32(p_lo);
#pragma unroll
    for (int j = 0; j < WN; ++j) wa[j][0] = wa[j][1] = wa[j][2] = wa[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < UN; ++j) ua[j][0] = ua[j][1] = ua[j][2] = ua[j][3] = 0.f;
    for (int kk = 0; kk <= mi; ++kk) {
      uint32_t ah[4], al[4];
      const uint32_t off = swz<CH>(mi * 16 + (lane & 15), kk * 2 + (lane >> 4));
      ldmatrix_x4(ah[0], ah[1], ah[2], ah[3], ph + off);
      ldmatrix_x4(al[0], al[1], al[2], al[3], pl + off);
      auto three = [&](float (&acc0)[4], float (&acc1)[4], uint32_t hi_at, uint32_t lo_at) {
        uint32_t b[4], bl[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], hi_at);
        ldmatrix_x4_trans(bl[0], bl[1], bl[2], bl[3], lo_at);
        mma_bf16(acc0, ah, b[0], b[1]);
        mma_bf16(acc1, ah, b[2], b[3]);
        mma_bf16(acc0, ah, bl[0], bl[1]);
        mma_bf16(acc1, ah, bl[2], bl[3]);
        mma_bf16(acc0, al, b[0], b[1]);
        mma_bf16(acc1, al, b[2], b[3]);
      };
#pragma unroll
      for (int j = 0; j < WN; j += 2) {
        const uint32_t o = swz<DK>(kk * 16 + (m & 1) * 8 + (lane & 7), ng * WN + j + (m >> 1));
        three(wa[j], wa[j + 1], wh + o, wl + o);
      }
#pragma unroll
      for (int j = 0; j < UN; j += 2) {
        const uint32_t o = swz<DV>(kk * 16 + (m & 1) * 8 + (lane & 7), ng * UN + j + (m >> 1));
        three(ua[j], ua[j + 1], uh + o, ul + o);
      }
    }
#pragma unroll
    for (int j = 0; j < WN; j += 2) {     // two column tiles of C fragments are one A fragment of 16 columns
      uint4 hi, lo;
      uint32_t *H = &hi.x, *Lo = &lo.x;
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int row = mi * 16 + g4 + (f & 1) * 8, d = (ng * WN + j + (f >> 1)) * 8 + t4 * 2;
        const uint32_t w = *reinterpret_cast<const uint32_t*>(qs + row * KP + d);
        const float x = __uint_as_float(w << 16) * rq[row] * fast_exp2(from_start(row, d));
        const float y = __uint_as_float(w & 0xffff0000u) * rq[row] * fast_exp2(from_start(row, d + 1));
        split_pack(x - wa[j + (f >> 1)][(f & 1) * 2], y - wa[j + (f >> 1)][(f & 1) * 2 + 1], H[f], Lo[f]);
      }
      uint4* dst = mq_c + ((size_t(DK / 16 + mi) * (DK / 16) + (ng * WN + j) / 2) * 2) * 32 + lane;
      dst[0] = hi;
      dst[32] = lo;
    }
#pragma unroll
    for (int j = 0; j < UN; ++j)
      bo_c[(size_t(DK / 16 + mi) * (DV / 8) + ng * UN + j) * 32 + lane] = make_float4(ua[j][0], ua[j][1], ua[j][2], ua[j][3]);
  }
  // ---- M = -Kd^T W and B = Kd^T U_0: row tile mt of the key channels, half of the columns
  {
    constexpr int MN = DK / 16, BN = DV / 16;      // column tiles of half the columns
    const int mt = warp % (DK / 16), half = warp / (DK / 16);
    const uint32_t kh = smem_u32(kd_hi), kl = smem_u32(kd_lo);
    float ma[MN][4] = {}, ba[BN][4] = {};
#pragma unroll
    for (int kk = 0; kk < CH / 16; ++kk) {
      uint32_t ah[4], al[4];
      const uint32_t off = swz<DK>(kk * 16 + (m >> 1) * 8 + (lane & 7), mt * 2 + (m & 1));
      ldmatrix_x4_trans(ah[0], ah[1], ah[2], ah[3], kh + off);
      ldmatrix_x4_trans(al[0], al[1], al[2], al[3], kl + off);
      auto three = [&](float (&acc0)[4], float (&acc1)[4], uint32_t hi_at, uint32_t lo_at) {
        uint32_t b[4], bl[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], hi_at);
        ldmatrix_x4_trans(bl[0], bl[1], bl[2], bl[3], lo_at);
        mma_bf16(acc0, ah, b[0], b[1]);
        mma_bf16(acc1, ah, b[2], b[3]);
        mma_bf16(acc0, ah, bl[0], bl[1]);
        mma_bf16(acc1, ah, bl[2], bl[3]);
        mma_bf16(acc0, al, b[0], b[1]);
        mma_bf16(acc1, al, b[2], b[3]);
      };
#pragma unroll
      for (int j = 0; j < MN; j += 2) {
        const uint32_t o = swz<DK>(kk * 16 + (m & 1) * 8 + (lane & 7), half * MN + j + (m >> 1));
        three(ma[j], ma[j + 1], wh + o, wl + o);
      }
#pragma unroll
      for (int j = 0; j < BN; j += 2) {
        const uint32_t o = swz<DV>(kk * 16 + (m & 1) * 8 + (lane & 7), half * BN + j + (m >> 1));
        three(ba[j], ba[j + 1], uh + o, ul + o);
      }
    }
#pragma unroll
    for (int j = 0; j < MN; j += 2) {
      uint4 hi, lo;
      split_pack(-ma[j][0], -ma[j][1], hi.x, lo.x);
      split_pack(-ma[j][2], -ma[j][3], hi.y, lo.y);
      split_pack(-ma[j + 1][0], -ma[j + 1][1], hi.z, lo.z);
      split_pack(-ma[j + 1][2], -ma[j + 1][3], hi.w, lo.w);
      uint4* dst = mq_c + ((size_t(mt) * (DK / 16) + (half * MN + j) / 2) * 2) * 32 + lane;
      dst[0] = hi;
      dst[32] = lo;
    }
#pragma unroll
    for (int j = 0; j < BN; ++j)
      bo_c[(size_t(mt) * (DV / 8) + half * BN + j) * 32 + lane] = make_float4(ba[j][0], ba[j][1], ba[j][2], ba[j][3]);
  }
}

// One block = one sequence x one head x 8 NTILE value columns; a warp per row tile of [M; Q]. The chunks in order: the
// warps of M hold the state's float32 values and leave them split in shared memory for all; a chunk's fragments are read
// from memory while the chunk before is multiplied.
template <int DK, int DV, int NTILE>
__global__ void __launch_bounds__((DK / 16 + 4) * 32)
delta_chunk_join_kernel(const uint4* __restrict__ mq, const float4* __restrict__ bo, const float* __restrict__ dec,
                        float* __restrict__ state, int state_stride, int state_off, const int* __restrict__ slots, StepBatch sb,
                        const int* __restrict__ seq_chunk0, float* __restrict__ out, int heads) {
  constexpr int MT = DK / 16 + 4, KS = DK / 16, PITCH = NTILE * 16 + 16;       // bytes of a state row: 16 more than its values
  __shared__ __align__(128) unsigned char s_sm[2][2][DK * PITCH];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3, m = lane >> 3;
  const int seq = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * NTILE * 8;
  const int n_new = sb.seq_new[seq], c0 = seq_chunk0[seq], start = sb.seq_start[seq];
  const int n_chunks = (n_new + CH - 1) / CH;
  if (n_chunks <= 0) return;
  const bool is_state = warp < KS;
  float* st = state + size_t(slots[seq]) * state_stride + state_off + (size_t(h) * DV + j0) * DK;
  float S[NTILE][4];
  const int d0 = warp * 16 + g4;
#pragma unroll
  for (int nt = 0; nt < NTILE; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      S[nt][e] = is_state ? st[size_t(nt * 8 + t4 * 2 + (e & 1)) * DK + d0 + (e >> 1) * 8] : 0.f;
  uint4 a[KS][2];
  float4 init[NTILE];
  float dc0 = 1.f, dc1 = 1.f;
  auto frag = [&](int chunk) { return mq + (((size_t(chunk) * heads + h) * MT + warp) * KS * 2) * 32 + lane; };
  auto rest = [&](int chunk) { return bo + ((size_t(chunk) * heads + h) * MT + warp) * (DV / 8) * 32 + (j0 / 8) * 32 + lane; };
  {
    const uint4* f = frag(c0);
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      a[ks][0] = f[(ks * 2) * 32];
      a[ks][1] = f[(ks * 2 + 1) * 32];
    }
    const float4* r = rest(c0);
#pragma unroll
    for (int nt = 0; nt < NTILE; ++nt) init[nt] = r[nt * 32];
    if (is_state) {
      dc0 = dec[(size_t(c0) * heads + h) * DK + d0];
      dc1 = dec[(size_t(c0) * heads + h) * DK + d0 + 8];
    }
  }
  for (int i = 0; i < n_chunks; ++i) {
    unsigned char* hi_s = s_sm[i & 1][0];
    unsigned char* lo_s = s_sm[i & 1][1];
    if (is_state) {
#pragma unroll
      for (int nt = 0; nt < NTILE; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split_pack(S[nt][half * 2], S[nt][half * 2 + 1], hi, lo);
          const int at = (d0 + half * 8) * PITCH + nt * 16 + t4 * 4;
          *reinterpret_cast<uint32_t*>(hi_s + at) = hi;
          *reinterpret_cast<uint32_t*>(lo_s + at) = lo;
        }
    }
    // one barrier a chunk: the buffer written next was last read before this barrier
    __syncthreads();
    float acc[NTILE][4];
#pragma unroll
    for (int nt = 0; nt < NTILE; ++nt) {
      acc[nt][0] = init[nt].x; acc[nt][1] = init[nt].y; acc[nt][2] = init[nt].z; acc[nt][3] = init[nt].w;
    }
    const float e0 = dc0, e1 = dc1;
    const bool more = i + 1 < n_chunks;
    const int nxt = c0 + (more ? i + 1 : i);       // after the last chunk its own fragments are read once more and not used
    const uint4* f = frag(nxt);
    {
      const float4* r = rest(nxt);
#pragma unroll
      for (int nt = 0; nt < NTILE; ++nt) init[nt] = r[nt * 32];
      if (is_state) {
        dc0 = dec[(size_t(nxt) * heads + h) * DK + d0];
        dc1 = dec[(size_t(nxt) * heads + h) * DK + d0 + 8];
      }
    }
    const uint32_t hb = smem_u32(hi_s), lb = smem_u32(lo_s);
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const uint32_t ah[4] = {a[ks][0].x, a[ks][0].y, a[ks][0].z, a[ks][0].w};
      const uint32_t al[4] = {a[ks][1].x, a[ks][1].y, a[ks][1].z, a[ks][1].w};
      a[ks][0] = f[(ks * 2) * 32];
      a[ks][1] = f[(ks * 2 + 1) * 32];
      const uint32_t row = uint32_t(ks * 16 + (m & 1) * 8 + (lane & 7)) * PITCH + (m >> 1) * 16;
#pragma unroll
      for (int j = 0; j < NTILE; j += 2) {
        uint32_t b[4], bl[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], hb + row + j * 16);
        ldmatrix_x4_trans(bl[0], bl[1], bl[2], bl[3], lb + row + j * 16);
        mma_bf16(acc[j], ah, b[0], b[1]);
        mma_bf16(acc[j + 1], ah, b[2], b[3]);
        mma_bf16(acc[j], ah, bl[0], bl[1]);
        mma_bf16(acc[j + 1], ah, bl[2], bl[3]);
        mma_bf16(acc[j], al, b[0], b[1]);
        mma_bf16(acc[j + 1], al, b[2], b[3]);
      }
    }
    if (is_state) {
#pragma unroll
      for (int nt = 0; nt < NTILE; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] = fmaf(e < 2 ? e0 : e1, S[nt][e], acc[nt][e]);
    } else {
      const int t0 = (warp - KS) * 16 + g4;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = i * CH + t0 + half * 8;
        if (t < n_new) {
          float* o = out + (size_t(start + t) * heads + h) * DV + j0 + t4 * 2;
#pragma unroll
          for (int nt = 0; nt < NTILE; ++nt) *reinterpret_cast<float2*>(o + nt * 8) = make_float2(acc[nt][half * 2], acc[nt][half * 2 + 1]);
        }
      }
    }
  }
  if (is_state) {
#pragma unroll
    for (int nt = 0; nt < NTILE; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[size_t(nt * 8 + t4 * 2 + (e & 1)) * DK + d0 + (e >> 1) * 8] = S[nt][e];
  }
}

size_t scratch_part(int n_chunks, int heads, int dk, int dv, int which) {
  const size_t ch = size_t(n_chunks) * heads, mt = dk / 16 + 4;
  const size_t mq = ch * mt * (dk / 16) * 2 * 32 * sizeof(uint4), bo = ch * mt * (dv / 8) * 32 * sizeof(float4);
  return which == 0 ? mq : (which == 1 ? bo : ch * dk * sizeof(float));
}

template <int DK, int DV, bool PER_HEAD>
int launch_local(const void* act, const float* inv, const float* logd, const float* beta, const StepBatch& sb,
                 const int* chunk_seq, const int* chunk_q0, int n_chunks, void* mq, void* bo, float* dec, int heads, int kv_heads,
                 cudaStream_t stream) {
  constexpr int smem = LocalSmem<DK, DV, PER_HEAD>::bytes;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(delta_chunk_local_kernel<DK, DV, PER_HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return PTB_ERR_LAUNCH;
    configured = true;
  }
  delta_chunk_local_kernel<DK, DV, PER_HEAD><<<dim3(n_chunks, heads), DK * 4, smem, stream>>>(
      (const __nv_bfloat16*)act, inv, logd, beta, sb, chunk_seq, chunk_q0, (uint4*)mq, (float4*)bo, dec, heads, kv_heads);
  return launch_status();
}

template <int DK, int DV>
int launch_chunks(const void* act, const float* inv, const float* logd, const float* beta, float* state, int state_stride,
                  const int* slots, const StepBatch& sb, const int* chunk_seq, const int* chunk_q0, const int* seq_chunk0,
                  int n_chunks, unsigned char* scratch, float* out, int heads, int kv_heads, int taps, int per_head,
                  cudaStream_t stream) {
  unsigned char* mq = scratch;
  unsigned char* bo = mq + scratch_part(n_chunks, heads, DK, DV, 0);
  float* dec = reinterpret_cast<float*>(bo + scratch_part(n_chunks, heads, DK, DV, 1));
  const int rc = per_head ? launch_local<DK, DV, true>(act, inv, logd, beta, sb, chunk_seq, chunk_q0, n_chunks, mq, bo, dec, heads, kv_heads, stream)
                          : launch_local<DK, DV, false>(act, inv, logd, beta, sb, chunk_seq, chunk_q0, n_chunks, mq, bo, dec, heads, kv_heads, stream);
  if (rc != PTB_OK) return rc;
  const int state_off = (taps - 1) * (2 * kv_heads * DK + heads * DV);
  // 32 value columns a block, or 16 where that many blocks would leave half of the device idle (2,048 tokens of 16 heads of
  // 128 x 128: 245 -> 222 us both passes; of 32 heads 16 columns were slower, 362 -> 406). A column's sums are the same.
#define PTB_JOIN(NTILE)                                                                                                        \
  delta_chunk_join_kernel<DK, DV, NTILE><<<dim3(DV / (8 * NTILE), heads, sb.n_seqs), (DK / 16 + 4) * 32, 0, stream>>>(         \
      (const uint4*)mq, (const float4*)bo, dec, state, state_stride, state_off, slots, sb, seq_chunk0, out, heads)
  if ((long long)(DV / 32) * heads * sb.n_seqs * 2 <= sm_count()) PTB_JOIN(2);
  else PTB_JOIN(4);
#undef PTB_JOIN
  return launch_status();
}

}  // namespace

PTB_API int ptb_delta_chunk_tokens() { return CH; }
PTB_API int ptb_delta_chunks_supports(int dim, int v_dim) { return (dim == 64 || dim == 128) && (v_dim == 64 || v_dim == 128); }
PTB_API long long ptb_delta_chunks_scratch_bytes(int n_chunks, int heads, int dim, int v_dim) {
  long long total = 0;
  for (int w = 0; w < 3; ++w) total += (long long)scratch_part(n_chunks, heads, dim, v_dim, w);
  return total;
}

// The step's tokens in chunks: arguments as ptb_delta_walk takes them (bfloat16), and the step's chunks: chunk_seq, chunk_q0
// (sequence and first of its new tokens of every chunk), seq_chunk0 (a sequence's first chunk). scratch: as many bytes as
// ptb_delta_chunks_scratch_bytes says, on a 16-byte boundary.
PTB_API int ptb_delta_chunks(const void* act, const float* inv, const float* logd, const float* beta, float* state,
                             int state_stride, const int* slots, const StepBatch* sb, const int* chunk_seq, const int* chunk_q0,
                             const int* seq_chunk0, int n_chunks, void* scratch, float* out, int heads, int kv_heads, int dim,
                             int v_dim, int taps, int per_head, cudaStream_t stream) {
  if (sb->n_tokens <= 0 || n_chunks <= 0) return PTB_OK;
  if (!ptb_delta_chunks_supports(dim, v_dim) || heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads != 0 || taps < 1 ||
      sb->n_seqs > 65535 || state_stride < (taps - 1) * (2 * kv_heads * dim + heads * v_dim) + heads * dim * v_dim)
    return PTB_ERR_SIZE;
  if (!aligned16(act) || !aligned16(scratch) || !aligned16(logd)) return PTB_ERR_ALIGN;
#define PTB_DC(DK, DV)                                                                                                       \
  return launch_chunks<DK, DV>(act, inv, logd, beta, state, state_stride, slots, *sb, chunk_seq, chunk_q0, seq_chunk0, n_chunks, \
                               (unsigned char*)scratch, out, heads, kv_heads, taps, per_head, stream)
  if (dim == 64 && v_dim == 64) PTB_DC(64, 64);
  if (dim == 64 && v_dim == 128) PTB_DC(64, 128);
  if (dim == 128 && v_dim == 64) PTB_DC(128, 64);
  PTB_DC(128, 128);
#undef PTB_DC
}
