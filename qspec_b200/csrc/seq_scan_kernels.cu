// Sequence-mixer kernels, sixth file: matrix states with one decay per head and token (linear attention with fixed decays, Mamba-2),
// in a form that walks short segments token by token and a form that takes 64 tokens at a time on the tensor cores; the norm of the
// read-outs in equal parts with a gate before or after it; the residual sum between two norms. bfloat16 / float32 activations
// (template T); everything that is normed, exponentiated or carried from token to token is float32.
#include "seq_common.cuh"
#include "../../include/qspec_b200_seq.h"
#include <stdint.h>

namespace qspec {

typedef __nv_bfloat16 bf16_t;

// ---- residual sum between a norm of the sublayer's result and the norm of the next sublayer's input ------------------------------
// v = sum_p y_w[t, p] y[t, p] + y2[t]; r = x_in + v / rms(v) * (w_offset + post_w); out = r / rms(r) * (w_offset + pre_w). One CTA
// per token, the row in registers from the first load to the last store.
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(256)
sandwich_norm_kernel(const float* __restrict__ x_in, float* __restrict__ x_out, const T* __restrict__ y, int y_parts, long long y_part_stride,
                     long long y_tok_stride, const float* __restrict__ y_w, const T* __restrict__ y2, const float* __restrict__ post_w,
                     const float* __restrict__ pre_w, float w_offset, T* __restrict__ out, int W, float eps) {
  pdl_enter();
  __shared__ float red[8];
  const int i = blockIdx.x, tid = threadIdx.x;
  const float inv_w = 1.0f / (float)W;
  VecF<VEC> v[NV], x[NV];
  float ss = 0.f;
#pragma unroll
  for (int q = 0; q < NV; ++q) {
    const int c = (tid + q * 256) * VEC;
#pragma unroll
    for (int e = 0; e < VEC; ++e) { v[q].v[e] = 0.f; x[q].v[e] = 0.f; }
    if (c >= W) continue;
    x[q] = ldv<VEC>(x_in + (size_t)i * W + c);
    if (!y) continue;
    if (y2) v[q] = ldv<VEC>(y2 + (size_t)i * W + c);
#pragma unroll 4
    for (int p = 0; p < y_parts; ++p) {
      const float wp = y_w ? y_w[(size_t)i * y_parts + p] : 1.0f;
      const VecF<VEC> t = ldv<VEC>(y + (size_t)i * y_tok_stride + (size_t)p * y_part_stride + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[q].v[e] += wp * t.v[e];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v[q].v[e] * v[q].v[e];
  }
  if (y) {
    const float r = 1.0f / sqrtf(block_sum_256(ss, red) * inv_w + eps);
#pragma unroll
    for (int q = 0; q < NV; ++q) {
      const int c = (tid + q * 256) * VEC;
      if (c >= W) continue;
      const VecF<VEC> pw = ldv<VEC>(post_w + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[q].v[e] += v[q].v[e] * r * (w_offset + pw.v[e]);
    }
  }
  if (x_out && (y || x_out != x_in)) {
#pragma unroll
    for (int q = 0; q < NV; ++q) {
      const int c = (tid + q * 256) * VEC;
      if (c < W) stv<VEC>(x_out + (size_t)i * W + c, x[q]);
    }
  }
  if (!out) return;
  ss = 0.f;
#pragma unroll
  for (int q = 0; q < NV; ++q)
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += x[q].v[e] * x[q].v[e];
  const float r = 1.0f / sqrtf(block_sum_256(ss, red) * inv_w + eps);
#pragma unroll
  for (int q = 0; q < NV; ++q) {
    const int c = (tid + q * 256) * VEC;
    if (c >= W) continue;
    const VecF<VEC> pw = ldv<VEC>(pre_w + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[q].v[e] *= r * (w_offset + pw.v[e]);
    stv<VEC>(out + (size_t)i * W + c, x[q]);
  }
}

// ---- norm of a row in equal parts, with a gate ----------------------------------------------------------------------------------
// QSPEC_GATE_SIGMOID_AFTER: out = out_scale * unit_rms(src) * w * sigmoid(gate); QSPEC_GATE_SILU_BEFORE: out = out_scale *
// unit_rms(src * silu(gate)) * w. unit_rms over each of `parts` equal parts. One group of TPP threads per (token, part): a warp for
// parts of up to 1024 entries, a CTA for larger ones. Each thread's first KEEP groups of VEC entries wait in registers with their gates
// and weights, so that nothing is loaded after the reduction; longer rows read the rest again.
template <typename T, int VEC, int TPP, int KEEP>
__global__ void __launch_bounds__(256)
part_norm_kernel(const float* __restrict__ src, const float* __restrict__ w, const T* __restrict__ gate, int gate_ld, int gate_mode,
                 T* __restrict__ out, int out_ld, long long rows, int parts, int n, float eps, float out_scale) {
  pdl_enter();
  __shared__ float red[8];
  const long long r = (long long)blockIdx.x * (256 / TPP) + threadIdx.x / TPP;
  if (r >= rows) return;                                          // whole warps; TPP = 256 has one row per CTA and never leaves here
  const int l = threadIdx.x % TPP;
  const long long t = r / parts;
  const int p = (int)(r - t * parts);
  const float* s = src + (size_t)r * n;
  const T* g = gate + (size_t)t * gate_ld + (size_t)p * n;
  const float* wr = w + (size_t)p * n;
  T* o = out + (size_t)t * out_ld + (size_t)p * n;
  const bool before = gate_mode == QSPEC_GATE_SILU_BEFORE;
  auto enter = [&](VecF<VEC>& v, const VecF<VEC>& z) {
    float q = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (before) v.v[e] *= silu_act<T>(z.v[e]);
      q += v.v[e] * v.v[e];
    }
    return q;
  };
  auto leave = [&](int c, VecF<VEC> v, const VecF<VEC>& z, const VecF<VEC>& wv, float f) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= (before ? f : f / (1.0f + expf(-z.v[e]))) * wv.v[e];
    stv<VEC>(o + c, v);
  };
  VecF<VEC> kv[KEEP], kz[KEEP], kw[KEEP];
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (l + k * TPP) * VEC;
#pragma unroll
    for (int e = 0; e < VEC; ++e) kv[k].v[e] = kz[k].v[e] = kw[k].v[e] = 0.f;
    if (c < n) { kv[k] = ldv<VEC>(s + c); kz[k] = ldv<VEC>(g + c); kw[k] = ldv<VEC>(wr + c); }
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) ss += enter(kv[k], kz[k]);
  for (int c = (l + KEEP * TPP) * VEC; c < n; c += TPP * VEC) {
    VecF<VEC> v = ldv<VEC>(s + c);
    ss += enter(v, ldv<VEC>(g + c));
  }
  const float sum = TPP == 32 ? warp_xor_sum(ss) : block_sum_256(ss, red);
  const float rr = out_scale / sqrtf(sum / (float)n + eps);
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (l + k * TPP) * VEC;
    if (c < n) leave(c, kv[k], kz[k], kw[k], rr);
  }
  for (int c = (l + KEEP * TPP) * VEC; c < n; c += TPP * VEC) {
    VecF<VEC> v = ldv<VEC>(s + c);
    const VecF<VEC> z = ldv<VEC>(g + c);
    enter(v, z);
    leave(c, v, z, ldv<VEC>(wr + c), rr);
  }
}

// ---- matrix state with one decay per head and token -------------------------------------------------------------------------------
//   S <- a_t S + dt_t k_t v_t^T,   y_t = S^T q_t + D v_t                 (S [D, DV] float32 per head)
// a_t = decay[h] and dt_t = 1, or dt_t = softplus(dt + dt_bias) and a_t = exp(-exp(A_log) dt_t).
//
// Token form: one CTA of eight warps per (segment, head, LPR * VEC value columns) walks the segment. LPR neighbouring lanes share NRW
// neighbouring rows of the state, VEC columns each, so that whole rows are read and written; the state stays in registers from the first
// token to the last. A token's vectors come from the projection: convolved and activated, activated, or as they are. The vectors are
// double-buffered: two barriers per token. KT > 0: a convolution of at most KT taps, whose weights and last inputs every thread keeps in
// registers for the entries it prepares; KT = 0: filters of any length, or none.
template <typename T, int NRW, int VEC, int LPR, int KT>
__global__ void __launch_bounds__(256, NRW * VEC <= 32 ? 3 : NRW * VEC <= 64 ? 2 : 1)
scalar_decay_token_kernel(const qspec_scalar_decay_args a, int max_len) {
  pdl_enter();
  constexpr int DP = (256 / LPR) * NRW, CW = LPR * VEC;
  __shared__ __align__(16) float sq[2][DP], sk[2][DP], sv[2][CW];
  __shared__ __align__(16) float red[8][CW];
  const int h = blockIdx.y, v0 = blockIdx.z * CW, tid = threadIdx.x, warp = tid >> 5, r0 = (tid / LPR) * NRW, lc = (tid % LPR) * VEC;
  const int i0 = a.seg_starts[blockIdx.x];
  const TokMeta mt = load_meta(a.meta, a.ntok, i0);
  const int len = mt.seg_end - mt.seg_begin;
  if (len > max_len) return;
  const int H = a.H, D = a.D, DV = a.DV, rep = H / a.G, g = h / rep, K1 = a.taps - 1, C = a.conv_c;
  float* st = a.state + ((size_t)mt.slot * H + h) * D * DV;
  const int col = v0 + lc;
  VecF<VEC> S[NRW];
#pragma unroll
  for (int r = 0; r < NRW; ++r) {                                 // in flight while the first token is prepared
    const int d = r0 + r;
    if (mt.pos > 0 && d < D && col < DV) S[r] = ldv<VEC>(st + (size_t)d * DV + col);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[r].v[e] = 0.f;
    }
  }
  ConvRows<T> cv;
  cv.in = (const T*)a.p + (size_t)mt.seg_begin * a.ld + a.conv_off;
  cv.ld = a.ld; cv.first_pos = mt.pos; cv.K1 = K1; cv.C = C;
  cv.told = a.conv_w ? a.tail + ((size_t)mt.phase * a.slots + mt.slot) * K1 * C : nullptr;
  float* tnew = a.conv_w ? a.tail + ((size_t)(1 - mt.phase) * a.slots + mt.slot) * K1 * C : nullptr;
  const float rate = a.A_log ? expf(a.A_log[h]) : 0.f, dtb = a.A_log ? a.dt_bias[h] : 0.f;
  const float fixed = a.A_log ? 0.f : a.decay[h], skip = a.D_skip ? a.D_skip[h] : 0.f;
  const bool group_owner = h % rep == 0 && blockIdx.z == 0;       // writes the tail of the channels that the group's heads share
  constexpr int NE = (2 * DP + CW + 255) / 256;
  float hist[KT ? NE : 1][KT ? KT : 1], cwt[KT ? NE : 1][KT ? KT : 1], cbias[KT ? NE : 1];
  int ecol[KT ? NE : 1];                                          // columns of the entries this thread prepares, -1: padding
  if (KT) {
#pragma unroll
    for (int n = 0; n < NE; ++n) {
      const int e = tid + n * 256;
      int c = -1;
      if (e < DP) c = e < D ? a.q_off + g * D + e : -1;
      else if (e < 2 * DP) c = e - DP < D ? a.k_off + g * D + e - DP : -1;
      else if (e < 2 * DP + CW) c = v0 + e - 2 * DP < DV ? a.v_off + h * DV + v0 + e - 2 * DP : -1;
      ecol[n] = c;
      const int ch = max(c - a.conv_off, 0);
      cbias[n] = a.conv_b ? a.conv_b[ch] : 0.f;
#pragma unroll
      for (int j = 0; j < KT; ++j) {                              // leading weights of a shorter filter are zero
        const int jr = j - (KT - a.taps);
        const float w = a.conv_w[(size_t)ch * a.taps + max(jr, 0)];
        cwt[n][j] = jr >= 0 ? w : 0.f;
      }
#pragma unroll
      for (int j = 0; j < KT - 1; ++j) {                          // inputs before the step: position pos - (KT - 1) + j
        const int r = j - (KT - 1 - K1);                          // row of the tail
        const float v = K1 > 0 ? cv.told[(size_t)max(r, 0) * C + ch] : 0.f;
        hist[n][j] = r >= 0 && mt.pos - (KT - 1) + j >= 0 ? v : 0.f;
      }
    }
  }
  for (int tt = 0; tt < len; ++tt) {
    const int i = i0 + tt, pos = mt.pos + tt, buf = tt & 1;
    const T* row = (const T*)a.p + (size_t)i * a.ld;
    auto value = [&](int c, bool owner) {                         // column c of the row
      float z;
      if (a.conv_w) {
        const int ch = c - a.conv_off;
        z = a.conv_b ? a.conv_b[ch] : 0.f;
        for (int j = 0; j <= K1; ++j) z += a.conv_w[(size_t)ch * a.taps + j] * cv.get(pos - K1 + j, ch);
        if (owner && tt == len - 1) cv.write_tail(tnew, pos, ch);
      } else z = to_f(row[c]);
      if (a.silu) z = to_f(from_f<T>(silu_act<T>(z)));            // the activated value has the activation type, as from the convolution kernel
      return z;
    };
    if (KT) {
#pragma unroll
      for (int n = 0; n < NE; ++n) {
        const int e = tid + n * 256;
        if (e >= 2 * DP + CW) continue;
        hist[n][KT ? KT - 1 : 0] = to_f(row[max(ecol[n], 0)]);
        float z = cbias[n];
#pragma unroll
        for (int j = 0; j < KT; ++j) z += cwt[n][j] * hist[n][j];
        if (a.silu) z = to_f(from_f<T>(silu_act<T>(z)));
        float* dst = e < DP ? &sq[buf][e] : e < 2 * DP ? &sk[buf][e - DP] : &sv[buf][e - 2 * DP];
        *dst = ecol[n] >= 0 ? z : 0.f;
        if (tt == len - 1 && ecol[n] >= 0 && (e >= 2 * DP || group_owner))
#pragma unroll
          for (int j = 1; j < KT; ++j)
            if (j >= KT - K1) tnew[(size_t)(j - (KT - K1)) * C + ecol[n] - a.conv_off] = hist[n][j];
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j) hist[n][j] = hist[n][j + 1];
      }
    } else
    for (int e = tid; e < 2 * DP + CW; e += 256) {
      if (e < DP) sq[buf][e] = e < D ? value(a.q_off + g * D + e, group_owner) : 0.f;
      else if (e < 2 * DP) sk[buf][e - DP] = e - DP < D ? value(a.k_off + g * D + e - DP, group_owner) : 0.f;
      else sv[buf][e - 2 * DP] = v0 + e - 2 * DP < DV ? value(a.v_off + h * DV + v0 + e - 2 * DP, true) : 0.f;
    }
    float dt = 1.f, decay = fixed;
    if (a.A_log) {
      dt = softplus_f(to_f(((const T*)a.dt)[(size_t)i * a.dt_ld + h]) + dtb);
      decay = expf(-rate * dt);
    }
    __syncthreads();
    VecF<VEC> v = ldv<VEC>(&sv[buf][lc]), acc;
#pragma unroll
    for (int e = 0; e < VEC; ++e) { v.v[e] *= dt; acc.v[e] = 0.f; }
#pragma unroll
    for (int r = 0; r < NRW; ++r) {
      const float k = sk[buf][r0 + r], q = sq[buf][r0 + r];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        S[r].v[e] = decay * S[r].v[e] + k * v.v[e];
        acc.v[e] += q * S[r].v[e];
      }
    }
#pragma unroll
    for (int off = LPR; off < 32; off <<= 1)                      // the row groups of a warp
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc.v[e] += __shfl_xor_sync(0xffffffffu, acc.v[e], off);
    if ((tid & 31) < LPR) stv<VEC>(&red[warp][lc], acc);
    __syncthreads();
    for (int c = tid; c < CW; c += 256) {
      if (v0 + c >= DV) continue;
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) s += red[k][c];
      a.y[((size_t)i * H + h) * DV + v0 + c] = s + skip * sv[buf][c];
    }
  }
  if (col < DV) {
#pragma unroll
    for (int r = 0; r < NRW; ++r) {
      const int d = r0 + r;
      if (d < D) stv<VEC>(st + (size_t)d * DV + col, S[r]);
    }
  }
}

// Chunk form (bfloat16). With L_t the sum of the log decays of a chunk of 64 tokens up to and including token t, and S0 the state
// before the chunk,
//   y_t = exp(L_t) S0^T q_t + sum_{s<=t} exp(L_t - L_s) dt_s (q_t . k_s) v_s + D v_t,
//   S   = exp(L_63) S0 + sum_s exp(L_63 - L_s) dt_s k_s v_s^T.
// Every exponent is a difference of a later and an earlier sum, never positive: nothing overflows however strong the decay. Three
// launches: the second sum of every chunk at once (scalar_decay_chunk_kernel), the walk over the chunks of each sequence, which leaves
// the state before every chunk as a two-term bfloat16 split in the same place (scalar_decay_walk_kernel), and the read-outs of all
// chunks (scalar_decay_out_kernel). The products run on the tensor cores with float32 accumulators; q, k and v are bfloat16 by
// themselves, the float32 factors enter as two-term splits.
constexpr int CHK = 64, CPAD = 8;

struct ChunkHead {
  int i0, nb;                                                     // first batch row, tokens
};

// dt and running log decays of a chunk's tokens for head h into sdt[64], sL[64] (threads 0 .. 63; a barrier follows at the caller)
template <typename T>
__device__ __forceinline__ void chunk_decays(const qspec_scalar_decay_args& a, const ChunkHead& ch, int h, float* sdt, float* sL, float* swarp) {
  const int tid = threadIdx.x, lane = tid & 31;
  float l = 0.f;
  if (tid < CHK) {
    float dt = 0.f;
    if (tid < ch.nb) {
      dt = 1.f;
      if (a.A_log) {
        dt = softplus_f(to_f(((const T*)a.dt)[(size_t)(ch.i0 + tid) * a.dt_ld + h]) + a.dt_bias[h]);
        l = -expf(a.A_log[h]) * dt;
      } else l = a.log_decay[h];
    }
    sdt[tid] = dt;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const float o = __shfl_up_sync(0xffffffffu, l, off);
      if (lane >= off) l += o;
    }
    if (tid == 31) *swarp = l;
  }
  __syncthreads();
  if (tid < CHK) sL[tid] = tid < 32 ? l : l + *swarp;
}

__device__ __forceinline__ uint32_t silu_bf2(uint32_t p) {
  const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&p));
  const __nv_bfloat162 r = __floats2bfloat162_rn(silu_act<bf16_t>(f.x), silu_act<bf16_t>(f.y));
  return *reinterpret_cast<const uint32_t*>(&r);
}
// 64 rows x N columns of a bfloat16 section into shared memory by NT threads, eight columns per load; rows past the chunk and columns
// past `lim` zero. Without silu the copies are asynchronous (the caller commits and waits); with it they pass through registers, all
// loads of a batch before the first store.
template <int N, int NT>
__device__ __forceinline__ void stage_rows(bf16_t* dst, int ds, const bf16_t* src, int ld, int lim, int nb, bool silu) {
  constexpr int PER = N / 8, TOTAL = CHK * PER / NT, BATCH = TOTAL < 8 ? TOTAL : 8;
  if (!silu) {
#pragma unroll
    for (int r = 0; r < TOTAL; ++r) {
      const int e = threadIdx.x + r * NT, t = e / PER, c = (e % PER) * 8;
      const bool ok = t < nb && c < lim;
      cp_async_16z(dst + t * ds + c, ok ? src + (size_t)t * ld + c : src, ok);
    }
    return;
  }
#pragma unroll
  for (int r0 = 0; r0 < TOTAL; r0 += BATCH) {
    uint4 v[BATCH];
#pragma unroll
    for (int r = 0; r < BATCH; ++r) {
      const int e = threadIdx.x + (r0 + r) * NT, t = e / PER, c = (e % PER) * 8;
      v[r] = *reinterpret_cast<const uint4*>(src + (size_t)min(t, nb - 1) * ld + (c < lim ? c : 0));
    }
#pragma unroll
    for (int r = 0; r < BATCH; ++r) {
      const int e = threadIdx.x + (r0 + r) * NT, t = e / PER, c = (e % PER) * 8;
      uint4 w = make_uint4(silu_bf2(v[r].x), silu_bf2(v[r].y), silu_bf2(v[r].z), silu_bf2(v[r].w));
      if (t >= nb || c >= lim) w = make_uint4(0u, 0u, 0u, 0u);
      *reinterpret_cast<uint4*>(dst + t * ds + c) = w;
    }
  }
}

// What a chunk adds to the state: [D x 64 tokens] x [64 tokens x 64 value columns], warps over the rows in tiles of 16. The values
// carry the factor exp(L_63 - L_s) dt_s, as a two-term split.
template <int DP>
__global__ void __launch_bounds__(128)
scalar_decay_chunk_kernel(const qspec_scalar_decay_args a, const int* __restrict__ chunk_rows, float* __restrict__ add, float* __restrict__ total) {
  pdl_enter();
  extern __shared__ __align__(16) unsigned char sm_sc[];
  constexpr int KS = DP + CPAD, VS = 64 + CPAD;
  bf16_t* sk = reinterpret_cast<bf16_t*>(sm_sc);                  // [64][KS]
  bf16_t* sh = sk + CHK * KS;                                     // [64][VS] high parts
  bf16_t* sl = sh + CHK * VS;                                     // [64][VS] low parts
  __shared__ float sdt[CHK], sL[CHK], swarp;
  const int x = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int H = a.H, D = a.D, DV = a.DV, g = h / (H / a.G);
  ChunkHead ch;
  ch.i0 = chunk_rows[x];
  ch.nb = min(CHK, a.meta[3 * a.ntok + ch.i0] - ch.i0);
  const bf16_t* base = (const bf16_t*)a.p + (size_t)ch.i0 * a.ld;
  const int nv = min(64, DV - v0);
  stage_rows<DP, 128>(sk, KS, base + a.k_off + g * D, a.ld, D, ch.nb, a.silu);
  cp_async_commit();
  uint4 val[4];                                                   // this thread's values, in flight during the decays
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int e = tid + r * 128, t = min(e >> 3, ch.nb - 1), c = (e & 7) * 8;
    val[r] = *reinterpret_cast<const uint4*>(base + (size_t)t * a.ld + a.v_off + h * DV + v0 + (c < nv ? c : 0));
  }
  chunk_decays<bf16_t>(a, ch, h, sdt, sL, &swarp);
  __syncthreads();                                                // sL is complete
  const float end = sL[CHK - 1];
  if (tid == 0 && blockIdx.z == 0) total[(size_t)x * H + h] = expf(end);
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int e = tid + r * 128, t = e >> 3, c = (e & 7) * 8;
    uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
    if (t < ch.nb && c < nv) {
      uint4 v = val[r];
      if (a.silu) { v.x = silu_bf2(v.x); v.y = silu_bf2(v.y); v.z = silu_bf2(v.z); v.w = silu_bf2(v.w); }
      const float f = expf(end - sL[t]) * sdt[t];
      const uint32_t in[4] = {v.x, v.y, v.z, v.w};
      uint32_t hp[4], lp[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in[k]));
        tk_split_bf2(w.x * f, w.y * f, hp[k], lp[k]);
      }
      hi = make_uint4(hp[0], hp[1], hp[2], hp[3]);
      lo = make_uint4(lp[0], lp[1], lp[2], lp[3]);
    }
    *reinterpret_cast<uint4*>(sh + t * VS + c) = hi;
    *reinterpret_cast<uint4*>(sl + t * VS + c) = lo;
  }
  cp_async_wait<0>();
  __syncthreads();
  const int mr = lane & 7, mm = lane >> 3;
  float* dst = add + ((size_t)x * H + h) * D * DV;
  for (int d0 = warp * 16; d0 < D; d0 += 64) {
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
#pragma unroll
    for (int s0 = 0; s0 < CHK; s0 += 16) {
      uint32_t A[4];
      tk_ldmatrix_x4_trans(A, sk + (s0 + (mm >> 1) * 8 + mr) * KS + d0 + (mm & 1) * 8);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        uint32_t B[4];
        const int at = (s0 + (mm & 1) * 8 + mr) * VS + n * 8 + (mm >> 1) * 8;
        tk_ldmatrix_x4_trans(B, sh + at);
        tk_mma_16816(acc[n], A, B[0], B[1]);
        tk_mma_16816(acc[n + 1], A, B[2], B[3]);
        tk_ldmatrix_x4_trans(B, sl + at);
        tk_mma_16816(acc[n], A, B[0], B[1]);
        tk_mma_16816(acc[n + 1], A, B[2], B[3]);
      }
    }
    const int d = d0 + (lane >> 2);
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int c = n * 8 + (lane & 3) * 2;
      if (c >= nv) continue;
      if (d < D) *reinterpret_cast<float2*>(dst + (size_t)d * DV + v0 + c) = make_float2(acc[n][0], acc[n][1]);
      if (d + 8 < D) *reinterpret_cast<float2*>(dst + (size_t)(d + 8) * DV + v0 + c) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

// The walk over a sequence's chunks, four neighbouring entries of the state per thread: what a chunk adds is replaced by the state
// before the chunk, high part in the lower half of the word and low part in the upper. Four chunks are in flight.
__global__ void __launch_bounds__(256)
scalar_decay_walk_kernel(const qspec_scalar_decay_args a, const int* __restrict__ starts, const int* __restrict__ chunk0, float* add,
                         const float* __restrict__ total) {
  pdl_enter();
  const int n = a.D * a.DV, c = (blockIdx.x * 256 + threadIdx.x) * 4, h = blockIdx.y;
  if (c >= n) return;
  const int i0 = starts[blockIdx.z], x0 = chunk0[blockIdx.z];
  const TokMeta mt = load_meta(a.meta, a.ntok, i0);
  const int nch = (mt.seg_end - mt.seg_begin + CHK - 1) / CHK;
  float* st = a.state + ((size_t)mt.slot * a.H + h) * n + c;
  float4 S = mt.pos > 0 ? *reinterpret_cast<const float4*>(st) : make_float4(0.f, 0.f, 0.f, 0.f);
  const size_t step = (size_t)a.H * n;
  float* p = add + ((size_t)x0 * a.H + h) * n + c;
  const float* tp = total + (size_t)x0 * a.H + h;
  constexpr int AHEAD = 4;
  for (int b0 = 0; b0 < nch; b0 += AHEAD) {
    float4 v[AHEAD];
    float f[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int b = min(b0 + u, nch - 1);
      v[u] = *reinterpret_cast<const float4*>(p + (size_t)b * step);
      f[u] = tp[(size_t)b * a.H];
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      if (b0 + u >= nch) break;
      uint32_t h0, l0, h1, l1;
      tk_split_bf2(S.x, S.y, h0, l0);
      tk_split_bf2(S.z, S.w, h1, l1);
      uint4 w;
      w.x = __byte_perm(h0, l0, 0x5410); w.y = __byte_perm(h0, l0, 0x7632);
      w.z = __byte_perm(h1, l1, 0x5410); w.w = __byte_perm(h1, l1, 0x7632);
      *reinterpret_cast<uint4*>(p + (size_t)(b0 + u) * step) = w;
      S.x = f[u] * S.x + v[u].x; S.y = f[u] * S.y + v[u].y;
      S.z = f[u] * S.z + v[u].z; S.w = f[u] * S.w + v[u].w;
    }
  }
  *reinterpret_cast<float4*>(st) = S;
}

// The read-outs of a chunk: eight warps of 16 tokens and 32 of the CTA's 64 value columns each. First q S0, whose rows are scaled by exp(L_t) in the
// accumulators; then the masked, decayed scores go from the accumulators of q k^T straight into the product with the values.
template <int DP>
__global__ void __launch_bounds__(256)
scalar_decay_out_kernel(const qspec_scalar_decay_args a, const int* __restrict__ chunk_rows, const float* __restrict__ states) {
  pdl_enter();
  extern __shared__ __align__(16) unsigned char sm_so[];
  constexpr int KS = DP + CPAD, VS = 64 + CPAD;
  bf16_t* sq = reinterpret_cast<bf16_t*>(sm_so);                  // [64][KS]
  bf16_t* sk = sq + CHK * KS;                                     // [64][KS]
  bf16_t* sv = sk + CHK * KS;                                     // [64][VS]
  bf16_t* sh = sv + CHK * VS;                                     // [DP][VS] state, high parts
  bf16_t* sl = sh + DP * VS;                                      // [DP][VS] low parts
  __shared__ float sdt[CHK], sL[CHK], swarp;
  const int x = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int H = a.H, D = a.D, DV = a.DV, g = h / (H / a.G), nv = min(64, DV - v0);
  ChunkHead ch;
  ch.i0 = chunk_rows[x];
  ch.nb = min(CHK, a.meta[3 * a.ntok + ch.i0] - ch.i0);
  const bf16_t* base = (const bf16_t*)a.p + (size_t)ch.i0 * a.ld;
  const float* src = states + ((size_t)x * H + h) * D * DV + v0;
  stage_rows<DP, 256>(sq, KS, base + a.q_off + g * D, a.ld, D, ch.nb, a.silu);
  stage_rows<DP, 256>(sk, KS, base + a.k_off + g * D, a.ld, D, ch.nb, a.silu);
  stage_rows<64, 256>(sv, VS, base + a.v_off + h * DV + v0, a.ld, nv, ch.nb, a.silu);
  cp_async_commit();
#pragma unroll
  for (int r0 = 0; r0 < DP / 16; r0 += 4) {                        // the state before the chunk, its halves apart
    uint4 v[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int e = tid + (r0 + r) * 256, d = e >> 4, c = (e & 15) * 4;
      v[r] = *reinterpret_cast<const uint4*>(src + (size_t)min(d, D - 1) * DV + (c < nv ? c : 0));
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int e = tid + (r0 + r) * 256, d = e >> 4, c = (e & 15) * 4;
      const bool ok = d < D && c < nv;
      uint2 hi = make_uint2(__byte_perm(v[r].x, v[r].y, 0x5410), __byte_perm(v[r].z, v[r].w, 0x5410));
      uint2 lo = make_uint2(__byte_perm(v[r].x, v[r].y, 0x7632), __byte_perm(v[r].z, v[r].w, 0x7632));
      if (!ok) hi = lo = make_uint2(0u, 0u);
      *reinterpret_cast<uint2*>(sh + d * VS + c) = hi;
      *reinterpret_cast<uint2*>(sl + d * VS + c) = lo;
    }
  }
  chunk_decays<bf16_t>(a, ch, h, sdt, sL, &swarp);
  cp_async_wait<0>();
  __syncthreads();
  const int t0 = (warp & 3) * 16, n0 = (warp >> 2) * 32, mr = lane & 7, mm = lane >> 3, ra = t0 + (lane >> 2), rb = ra + 8, cq = (lane & 3) * 2;
  if (t0 >= ch.nb) return;                                        // (uniform over the warp; no barrier follows)
  float y[4][4], s[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) y[n & 3][e] = s[n][e] = 0.f;
  for (int d0 = 0; d0 < D; d0 += 16) {
    uint32_t A[4], B[4];
    tk_ldmatrix_x4(A, sq + (t0 + (mm & 1) * 8 + mr) * KS + d0 + (mm >> 1) * 8);
#pragma unroll
    for (int n = 0; n < 4; n += 2) {
      const int at = (d0 + (mm & 1) * 8 + mr) * VS + n0 + n * 8 + (mm >> 1) * 8;
      tk_ldmatrix_x4_trans(B, sh + at);
      tk_mma_16816(y[n], A, B[0], B[1]);
      tk_mma_16816(y[n + 1], A, B[2], B[3]);
      tk_ldmatrix_x4_trans(B, sl + at);
      tk_mma_16816(y[n], A, B[0], B[1]);
      tk_mma_16816(y[n + 1], A, B[2], B[3]);
    }
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      if (n * 8 <= t0 + 15) {                                     // token columns the warp's rows can see
        tk_ldmatrix_x4(B, sk + (n * 8 + (mm >> 1) * 8 + mr) * KS + d0 + (mm & 1) * 8);
        tk_mma_16816(s[n], A, B[0], B[1]);
        tk_mma_16816(s[n + 1], A, B[2], B[3]);
      }
    }
  }
  const float La = sL[ra], Lb = sL[rb], ea = expf(La), eb = expf(Lb);
#pragma unroll
  for (int n = 0; n < 4; ++n) { y[n][0] *= ea; y[n][1] *= ea; y[n][2] *= eb; y[n][3] *= eb; }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    if (j * 16 > t0 + 15) break;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      float wgt[4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = (2 * j + u) * 8 + cq + e;
        const float Lc = sL[c], dc = sdt[c];
        wgt[e] = c <= ra ? s[2 * j + u][e] * (expf(La - Lc) * dc) : 0.f;
        wgt[2 + e] = c <= rb ? s[2 * j + u][2 + e] * (expf(Lb - Lc) * dc) : 0.f;
      }
      tk_split_bf2(wgt[0], wgt[1], hi[2 * u], lo[2 * u]);
      tk_split_bf2(wgt[2], wgt[3], hi[2 * u + 1], lo[2 * u + 1]);
    }
#pragma unroll
    for (int n = 0; n < 4; n += 2) {
      uint32_t B[4];
      tk_ldmatrix_x4_trans(B, sv + (j * 16 + (mm & 1) * 8 + mr) * VS + n0 + n * 8 + (mm >> 1) * 8);
      tk_mma_16816(y[n], hi, B[0], B[1]);
      tk_mma_16816(y[n], lo, B[0], B[1]);
      tk_mma_16816(y[n + 1], hi, B[2], B[3]);
      tk_mma_16816(y[n + 1], lo, B[2], B[3]);
    }
  }
  const float skip = a.D_skip ? a.D_skip[h] : 0.f;
#pragma unroll
  for (int n = 0; n < 4; ++n) {
    const int c = n0 + n * 8 + cq;
    if (c >= nv) continue;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = u ? rb : ra;
      if (t >= ch.nb) continue;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + t * VS + c));
      *reinterpret_cast<float2*>(a.y + ((size_t)(ch.i0 + t) * H + h) * DV + v0 + c) =
          make_float2(y[n][2 * u] + skip * v.x, y[n][2 * u + 1] + skip * v.y);
    }
  }
}

}  // namespace qspec

using namespace qspec;
#define SC_DTYPE_OK(dtype) QSPEC_REQUIRE((dtype) == QSPEC_DTYPE_BF16 || (dtype) == QSPEC_DTYPE_F32, QSPEC_ERR_UNSUPPORTED, \
                                         "dtype %d: bfloat16 (1) or float32 (2) expected", (dtype))

template <typename T, int VEC, int NV>
static int launch_sandwich(const float* x_in, float* x_out, const void* y, int y_parts, long long y_part_stride, long long y_tok_stride,
                           const float* y_w, const void* y2, const float* post_w, const float* pre_w, float w_offset, void* out, int ntok, int W,
                           float eps, cudaStream_t st) {
  launch_pdl(sandwich_norm_kernel<T, VEC, NV>, dim3(ntok), dim3(256), 0, st, x_in, x_out, (const T*)y, y_parts, y_part_stride, y_tok_stride, y_w,
             (const T*)y2, post_w, pre_w, w_offset, (T*)out, W, eps);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <typename T>
static int launch_sandwich_n(const float* x_in, float* x_out, const void* y, int y_parts, long long y_part_stride, long long y_tok_stride,
                             const float* y_w, const void* y2, const float* post_w, const float* pre_w, float w_offset, void* out, int ntok,
                             int W, float eps, cudaStream_t st) {
  const bool vec = W % 4 == 0 && y_part_stride % 4 == 0 && y_tok_stride % 4 == 0 &&
                   (((uintptr_t)x_in | (uintptr_t)x_out | (uintptr_t)post_w | (uintptr_t)pre_w) & 15) == 0 &&
                   (((uintptr_t)y | (uintptr_t)y2 | (uintptr_t)out) & (4 * sizeof(T) - 1)) == 0;
  const int nv = vec ? (W + 1023) / 1024 : (W + 255) / 256;
#define SN_ARGS x_in, x_out, y, y_parts, y_part_stride, y_tok_stride, y_w, y2, post_w, pre_w, w_offset, out, ntok, W, eps, st
  if (vec) {
    if (nv <= 1) return launch_sandwich<T, 4, 1>(SN_ARGS);
    if (nv <= 2) return launch_sandwich<T, 4, 2>(SN_ARGS);
    if (nv <= 4) return launch_sandwich<T, 4, 4>(SN_ARGS);
    if (nv <= 8) return launch_sandwich<T, 4, 8>(SN_ARGS);
    return launch_sandwich<T, 4, 16>(SN_ARGS);
  }
  if (nv <= 2) return launch_sandwich<T, 1, 2>(SN_ARGS);
  if (nv <= 8) return launch_sandwich<T, 1, 8>(SN_ARGS);
  return launch_sandwich<T, 1, 64>(SN_ARGS);
#undef SN_ARGS
}

extern "C" int qspec_seq_sandwich_norm(const float* x_in, float* x_out, const void* y, int y_parts, long long y_part_stride,
                                       long long y_tok_stride, const float* y_w, const void* y2, const float* post_w, const float* pre_w,
                                       float w_offset, void* out, int ntok, int W, float eps, int dtype, void* stream) {
  QSPEC_REQUIRE(x_in && (x_out || out) && (!y || post_w) && (!out || pre_w) && (y || !y2), QSPEC_ERR_INVALID_ARG, "seq_sandwich_norm: null pointer");
  QSPEC_REQUIRE(ntok >= 0 && W > 0 && W <= 16384 && y_parts >= 1, QSPEC_ERR_UNSUPPORTED, "seq_sandwich_norm: width %d (<= 16384)", W);
  SC_DTYPE_OK(dtype);
  if (ntok == 0) return QSPEC_OK;
#define SN_CALL x_in, x_out, y, y_parts, y_part_stride, y_tok_stride, y_w, y2, post_w, pre_w, w_offset, out, ntok, W, eps, (cudaStream_t)stream
  if (dtype == QSPEC_DTYPE_F32) return launch_sandwich_n<float>(SN_CALL);
  return launch_sandwich_n<bf16_t>(SN_CALL);
#undef SN_CALL
}

template <typename T, int VEC>
static int launch_part_norm(const float* src, const float* w, const void* gate, int gate_ld, int gate_mode, void* out, int out_ld, int ntok,
                            int parts, int n, float eps, float out_scale, cudaStream_t st) {
  const long long rows = (long long)ntok * parts;
#define PN_ARGS src, w, (const T*)gate, gate_ld, gate_mode, (T*)out, out_ld, rows, parts, n, eps, out_scale
  const int tpp = n <= 1024 ? 32 : 256, keep = (n + tpp * VEC - 1) / (tpp * VEC);
  const dim3 grid((unsigned)((rows + 256 / tpp - 1) / (256 / tpp)));
#define PN_KEEP(TPP)                                                                                                 \
  do {                                                                                                               \
    if (keep <= 2) launch_pdl(part_norm_kernel<T, VEC, TPP, 2>, grid, dim3(256), 0, st, PN_ARGS);                    \
    else if (keep <= 4) launch_pdl(part_norm_kernel<T, VEC, TPP, 4>, grid, dim3(256), 0, st, PN_ARGS);               \
    else launch_pdl(part_norm_kernel<T, VEC, TPP, 8>, grid, dim3(256), 0, st, PN_ARGS);                              \
  } while (0)
  if (tpp == 32) PN_KEEP(32);
  else PN_KEEP(256);
#undef PN_KEEP
#undef PN_ARGS
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

extern "C" int qspec_seq_part_norm(const float* src, const float* w, const void* gate, int gate_ld, int gate_mode, void* out, int out_ld,
                                   int ntok, int N, int parts, float eps, float out_scale, int dtype, void* stream) {
  QSPEC_REQUIRE(src && w && gate && out, QSPEC_ERR_INVALID_ARG, "seq_part_norm: null pointer");
  QSPEC_REQUIRE(ntok >= 0 && N > 0 && parts >= 1 && N % parts == 0 && gate_ld >= N && out_ld >= N, QSPEC_ERR_INVALID_ARG,
                "seq_part_norm: %d entries in %d parts", N, parts);
  QSPEC_REQUIRE(gate_mode == QSPEC_GATE_SIGMOID_AFTER || gate_mode == QSPEC_GATE_SILU_BEFORE, QSPEC_ERR_INVALID_ARG, "seq_part_norm: gate mode %d",
                gate_mode);
  SC_DTYPE_OK(dtype);
  if (ntok == 0) return QSPEC_OK;
  const int n = N / parts;
  const size_t es = dtype == QSPEC_DTYPE_F32 ? 4 : 2;
  const bool vec = n % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && (((uintptr_t)src | (uintptr_t)w) & 15) == 0 &&
                   (((uintptr_t)gate | (uintptr_t)out) & (4 * es - 1)) == 0;
#define PN_CALL src, w, gate, gate_ld, gate_mode, out, out_ld, ntok, parts, n, eps, out_scale, (cudaStream_t)stream
  if (dtype == QSPEC_DTYPE_F32) return vec ? launch_part_norm<float, 4>(PN_CALL) : launch_part_norm<float, 1>(PN_CALL);
  return vec ? launch_part_norm<bf16_t, 4>(PN_CALL) : launch_part_norm<bf16_t, 1>(PN_CALL);
#undef PN_CALL
}

template <typename T, int NRW, int VEC, int LPR>
static int launch_sd_token(const qspec_scalar_decay_args& a, int max_len, cudaStream_t st) {
  constexpr int CW = LPR * VEC;
  const dim3 grid(a.nseg, a.H, (a.DV + CW - 1) / CW);
  if (NRW * LPR <= 256 && a.conv_w && a.taps <= 4) launch_pdl(scalar_decay_token_kernel<T, NRW, VEC, LPR, NRW * LPR <= 256 ? 4 : 0>, grid, dim3(256), 0, st, a, max_len);
  else launch_pdl(scalar_decay_token_kernel<T, NRW, VEC, LPR, 0>, grid, dim3(256), 0, st, a, max_len);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <typename T, int VEC, int LPR>
static int launch_sd_token_n(const qspec_scalar_decay_args& a, int max_len, cudaStream_t st) {
  constexpr int F = LPR / 8;                                      // rows per group for 32 state rows in all
  if (a.D <= 32) return launch_sd_token<T, F, VEC, LPR>(a, max_len, st);
  if (a.D <= 64) return launch_sd_token<T, 2 * F, VEC, LPR>(a, max_len, st);
  if (a.D <= 128) return launch_sd_token<T, 4 * F, VEC, LPR>(a, max_len, st);
  return launch_sd_token<T, 8 * F, VEC, LPR>(a, max_len, st);
}

template <typename T>
static int launch_sd_tokens(const qspec_scalar_decay_args& a, int max_len, cudaStream_t st) {
  if (a.D > 256) {                                                // many rows: eight lanes share a row group
    if (a.DV % 4 == 0 && ((uintptr_t)a.state & 15) == 0) return a.D <= 512 ? launch_sd_token<T, 16, 4, 8>(a, max_len, st) : launch_sd_token<T, 32, 4, 8>(a, max_len, st);
    return a.D <= 512 ? launch_sd_token<T, 16, 1, 8>(a, max_len, st) : launch_sd_token<T, 32, 1, 8>(a, max_len, st);
  }
  if (a.DV % 4 == 0 && ((uintptr_t)a.state & 15) == 0) {          // four columns per lane, as many lanes per row as it needs
    if (a.DV <= 32) return launch_sd_token_n<T, 4, 8>(a, max_len, st);
    if (a.DV <= 64) return launch_sd_token_n<T, 4, 16>(a, max_len, st);
    return launch_sd_token_n<T, 4, 32>(a, max_len, st);
  }
  return launch_sd_token_n<T, 1, 32>(a, max_len, st);
}

template <int DP>
static int launch_sd_chunks(const qspec_scalar_decay_args& a, const int* chunk_rows, int nchunks, const int* starts, const int* chunk0, int nlong,
                            float* add, float* total, cudaStream_t st) {
  constexpr int KS = DP + CPAD, VS = 64 + CPAD;
  constexpr size_t smem_add = (size_t)(CHK * KS + 2 * CHK * VS) * 2, smem_out = (size_t)(2 * CHK * KS + CHK * VS + 2 * DP * VS) * 2;
  static bool configured = false;
  if (!configured) {
    QSPEC_CUDA(cudaFuncSetAttribute(scalar_decay_chunk_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_add));
    QSPEC_CUDA(cudaFuncSetAttribute(scalar_decay_out_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out));
    configured = true;
  }
  const dim3 grid(nchunks, a.H, (a.DV + 63) / 64);
  launch_pdl(scalar_decay_chunk_kernel<DP>, grid, dim3(128), smem_add, st, a, chunk_rows, add, total);
  QSPEC_CHECK_LAUNCH(1);
  launch_pdl(scalar_decay_walk_kernel, dim3((a.D * a.DV + 1023) / 1024, a.H, nlong), dim3(256), 0, st, a, starts, chunk0, add, (const float*)total);
  QSPEC_CHECK_LAUNCH(1);
  launch_pdl(scalar_decay_out_kernel<DP>, grid, dim3(256), smem_out, st, a, chunk_rows, (const float*)add);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

extern "C" size_t qspec_seq_scalar_decay_scratch_bytes(int nchunks, int H, int D, int DV) {
  if (nchunks <= 0) return 0;
  return ((size_t)nchunks * H * D * DV + (size_t)nchunks * H) * sizeof(float);
}

extern "C" int qspec_seq_scalar_decay_chunks_supported(int ld, int q_off, int k_off, int v_off, int D, int DV) {
  return D > 0 && D <= 256 && D % 8 == 0 && DV > 0 && DV % 8 == 0 && ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0;
}

static int check_scalar_decay(const qspec_scalar_decay_args* a, int dtype) {
  QSPEC_REQUIRE(a && a->p && a->state && a->y && a->meta && a->seg_starts && (a->A_log ? (a->dt && a->dt_bias) : (a->decay && a->log_decay)),
                QSPEC_ERR_INVALID_ARG, "seq_scalar_decay: null pointer");
  QSPEC_REQUIRE(a->ntok >= 0 && a->nseg >= 0 && a->H > 0 && a->H <= 65535 && a->G > 0 && a->H % a->G == 0 && a->D > 0 && a->D <= 1024 && a->DV > 0 &&
                    a->DV <= 65535 * 8,
                QSPEC_ERR_UNSUPPORTED, "seq_scalar_decay: heads %d / %d, key size %d (<= 1024), value size %d", a->H, a->G, a->D, a->DV);
  QSPEC_REQUIRE(a->q_off >= 0 && a->k_off >= 0 && a->v_off >= 0 && a->q_off + a->G * a->D <= a->ld && a->k_off + a->G * a->D <= a->ld &&
                    a->v_off + a->H * a->DV <= a->ld,
                QSPEC_ERR_INVALID_ARG, "seq_scalar_decay: sections outside the row");
  SC_DTYPE_OK(dtype);
  return QSPEC_OK;
}

extern "C" int qspec_seq_scalar_decay_tokens(const qspec_scalar_decay_args* a, int max_len, int dtype, void* stream) {
  const int s = check_scalar_decay(a, dtype);
  if (s) return s;
  if (a->conv_w) {
    const int lo = a->q_off < a->k_off ? (a->q_off < a->v_off ? a->q_off : a->v_off) : (a->k_off < a->v_off ? a->k_off : a->v_off);
    QSPEC_REQUIRE(a->taps >= 1 && a->taps <= 64 && (a->tail || a->taps == 1) && a->slots > 0 && a->conv_off >= 0 && a->conv_off <= lo &&
                      a->q_off + a->G * a->D <= a->conv_off + a->conv_c && a->k_off + a->G * a->D <= a->conv_off + a->conv_c &&
                      a->v_off + a->H * a->DV <= a->conv_off + a->conv_c,
                  QSPEC_ERR_INVALID_ARG, "seq_scalar_decay: a convolution of %d taps over %d channels", a->taps, a->conv_c);
  }
  if (a->ntok == 0 || a->nseg == 0) return QSPEC_OK;
  if (dtype == QSPEC_DTYPE_F32) return launch_sd_tokens<float>(*a, max_len, (cudaStream_t)stream);
  return launch_sd_tokens<bf16_t>(*a, max_len, (cudaStream_t)stream);
}

extern "C" int qspec_seq_scalar_decay_chunks(const qspec_scalar_decay_args* a, const int* chunk_rows, int nchunks, const int* starts,
                                             const int* chunk0, int nlong, void* scratch, size_t scratch_bytes, void* stream) {
  const int s = check_scalar_decay(a, QSPEC_DTYPE_BF16);
  if (s) return s;
  QSPEC_REQUIRE(qspec_seq_scalar_decay_chunks_supported(a->ld, a->q_off, a->k_off, a->v_off, a->D, a->DV) && !a->conv_w &&
                    (((uintptr_t)a->p | (uintptr_t)a->state) & 15) == 0 && ((uintptr_t)a->y & 7) == 0,
                QSPEC_ERR_UNSUPPORTED, "seq_scalar_decay: sizes or addresses off the boundaries of the chunk form");
  if (a->ntok == 0 || nlong == 0) return QSPEC_OK;
  QSPEC_REQUIRE(chunk_rows && starts && chunk0 && nchunks >= nlong && nlong <= 65535 && scratch && ((uintptr_t)scratch & 15) == 0 &&
                    scratch_bytes >= qspec_seq_scalar_decay_scratch_bytes(nchunks, a->H, a->D, a->DV),
                QSPEC_ERR_INVALID_ARG, "seq_scalar_decay: chunk table or scratch missing for %d segments", nlong);
  float* add = (float*)scratch;
  float* total = add + (size_t)nchunks * a->H * a->D * a->DV;
  cudaStream_t st = (cudaStream_t)stream;
  if (a->D <= 64) return launch_sd_chunks<64>(*a, chunk_rows, nchunks, starts, chunk0, nlong, add, total, st);
  if (a->D <= 128) return launch_sd_chunks<128>(*a, chunk_rows, nchunks, starts, chunk0, nlong, add, total, st);
  return launch_sd_chunks<256>(*a, chunk_rows, nchunks, starts, chunk0, nlong, add, total, st);
}
