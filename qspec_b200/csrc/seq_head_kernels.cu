// Sequence-mixer kernels, fifth file: a norm without statistics fused with the residual sum, attention heads prepared straight from
// the projection (short convolution, norm, rotation, position-dependent temperature, cache rows), the gated delta rule with one
// decay per key channel (a one-launch form for decoding, a block form for prompts), and the logit soft cap. bfloat16 / float32
// activations (template T); everything that is normed, exponentiated or carried from token to token is float32.
#include "seq_common.cuh"
#include "../../include/qspec_b200_seq.h"
#include <stdint.h>
#include <stdlib.h>

namespace qspec {

typedef __nv_bfloat16 bf16_t;

// ---- residual sum and a tanh norm of the result -------------------------------------------------------------------------------
// r = x_in + mult * (sum_p y_w[t, p] y[t, p] + y_bias); out = tanh(alpha r) * w + b. No statistic of the row is needed, so the work
// is cut by columns as well as by rows.
template <typename T, typename YT, int VEC>
__global__ void __launch_bounds__(256)
residual_tanh_kernel(const float* __restrict__ x_in, float* __restrict__ x_out, const YT* __restrict__ y, int y_parts,
                     long long y_part_stride, long long y_tok_stride, const float* __restrict__ y_w, const float* __restrict__ y_bias,
                     float mult, float alpha, const float* __restrict__ w, const float* __restrict__ b, T* __restrict__ out, int W) {
  pdl_enter();
  const int i = blockIdx.x, c = ((int)blockIdx.y * 256 + (int)threadIdx.x) * VEC;
  if (c >= W) return;
  VecF<VEC> r = ldv<VEC>(x_in + (size_t)i * W + c);
  if (y) {
    const YT* yr = y + (size_t)i * y_tok_stride + c;
    VecF<VEC> v;
    if (y_bias) v = ldv<VEC>(y_bias + c);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] = 0.f;
    }
#pragma unroll 4
    for (int p = 0; p < y_parts; ++p) {
      const float wp = y_w ? y_w[(size_t)i * y_parts + p] : 1.0f;
      const VecF<VEC> t = ldv<VEC>(yr + (size_t)p * y_part_stride);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += wp * t.v[e];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) r.v[e] += mult * v.v[e];
  }
  if (x_out) stv<VEC>(x_out + (size_t)i * W + c, r);
  if (out) {
    const VecF<VEC> wv = ldv<VEC>(w + c), bv = ldv<VEC>(b + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) r.v[e] = tanhf(alpha * r.v[e]) * wv.v[e] + bv.v[e];
    stv<VEC>(out + (size_t)i * W + c, r);
  }
}

template <int VEC> __global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ a, long long n, float cap) {
  pdl_enter();
  for (long long k = ((long long)blockIdx.x * 256 + threadIdx.x) * VEC; k < n; k += (long long)gridDim.x * 256 * VEC) {
    VecF<VEC> v = ldv<VEC>(a + k);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] = cap * tanhf(v.v[e] / cap);
    stv<VEC>(a + k, v);
  }
}

// ---- attention heads from the projection ----------------------------------------------------------------------------------------
// One warp per token, eight consecutive tokens per CTA, the heads in turn (query heads, key heads, value heads); lanes hold VEC
// neighbouring channels NCV times. Per head: convolution (optional), unit-RMS norm with a weight before the rotation or without
// one after it or none, rotation of the first rot_dims entries (entry i with i + rot_dims / 2, or 2i with 2i + 1; angle pos *
// inv_freq[i], cosine and sine times an amplitude), temperature of the queries. Values are a section of their own or the key heads as projected.
template <typename T, int VEC, int NCV>
__global__ void __launch_bounds__(256)
head_prep_kernel(const qspec_head_prep_args a) {
  pdl_enter();
  extern __shared__ float sm_hp[];                                // per warp: row [D] (rotation only) | cos [half] | sin [half]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, i = blockIdx.x * 8 + warp;
  if (i >= a.ntok) return;                                        // warps are independent: no block barrier below
  const TokMeta mt = load_meta(a.meta, a.ntok, i);
  const int half = a.rot_dims / 2, D = a.D, DV = a.DV, H = a.H, G = a.G;
  float* buf = sm_hp + (size_t)warp * (half ? D + 2 * half : 0);
  float* s_cos = buf + D;
  float* s_sin = s_cos + half;
  for (int f = lane; f < half; f += 32) {                         // once per token, for all its heads
    float sn, cs;
    sincosf((float)mt.pos * a.inv_freq[f], &sn, &cs);
    s_cos[f] = cs * a.rot_amp;
    s_sin[f] = sn * a.rot_amp;
  }
  __syncwarp();
  const T* prow = (const T*)a.p + (size_t)i * a.ld;
  const int first_pos = mt.pos - (i - mt.seg_begin);
  const int HD = H * D, GD = G * D, K1 = a.taps - 1, C = HD + GD + G * DV;
  const float* told = a.conv_w ? a.tail + ((size_t)mt.phase * a.slots + mt.slot) * K1 * C : nullptr;
  float* tnew = a.conv_w ? a.tail + ((size_t)(1 - mt.phase) * a.slots + mt.slot) * K1 * C : nullptr;
  const bool last = i == mt.seg_end - 1, inside = i - mt.seg_begin >= K1 && K1 < 4;
  const float temp = a.temp_every > 0 ? 1.0f + a.temp_coef * logf((float)((mt.pos + 1) / a.temp_every + 1)) : 1.0f;
  const size_t crow = (size_t)mt.slot * a.cap + (size_t)ring_row(mt.pos, a.keep_first, a.cap);
  const int NH = H + G + (a.v_off >= 0 ? G : 0);
  for (int hh = blockIdx.y; hh < NH; hh += gridDim.y) {
    const int kind = hh < H ? 0 : (hh < H + G ? 1 : 2), head = kind == 0 ? hh : (kind == 1 ? hh - H : hh - H - G);
    const int n = kind == 2 ? DV : D;                             // channels of this head
    const int col = (kind == 0 ? a.q_off : (kind == 1 ? a.k_off : a.v_off)) + head * n;             // its columns in the row
    const int ch = (kind == 0 ? 0 : (kind == 1 ? HD : HD + GD)) + head * n;                         // its channels in the convolution
    VecF<VEC> x[NCV];
#pragma unroll
    for (int s = 0; s < NCV; ++s) {
      const int c = (s * 32 + lane) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[s].v[e] = 0.f;
      if (c >= n) continue;
      if (!a.conv_w) { x[s] = ldv<VEC>(prow + col + c); continue; }
      if (inside) {                                               // (uniform over the warp) every tap lies in the step: loads without branches
        VecF<VEC> u[4], wv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int back = min(j, K1);
          u[j] = ldv<VEC>(prow - (size_t)back * a.ld + col + c);
          wv[j] = ldv<VEC>(a.conv_w + (size_t)(K1 - back) * C + ch + c);
        }
#pragma unroll
        for (int j = 3; j >= 0; --j)                              // oldest first, as below
          if (j <= K1) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[s].v[e] += wv[j].v[e] * u[j].v[e];
          }
      } else
      for (int j = 0; j <= K1; ++j) {
        const int back = K1 - j, sp = mt.pos - back;              // source position
        VecF<VEC> u;
        if (sp >= first_pos) u = ldv<VEC>(prow - (size_t)back * a.ld + col + c);
        else if (sp >= 0) u = ldv<VEC>(told + (size_t)(sp - first_pos + K1) * C + ch + c);
        else continue;
        const VecF<VEC> wv = ldv<VEC>(a.conv_w + (size_t)j * C + ch + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[s].v[e] += wv.v[e] * u.v[e];
      }
      if (last)
        for (int r = 0; r < K1; ++r) {                            // the sequence's last inputs, into the other buffer
          const int back = K1 - 1 - r, sp = mt.pos - back;
          VecF<VEC> u;
          if (sp >= first_pos) u = ldv<VEC>(prow - (size_t)back * a.ld + col + c);
          else if (sp >= 0) u = ldv<VEC>(told + (size_t)(sp - first_pos + K1) * C + ch + c);
          else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
          }
          stv<VEC>(tnew + (size_t)r * C + ch + c, u);
        }
    }
    if (kind == 2 || (kind == 1 && a.v_off < 0)) {
      T* vdst = (T*)a.cache_v + (crow * G + head) * DV;
#pragma unroll
      for (int s = 0; s < NCV; ++s) {
        const int c = (s * 32 + lane) * VEC;
        if (c < n) stv<VEC>(vdst + c, x[s]);
      }
      if (kind == 2) continue;
    }
    const float* nw = kind == 0 ? a.qn_w : a.kn_w;
    auto unit = [&](const float* weight) {
      float ss = 0.f;
#pragma unroll
      for (int s = 0; s < NCV; ++s)
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += x[s].v[e] * x[s].v[e];      // channels past the head are zero
      const float rr = 1.0f / sqrtf(warp_xor_sum(ss) / (float)D + a.eps);
#pragma unroll
      for (int s = 0; s < NCV; ++s) {
        const int c = (s * 32 + lane) * VEC;
        if (c >= D) continue;
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[s].v[e] *= weight ? rr * weight[c + e] : rr;
      }
    };
    if (a.norm_last == QSPEC_HEAD_NORM_FIRST) unit(nw);
    if (half && VEC == 4 && a.pairing == QSPEC_ROTARY_INTERLEAVED) {       // both entries of a pair lie in one lane
#pragma unroll
      for (int s = 0; s < NCV; ++s)
#pragma unroll
        for (int e = 0; e + 1 < VEC; e += 2) {
          const int f = ((s * 32 + lane) * VEC + e) >> 1;
          if (f < half) {
            const float u = x[s].v[e], v = x[s].v[e + 1];
            x[s].v[e] = u * s_cos[f] - v * s_sin[f];
            x[s].v[e + 1] = v * s_cos[f] + u * s_sin[f];
          }
        }
    } else if (half) {
#pragma unroll
      for (int s = 0; s < NCV; ++s) {
        const int c = (s * 32 + lane) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e)
          if (c + e < D) buf[c + e] = x[s].v[e];
      }
      __syncwarp();
#pragma unroll
      for (int s = 0; s < NCV; ++s)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const int c = (s * 32 + lane) * VEC + e;
          if (c < 2 * half) {
            if (a.pairing == QSPEC_ROTARY_INTERLEAVED) {
              const int f = c >> 1;
              x[s].v[e] = (c & 1) ? buf[c] * s_cos[f] + buf[c - 1] * s_sin[f] : buf[c] * s_cos[f] - buf[c + 1] * s_sin[f];
              continue;
            }
            const int f = c < half ? c : c - half;
            x[s].v[e] = c < half ? buf[c] * s_cos[f] - buf[c + half] * s_sin[f] : buf[c] * s_cos[f] + buf[c - half] * s_sin[f];
          }
        }
      __syncwarp();
    }
    if (a.norm_last == QSPEC_HEAD_NORM_LAST) unit(nw);
    if (kind == 0) {
      float* qdst = a.qout + ((size_t)i * H + head) * D;
#pragma unroll
      for (int s = 0; s < NCV; ++s) {
        const int c = (s * 32 + lane) * VEC;
        if (c >= D) continue;
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[s].v[e] *= temp;
        stv<VEC>(qdst + c, x[s]);
      }
    } else {
      T* kdst = (T*)a.cache_k + (crow * G + head) * D;
#pragma unroll
      for (int s = 0; s < NCV; ++s) {
        const int c = (s * 32 + lane) * VEC;
        if (c < D) stv<VEC>(kdst + c, x[s]);
      }
    }
  }
}

// ---- gated delta rule with one decay per key channel ------------------------------------------------------------------------------
//   S <- diag(g_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t        (S [D, DV] float32 per head)
// q, k, v = silu(convolution of the projection), q and k unit vectors per head, g = exp(-exp(A_log) softplus(a + dt_bias)).
//
// Token form: one CTA of eight warps per (segment, head), for segments of at most max_len tokens. Everything of a token happens in
// this one launch: convolution, unit vectors, gates, the state's step, the output's norm and gate. The state passes through
// registers once per segment (warp = NRW neighbouring rows, lane = VEC neighbouring columns: whole rows are read and written);
// where a head has more value columns than one pass covers, it passes once per token and column chunk.
template <typename T, int NRW, int VEC>
__global__ void __launch_bounds__(256, NRW * VEC <= 64 ? 2 : 1)
delta_channel_token_kernel(const qspec_delta_channel_args a, int max_len) {
  pdl_enter();
  constexpr int DP = 8 * NRW, CW = 32 * VEC;
  extern __shared__ __align__(16) float sm_dt[];                  // v [DV] | o [DV]
  __shared__ __align__(16) float sq[DP], sk[DP], sg[DP];
  __shared__ __align__(16) float red[8][2][CW];
  __shared__ float rqk[8];
  const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i0 = a.seg_starts[blockIdx.x];
  const TokMeta mt = load_meta(a.meta, a.ntok, i0);
  const int len = mt.seg_end - mt.seg_begin;
  if (len > max_len) return;
  const int H = a.H, G = a.G, D = a.D, DV = a.DV, rep = H / G, kq = h / rep;
  const int GD = G * D, K1 = a.taps - 1, C = 2 * GD + H * DV;
  float* sv = sm_dt;
  float* so = sm_dt + DV;
  const int nch = (DV + CW - 1) / CW;
  float* st = a.state + ((size_t)mt.slot * H + h) * D * DV;
  const bool fresh = mt.pos == 0;
  VecF<VEC> S[NRW];
  auto load_state = [&](int ck, bool zero) {
    const int c = ck * CW + lane * VEC;
#pragma unroll
    for (int r = 0; r < NRW; ++r) {
      const int d = warp * NRW + r;
      if (!zero && d < D && c < DV) S[r] = ldv<VEC>(st + (size_t)d * DV + c);
      else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) S[r].v[e] = 0.f;
      }
    }
  };
  load_state(0, fresh);                                           // in flight while the first token is prepared
  ConvRows<T> cv;
  cv.in = (const T*)a.p + (size_t)mt.seg_begin * a.ld;
  cv.ld = a.ld; cv.first_pos = mt.pos; cv.K1 = K1; cv.C = C;
  cv.told = a.tail + ((size_t)mt.phase * a.slots + mt.slot) * K1 * C;
  float* tnew = a.tail + ((size_t)(1 - mt.phase) * a.slots + mt.slot) * K1 * C;
  const float rate = expf(a.A_log[h]);
  for (int tt = 0; tt < len; ++tt) {
    const int i = i0 + tt, pos = mt.pos + tt;
    auto conv = [&](int ch) {
      float acc = 0.f;
      for (int j = 0; j <= K1; ++j) acc += a.conv_w[(size_t)j * C + ch] * cv.get(pos - K1 + j, ch);
      if (tt == len - 1) cv.write_tail(tnew, pos, ch);            // every head of a group writes the same query / key tail
      return silu_act<T>(acc);
    };
    if (warp < 2) {                                               // unit query (warp 0) and key (warp 1)
      float* dst = warp ? sk : sq;
      float ss = 0.f;
      for (int c = lane; c < DP; c += 32) {
        const float v = c < D ? conv(warp * GD + kq * D + c) : 0.f;
        dst[c] = v;
        ss += v * v;
      }
      const float rr = (warp ? 1.0f : a.q_mult) / sqrtf(warp_xor_sum(ss) + a.unit_eps);
      for (int c = lane; c < DP; c += 32) dst[c] *= rr;
    } else if (warp < 5) {
      for (int c = (warp - 2) * 32 + lane; c < DV; c += 96) sv[c] = conv(2 * GD + h * DV + c);
    } else {
      for (int c = (warp - 5) * 32 + lane; c < DP; c += 96)
        sg[c] = c < D ? expf(-rate * softplus_f(a.decay[(size_t)i * a.decay_ld + (size_t)h * D + c] + a.dt_bias[h * D + c])) : 0.f;
    }
    const float beta = 1.0f / (1.0f + expf(-to_f(((const T*)a.p)[(size_t)i * a.ld + a.beta_off + h])));
    __syncthreads();
    for (int ck = 0; ck < nch; ++ck) {
      if (nch > 1 && (tt || ck)) load_state(ck, fresh && tt == 0);
      VecF<VEC> pa, pb;
      float qk = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) { pa.v[e] = 0.f; pb.v[e] = 0.f; }
#pragma unroll
      for (int r = 0; r < NRW; ++r) {
        const int d = warp * NRW + r;
        const float g = sg[d], k = sk[d], q = sq[d];
        qk += q * k;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[r].v[e] *= g;
          pa.v[e] += k * S[r].v[e];
          pb.v[e] += q * S[r].v[e];
        }
      }
      stv<VEC>(&red[warp][0][lane * VEC], pa);
      stv<VEC>(&red[warp][1][lane * VEC], pb);
      if (lane == 0) rqk[warp] = qk;
      __syncthreads();
      VecF<VEC> u, o;
      qk = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) { u.v[e] = 0.f; o.v[e] = 0.f; }
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const VecF<VEC> ra = ldv<VEC>(&red[w][0][lane * VEC]), rb = ldv<VEC>(&red[w][1][lane * VEC]);
        qk += rqk[w];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { u.v[e] += ra.v[e]; o.v[e] += rb.v[e]; }
      }
      const int c = ck * CW + lane * VEC;
      if (c < DV) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          u.v[e] = beta * (sv[c + e] - u.v[e]);
          o.v[e] += qk * u.v[e];
        }
        if (warp == 0) stv<VEC>(so + c, o);
#pragma unroll
        for (int r = 0; r < NRW; ++r) {
          const int d = warp * NRW + r;
          const float k = sk[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) S[r].v[e] += k * u.v[e];
          if (d < D && (nch > 1 || tt == len - 1)) stv<VEC>(st + (size_t)d * DV + c, S[r]);
        }
      }
      __syncthreads();                                            // the partial sums are used again; so is complete after the last chunk
    }
    float ss = 0.f;
    for (int c = lane; c < DV; c += 32) ss += so[c] * so[c];
    const float rr = a.out_scale / sqrtf(warp_xor_sum(ss) / (float)DV + a.eps);
    const T* gate = a.gate ? (const T*)a.gate + (size_t)i * a.gate_ld + (size_t)h * DV : nullptr;
    T* out = (T*)a.out + (size_t)i * a.out_ld + (size_t)h * DV;
    for (int c = tid; c < DV; c += 256) {
      float v = so[c] * rr * a.norm_w[c];
      if (gate) v *= 1.0f / (1.0f + expf(-to_f(gate[c])));
      out[c] = from_f<T>(v);
    }
    __syncthreads();                                              // the next token's vectors replace this one's
  }
}

// Block form for longer segments. With S0 the state before a block of 16 tokens and, per key channel, P_t = g_1 ... g_t the decay
// since then, the recurrence over the block is linear in S0 and in the corrections u_t:
//   u_t = beta_t (v_t - S0^T (P_t k_t) - sum_{s<t} A[t,s] u_s),   A[t,s] = sum_d k_t k_s P_t / P_s
//   o_t = S0^T (P_t q_t) + sum_{s<=t} B[t,s] u_s,                   B[t,s] = sum_d q_t k_s P_t / P_s
//   S   = diag(P_16) S0 + sum_s (P_16 / P_s k_s) u_s^T
// Everything that does not contain S0 is found for all blocks at once (delta_channel_block_kernel): with X the inverse of
// I + diag(beta) A (unit lower triangular), Tb = X diag(beta) and M = B Tb,
//   u = Tb v - (Tb Pk) S0 = Uv - Wk S0,     o = M v + (Pq - M Pk) S0 = Ov + Qk S0.
// The ratios P_t / P_s are running products of the decays between s and t: no division, no overflow however strong the decay.
// What remains in sequence order (delta_channel_scan_kernel) are products of 16-token blocks with a slice of the state.
// Block layout (float32), for every (block, head): [Wk, Qk: 16 rows of (token pair, channel, parity)] [K: 8 rows of the same, P_16 /
// P_s k_s] [P_16 per channel] with DP (a multiple of 64) channels per row, then per slice of 16 value columns [Uv, Ov][token][16].
constexpr int DBLK = 16;
__host__ __device__ constexpr size_t delta_block_floats(int DP, int nsl) { return (size_t)49 * DP + (size_t)nsl * 512; }

template <typename T, int KT>
__global__ void __launch_bounds__(256, 2)
delta_channel_block_kernel(const qspec_delta_channel_args a, const int* __restrict__ block_rows, float* __restrict__ blocks, int DP) {
  pdl_enter_hold();
  extern __shared__ __align__(16) float sm_db[];
  const int x = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i0 = block_rows[x];
  const TokMeta mt = load_meta(a.meta, a.ntok, i0);               // of the block's first token
  const int nb = min(DBLK, mt.seg_end - i0);
  const int H = a.H, G = a.G, D = a.D, DV = a.DV, rep = H / G, kq = h / rep, GD = G * D, K1 = a.taps - 1, C = 2 * GD + H * DV;
  const int nsl = (DV + 15) / 16, DS = DP + 4, VS = nsl * 16;
  float* sQ = sm_db;                                              // [16][DS] queries, then P q
  float* sK = sQ + DBLK * DS;                                     // keys, then P k
  float* sG = sK + DBLK * DS;                                     // decays
  float* sV = sG + DBLK * DS;                                     // [16][VS]
  float* sA = sV + DBLK * VS;                                     // [s][t] (column s contiguous): beta_t A[t, s], t > s
  float* sB = sA + 256;                                           // [t][s]: B[t, s], s <= t
  float* sX = sB + 256;                                           // [t][s]: Tb
  float* sM = sX + 256;                                           // [t][s]: M
  float* sbeta = sM + 256;                                        // [16]
  ConvRows<T> cv;
  cv.in = (const T*)a.p + (size_t)mt.seg_begin * a.ld;
  cv.ld = a.ld; cv.first_pos = mt.pos - (i0 - mt.seg_begin); cv.K1 = K1; cv.C = C;
  cv.told = a.tail + ((size_t)mt.phase * a.slots + mt.slot) * K1 * C;
  float* tnew = a.tail + ((size_t)(1 - mt.phase) * a.slots + mt.slot) * K1 * C;
  const bool last = i0 + nb == mt.seg_end;
  // ---- convolved queries, keys, values and decays: a thread per channel, the block's rows in flight together
  for (int e = tid; e < 2 * DP + VS; e += 256) {
    const int kind = e < DP ? 0 : (e < 2 * DP ? 1 : 2), c = kind == 0 ? e : (kind == 1 ? e - DP : e - 2 * DP);
    float* dst = (kind == 0 ? sQ : (kind == 1 ? sK : sV)) + c;
    const int ds = kind == 2 ? VS : DS;
    if (c >= (kind == 2 ? DV : D)) {
#pragma unroll
      for (int t = 0; t < DBLK; ++t) dst[t * ds] = 0.f;
      continue;
    }
    const int ch = kind == 2 ? 2 * GD + h * DV + c : kind * GD + kq * D + c;
    if (KT) {                                                     // at most KT taps: leading weights of a shorter filter are zero
      float w[KT ? KT : 1], in[DBLK + (KT ? KT : 1) - 1];
#pragma unroll
      for (int j = 0; j < KT; ++j) { const int jr = j - (KT - 1 - K1); w[j] = jr >= 0 ? a.conv_w[(size_t)jr * C + ch] : 0.f; }
      // the block's rows: every load is issued before the first is used (rows past the end repeat the last one and are dropped)
      const T* src = (const T*)a.p + (size_t)i0 * a.ld + ch;
#pragma unroll
      for (int t = 0; t < DBLK; ++t) in[t + KT - 1] = to_f(src[(size_t)min(t, nb - 1) * a.ld]);
      if (i0 == mt.seg_begin) {                                   // the rows before the step
#pragma unroll
        for (int t = 0; t < KT - 1; ++t) in[t] = t < KT - 1 - K1 ? 0.f : cv.get(mt.pos - (KT - 1 - t), ch);
      } else {
#pragma unroll
        for (int t = 0; t < KT - 1; ++t) in[t] = to_f(*(src - (size_t)(KT - 1 - t) * a.ld));
      }
#pragma unroll
      for (int t = 0; t < DBLK; ++t) {
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < KT; ++j) acc += w[j] * in[t + j];
        dst[t * ds] = t < nb ? silu_act<T>(acc) : 0.f;
      }
    } else {
      for (int t = 0; t < DBLK; ++t) {
        float acc = 0.f;
        if (t < nb)
          for (int j = 0; j <= K1; ++j) acc += a.conv_w[(size_t)j * C + ch] * cv.get(mt.pos + t - K1 + j, ch);
        dst[t * ds] = silu_act<T>(acc);
      }
    }
    if (last && (kind == 2 || h % rep == 0)) cv.write_tail(tnew, mt.pos + nb - 1, ch);
  }
  const float rate = expf(a.A_log[h]);
  for (int c = tid; c < DP; c += 256) {
    const bool ok = c < D;
    const float db = ok ? a.dt_bias[h * D + c] : 0.f;
    float z[DBLK];
#pragma unroll
    for (int t = 0; t < DBLK; ++t) z[t] = a.decay[(size_t)(i0 + min(t, nb - 1)) * a.decay_ld + (size_t)h * D + (ok ? c : 0)];
#pragma unroll
    for (int t = 0; t < DBLK; ++t) sG[t * DS + c] = ok && t < nb ? expf(-rate * softplus_f(z[t] + db)) : 1.f;
  }
  if (tid < DBLK) sbeta[tid] = tid < nb ? 1.0f / (1.0f + expf(-to_f(((const T*)a.p)[(size_t)(i0 + tid) * a.ld + a.beta_off + h]))) : 0.f;
  for (int e = tid; e < 512; e += 256) sA[e] = 0.f;               // sA and sB
  __syncthreads();
  // ---- unit vectors
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int rr = warp * 4 + r;
    float* row = (rr < DBLK ? sQ : sK) + (rr & 15) * DS;
    float ss = 0.f;
    for (int c = lane; c < DP; c += 32) ss += row[c] * row[c];
    const float f = (rr < DBLK ? a.q_mult : 1.0f) / sqrtf(warp_xor_sum(ss) + a.unit_eps);
    for (int c = lane; c < DP; c += 32) row[c] *= f;
  }
  __syncthreads();
  // ---- A and B: 16 lanes per s; the running product k_s g_(s+1) .. g_t meets k_t and q_t
  {
    const int s = tid >> 4, l = tid & 15;
    float4 w[4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
      w[m] = m * 64 < DP ? *reinterpret_cast<const float4*>(sK + s * DS + m * 64 + 4 * l) : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int t0 = (2 * warp) & ~3; t0 < nb; t0 += 4) {            // four tokens' sums at a time
      float p[8];                                                 // [token][key, query]
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int t = t0 + u;
        float dk = 0.f, dq = 0.f;
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          if (m * 64 >= DP) break;
          const int at = t * DS + m * 64 + 4 * l;
          const float4 k = *reinterpret_cast<const float4*>(sK + at), q = *reinterpret_cast<const float4*>(sQ + at);
          if (t > s) {
            const float4 g = *reinterpret_cast<const float4*>(sG + at);
            w[m].x *= g.x; w[m].y *= g.y; w[m].z *= g.z; w[m].w *= g.w;
          }
          dk += (w[m].x * k.x + w[m].y * k.y) + (w[m].z * k.z + w[m].w * k.w);
          dq += (w[m].x * q.x + w[m].y * q.y) + (w[m].z * q.z + w[m].w * q.w);
        }
        p[2 * u] = dk;
        p[2 * u + 1] = dq;
      }
      // eight sums over 16 lanes by halving exchanges: lane bits 3, 2, 1 select the sum a lane ends with, bit 0 adds the last two
#pragma unroll
      for (int n = 4; n >= 1; n >>= 1) {
        const bool hi = (l & (2 * n)) != 0;
#pragma unroll
        for (int j = 0; j < n; ++j) {
          const float send = hi ? p[j] : p[j + n], keep = hi ? p[j + n] : p[j];
          p[j] = keep + __shfl_xor_sync(0xffffffffu, send, 2 * n);
        }
      }
      p[0] += __shfl_xor_sync(0xffffffffu, p[0], 1);
      const int t = t0 + (l >> 2);                                // sum index l >> 1 = 2 u + (0 key, 1 query)
      if ((l & 1) == 0 && t >= s && t < nb) {
        if (l & 2) sB[t * 16 + s] = p[0];
        else if (t > s) sA[s * 16 + t] = sbeta[t] * p[0];
      }
    }
  }
  __syncthreads();
  float* blk = blocks + ((size_t)x * H + h) * delta_block_floats(DP, nsl);
  // ---- warp 0: the inverse, a column per lane; the other warps: decayed keys and queries
  if (warp == 0) {
    if (lane < DBLK) {
      float xc[DBLK];
#pragma unroll
      for (int t = 0; t < DBLK; ++t) xc[t] = t == lane ? 1.f : 0.f;
#pragma unroll
      for (int r = 0; r < DBLK - 1; ++r) {
        float col[DBLK];
#pragma unroll
        for (int v = 0; v < 4; ++v) {
          const float4 f = *reinterpret_cast<const float4*>(sA + r * 16 + 4 * v);
          col[4 * v] = f.x; col[4 * v + 1] = f.y; col[4 * v + 2] = f.z; col[4 * v + 3] = f.w;
        }
#pragma unroll
        for (int t = r + 1; t < DBLK; ++t) xc[t] -= col[t] * xc[r];
      }
      const float be = sbeta[lane];
#pragma unroll
      for (int t = 0; t < DBLK; ++t) sX[t * 16 + lane] = xc[t] * be;
    }
  } else {
    for (int c = tid - 32; c < DP; c += 224) {
      float k[DBLK], g[DBLK];
#pragma unroll
      for (int t = 0; t < DBLK; ++t) { k[t] = sK[t * DS + c]; g[t] = sG[t * DS + c]; }
      float p = 1.f;
#pragma unroll
      for (int t = 0; t < DBLK; ++t) {                            // decay since the block's start
        p *= g[t];
        sK[t * DS + c] = p * k[t];
        sQ[t * DS + c] *= p;
      }
      blk[(size_t)48 * DP + c] = p;
      p = 1.f;
#pragma unroll
      for (int t = DBLK - 1; t >= 0; --t) {                       // decay until the block's end
        k[t] *= p;
        p *= g[t];
      }
#pragma unroll
      for (int tp = 0; tp < 8; ++tp)
        *reinterpret_cast<float2*>(blk + (size_t)32 * DP + ((size_t)tp * DP + c) * 2) = make_float2(k[2 * tp], k[2 * tp + 1]);
    }
  }
  __syncthreads();
  {
    const int t = tid >> 4, s = tid & 15;
    float m = 0.f;
    for (int r = s; r <= t; ++r) m += sB[t * 16 + r] * sX[r * 16 + s];
    sM[t * 16 + s] = m;
  }
  __syncthreads();
  // ---- products with the keys (a thread per key channel) and the values (a thread per value column)
  for (int e = tid; e < DP + VS; e += 256) {
    const bool keys = e < DP;
    const int c = keys ? e : e - DP;
    const float* src = keys ? sK + c : sV + c;
    const int ss = keys ? DS : VS;
    float v[DBLK];
#pragma unroll
    for (int t = 0; t < DBLK; ++t) v[t] = src[t * ss];
#pragma unroll
    for (int tp = 0; tp < 8; ++tp) {
      float rx[2], rm[2];
#pragma unroll
      for (int par = 0; par < 2; ++par) {
        const int t = 2 * tp + par;
        float ax = 0.f, am = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (4 * q > t) break;
          const float4 fx = *reinterpret_cast<const float4*>(sX + t * 16 + 4 * q), fm = *reinterpret_cast<const float4*>(sM + t * 16 + 4 * q);
          ax += (fx.x * v[4 * q] + fx.y * v[4 * q + 1]) + (fx.z * v[4 * q + 2] + fx.w * v[4 * q + 3]);      // zero above the diagonal
          am += (fm.x * v[4 * q] + fm.y * v[4 * q + 1]) + (fm.z * v[4 * q + 2] + fm.w * v[4 * q + 3]);
        }
        rx[par] = ax;
        rm[par] = am;
      }
      if (keys) {
        *reinterpret_cast<float2*>(blk + ((size_t)tp * DP + c) * 2) = make_float2(rx[0], rx[1]);
        *reinterpret_cast<float2*>(blk + ((size_t)(8 + tp) * DP + c) * 2) =
            make_float2(sQ[2 * tp * DS + c] - rm[0], sQ[(2 * tp + 1) * DS + c] - rm[1]);
      } else {
        float* uo = blk + (size_t)49 * DP + (size_t)(c >> 4) * 512 + (c & 15);
        uo[2 * tp * 16] = rx[0]; uo[(2 * tp + 1) * 16] = rx[1];
        uo[256 + 2 * tp * 16] = rm[0]; uo[256 + (2 * tp + 1) * 16] = rm[1];
      }
    }
  }
}

__device__ __forceinline__ unsigned long long f2_dup(float v) { return pack_f2(v, v); }

// The part in sequence order. One CTA of eight warps per (segment, head, 16 value columns); two warps share four columns, one for the
// corrections (Wk) and one for the read-outs (Qk), each with its own copy of the columns; lanes own key channels hx * 64 + 2 lane +
// {0, 1}. Products run as packed pairs of float32 (two tokens of the block at a time, the state kept
// as duplicated pairs). The sums over the channels of 8 token pairs x 4 columns x 2 tokens are taken by halving exchanges: accumulator slot j of
// lane L belongs to token pair j ^ (L >> 2), so that the exchanges over token pairs send the slots the lane does not keep and need no
// selection. The blocks' operands arrive one block ahead by cp.async.
template <int NHR>
__global__ void __launch_bounds__(256)
delta_channel_scan_kernel(const qspec_delta_channel_args a, const int* __restrict__ long_starts, const int* __restrict__ long_block0,
                          const float* __restrict__ blocks, float* __restrict__ o) {
  pdl_enter();
  constexpr int DP = 64 * NHR, ROW = DP * 2;                      // floats of one (token pair) row
  constexpr int NF = 49 * DP + 512;                               // floats of a staged block: shared operands, this slice's Uv and Ov
  extern __shared__ __align__(16) float sm_ds[];                  // [2][NF]
  __shared__ __align__(16) float su[4][8][4][2];                  // per warp: u as [token pair][column][parity]
  const int i0 = long_starts[blockIdx.x], x0 = long_block0[blockIdx.x], h = blockIdx.y, sl = blockIdx.z;
  const TokMeta mt = load_meta(a.meta, a.ntok, i0);
  const int H = a.H, D = a.D, DV = a.DV, nsl = gridDim.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, kind = tid >> 7, xl = lane >> 2;
  const int len = mt.seg_end - mt.seg_begin, nblk = (len + DBLK - 1) / DBLK, c0 = sl * 16 + warp * 4;
  const size_t bf = delta_block_floats(DP, nsl);
  auto stage = [&](int buf, int b) {
    const float* src = blocks + ((size_t)(x0 + b) * H + h) * bf;
    float* dst = sm_ds + buf * NF;
    for (int e = tid; e < 49 * DP / 4; e += 256) cp_async_16z(dst + 4 * e, src + 4 * e, true);
    if (tid < 128) cp_async_16z(dst + 49 * DP + 4 * tid, src + 49 * DP + (size_t)sl * 512 + 4 * tid, true);       // 512 floats = 128 x 16 bytes
    cp_async_commit();
  };
  stage(0, 0);
  float* st = a.state + ((size_t)mt.slot * H + h) * D * DV;
  unsigned long long S[NHR][2][4];
#pragma unroll
  for (int hx = 0; hx < NHR; ++hx)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = hx * 64 + 2 * lane + e;
#pragma unroll
      for (int c = 0; c < 4; ++c) S[hx][e][c] = f2_dup(mt.pos > 0 && d < D && c0 + c < DV ? st[(size_t)d * DV + c0 + c] : 0.f);
    }
  for (int b = 0; b < nblk; ++b) {
    const int buf = b & 1;
    cp_async_wait<0>();
    __syncthreads();                                              // block b has arrived, and nobody reads block b - 1 any more
    if (b + 1 < nblk) stage(buf ^ 1, b + 1);
    const float* B = sm_ds + buf * NF;
    unsigned long long acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[j][c] = 0ull;
    const uint32_t perm = (uint32_t)(xl * ROW * 4 + lane * 16);   // a row is a power of two of bytes: row j ^ xl = (j rows) ^ (xl rows)
    const char* Bc = reinterpret_cast<const char*>(B + kind * 8 * ROW);
#pragma unroll
    for (int hx = 0; hx < NHR; ++hx)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(Bc + (((uint32_t)(j * ROW * 4) ^ perm) + hx * 512));
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[j][c] = ffma2_rn(w.x, S[hx][0][c], acc[j][c]);
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[j][c] = ffma2_rn(w.y, S[hx][1][c], acc[j][c]);
      }
    float v[8][4][2];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) { const float2 f = unpack_f2(acc[j][c]); v[j][c][0] = f.x; v[j][c][1] = f.y; }
#pragma unroll
    for (int n = 4; n >= 1; n >>= 1)                              // lane bit of the exchange: n << 2
#pragma unroll
      for (int j = 0; j < n; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          v[j][c][0] += __shfl_xor_sync(0xffffffffu, v[j + n][c][0], n << 2);
          v[j][c][1] += __shfl_xor_sync(0xffffffffu, v[j + n][c][1], n << 2);
        }
    // two more exchanges: over the column pairs (lane bit 1), then over the columns of a pair (lane bit 0)
    const int hp = (lane >> 1) & 1, hc = lane & 1;
    float r[2], m[2][2];
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
      for (int par = 0; par < 2; ++par) {
        const float send = hp ? v[0][c][par] : v[0][2 + c][par], keep = hp ? v[0][2 + c][par] : v[0][c][par];
        m[c][par] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
      }
#pragma unroll
    for (int par = 0; par < 2; ++par) {
      const float send = hc ? m[0][par] : m[1][par], keep = hc ? m[1][par] : m[0][par];
      r[par] = keep + __shfl_xor_sync(0xffffffffu, send, 1);
    }
    // this lane holds the two tokens of pair xl for column 2 hp + hc of its warp
    {
      const int cl = warp * 4 + (lane & 3);
      const float* uo = B + 49 * DP + kind * 256 + cl;
#pragma unroll
      for (int par = 0; par < 2; ++par) {
        const int t = 2 * xl + par;
        if (kind == 0) su[warp][xl][lane & 3][par] = uo[t * 16] - r[par];
        else if (b * DBLK + t < len && sl * 16 + cl < DV) o[((size_t)(i0 + b * DBLK + t) * H + h) * DV + sl * 16 + cl] = uo[t * 16] + r[par];
      }
    }
    __syncthreads();                                              // the corrections are complete
    unsigned long long add[NHR][2][4];
#pragma unroll
    for (int hx = 0; hx < NHR; ++hx)
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int c = 0; c < 4; ++c) add[hx][e][c] = 0ull;
#pragma unroll
    for (int tp = 0; tp < 8; ++tp) {
      const ulonglong2 u01 = *reinterpret_cast<const ulonglong2*>(&su[warp][tp][0][0]), u23 = *reinterpret_cast<const ulonglong2*>(&su[warp][tp][2][0]);
#pragma unroll
      for (int hx = 0; hx < NHR; ++hx) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(B + 32 * DP + tp * ROW + hx * 128 + 4 * lane);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const unsigned long long ke = e ? k.y : k.x;
          add[hx][e][0] = ffma2_rn(ke, u01.x, add[hx][e][0]);
          add[hx][e][1] = ffma2_rn(ke, u01.y, add[hx][e][1]);
          add[hx][e][2] = ffma2_rn(ke, u23.x, add[hx][e][2]);
          add[hx][e][3] = ffma2_rn(ke, u23.y, add[hx][e][3]);
        }
      }
    }
#pragma unroll
    for (int hx = 0; hx < NHR; ++hx) {
      const float2 g = *reinterpret_cast<const float2*>(B + 48 * DP + hx * 64 + 2 * lane);
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float2 ad = unpack_f2(add[hx][e][c]);
          S[hx][e][c] = f2_dup((e ? g.y : g.x) * unpack_f2(S[hx][e][c]).x + (ad.x + ad.y));
        }
    }
  }
  if (kind) return;                                               // both copies are the same
#pragma unroll
  for (int hx = 0; hx < NHR; ++hx)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = hx * 64 + 2 * lane + e;
#pragma unroll
      for (int c = 0; c < 4; ++c)
        if (d < D && c0 + c < DV) st[(size_t)d * DV + c0 + c] = unpack_f2(S[hx][e][c]).x;
    }
}

// Per-head norm and gate of the block form's read-outs, for the tokens of segments longer than max_len: a warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
delta_channel_out_kernel(const qspec_delta_channel_args a, const float* __restrict__ o, int max_len) {
  pdl_enter();
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= (long long)a.ntok * a.H) return;
  const int lane = threadIdx.x & 31, DV = a.DV;
  const int t = (int)(r / a.H), h = (int)(r - (long long)t * a.H);
  if (a.meta[3 * a.ntok + t] - a.meta[2 * a.ntok + t] <= max_len) return;
  const float* s = o + r * DV;
  float ss = 0.f;
  for (int c = lane; c < DV; c += 32) ss += s[c] * s[c];
  const float rr = a.out_scale / sqrtf(warp_xor_sum(ss) / (float)DV + a.eps);
  const T* gate = a.gate ? (const T*)a.gate + (size_t)t * a.gate_ld + (size_t)h * DV : nullptr;
  T* out = (T*)a.out + (size_t)t * a.out_ld + (size_t)h * DV;
  for (int c = lane; c < DV; c += 32) {
    float v = s[c] * rr * a.norm_w[c];
    if (gate) v *= 1.0f / (1.0f + expf(-to_f(gate[c])));
    out[c] = from_f<T>(v);
  }
}

}  // namespace qspec

using namespace qspec;
#define HD_DTYPE_OK(dtype) QSPEC_REQUIRE((dtype) == QSPEC_DTYPE_BF16 || (dtype) == QSPEC_DTYPE_F32, QSPEC_ERR_UNSUPPORTED, \
                                         "dtype %d: bfloat16 (1) or float32 (2) expected", (dtype))

template <typename T, typename YT>
static int launch_residual_tanh(const float* x_in, float* x_out, const void* y, int y_parts, long long y_part_stride, long long y_tok_stride,
                                const float* y_w, const float* y_bias, float mult, float alpha, const float* w, const float* b, void* out,
                                int ntok, int W, cudaStream_t st) {
  const bool vec = W % 4 == 0 && y_part_stride % 4 == 0 && y_tok_stride % 4 == 0 &&
                   (((uintptr_t)x_in | (uintptr_t)x_out | (uintptr_t)w | (uintptr_t)b | (uintptr_t)y_bias) & 15) == 0 &&
                   ((uintptr_t)y & (4 * sizeof(YT) - 1)) == 0 && ((uintptr_t)out & (4 * sizeof(T) - 1)) == 0;
#define RT_ARGS x_in, x_out, (const YT*)y, y_parts, y_part_stride, y_tok_stride, y_w, y_bias, mult, alpha, w, b, (T*)out, W
  if (vec) launch_pdl(residual_tanh_kernel<T, YT, 4>, dim3(ntok, (W + 1023) / 1024), dim3(256), 0, st, RT_ARGS);
  else launch_pdl(residual_tanh_kernel<T, YT, 1>, dim3(ntok, (W + 255) / 256), dim3(256), 0, st, RT_ARGS);
#undef RT_ARGS
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

extern "C" int qspec_seq_residual_tanh(const float* x_in, float* x_out, const void* y, int y_parts, long long y_part_stride,
                                       long long y_tok_stride, const float* y_w, const float* y_bias, float mult, float alpha,
                                       const float* w, const float* b, void* out, int ntok, int W, int y_dtype, int dtype, void* stream) {
  QSPEC_REQUIRE(x_in && (x_out || out) && (!out || (w && b)), QSPEC_ERR_INVALID_ARG, "seq_residual_tanh: null pointer");
  QSPEC_REQUIRE(ntok >= 0 && W > 0 && W <= 65535 * 256 && y_parts >= 1, QSPEC_ERR_INVALID_ARG, "seq_residual_tanh: bad sizes");
  HD_DTYPE_OK(dtype);
  QSPEC_REQUIRE(y_dtype == dtype || y_dtype == QSPEC_DTYPE_F32, QSPEC_ERR_UNSUPPORTED, "seq_residual_tanh: y is of the activation type or float32");
  if (ntok == 0) return QSPEC_OK;
  cudaStream_t st = (cudaStream_t)stream;
#define RT_CALL x_in, x_out, y, y_parts, y_part_stride, y_tok_stride, y_w, y_bias, mult, alpha, w, b, out, ntok, W, st
  if (dtype == QSPEC_DTYPE_F32) return launch_residual_tanh<float, float>(RT_CALL);
  if (y_dtype == QSPEC_DTYPE_F32) return launch_residual_tanh<bf16_t, float>(RT_CALL);
  return launch_residual_tanh<bf16_t, bf16_t>(RT_CALL);
#undef RT_CALL
}

extern "C" int qspec_seq_softcap_f32(float* a, long long n, float cap, void* stream) {
  QSPEC_REQUIRE(a && n >= 0 && cap > 0.f, QSPEC_ERR_INVALID_ARG, "seq_softcap: bad arguments");
  if (n == 0) return QSPEC_OK;
  const bool vec = n % 4 == 0 && ((uintptr_t)a & 15) == 0;
  const long long per = vec ? 1024 : 256, want = (n + per - 1) / per;
  const unsigned blocks = (unsigned)(want > 148 * 16 ? 148 * 16 : want);
  if (vec) launch_pdl(softcap_kernel<4>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, a, n, cap);
  else launch_pdl(softcap_kernel<1>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, a, n, cap);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <typename T, int VEC, int NCV>
static int launch_head_prep(const qspec_head_prep_args& a, cudaStream_t st) {
  const size_t smem = a.rot_dims ? (size_t)8 * (a.D + a.rot_dims) * sizeof(float) : 0;
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    QSPEC_CUDA(cudaFuncSetAttribute(head_prep_kernel<T, VEC, NCV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  // heads of a token go round grid y: enough CTAs to fill the GPU, few enough that a token's angles serve several heads
  const int nh = a.H + a.G + (a.v_off >= 0 ? a.G : 0), rows = (a.ntok + 7) / 8;
  int gy = (148 * 16 + rows - 1) / rows;
  if (gy > nh) gy = nh;
  if (gy > 65535) gy = 65535;
  launch_pdl(head_prep_kernel<T, VEC, NCV>, dim3(rows, gy), dim3(256), smem, st, a);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <typename T>
static int launch_head_prep_n(const qspec_head_prep_args& a, cudaStream_t st) {
  const size_t es = sizeof(T);
  const int dm = a.D > a.DV ? a.D : a.DV;
  const uintptr_t f32s = (uintptr_t)a.conv_w | (uintptr_t)a.tail | (uintptr_t)a.qout;
  const bool vec = a.D % 4 == 0 && a.DV % 4 == 0 && a.ld % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 && (a.v_off < 0 || a.v_off % 4 == 0) &&
                   (f32s & 15) == 0 && (((uintptr_t)a.p | (uintptr_t)a.cache_k | (uintptr_t)a.cache_v) & (4 * es - 1)) == 0;
  if (vec) {
    if (dm <= 128) return launch_head_prep<T, 4, 1>(a, st);
    if (dm <= 256) return launch_head_prep<T, 4, 2>(a, st);
    return launch_head_prep<T, 4, 8>(a, st);
  }
  if (dm <= 64) return launch_head_prep<T, 1, 2>(a, st);
  if (dm <= 256) return launch_head_prep<T, 1, 8>(a, st);
  return launch_head_prep<T, 1, 32>(a, st);
}

extern "C" int qspec_seq_head_prep(const qspec_head_prep_args* a, int dtype, void* stream) {
  QSPEC_REQUIRE(a && a->p && a->qout && a->cache_k && a->cache_v && a->meta && (a->rot_dims == 0 || a->inv_freq), QSPEC_ERR_INVALID_ARG,
                "seq_head_prep: null pointer");
  QSPEC_REQUIRE(a->ntok >= 0 && a->H > 0 && a->G > 0 && a->H % a->G == 0 && a->D > 0 && a->D <= 1024 && a->DV > 0 && a->DV <= 1024 &&
                    a->cap > 0 && a->keep_first >= 0 && a->keep_first < a->cap && a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->D,
                QSPEC_ERR_UNSUPPORTED, "seq_head_prep: heads %d / %d, key size %d, value size %d (<= 1024), %d rotated entries", a->H, a->G, a->D,
                a->DV, a->rot_dims);
  QSPEC_REQUIRE(a->q_off >= 0 && a->k_off >= 0 && a->q_off + a->H * a->D <= a->ld && a->k_off + a->G * a->D <= a->ld &&
                    (a->v_off < 0 ? a->DV == a->D && !a->conv_w : a->v_off + a->G * a->DV <= a->ld),
                QSPEC_ERR_INVALID_ARG, "seq_head_prep: sections outside the row (values taken from the keys need equal sizes and no convolution)");
  QSPEC_REQUIRE(!a->conv_w || (a->taps >= 1 && a->taps <= 64 && (a->tail || a->taps == 1) && a->slots > 0), QSPEC_ERR_INVALID_ARG,
                "seq_head_prep: a convolution of %d taps", a->taps);
  QSPEC_REQUIRE(a->norm_last >= QSPEC_HEAD_NORM_FIRST && a->norm_last <= QSPEC_HEAD_NORM_NONE &&
                    (a->pairing == QSPEC_ROTARY_HALVES || a->pairing == QSPEC_ROTARY_INTERLEAVED), QSPEC_ERR_INVALID_ARG,
                "seq_head_prep: norm %d, pairing %d", a->norm_last, a->pairing);
  HD_DTYPE_OK(dtype);
  if (a->ntok == 0) return QSPEC_OK;
  if (dtype == QSPEC_DTYPE_F32) return launch_head_prep_n<float>(*a, (cudaStream_t)stream);
  return launch_head_prep_n<bf16_t>(*a, (cudaStream_t)stream);
}

template <typename T, int NRW, int VEC>
static int launch_delta_token(const qspec_delta_channel_args& a, int max_len, cudaStream_t st) {
  launch_pdl(delta_channel_token_kernel<T, NRW, VEC>, dim3(a.nseg, a.H), dim3(256), (size_t)2 * a.DV * sizeof(float), st, a, max_len);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <typename T>
static int launch_delta_token_n(const qspec_delta_channel_args& a, int max_len, cudaStream_t st) {
  const bool vec = a.DV % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
  if (vec) {
    if (a.D <= 32) return launch_delta_token<T, 4, 4>(a, max_len, st);
    if (a.D <= 64) return launch_delta_token<T, 8, 4>(a, max_len, st);
    if (a.D <= 128) return launch_delta_token<T, 16, 4>(a, max_len, st);
    return launch_delta_token<T, 32, 4>(a, max_len, st);
  }
  if (a.D <= 32) return launch_delta_token<T, 4, 1>(a, max_len, st);
  if (a.D <= 64) return launch_delta_token<T, 8, 1>(a, max_len, st);
  if (a.D <= 128) return launch_delta_token<T, 16, 1>(a, max_len, st);
  return launch_delta_token<T, 32, 1>(a, max_len, st);
}

static int delta_padded(int D) { return D <= 64 ? 64 : D <= 128 ? 128 : 256; }

template <typename T, int KT>
static int launch_delta_block(const qspec_delta_channel_args& a, const int* block_rows, int nblocks, float* blocks, cudaStream_t st) {
  const int DP = delta_padded(a.D), VS = (a.DV + 15) / 16 * 16;
  const size_t smem = ((size_t)3 * DBLK * (DP + 4) + (size_t)DBLK * VS + 4 * 256 + 16) * sizeof(float);
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    QSPEC_CUDA(cudaFuncSetAttribute(delta_channel_block_kernel<T, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  launch_pdl(delta_channel_block_kernel<T, KT>, dim3(nblocks, a.H), dim3(256), smem, st, a, block_rows, blocks, DP);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

template <int NHR>
static int launch_delta_scan_blocks(const qspec_delta_channel_args& a, const int* long_starts, const int* long_block0, int nlong,
                                    const float* blocks, float* o, cudaStream_t st) {
  constexpr size_t smem = (size_t)2 * (49 * 64 * NHR + 512) * sizeof(float);
  static bool configured = false;
  if (!configured) {
    QSPEC_CUDA(cudaFuncSetAttribute(delta_channel_scan_kernel<NHR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = true;
  }
  launch_pdl(delta_channel_scan_kernel<NHR>, dim3(nlong, a.H, (a.DV + 15) / 16), dim3(256), smem, st, a, long_starts, long_block0, blocks, o);
  QSPEC_CHECK_LAUNCH(1);
  return QSPEC_OK;
}

extern "C" size_t qspec_seq_delta_channel_scratch_bytes(int nblocks, int ntok, int H, int D, int DV) {
  if (nblocks <= 0 || D > 256) return 0;
  return (delta_block_floats(delta_padded(D), (DV + 15) / 16) * (size_t)nblocks * H + (size_t)ntok * H * DV) * sizeof(float);
}

extern "C" int qspec_seq_delta_channel(const qspec_delta_channel_args* args, const int* block_rows, int nblocks, const int* long_starts,
                                       const int* long_block0, int nlong, int max_len, void* scratch, size_t scratch_bytes, int dtype,
                                       void* stream) {
  QSPEC_REQUIRE(args, QSPEC_ERR_INVALID_ARG, "seq_delta_channel: null pointer");
  const qspec_delta_channel_args& a = *args;
  QSPEC_REQUIRE(a.p && a.conv_w && a.decay && a.A_log && a.dt_bias && a.norm_w && a.state && a.out && a.meta && a.seg_starts &&
                    (a.tail || a.taps == 1), QSPEC_ERR_INVALID_ARG, "seq_delta_channel: null pointer");
  QSPEC_REQUIRE(a.ntok >= 0 && a.nseg >= 0 && a.H > 0 && a.H <= 65535 && a.G > 0 && a.H % a.G == 0 && a.D > 0 && a.D <= 256 && a.DV > 0 &&
                    a.DV <= 4096 && a.taps >= 1 && a.taps <= 64 && a.slots > 0 && a.ld >= 2 * a.G * a.D + a.H * a.DV && a.beta_off >= 0 && max_len >= 1,
                QSPEC_ERR_UNSUPPORTED, "seq_delta_channel: heads %d / %d, key size %d (<= 256), value size %d (<= 4096), %d taps", a.H, a.G, a.D,
                a.DV, a.taps);
  HD_DTYPE_OK(dtype);
  if (a.ntok == 0 || a.nseg == 0) return QSPEC_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (nlong > 0) {
    QSPEC_REQUIRE(block_rows && long_starts && long_block0 && scratch && nblocks > 0 && ((uintptr_t)scratch & 15) == 0 &&
                      scratch_bytes >= qspec_seq_delta_channel_scratch_bytes(nblocks, a.ntok, a.H, a.D, a.DV),
                  QSPEC_ERR_INVALID_ARG, "seq_delta_channel: block table or scratch missing for %d long segments", nlong);
    QSPEC_REQUIRE((a.DV + 15) / 16 * 16 * DBLK * 4 + 3 * DBLK * (delta_padded(a.D) + 4) * 4 + 4200 <= 220 * 1024, QSPEC_ERR_UNSUPPORTED,
                  "seq_delta_channel: key size %d with value size %d exceed shared memory", a.D, a.DV);
    const int DP = delta_padded(a.D);
    float* blocks = (float*)scratch;
    float* o = blocks + delta_block_floats(DP, (a.DV + 15) / 16) * (size_t)nblocks * a.H;
    int s;
    if (dtype == QSPEC_DTYPE_F32)
      s = a.taps <= 4 ? launch_delta_block<float, 4>(a, block_rows, nblocks, blocks, st) : launch_delta_block<float, 0>(a, block_rows, nblocks, blocks, st);
    else
      s = a.taps <= 4 ? launch_delta_block<bf16_t, 4>(a, block_rows, nblocks, blocks, st) : launch_delta_block<bf16_t, 0>(a, block_rows, nblocks, blocks, st);
    if (s) return s;
    s = DP == 64 ? launch_delta_scan_blocks<1>(a, long_starts, long_block0, nlong, blocks, o, st)
                 : DP == 128 ? launch_delta_scan_blocks<2>(a, long_starts, long_block0, nlong, blocks, o, st)
                             : launch_delta_scan_blocks<4>(a, long_starts, long_block0, nlong, blocks, o, st);
    if (s) return s;
    const long long rows = (long long)a.ntok * a.H;
    const dim3 grid((unsigned)((rows + 7) / 8));
    if (dtype == QSPEC_DTYPE_F32) launch_pdl(delta_channel_out_kernel<float>, grid, dim3(256), 0, st, a, (const float*)o, max_len);
    else launch_pdl(delta_channel_out_kernel<bf16_t>, grid, dim3(256), 0, st, a, (const float*)o, max_len);
    QSPEC_CHECK_LAUNCH(1);
  }
  if (nlong < a.nseg) {
    if (dtype == QSPEC_DTYPE_F32) return launch_delta_token_n<float>(a, max_len, st);
    return launch_delta_token_n<bf16_t>(a, max_len, st);
  }
  return QSPEC_OK;
}
