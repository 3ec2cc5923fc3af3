// Linear recurrences over a matrix state per head with value channels outermost, [Dv, D] (the key channels of a value channel are contiguous):
//   * the gated delta rule with one decay per head and key channel, and the kernel that makes its rows (convolution, SiLU, unit norms,
//     decays, write strengths);
//   * linear attention with a fixed decay per head;
//   * matrix memory with exponential input gates, a running maximum and a key sum as denominator;
// and routing by token id.  States, decays, unit norms and everything else inside a recurrence are fp32; compiled WITHOUT fast-math.
#include <cuda_bf16.h>
#include <math.h>

#include <stdexcept>
#include <type_traits>

#include "common.cuh"
#include "seqmix.h"

namespace nxdi {
namespace {

template <typename T> __device__ __forceinline__ float ldf1(const T* p);
template <> __device__ __forceinline__ float ldf1<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf1<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf1(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf1(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float sigmoid_acc(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float silu_acc(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_acc(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// VEC consecutive values as one access
template <int VEC> __device__ __forceinline__ void ldvec(const float* p, float* x) {
  if constexpr (VEC == 4) { const float4 v = *reinterpret_cast<const float4*>(p); x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w; }
  else x[0] = *p;
}
template <int VEC> __device__ __forceinline__ void ldvec(const __nv_bfloat16* p, float* x) {
  if constexpr (VEC == 4) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    x[0] = bf16lo(r.x); x[1] = bf16hi(r.x); x[2] = bf16lo(r.y); x[3] = bf16hi(r.y);
  } else x[0] = __bfloat162float(*p);
}
template <int VEC> __device__ __forceinline__ void stvec(float* p, const float* x) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  else *p = x[0];
}
template <int VEC> __device__ __forceinline__ void stvec(__nv_bfloat16* p, const float* x) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]));
  else *p = __float2bfloat16_rn(x[0]);
}

// ---- rows of the per-channel delta rule -------------------------------------------------------------------------------------------------
// A warp takes one segment of channels over a tile of tokens: a q or k head (unit norm), a run of v channels, a run of decays, or all write
// strengths.  The convolution's window stays in registers while the warp marches over its tokens; only the first tile of a row reads the
// carried rows, and it writes them back at the end (from the projection rows themselves), so no other warp touches them.
constexpr int FRONT_WARPS = 8;
template <typename T, int VEC, int NI, int KM>
__global__ void __launch_bounds__(FRONT_WARPS * 32) delta_front_kernel(DeltaFrontParams p, int TT, int vsegs, int gsegs) {
  constexpr int SEG = 32 * VEC * NI, N = VEC * NI;
  const int b = blockIdx.z, t0 = blockIdx.x * TT, lane = threadIdx.x & 31;
  const int seg = blockIdx.y * FRONT_WARPS + (threadIdx.x >> 5);
  const int qn = p.q_len[b], live = min(t0 + TT, qn);
  if (t0 >= qn) return;
  const int K = p.K, D = p.D, Cq = p.n_qk * D, Cv = p.nh * p.Dv, C = 2 * Cq + Cv, Cg = p.nh * D;
  const long long row0 = (long long)b * p.T;
  if (seg < 2 * p.n_qk + vsegs) {
    const bool unit = seg < 2 * p.n_qk, isq = seg < p.n_qk;
    const int first = unit ? seg * D : 2 * Cq + (seg - 2 * p.n_qk) * SEG;              // channel of the row
    const int width = unit ? D : min(SEG, C - first);
    const T* src = (const T*)p.p + (long long)b * p.p_sb + first;
    float ring[KM - 1 > 0 ? KM - 1 : 1][N], cw[KM][N], x[N];
    bool in[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * 32 + lane) * VEC;
      in[i] = c < width;
#pragma unroll
      for (int e = 0; e < VEC; ++e)
#pragma unroll
        for (int d = 0; d < KM; ++d) cw[d][i * VEC + e] = (in[i] && d < K) ? p.conv_w[(long long)(first + c + e) * K + (K - 1 - d)] : 0.f;
    }
    T* state = K > 1 ? (T*)p.state + (long long)p.lines[b] * (K - 1) * C + first : nullptr;
    const bool carried = K > 1 && p.ctx_len[b] > 0;
    auto load = [&](const T* row, float* dst, bool on) {
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        if (in[i] && on) ldvec<VEC>(row + (i * 32 + lane) * VEC, dst + i * VEC);
        else
#pragma unroll
          for (int e = 0; e < VEC; ++e) dst[i * VEC + e] = 0.f;
      }
    };
    // ring[d]: the input of d + 1 tokens ago
#pragma unroll
    for (int d = 0; d < KM - 1; ++d) {
      const int t = t0 - 1 - d;
      if (d >= K - 1) load(src, ring[d], false);
      else if (t >= 0) load(src + (long long)t * p.p_st, ring[d], true);
      else load(K > 1 ? state + (long long)(K - 1 + t) * C : src, ring[d], carried);
    }
    const float qmul = isq ? 1.f / sqrtf((float)D) : 1.f;
    load(src + (long long)t0 * p.p_st, x, true);
    for (int t = t0; t < live; ++t) {
      float y[N], ss = 0.f, cur[N];
#pragma unroll
      for (int i = 0; i < N; ++i) {
        cur[i] = x[i];
        float a = cw[0][i] * x[i];
#pragma unroll
        for (int d = 1; d < KM; ++d) a += cw[d][i] * ring[d - 1][i];
        y[i] = silu_acc(a);
        ss += y[i] * y[i];
      }
      if (t + 1 < live) load(src + (long long)(t + 1) * p.p_st, x, true);
#pragma unroll
      for (int i = 0; i < N; ++i) {
#pragma unroll
        for (int d = KM - 2; d > 0; --d) ring[d][i] = ring[d - 1][i];
        if (KM > 1) ring[0][i] = cur[i];
      }
      if (unit) {
        const float r = qmul / sqrtf(warp_sum(ss) + p.unit_eps);
#pragma unroll
        for (int i = 0; i < N; ++i) y[i] *= r;
      }
      float* out = p.qkv + (row0 + t) * C + first;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (in[i]) stvec<VEC>(out + (i * 32 + lane) * VEC, y + i * VEC);
    }
    if (t0 == 0 && K > 1) {
      // the last K - 1 inputs of (carried rows, this portion); oldest first, so a carried row is read before its place is overwritten
      for (int j = 0; j < K - 1; ++j) {
        const int t = qn - (K - 1) + j;
        float v[N];
        if (t >= 0) load(src + (long long)t * p.p_st, v, true);
        else load(state + (long long)(K - 1 + t) * C, v, carried);
#pragma unroll
        for (int i = 0; i < NI; ++i)
          if (in[i]) stvec<VEC>(state + (long long)j * C + (i * 32 + lane) * VEC, v + i * VEC);
      }
    }
  } else if (seg < 2 * p.n_qk + vsegs + gsegs) {
    const int first = (seg - 2 * p.n_qk - vsegs) * SEG;
    float nA[N], dt[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + (i / VEC * 32 + lane) * VEC + i % VEC;
      nA[i] = c < Cg ? -expf(p.A_log[c / D]) : 0.f;
      dt[i] = c < Cg ? p.dt_bias[c] : 0.f;
    }
    for (int t = t0; t < live; ++t) {
      const T* src = (const T*)p.a_raw + (long long)b * p.a_sb + (long long)t * p.a_st + first;
      float* out = p.decay + (row0 + t) * Cg + first;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = (i * 32 + lane) * VEC;
        if (first + c < Cg) {
          float v[VEC];
          ldvec<VEC>(src + c, v);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[e] = expf(nA[i * VEC + e] * softplus_acc(v[e] + dt[i * VEC + e]));
          stvec<VEC>(out + c, v);
        }
      }
    }
  } else if (seg == 2 * p.n_qk + vsegs + gsegs) {
    for (int t = t0; t < live; ++t)
      for (int h = lane; h < p.nh; h += 32)
        p.beta[(row0 + t) * p.nh + h] = sigmoid_acc(ldf1((const T*)p.b_raw + (long long)b * p.b_sb + (long long)t * p.b_st + h));
  }
}

// ---- recurrent form ---------------------------------------------------------------------------------------------------------------------
// Block = (batch row, head, 16 value channels).  A thread holds two value channels and, of each, the key channels j * 32 + ns * 4 .. + 3 (ns = its
// place among eight lanes), so a lane's 16-byte shared-memory reads of k / q / decay serve both channels, the eight lanes read 128 contiguous
// bytes, and the state moves in 16-byte pieces.  Time runs in rounds of 16 steps; the rows of the next round land in a second shared-memory
// stage (cp.async) meanwhile.
//   delta: s <- decay * s per key channel; r = s . k, o = s . q on the shrunk state share one lane reduction; u = beta (v - r); s += u k;
//          o += u (k . q), k . q formed once per step and round
//   fixed: s <- decay_h s + v k;  o = s . q
//   gated: s <- fade_t s + (put_t v) k;  o = s . q / den_t.  A third warp of the block forms the gates one round ahead (running maximum step by
//          step), keeps the key sum n and the denominators den_t = max(|n . q|, exp(-m)) + 1e-6
constexpr int LS_FIXED = 0, LS_DELTA = 1, LS_GATED = 2;
constexpr float MLSTM_DEN_EPS = 1e-6f;
constexpr int LS_PT = 16, LS_TT = 16, LS_NS = 8, LS_CPT = 2, LS_THREADS = (LS_PT / LS_CPT) * LS_NS;

// capped log input gate and log forget gate
__device__ __forceinline__ float2 log_gates(float i, float f, float cap) {
  const float z = cap * tanhf(f / cap);
  return make_float2(cap * tanhf(i / cap), fminf(z, 0.f) - log1pf(expf(-fabsf(z))));
}

template <typename T, int KIND, int NJ, bool ALIGNED>
__global__ void __launch_bounds__(LS_THREADS + (KIND == LS_GATED ? 32 : 0)) linear_scan_kernel(LinearScanParams p) {
  extern __shared__ __align__(16) float lsm[];
  constexpr bool DELTA = KIND == LS_DELTA, GATED = KIND == LS_GATED;
  constexpr int NT = LS_THREADS + (GATED ? 32 : 0);
  constexpr int DP = NJ * 32, ROWS = DELTA ? 3 : 2, STAGE = ROWS * LS_TT * DP + LS_TT * LS_PT;
  float* kq = lsm + 2 * STAGE;                  // [TT] k . q
  float* bt = kq + LS_TT;                       // [TT] beta
  float* os = bt + LS_TT;                       // [TT][PT]
  float* gts = os + LS_TT * LS_PT;              // gated: two stages of fade, put, exp(-m) [TT] each, then the denominators [TT]
  float* den = gts + 6 * LS_TT;
  const int D = p.D, Dv = p.Dv, b = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * LS_PT;
  const int n_tok = p.q_len[b];
  if (n_tok <= 0) return;
  const int tid = threadIdx.x, pl = tid / LS_NS, ns = tid % LS_NS;
  const bool channels = !GATED || tid < LS_THREADS;      // false: the warp of gates and key sum
  const int gq = h / (p.nh / p.n_qk), Cq = p.n_qk * D;
  float* Sg = p.state + ((long long)p.lines[b] * p.nh + h) * Dv * D;
  const bool has_ctx = p.ctx_len[b] > 0;
  float4 S[LS_CPT][NJ];
#pragma unroll
  for (int c = 0; c < LS_CPT; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int d = j * 32 + ns * 4, pc = p0 + pl * LS_CPT + c;
      S[c][j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (has_ctx && channels && pc < Dv) {
        const float* s = Sg + (long long)pc * D + d;
        if (ALIGNED) { if (d < D) S[c][j] = *reinterpret_cast<const float4*>(s); }
        else {
          if (d < D) S[c][j].x = s[0];
          if (d + 1 < D) S[c][j].y = s[1];
          if (d + 2 < D) S[c][j].z = s[2];
          if (d + 3 < D) S[c][j].w = s[3];
        }
      }
    }
  const T* xrow = (const T*)p.x + (long long)b * p.x_sb;
  const float lam = KIND == LS_FIXED ? p.decay[h] : 0.f;
  // gated: this block's copy of the key sum (lane + 32 j of the third warp) and of the running maximum
  float nk[GATED ? NJ : 1], m_run = 0.f, i_b = 0.f, f_b = 0.f;
  const float q_scale = rsqrtf((float)D);
  const long long copy = (((long long)p.lines[b] * p.nh + h) * gridDim.x + blockIdx.x);
  auto gates = [&](int t0, int st) {
    const int lane = tid & 31, tt = min(LS_TT, n_tok - t0);
    float2 g = make_float2(0.f, 0.f);
    if (lane < tt) {
      const T* r = (const T*)p.x + (long long)b * p.x_sb + (long long)(t0 + lane) * p.x_st + p.gate_at + h;
      g = log_gates(ldf1(r) + i_b, ldf1(r + p.nh) + f_b, p.cap);
    }
    float before = 0.f, after = 0.f;
#pragma unroll 1
    for (int t = 0; t < tt; ++t) {
      const float it = __shfl_sync(0xffffffffu, g.x, t), ft = __shfl_sync(0xffffffffu, g.y, t);
      const float m = fmaxf(ft + m_run, it);
      if (lane == t) { before = m_run; after = m; }
      m_run = m;
    }
    if (lane < tt) {
      float* d = gts + st * 3 * LS_TT + lane;
      d[0] = expf(g.y + before - after);
      d[LS_TT] = expf(g.x - after);
      d[2 * LS_TT] = expf(-after);
    }
  };
  if constexpr (GATED) {
    if (!channels) {
      i_b = p.i_bias[h];
      f_b = p.f_bias[h];
      if (has_ctx) m_run = p.run_max[copy];
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int d = (tid & 31) + 32 * j;
        nk[j] = has_ctx && d < D ? p.key_sum[copy * D + d] : 0.f;
      }
      gates(0, 0);
    }
  }
  // rows of steps t0 .. into stage st; zeros past the key channels and past the live steps
  auto issue = [&](int t0, int st) {
    const int tt = min(LS_TT, n_tok - t0);
    float* qd = lsm + st * STAGE;
    float* kd = qd + LS_TT * DP;
    float* gd = kd + LS_TT * DP;                // delta only
    float* vd = qd + ROWS * LS_TT * DP;
    if constexpr (DELTA && ALIGNED) {
      constexpr int CPR = DP / 4;
      for (int i = tid; i < LS_TT * CPR; i += NT) {
        const int t = i / CPR, d = (i % CPR) * 4, at = t * DP + d;
        const bool on = t < tt && d < D;
        const float* q = on ? (const float*)xrow + (long long)(t0 + t) * p.x_st + gq * D + d : (const float*)xrow;
        cp_async16(qd + at, q, on);
        cp_async16(kd + at, on ? q + Cq : q, on);
        cp_async16(gd + at, on ? p.decay + ((long long)b * p.T + t0 + t) * p.nh * D + h * D + d : (const float*)xrow, on);
      }
      for (int i = tid; i < LS_TT * (LS_PT / 4); i += NT) {
        const int t = i / (LS_PT / 4), c = (i % (LS_PT / 4)) * 4;
        const bool on = t < tt && p0 + c < Dv;
        cp_async16(vd + t * LS_PT + c, on ? (const float*)xrow + (long long)(t0 + t) * p.x_st + 2 * Cq + h * Dv + p0 + c : (const float*)xrow, on);
      }
      cp_async_commit();
    } else {
      auto act = [&](float v) { return (KIND == LS_FIXED && p.silu) ? silu_acc(v) : v; };
      const int tl = (t0 == 0 && tt < LS_TT) ? tt : LS_TT;          // a lone short round touches its live steps only
      for (int i = tid; i < tl * DP; i += NT) {
        const int t = i / DP, d = i % DP;
        const bool on = t < tt && d < D;
        const T* r = xrow + (long long)(t0 + t) * p.x_st + gq * D + d;
        qd[i] = on ? act(ldf1(r)) : 0.f;
        kd[i] = on ? act(ldf1(r + Cq)) : 0.f;
        if (DELTA) gd[i] = on ? p.decay[((long long)b * p.T + t0 + t) * p.nh * D + h * D + d] : 0.f;
      }
      for (int i = tid; i < tl * LS_PT; i += NT) {
        const int t = i / LS_PT, c = p0 + i % LS_PT;
        vd[i] = (t < tt && c < Dv) ? act(ldf1(xrow + (long long)(t0 + t) * p.x_st + 2 * Cq + h * Dv + c)) : 0.f;
      }
    }
  };
  issue(0, 0);
  int st = 0;
  for (int t0 = 0; t0 < n_tok; t0 += LS_TT, st ^= 1) {
    const int tt = min(LS_TT, n_tok - t0);
    if constexpr (DELTA && ALIGNED) cp_async_wait<0>();
    __syncthreads();                            // these steps have landed; everyone is done with the other stage, kq, bt and os
    const float* qs = lsm + st * STAGE;
    const float* ks = qs + LS_TT * DP;
    const float* gs = ks + LS_TT * DP;
    const float* vs = qs + ROWS * LS_TT * DP;
    if constexpr (DELTA) {
      // four threads per step form k . q
      const int t = tid / 4, part = tid % 4;
      float s = 0.f;
      if (t < tt) {
#pragma unroll
        for (int j = 0; j < NJ * 2; ++j) {
          const int at = t * DP + (j * 4 + part) * 4;
          const float4 a = *reinterpret_cast<const float4*>(qs + at), k = *reinterpret_cast<const float4*>(ks + at);
          s += (a.x * k.x + a.z * k.z) + (a.y * k.y + a.w * k.w);
        }
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if (part == 0 && t < tt) {
        kq[t] = s;
        bt[t] = p.beta[((long long)b * p.T + t0 + t) * p.nh + h];
      }
      __syncthreads();
    }
    if (t0 + LS_TT < n_tok) issue(t0 + LS_TT, st ^ 1);
    const float* gt = gts + st * 3 * LS_TT;
    if constexpr (GATED) {
      if (!channels) {
#pragma unroll 1
        for (int t = 0; t < tt; ++t) {
          const float fade = gt[t], put = gt[LS_TT + t];
          float dot = 0.f;
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            const int d = t * DP + (tid & 31) + 32 * j;
            nk[j] = fade * nk[j] + put * ks[d];
            dot += nk[j] * qs[d];
          }
          dot = warp_sum(dot);
          if ((tid & 31) == 0) den[t] = fmaxf(fabsf(dot * q_scale), gt[2 * LS_TT + t]) + MLSTM_DEN_EPS;
        }
        if (t0 + LS_TT < n_tok) gates(t0 + LS_TT, st ^ 1);
      }
    }
#pragma unroll 1
    for (int t = 0; channels && t < tt; ++t) {
      const float4* Kt = reinterpret_cast<const float4*>(ks + t * DP) + ns;
      const float4* Qt = reinterpret_cast<const float4*>(qs + t * DP) + ns;
      float4 kv[NJ];
      float sq[LS_CPT], vt[LS_CPT];
#pragma unroll
      for (int c = 0; c < LS_CPT; ++c) { sq[c] = 0.f; vt[c] = vs[t * LS_PT + pl * LS_CPT + c]; }
      if constexpr (DELTA) {
        const float4* Gt = reinterpret_cast<const float4*>(gs + t * DP) + ns;
        float sk[LS_CPT];
#pragma unroll
        for (int c = 0; c < LS_CPT; ++c) sk[c] = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          kv[j] = Kt[j * 8];
          const float4 qv = Qt[j * 8], gv = Gt[j * 8];
#pragma unroll
          for (int c = 0; c < LS_CPT; ++c) {
            S[c][j].x *= gv.x; S[c][j].y *= gv.y; S[c][j].z *= gv.z; S[c][j].w *= gv.w;
            sk[c] += (S[c][j].x * kv[j].x + S[c][j].z * kv[j].z) + (S[c][j].y * kv[j].y + S[c][j].w * kv[j].w);
            sq[c] += (S[c][j].x * qv.x + S[c][j].z * qv.z) + (S[c][j].y * qv.y + S[c][j].w * qv.w);
          }
        }
#pragma unroll
        for (int o = LS_NS / 2; o > 0; o >>= 1)
#pragma unroll
          for (int c = 0; c < LS_CPT; ++c) {
            sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], o);
            sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], o);
          }
        const float be = bt[t], kqt = kq[t];
#pragma unroll
        for (int c = 0; c < LS_CPT; ++c) {
          const float u = be * (vt[c] - sk[c]);
#pragma unroll
          for (int j = 0; j < NJ; ++j) { S[c][j].x += u * kv[j].x; S[c][j].y += u * kv[j].y; S[c][j].z += u * kv[j].z; S[c][j].w += u * kv[j].w; }
          sq[c] += u * kqt;
        }
      } else {
        float lt = lam;
        if constexpr (GATED) {
          lt = gt[t];
#pragma unroll
          for (int c = 0; c < LS_CPT; ++c) vt[c] *= gt[LS_TT + t];
        }
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const float4 k4 = Kt[j * 8], qv = Qt[j * 8];
#pragma unroll
          for (int c = 0; c < LS_CPT; ++c) {
            S[c][j].x = lt * S[c][j].x + vt[c] * k4.x; S[c][j].y = lt * S[c][j].y + vt[c] * k4.y;
            S[c][j].z = lt * S[c][j].z + vt[c] * k4.z; S[c][j].w = lt * S[c][j].w + vt[c] * k4.w;
            sq[c] += (S[c][j].x * qv.x + S[c][j].z * qv.z) + (S[c][j].y * qv.y + S[c][j].w * qv.w);
          }
        }
#pragma unroll
        for (int o = LS_NS / 2; o > 0; o >>= 1)
#pragma unroll
          for (int c = 0; c < LS_CPT; ++c) sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], o);
      }
      if (ns == 0)
#pragma unroll
        for (int c = 0; c < LS_CPT; ++c) os[t * LS_PT + pl * LS_CPT + c] = sq[c];
    }
    __syncthreads();
    for (int i = tid; i < tt * LS_PT; i += NT) {
      const int t = i / LS_PT, c = p0 + i % LS_PT;
      if (c < Dv) p.y[((long long)b * p.T + t0 + t) * p.nh * Dv + h * Dv + c] = GATED ? os[i] * q_scale / den[t] : os[i];
    }
  }
  if constexpr (GATED) {
    if (!channels) {
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int d = (tid & 31) + 32 * j;
        if (d < D) p.key_sum[copy * D + d] = nk[j];
      }
      if ((tid & 31) == 0) p.run_max[copy] = m_run;
      return;
    }
  }
#pragma unroll
  for (int c = 0; c < LS_CPT; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int d = j * 32 + ns * 4, pc = p0 + pl * LS_CPT + c;
      if (pc < Dv) {
        float* s = Sg + (long long)pc * D + d;
        if (ALIGNED) { if (d < D) *reinterpret_cast<float4*>(s) = S[c][j]; }
        else {
          if (d < D) s[0] = S[c][j].x;
          if (d + 1 < D) s[1] = S[c][j].y;
          if (d + 2 < D) s[2] = S[c][j].z;
          if (d + 3 < D) s[3] = S[c][j].w;
        }
      }
    }
}

// ---- fixed decays and exponential gates, chunked form on tensor cores (bf16 rows, key sizes 64 / 128 / 256): prompt portions ---------------
// Block = (batch row, head, 32 value channels), 4 warps; time runs in chunks of 64 steps.  With q, k, v after SiLU (bf16) and the state M (fp32,
// in accumulator registers, [value, key]) before the chunk, for steps t, s counted inside the chunk of n live steps:
//     y_t = decay^(t+1) M q_t + sum_{s <= t} decay^(t-s) (q_t . k_s) v_s
//     M   = decay^n M + sum_s decay^(n-1-s) v_s k_s^T
// All products run on mma.sync m16n8k16 with fp32 accumulators.  The operands that are fp32 by nature — the state, the decayed scores and the
// decayed values — enter as a bf16 pair (value, remainder), two products each, so that they keep 16 bits.  Raw rows arrive through cp.async
// one chunk ahead; a thread applies SiLU in place to the pieces it copied itself.
// GATED: the powers of the decay become weights from the gates.  With F_t the sum of the log forget gates of the chunk up to t, g_s = i_s - F_s
// and x_t = max(m, max_{s <= t} g_s) (m: the running maximum before the chunk), the running maximum at t is F_t + x_t and
//     decay^(t+1) -> exp(m - x_t);   decay^(t-s) -> exp(g_s - x_t);   decay^(n-1-s) -> exp(g_s - x_n);   decay^n -> exp(m - x_n)
// (no exponent is positive).  The key sum n follows the state with the same weights, n_t . q_t = exp(m - x_t) n . q_t + the row sum of the
// weighted scores, and y_t is divided by max(|n_t . q_t|, exp(-F_t - x_t)) + 1e-6.  Warp 0 forms the gates one chunk ahead.
constexpr int CS_C = 64, CS_NV = 32, CS_THREADS = 128, CS_MIN_T = 16;

__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16lo(hi), b - bf16hi(hi));
}
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.f + __expf(-v)); }

template <int D, bool GATED>
__global__ void __launch_bounds__(CS_THREADS, D > 128 ? 1 : 2) linear_chunk_kernel(LinearScanParams p) {
  extern __shared__ __align__(16) unsigned char csm[];
  constexpr int DS = D + 8, VS = CS_NV + 8, STAGE = 2 * CS_C * DS + CS_C * VS, NTW = D / 32;
  __nv_bfloat16* stage0 = reinterpret_cast<__nv_bfloat16*>(csm);           // two stages of q [64][DS], k [64][DS], v [64][VS]
  __nv_bfloat16* Sh = stage0 + 2 * STAGE;                                  // state [32][DS]: value, then remainder
  __nv_bfloat16* Sl = Sh + CS_NV * DS;
  __nv_bfloat16* Wh = Sl + CS_NV * DS;                                     // decayed values [64][VS]: value, then remainder
  __nv_bfloat16* Wl = Wh + CS_C * VS;
  float* pw = reinterpret_cast<float*>(Wl + CS_C * VS);                    // fixed: powers of the decay, 0 .. 64
  // gated: two stages of g, x, exp(m - x), exp(-F - x) [64] each, of exp(m - x_n) and x_n, and of the key sum [D]; then exp(g - x_n) [64]
  float *gts = pw, *tot = gts + 8 * CS_C, *nsum = tot + 4, *wgt = nsum + 2 * D;
  const int b = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * CS_NV, Dv = p.Dv;
  const int n_tok = p.q_len[b];
  if (n_tok <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const __nv_bfloat16* xrow = (const __nv_bfloat16*)p.x + (long long)b * p.x_sb;
  const int Cq = p.nh * D;
  float* Sg = p.state + ((long long)p.lines[b] * p.nh + h) * Dv * D;
  const float q_scale = rsqrtf((float)D);
  float m_run = 0.f, i_b = 0.f, f_b = 0.f;
  const int slices = (Dv + MLSTM_SLICE - 1) / MLSTM_SLICE, sl0 = p0 / MLSTM_SLICE;
  const long long copy = ((long long)p.lines[b] * p.nh + h) * slices + sl0;      // of this block; the next one is its too when it exists
  auto gates = [&](int t0, int st) {
    const int n = min(CS_C, n_tok - t0);
    float *g = gts + st * 4 * CS_C, f_sum = 0.f, x_max = m_run;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = half * 32 + lane;
      float2 lg = make_float2(0.f, 0.f);
      if (t < n) {
        const __nv_bfloat16* r = xrow + (long long)(t0 + t) * p.x_st + p.gate_at + h;
        lg = log_gates(__bfloat162float(r[0]) + i_b, __bfloat162float(r[p.nh]) + f_b, p.cap);
      }
      float F = lg.y;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, F, o);
        if (lane >= o) F += v;
      }
      F += f_sum;
      const float gs = t < n ? lg.x - F : -INFINITY;
      float x = gs;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x = fmaxf(x, v);
      }
      x = fmaxf(x, x_max);
      g[t] = gs;
      g[CS_C + t] = x;
      g[2 * CS_C + t] = expf(m_run - x);
      g[3 * CS_C + t] = expf(-(F + x));
      f_sum = __shfl_sync(0xffffffffu, F, 31);
      x_max = __shfl_sync(0xffffffffu, x, 31);
    }
    if (lane == 0) {
      tot[st * 2] = expf(m_run - x_max);
      tot[st * 2 + 1] = x_max;
    }
    m_run = f_sum + x_max;
  };
  // this warp's share of the state: all 32 value channels x key channels [warp * D / 4, + D / 4)
  float S[2][NTW][4];
  const bool has_ctx = p.ctx_len[b] > 0;
  if constexpr (GATED) {
    for (int d = tid; d < D; d += CS_THREADS) nsum[d] = has_ctx ? p.key_sum[copy * D + d] : 0.f;
    if (warp == 0) {
      i_b = p.i_bias[h];
      f_b = p.f_bias[h];
      if (has_ctx) m_run = p.run_max[copy];
      gates(0, 0);
    }
  } else {
    if (tid <= CS_C) pw[tid] = powf(p.decay[h], (float)tid);
  }
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int v = p0 + mt * 16 + gid + r * 8, d = warp * (D / 4) + nt * 8 + tig * 2;
        float2 s = make_float2(0.f, 0.f);
        if (has_ctx && v < Dv) s = *reinterpret_cast<const float2*>(Sg + (long long)v * D + d);
        S[mt][nt][r * 2] = s.x;
        S[mt][nt][r * 2 + 1] = s.y;
      }
  constexpr int QP = CS_C * D / 8 / CS_THREADS, VP = CS_C * CS_NV / 8 / CS_THREADS;        // 16-byte pieces per thread
  auto issue = [&](int t0, int st) {
    __nv_bfloat16* qd = stage0 + st * STAGE;
    __nv_bfloat16* kd = qd + CS_C * DS;
    __nv_bfloat16* vd = kd + CS_C * DS;
    const int n = min(CS_C, n_tok - t0);
#pragma unroll
    for (int i = 0; i < QP; ++i) {
      const int c = tid + i * CS_THREADS, t = c / (D / 8), d = (c % (D / 8)) * 8;
      const bool on = t < n;
      const __nv_bfloat16* q = on ? xrow + (long long)(t0 + t) * p.x_st + h * D + d : xrow;
      cp_async16(qd + t * DS + d, q, on);
      cp_async16(kd + t * DS + d, on ? q + Cq : q, on);
    }
#pragma unroll
    for (int i = 0; i < VP; ++i) {
      const int c = tid + i * CS_THREADS, t = c / (CS_NV / 8), v = (c % (CS_NV / 8)) * 8;
      const bool on = t < n && p0 + v < Dv;
      cp_async16(vd + t * VS + v, on ? xrow + (long long)(t0 + t) * p.x_st + 2 * Cq + h * Dv + p0 + v : xrow, on);
    }
    cp_async_commit();
  };
  auto silu_piece = [&](__nv_bfloat16* at, float* f) {
    uint4 r = *reinterpret_cast<const uint4*>(at);
    f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y);
    f[4] = bf16lo(r.z); f[5] = bf16hi(r.z); f[6] = bf16lo(r.w); f[7] = bf16hi(r.w);
    if (!GATED && p.silu) {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = silu_fast(f[e]);
      r = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
      *reinterpret_cast<uint4*>(at) = r;
      f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y);
      f[4] = bf16lo(r.z); f[5] = bf16hi(r.z); f[6] = bf16lo(r.w); f[7] = bf16hi(r.w);
    }
  };
  issue(0, 0);
  __syncthreads();                              // pw (gates, key sum) is there
  int st = 0;
  for (int t0 = 0; t0 < n_tok; t0 += CS_C, st ^= 1) {
    const int n = min(CS_C, n_tok - t0);
    __nv_bfloat16* Q = stage0 + st * STAGE;
    __nv_bfloat16* K = Q + CS_C * DS;
    __nv_bfloat16* V = K + CS_C * DS;
    cp_async_wait<0>();
    {
      float f[8];
#pragma unroll 2
      for (int i = 0; !GATED && i < QP; ++i) {
        const int c = tid + i * CS_THREADS, t = c / (D / 8), d = (c % (D / 8)) * 8;
        silu_piece(Q + t * DS + d, f);
        silu_piece(K + t * DS + d, f);
      }
#pragma unroll
      for (int i = 0; i < VP; ++i) {
        const int c = tid + i * CS_THREADS, t = c / (CS_NV / 8), v = (c % (CS_NV / 8)) * 8;
        silu_piece(V + t * VS + v, f);
        float w = 0.f;
        if constexpr (GATED) {
          if (t < n) w = __expf(gts[st * 4 * CS_C + t] - tot[st * 2 + 1]);
          if (v == 0) wgt[t] = w;
        } else if (t < n) {
          w = pw[n - 1 - t];
        }
        uint4 hi, lo;
        split_bf16(f[0] * w, f[1] * w, hi.x, lo.x); split_bf16(f[2] * w, f[3] * w, hi.y, lo.y);
        split_bf16(f[4] * w, f[5] * w, hi.z, lo.z); split_bf16(f[6] * w, f[7] * w, hi.w, lo.w);
        *reinterpret_cast<uint4*>(Wh + t * VS + v) = hi;
        *reinterpret_cast<uint4*>(Wl + t * VS + v) = lo;
      }
    }
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int at = (mt * 16 + gid + r * 8) * DS + warp * (D / 4) + nt * 8 + tig * 2;
          uint32_t hi, lo;
          split_bf16(S[mt][nt][r * 2], S[mt][nt][r * 2 + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(Sh + at) = hi;
          *reinterpret_cast<uint32_t*>(Sl + at) = lo;
        }
    __syncthreads();
    if (t0 + CS_C < n_tok) issue(t0 + CS_C, st ^ 1);          // the other stage was last read before this barrier
    const int r0 = warp * 16 + gid, r1 = r0 + 8;              // this thread's two steps
    const float* gt = gts + st * 4 * CS_C;
    float nq0 = 0.f, nq1 = 0.f;                               // key sum before the chunk, times q, of the two steps
    if constexpr (GATED) {
      const float* ns = nsum + st * D;
      const __nv_bfloat16* qr = Q + (warp * 16 + (lane >> 1)) * DS + (lane & 1) * (D / 2);
      float s = 0.f;
#pragma unroll 4
      for (int d = 0; d < D / 2; d += 8) {
        const uint4 r = *reinterpret_cast<const uint4*>(qr + d);
        const float4 a = *reinterpret_cast<const float4*>(ns + (lane & 1) * (D / 2) + d), c = *reinterpret_cast<const float4*>(ns + (lane & 1) * (D / 2) + d + 4);
        s += (bf16lo(r.x) * a.x + bf16hi(r.x) * a.y) + (bf16lo(r.y) * a.z + bf16hi(r.y) * a.w) +
             (bf16lo(r.z) * c.x + bf16hi(r.z) * c.y) + (bf16lo(r.w) * c.z + bf16hi(r.w) * c.w);
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      nq0 = __shfl_sync(0xffffffffu, s, 2 * gid);
      nq1 = __shfl_sync(0xffffffffu, s, 2 * gid + 16);
      // key sum after the chunk, into the other stage
      constexpr int PARTS = CS_THREADS / (D / 2);             // threads per pair of channels
      const int d = tid / PARTS * 2, part = tid % PARTS;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll 8
      for (int t = part; t < CS_C; t += PARTS) {
        const uint32_t r = *reinterpret_cast<const uint32_t*>(K + t * DS + d);
        s0 += wgt[t] * bf16lo(r);
        s1 += wgt[t] * bf16hi(r);
      }
#pragma unroll
      for (int o = PARTS / 2; o > 0; o >>= 1) {
        s0 += __shfl_xor_sync(0xffffffffu, s0, o);
        s1 += __shfl_xor_sync(0xffffffffu, s1, o);
      }
      if (part == 0) {
        nsum[(st ^ 1) * D + d] = tot[st * 2] * ns[d] + s0;
        nsum[(st ^ 1) * D + d + 1] = tot[st * 2] * ns[d + 1] + s1;
      }
    }
    if (warp * 16 < n) {
      float o[CS_NV / 8][4], sc[CS_C / 8][4];
#pragma unroll
      for (int i = 0; i < CS_NV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
      for (int i = 0; i < CS_C / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        const __nv_bfloat16* qp = Q + r0 * DS + ks * 16 + tig * 2;
        const uint32_t qa[4] = {*reinterpret_cast<const uint32_t*>(qp), *reinterpret_cast<const uint32_t*>(qp + 8 * DS),
                                *reinterpret_cast<const uint32_t*>(qp + 8), *reinterpret_cast<const uint32_t*>(qp + 8 * DS + 8)};
#pragma unroll
        for (int nt = 0; nt < CS_NV / 8; ++nt) {
          const int at = (nt * 8 + gid) * DS + ks * 16 + tig * 2;
          const uint32_t bh[2] = {*reinterpret_cast<const uint32_t*>(Sh + at), *reinterpret_cast<const uint32_t*>(Sh + at + 8)};
          const uint32_t bl[2] = {*reinterpret_cast<const uint32_t*>(Sl + at), *reinterpret_cast<const uint32_t*>(Sl + at + 8)};
          mma_bf16_16816(o[nt], qa, bh);
          mma_bf16_16816(o[nt], qa, bl);
        }
#pragma unroll
        for (int nt = 0; nt < CS_C / 8; ++nt)
          if (nt <= 2 * warp + 1) {                           // later steps than this warp's last one are not seen
            const __nv_bfloat16* kp = K + (nt * 8 + gid) * DS + ks * 16 + tig * 2;
            const uint32_t bb[2] = {*reinterpret_cast<const uint32_t*>(kp), *reinterpret_cast<const uint32_t*>(kp + 8)};
            mma_bf16_16816(sc[nt], qa, bb);
          }
      }
      const float d0 = GATED ? gt[2 * CS_C + r0] : pw[r0 + 1], d1 = GATED ? gt[2 * CS_C + r1] : pw[r1 + 1];
      const float x0 = GATED ? gt[CS_C + r0] : 0.f, x1 = GATED ? gt[CS_C + r1] : 0.f;
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int i = 0; i < CS_NV / 8; ++i) { o[i][0] *= d0; o[i][1] *= d0; o[i][2] *= d1; o[i][3] *= d1; }
#pragma unroll
      for (int kk = 0; kk < CS_C / 16; ++kk)
        if (kk <= warp) {
          uint32_t ah[4], al[4];
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int nt = kk * 2 + half, s = nt * 8 + tig * 2;
            float f[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int gap = (e < 2 ? r0 : r1) - (s + (e & 1));
              if constexpr (GATED) f[e] = gap >= 0 ? sc[nt][e] * __expf(gt[s + (e & 1)] - (e < 2 ? x0 : x1)) : 0.f;
              else f[e] = gap >= 0 ? sc[nt][e] * pw[gap] : 0.f;
            }
            if constexpr (GATED) {
              sum0 += f[0] + f[1];
              sum1 += f[2] + f[3];
            }
            split_bf16(f[0], f[1], ah[half * 2], al[half * 2]);
            split_bf16(f[2], f[3], ah[half * 2 + 1], al[half * 2 + 1]);
          }
#pragma unroll
          for (int nv = 0; nv < CS_NV / 8; nv += 2) {
            uint32_t r[4];
            ldmatrix_x4_trans(r, V + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VS + (nv + (lane >> 4)) * 8);
            const uint32_t ba[2] = {r[0], r[1]}, bb[2] = {r[2], r[3]};
            mma_bf16_16816(o[nv], ah, ba);
            mma_bf16_16816(o[nv], al, ba);
            mma_bf16_16816(o[nv + 1], ah, bb);
            mma_bf16_16816(o[nv + 1], al, bb);
          }
        }
      if constexpr (GATED) {
#pragma unroll
        for (int o = 1; o <= 2; o <<= 1) {
          sum0 += __shfl_xor_sync(0xffffffffu, sum0, o);
          sum1 += __shfl_xor_sync(0xffffffffu, sum1, o);
        }
        const float m0 = q_scale / (fmaxf(fabsf((d0 * nq0 + sum0) * q_scale), gt[3 * CS_C + r0]) + MLSTM_DEN_EPS);
        const float m1 = q_scale / (fmaxf(fabsf((d1 * nq1 + sum1) * q_scale), gt[3 * CS_C + r1]) + MLSTM_DEN_EPS);
#pragma unroll
        for (int i = 0; i < CS_NV / 8; ++i) { o[i][0] *= m0; o[i][1] *= m0; o[i][2] *= m1; o[i][3] *= m1; }
      }
      float* y = p.y + ((long long)b * p.T + t0) * p.nh * Dv + h * Dv + p0;
#pragma unroll
      for (int nv = 0; nv < CS_NV / 8; ++nv) {
        const int col = nv * 8 + tig * 2;
        if (p0 + col < Dv) {
          if (r0 < n) *reinterpret_cast<float2*>(y + (long long)r0 * p.nh * Dv + col) = make_float2(o[nv][0], o[nv][1]);
          if (r1 < n) *reinterpret_cast<float2*>(y + (long long)r1 * p.nh * Dv + col) = make_float2(o[nv][2], o[nv][3]);
        }
      }
    }
    // state after the chunk
    const float dn = GATED ? tot[st * 2] : pw[n];
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int nt = 0; nt < NTW; ++nt) { S[mt][nt][0] *= dn; S[mt][nt][1] *= dn; S[mt][nt][2] *= dn; S[mt][nt][3] *= dn; }
#pragma unroll
    for (int kk = 0; kk < CS_C / 16; ++kk) {
      uint32_t kb[NTW / 2][4];
#pragma unroll
      for (int nt = 0; nt < NTW; nt += 2)
        ldmatrix_x4_trans(kb[nt / 2], K + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * DS + warp * (D / 4) + (nt + (lane >> 4)) * 8);
#pragma unroll
      for (int mt = 0; mt < 2; ++mt) {
        uint32_t wh[4], wl[4];
        const int at = (kk * 16 + (lane & 7) + (lane >> 4) * 8) * VS + mt * 16 + ((lane >> 3) & 1) * 8;
        ldmatrix_x4_trans(wh, Wh + at);
        ldmatrix_x4_trans(wl, Wl + at);
#pragma unroll
        for (int nt = 0; nt < NTW; ++nt) {
          const uint32_t bb[2] = {kb[nt / 2][(nt & 1) * 2], kb[nt / 2][(nt & 1) * 2 + 1]};
          mma_bf16_16816(S[mt][nt], wh, bb);
          mma_bf16_16816(S[mt][nt], wl, bb);
        }
      }
    }
    if (GATED && warp == 0 && t0 + CS_C < n_tok) gates(t0 + CS_C, st ^ 1);
    __syncthreads();                            // the state and decayed-value copies are rewritten at the top of the next chunk
  }
  if constexpr (GATED) {
    const int copies = min(CS_NV / MLSTM_SLICE, slices - sl0);
    for (int i = tid; i < copies * D; i += CS_THREADS) p.key_sum[copy * D + i] = nsum[st * D + i % D];
    if (tid == 0)
      for (int c = 0; c < copies; ++c) p.run_max[copy + c] = m_run;
  }
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int v = p0 + mt * 16 + gid + r * 8, d = warp * (D / 4) + nt * 8 + tig * 2;
        if (v < Dv) *reinterpret_cast<float2*>(Sg + (long long)v * D + d) = make_float2(S[mt][nt][r * 2], S[mt][nt][r * 2 + 1]);
      }
}

__global__ void __launch_bounds__(256) table_route_kernel(const int* __restrict__ table, const int* __restrict__ ids, const int* __restrict__ q_len,
                                                          float* __restrict__ w, int* __restrict__ idx, int B, int T, int k, int vocab) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)B * T * k) return;
  const long long tok = i / k;
  const int id = ids[tok];
  const bool on = (int)(tok % T) < q_len[tok / T] && id >= 0 && id < vocab;
  idx[i] = on ? table[(long long)id * k + i % k] : -1;
  w[i] = 1.f / (float)k;
}

template <typename K>
void opt_in(K kernel, size_t bytes) {
  if (bytes > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <typename T, int KIND>
void scan_go(const LinearScanParams& p, bool aligned, cudaStream_t st) {
  const dim3 grid((p.Dv + LS_PT - 1) / LS_PT, p.nh, p.B);
  auto go = [&](auto nj, auto al) {
    constexpr int NJ = decltype(nj)::value;
    constexpr bool AL = decltype(al)::value;
    constexpr size_t stage = (KIND == LS_DELTA ? 3 : 2) * LS_TT * NJ * 32 + LS_TT * LS_PT;
    const size_t smem = sizeof(float) * (2 * stage + 2 * LS_TT + LS_TT * LS_PT + (KIND == LS_GATED ? 7 * LS_TT : 0));
    auto kernel = linear_scan_kernel<T, KIND, NJ, AL>;
    opt_in(kernel, smem);
    kernel<<<grid, LS_THREADS + (KIND == LS_GATED ? 32 : 0), smem, st>>>(p);
  };
  auto by_size = [&](auto al) {
    if (p.D <= 64) go(std::integral_constant<int, 2>{}, al);
    else if (p.D <= 128) go(std::integral_constant<int, 4>{}, al);
    else go(std::integral_constant<int, 8>{}, al);
  };
  if (aligned) by_size(std::true_type{}); else by_size(std::false_type{});
}

// prompt portions in bf16 whose sizes fit the chunked form; false: not launched
template <bool GATED>
bool chunk_go(const LinearScanParams& p, bool lp, cudaStream_t st) {
  if (!lp || p.T < CS_MIN_T || (p.D != 64 && p.D != 128 && p.D != 256) || p.Dv % 8 != 0 || p.x_st % 8 != 0 || p.x_sb % 8 != 0 ||
      (((uintptr_t)p.x | (uintptr_t)p.state | (uintptr_t)p.y) & 15) != 0)
    return false;
  const dim3 grid((p.Dv + CS_NV - 1) / CS_NV, p.nh, p.B);
  auto go = [&](auto d) {
    constexpr int D = decltype(d)::value;
    const size_t smem = sizeof(__nv_bfloat16) * (2 * (2 * CS_C * (D + 8) + CS_C * (CS_NV + 8)) + 2 * CS_NV * (D + 8) + 2 * CS_C * (CS_NV + 8)) +
                        sizeof(float) * (GATED ? 9 * CS_C + 4 + 2 * D : CS_C + 1);
    opt_in(linear_chunk_kernel<D, GATED>, smem);
    linear_chunk_kernel<D, GATED><<<grid, CS_THREADS, smem, st>>>(p);
  };
  if (p.D == 64) go(std::integral_constant<int, 64>{});
  else if (p.D == 128) go(std::integral_constant<int, 128>{});
  else go(std::integral_constant<int, 256>{});
  return true;
}

static_assert(LS_PT == MLSTM_SLICE && CS_NV % MLSTM_SLICE == 0, "a block keeps whole copies of the key sum");

}  // namespace

void delta_front_launch(const DeltaFrontParams& p, bool lp, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  if (p.D > 256 || p.K > SEQMIX_MAX_TAPS || p.nh % p.n_qk != 0) throw std::runtime_error("delta_front: key size <= 256, taps <= 8, heads a multiple of q / k heads");
  const int C = 2 * p.n_qk * p.D + p.nh * p.Dv, Cg = p.nh * p.D;
  const size_t va = lp ? 8 : 16, esz = lp ? 2 : 4;
  auto al = [&](const void* q) { return ((uintptr_t)q % va) == 0; };
  const bool vec = p.D % 4 == 0 && C % 4 == 0 && al(p.p) && al(p.a_raw) && al(p.state) && (p.p_sb * esz) % va == 0 && (p.p_st * esz) % va == 0 &&
                   (p.a_sb * esz) % va == 0 && (p.a_st * esz) % va == 0 && ((uintptr_t)p.qkv % 16) == 0 && ((uintptr_t)p.decay % 16) == 0;
  auto go = [&](auto tag, auto ve, auto ni, auto km) {
    using T = decltype(tag);
    constexpr int VEC = decltype(ve)::value, NI = decltype(ni)::value, KM = decltype(km)::value, SEG = 32 * VEC * NI;
    // tiles hold at least K - 1 tokens: only the first one of a row needs the carried rows
    const int TT = p.T == 1 ? 1 : 8;
    const int vsegs = (p.nh * p.Dv + SEG - 1) / SEG, gsegs = (Cg + SEG - 1) / SEG, segs = 2 * p.n_qk + vsegs + gsegs + 1;
    const dim3 grid((p.T + TT - 1) / TT, (segs + FRONT_WARPS - 1) / FRONT_WARPS, p.B);
    delta_front_kernel<T, VEC, NI, KM><<<grid, FRONT_WARPS * 32, 0, st>>>(p, TT, vsegs, gsegs);
  };
  using std::integral_constant;
  auto by_taps = [&](auto tag, auto ve, auto ni) {
    if (p.K <= 4) go(tag, ve, ni, integral_constant<int, 4>{}); else go(tag, ve, ni, integral_constant<int, 8>{});
  };
  auto by_size = [&](auto tag) {
    if (vec && p.D <= 128) by_taps(tag, integral_constant<int, 4>{}, integral_constant<int, 1>{});
    else if (vec) by_taps(tag, integral_constant<int, 4>{}, integral_constant<int, 2>{});
    else by_taps(tag, integral_constant<int, 1>{}, integral_constant<int, 8>{});
  };
  if (lp) by_size(__nv_bfloat16{}); else by_size(float{});
}

void channel_delta_scan_launch(const LinearScanParams& p, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  if (p.D > 256 || p.nh % p.n_qk != 0) throw std::runtime_error("channel_delta_scan: key size <= 256, heads a multiple of q / k heads");
  const bool aligned = p.D % 4 == 0 && p.Dv % 4 == 0 && p.x_st % 4 == 0 && p.x_sb % 4 == 0 &&
                       (((uintptr_t)p.x | (uintptr_t)p.decay | (uintptr_t)p.state) & 15) == 0;
  scan_go<float, LS_DELTA>(p, aligned, st);
}

void decay_scan_launch(const LinearScanParams& p, bool lp, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  if (p.D > 256 || p.n_qk != p.nh) throw std::runtime_error("decay_scan: key size <= 256");
  if (chunk_go<false>(p, lp, st)) return;
  const bool aligned = p.D % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
  if (lp) scan_go<__nv_bfloat16, LS_FIXED>(p, aligned, st); else scan_go<float, LS_FIXED>(p, aligned, st);
}

void mlstm_scan_launch(const LinearScanParams& p, bool lp, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  if (p.D > 256 || p.n_qk != p.nh) throw std::runtime_error("mlstm_scan: key size <= 256");
  if (chunk_go<true>(p, lp, st)) return;
  const bool aligned = p.D % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
  if (lp) scan_go<__nv_bfloat16, LS_GATED>(p, aligned, st); else scan_go<float, LS_GATED>(p, aligned, st);
}

void table_route_launch(const int* table, const int* ids, const int* q_len, float* w, int* idx, int B, int T, int k, int vocab, cudaStream_t st) {
  const long long n = (long long)B * T * k;
  if (n <= 0) return;
  table_route_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(table, ids, q_len, w, idx, B, T, k, vocab);
}

}  // namespace nxdi
