// Several residual streams per token: write-back of a sublayer's result, mixing of the streams, the weighted sum the next sublayer reads,
// its RMS norm and its short causal convolution over time, with the carried rows, in one kernel:
//
//   x'_t = sum_s mix[s, t] x_s + out[t] y;   u = sum_s in[s] x'_s;   h = rms_unit(u) * w;   r_p = h_p + sum_j cw[:, j] h_(p - K + 1 + j)
//
// A block marches over a tile of consecutive tokens of one batch row.  The convolution's window (the last K - 1 rows h) stays in registers;
// a tile that does not start the row first re-forms the K - 1 rows before it from x and y (inputs, so no block depends on another).  Only the
// first tile of a row reads the sequence's carried rows, and it is also the one that writes them back when it is done (re-forming the row's
// last K - 1 rows h when they lie in later tiles), so carrying them needs no second kernel.  The loads of token t + 1 are issued before the
// block-wide sum of token t, with one barrier per token.  Everything is fp32; compiled WITHOUT fast-math.
#include <cuda_bf16.h>
#include <math.h>

#include <stdexcept>
#include <type_traits>

#include "common.cuh"
#include "seqmix.h"

namespace nxdi {
namespace {

__device__ __forceinline__ float4 ldv4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ldv4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16lo(r.x), bf16hi(r.x), bf16lo(r.y), bf16hi(r.y));
}
__device__ __forceinline__ void stv4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void stv4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }
__device__ __forceinline__ void fma4(float4& a, float s, const float4& b) { a.x += s * b.x; a.y += s * b.y; a.z += s * b.z; a.w += s * b.w; }
__device__ __forceinline__ float ldy(const void* y, int lp, long long i) {
  return lp ? __bfloat162float(((const __nv_bfloat16*)y)[i]) : ((const float*)y)[i];
}

// block-wide sum with ONE barrier: consecutive calls alternate between two halves of `red` (2 x 32 floats)
__device__ __forceinline__ float block_sum1(float v, float* red, int& flip) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float* r = red + flip * 32;
  flip ^= 1;
  if (lane == 0) r[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? r[lane] : 0.f);
}

// SM: streams (S <= SM, the rest count as zero), KM: taps (K <= KM), NCH: groups of four channels per thread; W a multiple of 4, W <= 4 * NCH * threads
template <typename TH, int SM, int KM, int NCH>
__global__ void __launch_bounds__(512) stream_mix_vec_kernel(StreamMixParams p, int TT) {
  __shared__ float red[64];
  const int b = blockIdx.y, t0 = blockIdx.x * TT, W = p.W, S = p.S, K = p.K;
  const int qn = p.q_len ? p.q_len[b] : p.T;
  const int t1 = min(t0 + TT, p.T), live = min(t1, qn);
  TH* hout = (TH*)p.h;
  int col[NCH];
#pragma unroll
  for (int c = 0; c < NCH; ++c) col[c] = (threadIdx.x + c * blockDim.x) * 4;
  for (int t = max(t0, qn); t < t1; ++t)          // rows past the live ones: zeros
#pragma unroll
    for (int c = 0; c < NCH; ++c)
      if (col[c] < W) stv4(hout + ((long long)b * p.T + t) * W + col[c], make_float4(0.f, 0.f, 0.f, 0.f));
  if (t0 >= qn) return;
  float mix[SM][SM], ow[SM], iw[SM];
#pragma unroll
  for (int s = 0; s < SM; ++s) {
    iw[s] = s < S ? p.in_w[s] : 0.f;
    ow[s] = (p.y && s < S) ? p.out_w[s] : 0.f;
#pragma unroll
    for (int d = 0; d < SM; ++d) mix[s][d] = (p.y && s < S && d < S) ? p.mix[s * S + d] : 0.f;
  }
  float4 nw[NCH], cw[KM][NCH], ring[KM][NCH];          // ring[d]: row h of d + 1 tokens ago; cw[d]: weight of lag d
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const bool in = col[c] < W;
    const float n1 = p.norm_n == 1 ? p.norm_w[0] : 1.f;
    nw[c] = (p.norm_n > 1 && in) ? ldv4(p.norm_w + col[c]) : make_float4(n1, n1, n1, n1);
#pragma unroll
    for (int d = 0; d < KM; ++d) {
      ring[d][c] = cw[d][c] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.conv_w && d < K && in) {
        const float* w = p.conv_w + (long long)col[c] * K + (K - 1 - d);
        cw[d][c] = make_float4(w[0], w[K], w[2 * K], w[3 * K]);
      }
    }
  }
  float* state = (p.conv_w && K > 1) ? p.state + (long long)p.lines[b] * (K - 1) * W : nullptr;
  if (state && t0 == 0 && p.ctx_len[b] > 0)
#pragma unroll
    for (int d = 0; d < KM - 1; ++d)
#pragma unroll
      for (int c = 0; c < NCH; ++c)
        if (d < K - 1 && col[c] < W) ring[d][c] = ldv4(state + (long long)(K - 2 - d) * W + col[c]);
  float4 xv[SM][NCH], yv[NCH];
  auto fetch = [&](int t) {
    const long long tok = (long long)b * p.T + t;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      const bool in = col[c] < W;
#pragma unroll
      for (int s = 0; s < SM; ++s)
        xv[s][c] = (in && s < S) ? ldv4(p.x + tok * p.x_tok + s * p.x_str + col[c]) : make_float4(0.f, 0.f, 0.f, 0.f);
      yv[c] = (p.y && in) ? (p.y_lp ? ldv4((const __nv_bfloat16*)p.y + tok * W + col[c]) : ldv4((const float*)p.y + tok * W + col[c]))
                          : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  int flip = 0;
  // tokens [ta, tb): update the streams, form h and push it into the ring; `emit`: write the streams and the convolved row
  auto march = [&](int ta, int tb, bool emit) {
    if (ta >= tb) return;
    fetch(ta);
    for (int t = ta; t < tb; ++t) {
      const long long tok = (long long)b * p.T + t;
      float4 u[NCH];
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        u[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (p.y) {
#pragma unroll
          for (int d = 0; d < SM; ++d) {
            float4 n = make_float4(ow[d] * yv[c].x, ow[d] * yv[c].y, ow[d] * yv[c].z, ow[d] * yv[c].w);
#pragma unroll
            for (int s = 0; s < SM; ++s) fma4(n, mix[s][d], xv[s][c]);
            if (emit && p.xn && d < S && col[c] < W) stv4(p.xn + (tok * S + d) * W + col[c], n);
            fma4(u[c], iw[d], n);
          }
        } else {
#pragma unroll
          for (int s = 0; s < SM; ++s) fma4(u[c], iw[s], xv[s][c]);
        }
        ss += u[c].x * u[c].x + u[c].y * u[c].y + u[c].z * u[c].z + u[c].w * u[c].w;
      }
      if (t + 1 < tb) fetch(t + 1);          // in flight during the block-wide sum
      float r = 1.f;
      if (p.norm_n) r = 1.f / sqrtf(block_sum1(ss, red, flip) / (float)W + p.eps);
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        const float4 h = make_float4(u[c].x * r * nw[c].x, u[c].y * r * nw[c].y, u[c].z * r * nw[c].z, u[c].w * r * nw[c].w);
        float4 o = h;
        if (KM > 1 || p.conv_w) {
          o.x += cw[0][c].x * h.x; o.y += cw[0][c].y * h.y; o.z += cw[0][c].z * h.z; o.w += cw[0][c].w * h.w;
#pragma unroll
          for (int d = 1; d < KM; ++d) {
            o.x += cw[d][c].x * ring[d - 1][c].x; o.y += cw[d][c].y * ring[d - 1][c].y;
            o.z += cw[d][c].z * ring[d - 1][c].z; o.w += cw[d][c].w * ring[d - 1][c].w;
          }
#pragma unroll
          for (int d = KM - 1; d > 0; --d) ring[d][c] = ring[d - 1][c];
          ring[0][c] = h;
        }
        if (emit && col[c] < W) stv4(hout + tok * W + col[c], o);
      }
    }
  };
  if (t0 > 0 && K > 1) march(max(t0 - (K - 1), 0), t0, false);
  march(t0, live, true);
  if (state && t0 == 0) {
    if (qn > live) march(qn - (K - 1), qn, false);          // the row's last rows h lie in later tiles (tiles hold at least K - 1 tokens)
#pragma unroll
    for (int d = 0; d < KM - 1; ++d)
#pragma unroll
      for (int c = 0; c < NCH; ++c)
        if (d < K - 1 && col[c] < W) stv4(state + (long long)(K - 2 - d) * W + col[c], ring[d][c]);
  }
}

// Any width, up to 8 streams and 8 taps: the window's rows live in shared memory, [K][W] floats used as a ring.
template <typename TH>
__global__ void __launch_bounds__(256) stream_mix_any_kernel(StreamMixParams p, int TT) {
  extern __shared__ float rows[];
  __shared__ float red[64];
  const int b = blockIdx.y, t0 = blockIdx.x * TT, W = p.W, S = p.S, K = p.K;
  const int qn = p.q_len ? p.q_len[b] : p.T;
  const int t1 = min(t0 + TT, p.T), live = min(t1, qn);
  TH* hout = (TH*)p.h;
  for (int t = max(t0, qn); t < t1; ++t)
    for (int c = threadIdx.x; c < W; c += blockDim.x) hout[((long long)b * p.T + t) * W + c] = (TH)0.f;
  if (t0 >= qn) return;
  float* state = (p.conv_w && K > 1) ? p.state + (long long)p.lines[b] * (K - 1) * W : nullptr;
  // a channel is handled by one thread throughout, so the ring needs no barriers; `head`: the slot of the next row
  int head = 0, flip = 0;
  const bool carried = state && t0 == 0 && p.ctx_len[b] > 0;
  for (int j = 0; j < K - 1; ++j)
    for (int c = threadIdx.x; c < W; c += blockDim.x) rows[j * W + c] = carried ? state[(long long)j * W + c] : 0.f;
  head = K - 1;
  auto march = [&](int ta, int tb, bool emit) {
    for (int t = ta; t < tb; ++t) {
      const long long tok = (long long)b * p.T + t;
      float* hr = rows + head * W;
      float ss = 0.f;
      for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float x[8], u = 0.f;
        for (int s = 0; s < S; ++s) x[s] = p.x[tok * p.x_tok + s * p.x_str + c];
        if (p.y) {
          const float y = ldy(p.y, p.y_lp, tok * W + c);
          for (int d = 0; d < S; ++d) {
            float n = p.out_w[d] * y;
            for (int s = 0; s < S; ++s) n += p.mix[s * S + d] * x[s];
            if (emit && p.xn) p.xn[(tok * S + d) * W + c] = n;
            u += p.in_w[d] * n;
          }
        } else {
          for (int s = 0; s < S; ++s) u += p.in_w[s] * x[s];
        }
        hr[c] = u;
        ss += u * u;
      }
      float r = 1.f;
      if (p.norm_n) r = 1.f / sqrtf(block_sum1(ss, red, flip) / (float)W + p.eps);
      for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const float h = hr[c] * r * (p.norm_n == 1 ? p.norm_w[0] : p.norm_n > 1 ? p.norm_w[c] : 1.f);
        hr[c] = h;
        float o = h;
        if (p.conv_w)
          for (int d = 0; d < K; ++d) o += p.conv_w[(long long)c * K + (K - 1 - d)] * rows[((head - d + K) % K) * W + c];
        if (emit) {
          if constexpr (std::is_same<TH, float>::value) hout[tok * W + c] = o;
          else hout[tok * W + c] = __float2bfloat16_rn(o);
        }
      }
      head = (head + 1) % K;
    }
  };
  if (t0 > 0 && K > 1) march(max(t0 - (K - 1), 0), t0, false);
  march(t0, live, true);
  if (state && t0 == 0) {
    if (qn > live) march(qn - (K - 1), qn, false);
    for (int j = 0; j < K - 1; ++j)          // oldest first: the row after the next free slot
      for (int c = threadIdx.x; c < W; c += blockDim.x) state[(long long)j * W + c] = rows[((head + 1 + j) % K) * W + c];
  }
}

}  // namespace

void stream_mix_norm_conv_launch(const StreamMixParams& p, bool h_lp, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  if (p.S < 1 || p.S > SEQMIX_MAX_STREAMS || p.K < 1 || p.K > SEQMIX_MAX_TAPS) throw std::runtime_error("stream_mix_norm_conv: at most 8 streams and 8 taps");
  // a tile holds at least K - 1 tokens, so that only the first one of a row needs the carried rows
  int TT = 1;
  if (p.K > 1 && p.T > 1) TT = p.K > 5 ? 8 : ((long long)p.B * ((p.T + 7) / 8) >= 2 * kNumSMs ? 8 : 4);
  const dim3 grid((p.T + TT - 1) / TT, p.B);
  auto al = [](const void* q, size_t a) { return ((uintptr_t)q & (a - 1)) == 0; };
  if (p.W % 4 == 0 && p.W <= 8192 && p.S <= 4 && p.K <= 4 && al(p.x, 16) && al(p.y, p.y_lp ? 8 : 16) && al(p.xn, 16) && al(p.h, h_lp ? 8 : 16) &&
      (p.norm_n <= 1 || al(p.norm_w, 16)) && al(p.state, 16)) {
    const int groups = p.W / 4, nch = groups <= 512 ? 1 : groups <= 1024 ? 2 : 4;
    const int threads = ((groups + nch - 1) / nch + 31) / 32 * 32;
    auto pick = [&](auto th, auto sm, auto km) {
      using TH = decltype(th);
      constexpr int SM = decltype(sm)::value, KM = decltype(km)::value;
      if (nch == 1) stream_mix_vec_kernel<TH, SM, KM, 1><<<grid, threads, 0, st>>>(p, TT);
      else if (nch == 2) stream_mix_vec_kernel<TH, SM, KM, 2><<<grid, threads, 0, st>>>(p, TT);
      else stream_mix_vec_kernel<TH, SM, KM, 4><<<grid, threads, 0, st>>>(p, TT);
    };
    auto by_taps = [&](auto th, auto sm) {
      if (p.K == 1) pick(th, sm, std::integral_constant<int, 1>{}); else pick(th, sm, std::integral_constant<int, 4>{});
    };
    auto by_streams = [&](auto th) {
      if (p.S == 1) by_taps(th, std::integral_constant<int, 1>{});
      else if (p.S == 2) by_taps(th, std::integral_constant<int, 2>{});
      else by_taps(th, std::integral_constant<int, 4>{});
    };
    if (h_lp) by_streams(__nv_bfloat16{}); else by_streams(float{});
    return;
  }
  const size_t smem = sizeof(float) * (size_t)p.K * p.W;
  if (smem > 200 * 1024) throw std::runtime_error("stream_mix_norm_conv: taps * width beyond the shared memory of a block");
  auto go = [&](auto kernel) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    kernel<<<grid, 256, smem, st>>>(p, TT);
  };
  if (h_lp) go(stream_mix_any_kernel<__nv_bfloat16>); else go(stream_mix_any_kernel<float>);
}

}  // namespace nxdi
