// Token embedding with a bigram term: the fp32 residual stream and its bf16 copy straight from the tables.
#include <cuda_bf16.h>

#include "common.cuh"
#include "seqmix.h"

namespace nxdi {
namespace {

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16lo(r.x), bf16hi(r.x), bf16lo(r.y), bf16hi(r.y));
}
__device__ __forceinline__ float load1(const float* p) { return *p; }
__device__ __forceinline__ float load1(const __nv_bfloat16* p) { return __bfloat162float(*p); }

// Block = one token.  The block of a row's first token is the only one that touches the sequence's line: it reads the carried token before it
// stores the portion's last one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) bigram_embed_kernel(BigramEmbedParams p) {
  const int b = blockIdx.y, t = blockIdx.x, n = p.q_len[b];
  const int W = p.W;
  const long long tok = (long long)b * p.T + t;
  __shared__ long long row_s;
  const bool live = t < n;
  const int id = live ? p.ids[tok] : -1;
  if (threadIdx.x == 0) {
    long long row = -1;
    if (live && p.bigram) {
      int* line = p.state + p.lines[b];
      if (t == 0 && p.ctx_len[b] == 0) {
        row = p.buckets;
      } else {
        const long long prev = t == 0 ? *line : p.ids[tok - 1];
        row = (prev * p.mul_prev + (long long)id * p.mul_cur) % p.buckets;
        if (row < 0) row += p.buckets;
      }
      if (t == 0) *line = p.ids[(long long)b * p.T + n - 1];
    }
    row_s = row;
  }
  __syncthreads();
  const T* e = id >= 0 && id < p.vocab ? (const T*)p.embed + (long long)id * W : nullptr;      // padding and unknown ids: no embedding
  const T* g = row_s >= 0 ? (const T*)p.bigram + row_s * W : nullptr;
  float* x = p.x + tok * W;
  __nv_bfloat16* lp = p.x_lp ? (__nv_bfloat16*)p.x_lp + tok * W : nullptr;
  if constexpr (VEC) {
    for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
      float4 v = e ? load4(e + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 a = g ? load4(g + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      v = make_float4(v.x * p.scale + a.x, v.y * p.scale + a.y, v.z * p.scale + a.z, v.w * p.scale + a.w);
      *reinterpret_cast<float4*>(x + c) = v;
      if (lp) *reinterpret_cast<uint2*>(lp + c) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = (e ? load1(e + c) * p.scale : 0.f) + (g ? load1(g + c) : 0.f);
      x[c] = v;
      if (lp) lp[c] = __float2bfloat16_rn(v);
    }
  }
}

}  // namespace

void bigram_embed_launch(const BigramEmbedParams& p, bool lp, cudaStream_t st) {
  if (p.B <= 0 || p.T <= 0) return;
  const dim3 grid(p.T, p.B);
  const bool vec = p.W % 4 == 0 && (((uintptr_t)p.embed | (uintptr_t)p.bigram) & (lp ? 7 : 15)) == 0;
  if (lp) {
    if (vec) bigram_embed_kernel<__nv_bfloat16, true><<<grid, 256, 0, st>>>(p); else bigram_embed_kernel<__nv_bfloat16, false><<<grid, 256, 0, st>>>(p);
  } else {
    if (vec) bigram_embed_kernel<float, true><<<grid, 256, 0, st>>>(p); else bigram_embed_kernel<float, false><<<grid, 256, 0, st>>>(p);
  }
}

}  // namespace nxdi
