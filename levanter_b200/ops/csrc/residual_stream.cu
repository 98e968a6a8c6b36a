// The two ends of a pre-norm block whose residual stream is kept in fp32: the token embedding that starts it and the RMS norm that
// reads it.  (The adds in between ride in the epilogues of the projections, which accumulate into the stream.)  Built without
// fast-math: norms of a 32-bit stream are 32-bit arithmetic throughout.
#include "common.cuh"

namespace lvb {
namespace stream32 {

__device__ __forceinline__ float ld1(const void* p, int f32, size_t i) {
  return f32 ? reinterpret_cast<const float*>(p)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}
__device__ __forceinline__ float4 ld4(const void* p, int f32, size_t i) {  // i a multiple of 4, aligned
  if (f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 w = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// out[t, :] = scale * weight[ids[t], :] in fp32
__global__ void embed_kernel(const int* __restrict__ ids, const void* __restrict__ weight, int w_f32, float* __restrict__ out, int dim,
                             int vocab, float scale, int vec, int* status) {
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) record_status(status, kBoundsCheck, 602, id);
  const size_t src = static_cast<size_t>(ok ? id : 0) * dim, dst = static_cast<size_t>(t) * dim;
  const float f = ok ? scale : 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = ld4(weight, w_f32, src + c);
      *reinterpret_cast<float4*>(out + dst + c) = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) out[dst + c] = ld1(weight, w_f32, src + c) * f;
  }
}

// y[r, :] = x[r, :] / sqrt(mean(x[r, :]^2) + eps) * (w + w_offset); x fp32, y fp32 or bf16.  rows: optional int64 gather of the rows.
// One CTA per row; the row's second read comes from L1.
__global__ void __launch_bounds__(256)
rms_kernel(const float* __restrict__ x, const long long* __restrict__ rows, const void* __restrict__ w, int w_f32, void* __restrict__ y,
           int y_f32, int dim, float eps, float w_offset, int vec) {
  __shared__ float s_red[8];
  const size_t src = static_cast<size_t>(rows != nullptr ? rows[blockIdx.x] : blockIdx.x) * dim;
  const size_t dst = static_cast<size_t>(blockIdx.x) * dim;
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(x + src + c);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) ss = fmaf(x[src + c], x[src + c], ss);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x) / 32; ++i) ss += s_red[i];
  const float r = 1.f / sqrtf(ss / static_cast<float>(dim) + eps);
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(x + src + c);
      const float4 g = ld4(w, w_f32, c);
      const float4 o = make_float4(v.x * r * (g.x + w_offset), v.y * r * (g.y + w_offset), v.z * r * (g.z + w_offset),
                                   v.w * r * (g.w + w_offset));
      if (y_f32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(y) + dst + c) = o;
      else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(y) + dst + c) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
      const float o = x[src + c] * r * (ld1(w, w_f32, c) + w_offset);
      if (y_f32) reinterpret_cast<float*>(y)[dst + c] = o;
      else reinterpret_cast<__nv_bfloat16*>(y)[dst + c] = __float2bfloat16(o);
    }
  }
}

inline int threads_for(int dim) {
  const int t = ((dim + 3) / 4 + 31) / 32 * 32;
  return t < 32 ? 32 : t > 256 ? 256 : t;
}

}  // namespace stream32
}  // namespace lvb

extern "C" int lvb_embed_stream(const int* ids, const void* weight, int w_f32, float* out, int tokens, int dim, int vocab, float scale,
                                int* status, void* stream) {
  using namespace lvb;
  if (tokens <= 0 || dim <= 0 || vocab <= 0) return kErrBadArg;
  const int vec = (dim & 3) == 0 && ((reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  stream32::embed_kernel<<<tokens, stream32::threads_for(dim), 0, reinterpret_cast<cudaStream_t>(stream)>>>(ids, weight, w_f32, out, dim, vocab,
                                                                                                        scale, vec, status);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// n_rows output rows; rows: int64 [n_rows] source rows (each in range: the caller's responsibility), or null for row i = i.
extern "C" int lvb_rms_stream(const float* x, const long long* rows, const void* w, int w_f32, void* y, int y_f32, int n_rows, int dim,
                              float eps, float w_offset, void* stream) {
  using namespace lvb;
  if (n_rows <= 0 || dim <= 0) return kErrBadArg;
  const int vec = (dim & 3) == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(y)) & 15) == 0;
  stream32::rms_kernel<<<n_rows, stream32::threads_for(dim), 0, reinterpret_cast<cudaStream_t>(stream)>>>(x, rows, w, w_f32, y, y_f32, dim, eps,
                                                                                                       w_offset, vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
