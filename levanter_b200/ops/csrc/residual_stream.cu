// The two ends of a pre-norm block whose residual stream is kept in fp32: the token embedding that starts it and the RMS norm that
// reads it.  (The adds in between ride in the epilogues of the projections, which accumulate into the stream.)  Where a block's
// output is normed before it is added, one kernel does both and the next block's norm.  Also here: the gated activation for fp32
// and for sizes that are not multiples of 8.  Built without fast-math: norms of a 32-bit stream are 32-bit arithmetic throughout.
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
// One CTA per row; the row's second read comes from L1.  kAdd: the vector `add` (w's type) joins the row first, and the sum is written
// back; every thread reads back the columns that it wrote.
template <bool kAdd>
__global__ void __launch_bounds__(256)
rms_kernel(float* x, const long long* __restrict__ rows, const void* __restrict__ add, const void* __restrict__ w, int w_f32, void* __restrict__ y,
           int y_f32, int dim, float eps, float w_offset, int vec) {
  __shared__ float s_red[8];
  const size_t src = static_cast<size_t>(rows != nullptr ? rows[blockIdx.x] : blockIdx.x) * dim;
  const size_t dst = static_cast<size_t>(blockIdx.x) * dim;
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      float4 v = *reinterpret_cast<const float4*>(x + src + c);
      if constexpr (kAdd) {
        const float4 a = ld4(add, w_f32, c);
        v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
        *reinterpret_cast<float4*>(x + src + c) = v;
      }
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
      float v = x[src + c];
      if constexpr (kAdd) {
        v += ld1(add, w_f32, c);
        x[src + c] = v;
      }
      ss = fmaf(v, v, ss);
    }
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

// x[r, :] += rms(y[r, :]) * w_post, then h[d, :] = rms(x[r, :]) * w_next, for r = rows[d] (or d).  With `rows` the stream is read only:
// the sum is what the last norm of a model sees.  The row stays in shared memory between the passes.
__global__ void __launch_bounds__(256)
add_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const long long* __restrict__ rows, const void* __restrict__ w_post,
                const void* __restrict__ w_next, int w_f32, void* __restrict__ h, int h_f32, int dim, float eps, int vec) {
  extern __shared__ __align__(16) float s_row[];  // [dim]
  __shared__ float s_red[2][8];
  const size_t src = static_cast<size_t>(rows != nullptr ? rows[blockIdx.x] : blockIdx.x) * dim;
  const size_t dst = static_cast<size_t>(blockIdx.x) * dim;
  auto block_sum = [&](float v, int slot) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) s_red[slot][threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < static_cast<int>(blockDim.x) / 32; ++i) t += s_red[slot][i];
    return t;
  };
  const float n = static_cast<float>(dim);
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(y + src + c);
      *reinterpret_cast<float4*>(s_row + c) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
      const float v = y[src + c];
      s_row[c] = v;
      ss = fmaf(v, v, ss);
    }
  }
  const float r1 = 1.f / sqrtf(block_sum(ss, 0) / n + eps);
  ss = 0.f;
  if (vec) {  // every thread reads back the columns that it wrote
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(s_row + c), g = ld4(w_post, w_f32, c);
      float4 o = *reinterpret_cast<const float4*>(x + src + c);
      o.x += v.x * r1 * g.x; o.y += v.y * r1 * g.y; o.z += v.z * r1 * g.z; o.w += v.w * r1 * g.w;
      *reinterpret_cast<float4*>(s_row + c) = o;
      if (rows == nullptr) *reinterpret_cast<float4*>(x + src + c) = o;
      ss = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, fmaf(o.w, o.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
      const float o = x[src + c] + s_row[c] * r1 * ld1(w_post, w_f32, c);
      s_row[c] = o;
      if (rows == nullptr) x[src + c] = o;
      ss = fmaf(o, o, ss);
    }
  }
  const float r2 = 1.f / sqrtf(block_sum(ss, 1) / n + eps);
  if (vec) {
    for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(s_row + c), g = ld4(w_next, w_f32, c);
      const float4 o = make_float4(v.x * r2 * g.x, v.y * r2 * g.y, v.z * r2 * g.z, v.w * r2 * g.w);
      if (h_f32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(h) + dst + c) = o;
      else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(h) + dst + c) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
    }
  } else {
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
      const float o = s_row[c] * r2 * ld1(w_next, w_f32, c);
      if (h_f32) reinterpret_cast<float*>(h)[dst + c] = o;
      else reinterpret_cast<__nv_bfloat16*>(h)[dst + c] = __float2bfloat16(o);
    }
  }
}

// act(g) * u: tanh-gelu (0) or silu (1); or (2) g sigmoid(1.702 g) (u + 1) with g at most `limit` and u within +-limit.  kFast: for results that
// are rounded to bf16.
template <bool kFast>
__device__ __forceinline__ float glu(int act, float limit, float g, float u) {
  if (act == 2) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit) + 1.f;
    return kFast ? g * u * __fdividef(1.f, 1.f + __expf(-1.702f * g)) : g / (1.f + expf(-1.702f * g)) * u;
  }
  if (act == 1) return kFast ? g * u * __fdividef(1.f, 1.f + __expf(-g)) : g / (1.f + expf(-g)) * u;
  return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
}

// out[r, c] = act(gate[r, c]) * up[r, c] (* sigmoid(row_gate[r * ldr])), any size; gate and up of one type, out of that type or bf16
template <bool kOutF32>
__global__ void __launch_bounds__(256)
glu_kernel(const void* __restrict__ gate, const void* __restrict__ up, const float* __restrict__ row_gate, void* __restrict__ out, int act, float limit,
           int f32, long long total, int cols, long long ldg, long long ldu, long long ldr, int vec) {
  auto factor = [&](long long r) { return row_gate != nullptr ? 1.f / (1.f + expf(-row_gate[r * ldr])) : 1.f; };
  const long long step = static_cast<long long>(gridDim.x) * blockDim.x;
  if constexpr (!kOutF32) {
    if (vec == 8) {  // groups of 8 columns, bf16 throughout
      const int per = cols / 8;
      for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total / 8; i += step) {
        const long long r = i / per, c = (i - r * per) * 8;
        const uint4 g = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(gate) + r * ldg + c);
        const uint4 u = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(up) + r * ldu + c);
        const float f = factor(r);
        const uint32_t gw[4] = {g.x, g.y, g.z, g.w}, uw[4] = {u.x, u.y, u.z, u.w};
        uint32_t o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
          const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&uw[e]));
          o[e] = pack_bf16x2(glu<true>(act, limit, a.x, b.x) * f, glu<true>(act, limit, a.y, b.y) * f);
        }
        reinterpret_cast<uint4*>(out)[i] = make_uint4(o[0], o[1], o[2], o[3]);
      }
      return;
    }
  }
  if (vec) {  // groups of 4 columns; cols is a multiple of 4
    const int per = cols / 4;
    for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total / 4; i += step) {
      const long long r = i / per, c = (i - r * per) * 4;
      const float4 g = ld4(gate, f32, r * ldg + c), u = ld4(up, f32, r * ldu + c);
      const float f = factor(r);
      const float4 o = make_float4(glu<!kOutF32>(act, limit, g.x, u.x) * f, glu<!kOutF32>(act, limit, g.y, u.y) * f, glu<!kOutF32>(act, limit, g.z, u.z) * f,
                                   glu<!kOutF32>(act, limit, g.w, u.w) * f);
      if constexpr (kOutF32) reinterpret_cast<float4*>(out)[i] = o;
      else reinterpret_cast<uint2*>(out)[i] = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
    }
    return;
  }
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += step) {
    const long long r = i / cols, c = i - r * cols;
    const float o = glu<!kOutF32>(act, limit, ld1(gate, f32, r * ldg + c), ld1(up, f32, r * ldu + c)) * factor(r);
    if constexpr (kOutF32) reinterpret_cast<float*>(out)[i] = o;
    else reinterpret_cast<__nv_bfloat16*>(out)[i] = __float2bfloat16(o);
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

// n_rows output rows; rows: int64 [n_rows] source rows (each in range: the caller's responsibility), or null for row i = i.  add: null, or a
// vector [dim] of w's type that is added to every row of x first (in place; rows must be null then).
extern "C" int lvb_rms_stream(float* x, const long long* rows, const void* add, const void* w, int w_f32, void* y, int y_f32, int n_rows, int dim,
                              float eps, float w_offset, void* stream) {
  using namespace lvb;
  if (n_rows <= 0 || dim <= 0 || (add != nullptr && rows != nullptr)) return kErrBadArg;
  const int vec = (dim & 3) == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(y) |
                                      reinterpret_cast<uintptr_t>(add)) & 15) == 0;
  auto kern = add != nullptr ? stream32::rms_kernel<true> : stream32::rms_kernel<false>;
  kern<<<n_rows, stream32::threads_for(dim), 0, reinterpret_cast<cudaStream_t>(stream)>>>(x, rows, add, w, w_f32, y, y_f32, dim, eps, w_offset, vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// x[rows] += rms(y) * w_post; h = rms(x) * w_next.  x, y fp32 [.., dim]; w_f32: type of both weights; h [n_rows, dim] fp32 or bf16.  rows: null, or
// int64 [n_rows] source rows (each in range), and then x is left as it is.
extern "C" int lvb_add_norm_stream(float* x, const float* y, const long long* rows, const void* w_post, const void* w_next, int w_f32, void* h,
                                   int h_f32, int n_rows, int dim, float eps, void* stream) {
  using namespace lvb;
  if (n_rows <= 0 || dim <= 0) return kErrBadArg;
  const size_t smem = static_cast<size_t>(dim) * 4;
  if (smem > 200 * 1024) return kErrTooLarge;
  if (smem > 40 * 1024 &&
      cudaFuncSetAttribute(stream32::add_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
    return kErrCuda;
  const uintptr_t mis = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w_post) |
                        reinterpret_cast<uintptr_t>(w_next) | reinterpret_cast<uintptr_t>(h);
  const int vec = (dim & 3) == 0 && (mis & 15) == 0;
  stream32::add_norm_kernel<<<n_rows, stream32::threads_for(dim), smem, reinterpret_cast<cudaStream_t>(stream)>>>(x, y, rows, w_post, w_next, w_f32,
                                                                                                             h, h_f32, dim, eps, vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// out [rows, cols] = act(gate) * up (* the sigmoid of row_gate[r * ldr], fp32, when given) with act = tanh-gelu (0), silu (1) or the clamped form
// (2: min(gate, limit) sigmoid(1.702 min(gate, limit)) (clamp(up, -limit, limit) + 1)); gate and up with row strides ldg and ldu; in_f32, out_f32:
// types (fp32 results need fp32 operands).
extern "C" int lvb_glu_any(const void* gate, const void* up, const float* row_gate, void* out, int act, float limit, int in_f32, int out_f32, int rows,
                           int cols, long long ldg, long long ldu, long long ldr, void* stream) {
  using namespace lvb;
  if (rows <= 0 || cols <= 0 || act < 0 || act > 2 || (out_f32 && !in_f32)) return kErrBadArg;
  const uintptr_t mis = reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(out);
  const int vec = (mis & 15) != 0 ? 0 : !in_f32 && ((cols | ldg | ldu) & 7) == 0 ? 8 : ((cols | ldg | ldu) & 3) == 0 ? 4 : 0;
  const long long total = static_cast<long long>(rows) * cols, cap = static_cast<long long>(num_sms()) * 16;
  long long blocks = (total / (vec ? vec : 1) + 255) / 256;
  if (blocks > cap) blocks = cap;
  auto kern = out_f32 ? stream32::glu_kernel<true> : stream32::glu_kernel<false>;
  kern<<<static_cast<int>(blocks), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(gate, up, row_gate, out, act, limit, in_f32, total, cols, ldg, ldu, ldr,
                                                                                   vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
