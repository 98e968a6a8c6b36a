// Rows whose elements are split into equal consecutive groups, each with a root mean square of its own: how a CTA holds a row in registers
// and forms the groups' factors.  All arithmetic is 32-bit; include it from files that are built without fast-math.
#pragma once
#include "common.cuh"

namespace lvb {
namespace rowg {

__device__ __forceinline__ float ld1(const void* p, int f32, size_t i) {
  return f32 ? reinterpret_cast<const float*>(p)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}

// kVec consecutive elements (4, aligned, or 1)
template <int kVec>
__device__ __forceinline__ void ld_unit(const void* p, int f32, size_t i, float (&v)[kVec]) {
  if constexpr (kVec == 4) {
    if (f32) {
      const float4 a = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
      const uint2 w = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
      v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
  } else {
    v[0] = ld1(p, f32, i);
  }
}
template <int kVec>
__device__ __forceinline__ void st_unit(void* p, int f32, size_t i, const float (&v)[kVec]) {
  if constexpr (kVec == 4) {
    if (f32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = make_float4(v[0], v[1], v[2], v[3]);
    else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p) + i) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  } else {
    if (f32) reinterpret_cast<float*>(p)[i] = v[0];
    else reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16(v[0]);
  }
}

// A row of `dim` elements over the threads of a CTA: unit u = threadIdx.x + n * blockDim.x holds elements [u * kVec, (u + 1) * kVec).  A group is
// `part` elements, a multiple of kVec.
template <int kN, int kVec>
struct Row {
  float a[kN][kVec];

  static __device__ __forceinline__ int column(int n) { return (threadIdx.x + n * blockDim.x) * kVec; }

  // Where the groups lie, for all rows of a CTA.
  struct Groups {
    int dim, part, per;  // per: partial sums of a group
    bool by_warp;        // the 32 units of a warp lie in one group: a partial sum per warp and n, else one per unit
    int first[kN];       // by_warp: first partial sum of the group of unit n; else the number of its group

    __device__ __forceinline__ Groups(int dim, int part) : dim(dim), part(part) {
      by_warp = part == dim || part % (32 * kVec) == 0;
      per = part == dim ? static_cast<int>(blockDim.x >> 5) * kN : by_warp ? part / (32 * kVec) : part / kVec;
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        const int g = part == dim || column(n) >= dim ? 0 : column(n) / part;
        first[n] = by_warp ? g * per : g;
      }
    }
  };

  // Multiplies every group by 1 / sqrt(mean of its squares + eps).  s: scratch of scratch_floats() floats, not in use by a slower warp (two
  // buffers in turn suffice).  Every thread of the CTA takes part.
  __device__ __forceinline__ void normalize(const Groups& g, float eps, float* s) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float ss[kN];
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      ss[n] = 0.f;
#pragma unroll
      for (int e = 0; e < kVec; ++e) ss[n] = fmaf(a[n][e], a[n][e], ss[n]);
    }
    const float inv = 1.f / static_cast<float>(g.part);
    if (g.by_warp) {
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        const float v = warp_sum(ss[n]);
        if (lane == 0) s[n * warps + warp] = v;
      }
      __syncthreads();
      float r = 0.f;
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        if (n == 0 || g.first[n] != g.first[n - 1]) {
          float t = 0.f;
          for (int i = 0; i < g.per; ++i) t += s[g.first[n] + i];
          r = 1.f / sqrtf(t * inv + eps);
        }
#pragma unroll
        for (int e = 0; e < kVec; ++e) a[n][e] *= r;
      }
      return;
    }
    float* s_r = s + kN * blockDim.x;
#pragma unroll
    for (int n = 0; n < kN; ++n) s[threadIdx.x + n * blockDim.x] = ss[n];
    __syncthreads();
    for (int j = warp; j < g.dim / g.part; j += warps) {
      float t = 0.f;
      for (int i = lane; i < g.per; i += 32) t += s[j * g.per + i];
      t = warp_sum(t);
      if (lane == 0) s_r[j] = 1.f / sqrtf(t * inv + eps);
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      const float r = s_r[g.first[n]];
#pragma unroll
      for (int e = 0; e < kVec; ++e) a[n][e] *= r;
    }
  }
  static size_t scratch_floats(int threads, int groups) { return static_cast<size_t>(kN) * threads + groups; }
};

// Threads and units per thread (1, 2, 4 or 16) for rows of `dim` elements; few_rows: the rows do not fill the GPU, so a row is spread over
// more threads.  False: too long.
inline bool shape_for(int dim, int vec, bool few_rows, int& n, int& threads) {
  const int units = (dim + vec - 1) / vec;
  const int choices[4] = {1, 2, 4, 16}, most[4] = {few_rows ? 1024 : 256, 512, 1024, 1024};
  for (int i = 0; i < 4; ++i) {
    n = choices[i];
    threads = ((units + n - 1) / n + 31) / 32 * 32;
    if (threads <= most[i]) return true;
  }
  return false;
}

}  // namespace rowg
}  // namespace lvb
