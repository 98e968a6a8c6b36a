// Serving kernels of a mixture of experts whose router scores the experts by a sigmoid or a softmax and picks within groups of neighbours:
//   route     one warp per token: scores, group choice, top-k, weights; tokens per expert
//   dispatch  positions in the expert-sorted, block-padded layout of the grouped GEMMs, and the copy of the token rows into it
//   combine   weighted sum of a token's expert outputs, added to the fp32 residual stream
// plus a grouped product for fp32 (and for sizes TMA cannot describe).  Nothing is read back by the host, so a decode round can be
// captured in a CUDA graph.  Built without fast-math: router scores and weights are 32-bit arithmetic.
#include "common.cuh"

namespace lvb {
namespace experts {

constexpr int kRouteWarps = 4;
constexpr int kMaxExperts = 1024;

__device__ __forceinline__ float ldv(const void* p, int f32, size_t i) {
  return f32 ? reinterpret_cast<const float*>(p)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}

// The largest of n values in shared memory and its index (the lower index on ties); every lane gets the result.
__device__ __forceinline__ int warp_argmax(const float* v, int n) {
  float best = -INFINITY;
  int at = 0x7fffffff;
  for (int i = threadIdx.x & 31; i < n; i += 32)
    if (v[i] > best || (v[i] == best && i < at)) { best = v[i]; at = i; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
    const int a2 = __shfl_xor_sync(0xffffffffu, at, o);
    if (b2 > best || (b2 == best && a2 < at)) { best = b2; at = a2; }
  }
  return at < n ? at : 0;
}

// kSoftmax: scores are the softmax over all experts of z + correction, a group counts by its best score, and the weights are the chosen
// scores divided by their sum.  Otherwise scores are sigmoids, a group counts by its two best choice scores, and the weights are scale * score.
template <bool kSoftmax>
__global__ void __launch_bounds__(kRouteWarps * 32)
route_kernel(const float* __restrict__ z, long long ldz, const void* __restrict__ correction, int c_f32, const int* __restrict__ live,
             int live_limit, int T, int E, int k, int groups, int keep, float scale, int* __restrict__ idx, float* __restrict__ w,
             int* __restrict__ counts) {
  extern __shared__ float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s_score = smem + warp * (2 * E + groups);  // sigmoid(z)
  float* s_choice = s_score + E;                    // + correction; -inf once taken or outside the kept groups
  float* s_group = s_choice + E;
  const int t = blockIdx.x * kRouteWarps + warp;
  if (t >= T) return;  // warps are independent: no block-wide barrier below
  if (live != nullptr && (live[t] < 0 || live[t] >= live_limit)) {  // padding token: no expert runs for it
    for (int j = lane; j < k; j += 32) { idx[static_cast<size_t>(t) * k + j] = -1; w[static_cast<size_t>(t) * k + j] = 0.f; }
    return;
  }
  auto corrected = [&](float s, int e) { return correction != nullptr ? s + ldv(correction, c_f32, e) : s; };
  float top = -INFINITY, inv = 1.f;
  if constexpr (kSoftmax) {
    for (int e = lane; e < E; e += 32) {
      s_score[e] = corrected(z[t * ldz + e], e);  // read back by this lane only
      top = fmaxf(top, s_score[e]);
    }
    top = warp_max(top);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) sum += expf(s_score[e] - top);
    inv = 1.f / warp_sum(sum);
  }
  for (int e = lane; e < E; e += 32) {
    const float s = kSoftmax ? expf(s_score[e] - top) * inv : 1.f / (1.f + expf(-z[t * ldz + e]));
    s_score[e] = s;
    s_choice[e] = kSoftmax ? s : corrected(s, e);
  }
  __syncwarp();
  if (groups > 1 && keep < groups) {
    const int size = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;  // the two largest choice scores of the group
      for (int e = g * size; e < (g + 1) * size; ++e) {
        const float c = s_choice[e];
        if (c > a) { b = a; a = c; } else if (c > b) b = c;
      }
      s_group[g] = size > 1 && !kSoftmax ? a + b : a;
    }
    __syncwarp();
    unsigned long long kept[kMaxExperts / 64] = {};
    for (int j = 0; j < keep; ++j) {
      const int g = warp_argmax(s_group, groups);
      kept[g >> 6] |= 1ull << (g & 63);
      __syncwarp();
      if (lane == 0) s_group[g] = -INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32) {
      const int g = e / size;
      if (!((kept[g >> 6] >> (g & 63)) & 1ull)) s_choice[e] = -INFINITY;
    }
    __syncwarp();
  }
  float chosen = 0.f;
  for (int j = 0; j < k; ++j) {
    const int e = warp_argmax(s_choice, E);
    chosen += s_score[e];
    __syncwarp();
    if (lane == 0) {
      idx[static_cast<size_t>(t) * k + j] = e;
      w[static_cast<size_t>(t) * k + j] = s_score[e] * scale;
      s_choice[e] = -INFINITY;
      atomicAdd(&counts[e], 1);
    }
    __syncwarp();
  }
  if constexpr (kSoftmax) {
    for (int j = lane; j < k; j += 32) w[static_cast<size_t>(t) * k + j] /= chosen + 1e-20f;
  }
}

// Every CTA derives the padded start of each expert from the counts, then places a share of the (token, choice) pairs and copies
// their rows (vec: 16-byte units per row, or 0 for `row_bytes` single bytes / 2).  cursor[e]: pairs of expert e placed so far.
__global__ void __launch_bounds__(256)
dispatch_kernel(const int* __restrict__ idx, const int* __restrict__ counts, int* __restrict__ cursor, int pairs, int k, int E, int block_rows,
                int blocks, const uint8_t* __restrict__ x, uint8_t* __restrict__ x_pad, int row_bytes, int vec, int* __restrict__ dest,
                int* __restrict__ tile_group) {
  __shared__ int s_off[kMaxExperts + 1];
  __shared__ int s_warp[8];
  // exclusive prefix sum of the padded counts, 256 experts at a time
  int base = 0;
  for (int e0 = 0; e0 < E; e0 += 256) {
    const int e = e0 + threadIdx.x;
    const int v = e < E ? (counts[e] + block_rows - 1) / block_rows * block_rows : 0;
    int inc = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, inc, o);
      if ((threadIdx.x & 31) >= o) inc += u;
    }
    if ((threadIdx.x & 31) == 31) s_warp[threadIdx.x >> 5] = inc;
    __syncthreads();
    int add = base;
    for (int i = 0; i < static_cast<int>(threadIdx.x >> 5); ++i) add += s_warp[i];
    if (e < E) s_off[e] = add + inc - v;
    for (int i = 0; i < 8; ++i) base += s_warp[i];
    __syncthreads();
  }
  if (threadIdx.x == 0) s_off[E] = base;
  __syncthreads();
  // expert of every row block: the last expert whose start is not beyond it
  for (int b = blockIdx.x * blockDim.x + threadIdx.x; b < blocks; b += gridDim.x * blockDim.x) {
    const int row = b * block_rows;
    int g = -1;
    if (row < s_off[E]) {
      int lo = 0, hi = E - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (s_off[mid] <= row) lo = mid; else hi = mid - 1;
      }
      g = lo;
    }
    tile_group[b] = g;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = blockIdx.x * 8 + warp; i < pairs; i += gridDim.x * 8) {
    const int e = idx[i];
    int d = -1;
    if (e >= 0) {
      if (lane == 0) d = s_off[e] + atomicAdd(&cursor[e], 1);
      d = __shfl_sync(0xffffffffu, d, 0);
    }
    if (lane == 0) dest[i] = d;
    if (d < 0) continue;
    const uint8_t* src = x + static_cast<size_t>(i / k) * row_bytes;
    uint8_t* dst = x_pad + static_cast<size_t>(d) * row_bytes;
    if (vec) {
      for (int c = lane; c < row_bytes / 16; c += 32) reinterpret_cast<uint4*>(dst)[c] = __ldg(reinterpret_cast<const uint4*>(src) + c);
    } else {
      for (int c = lane; c < row_bytes / 2; c += 32) reinterpret_cast<uint16_t*>(dst)[c] = reinterpret_cast<const uint16_t*>(src)[c];
    }
  }
}

// stream[t, :] += sum_j w[t, j] * y[dest[t, j], :]
__global__ void __launch_bounds__(256)
combine_kernel(const void* __restrict__ y, int y_f32, const int* __restrict__ dest, const float* __restrict__ w, int k, int dim,
               float* __restrict__ stream, int vec) {
  const int t = blockIdx.x;
  const int* d = dest + static_cast<size_t>(t) * k;
  const float* wt = w + static_cast<size_t>(t) * k;
  float* out = stream + static_cast<size_t>(t) * dim;
  if (vec) {  // bf16, dim a multiple of 8
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8; c < dim; c += gridDim.y * blockDim.x * 8) {
      float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      for (int j = 0; j < k; ++j) {
        const int r = d[j];
        if (r < 0) continue;
        const float f = wt[j];
        const uint4 u = __ldg(reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(y) + static_cast<size_t>(r) * dim + c));
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float2 v = __bfloat1622float2(h[q]);
          acc[2 * q] = fmaf(f, v.x, acc[2 * q]);
          acc[2 * q + 1] = fmaf(f, v.y, acc[2 * q + 1]);
        }
      }
      float4* o = reinterpret_cast<float4*>(out + c);
      float4 a = o[0], b = o[1];
      a.x += acc[0]; a.y += acc[1]; a.z += acc[2]; a.w += acc[3];
      b.x += acc[4]; b.y += acc[5]; b.z += acc[6]; b.w += acc[7];
      o[0] = a;
      o[1] = b;
    }
  } else {
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < dim; c += gridDim.y * blockDim.x) {
      float acc = 0.f;
      for (int j = 0; j < k; ++j)
        if (d[j] >= 0) acc = fmaf(wt[j], ldv(y, y_f32, static_cast<size_t>(d[j]) * dim + c), acc);
      out[c] += acc;
    }
  }
}

// C[Tp, N] = A[Tp, K] B[g][N, K]^T (squared relu if asked) with g = tile_group[row block of 64], fp32 FMA; blocks with g < 0 are skipped.
constexpr int kTile = 64, kDepth = 16;
template <typename T>
__global__ void __launch_bounds__(256)
grouped_fma_kernel(const T* __restrict__ A, const T* __restrict__ B, T* __restrict__ C, const int* __restrict__ tile_group, int N, int K,
                   int sq_relu) {
  __shared__ float s_a[kDepth][kTile + 4], s_b[kDepth][kTile + 4];
  const int g = tile_group[blockIdx.y];
  if (g < 0) return;
  const int m0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
  const T* Bg = B + static_cast<size_t>(g) * N * K;
  const int ty = threadIdx.x / 16, tx = threadIdx.x % 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kDepth) {
    for (int i = threadIdx.x; i < kTile * kDepth; i += 256) {
      const int r = i / kDepth, c = i % kDepth;
      const bool in_k = k0 + c < K;
      s_a[c][r] = in_k ? static_cast<float>(A[static_cast<size_t>(m0 + r) * K + k0 + c]) : 0.f;
      s_b[c][r] = in_k && n0 + r < N ? static_cast<float>(Bg[static_cast<size_t>(n0 + r) * K + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kDepth; ++c) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = s_a[c][ty * 4 + i]; b[i] = s_b[c][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = n0 + tx * 4 + j;
      float v = acc[i][j];
      if (sq_relu) { v = fmaxf(v, 0.f); v *= v; }
      if (col < N) C[static_cast<size_t>(m0 + ty * 4 + i) * N + col] = static_cast<T>(v);
    }
}

}  // namespace experts
}  // namespace lvb

// Routing of z [T, E] fp32 (row stride ldz).  kind 0: choice score sigmoid(z) + correction (optional, fp32 or bf16 [E]); groups > 1: only
// experts of the `keep` neighbour groups (E / groups experts each) with the largest sum of their two best choice scores can be
// chosen; idx, w [T, k]: the k best choice scores, best first, and scale * sigmoid(z) of each.  kind 1: the softmax of z + correction, groups by
// their best choice score, weights softmax(z) / (sum over the chosen + 1e-20).  live (optional) [T]: tokens with a value outside
// [0, live_limit) are padding and get idx = -1.  counts: int32 [2 * E], cleared here; the first E receive the tokens per expert, the
// rest are lvb_moe_dispatch's cursors.
extern "C" int lvb_moe_route_grouped(int kind, const float* z, long long ldz, const void* correction, int c_f32, const int* live, int live_limit, int T,
                                     int E, int k, int groups, int keep, float scale, int* idx, float* w, int* counts, void* stream) {
  using namespace lvb;
  using namespace lvb::experts;
  if (T <= 0 || E <= 0 || E > kMaxExperts || k <= 0 || k > E || groups <= 0 || E % groups != 0 || keep <= 0 || keep > groups ||
      static_cast<long long>(keep) * (E / groups) < k)
    return kErrBadArg;
  const size_t smem = static_cast<size_t>(kRouteWarps) * (2 * E + groups) * 4;
  if (smem > 48 * 1024) return kErrTooLarge;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (cudaMemsetAsync(counts, 0, 2 * static_cast<size_t>(E) * sizeof(int), s) != cudaSuccess) return kErrCuda;
  auto kern = kind == 1 ? route_kernel<true> : route_kernel<false>;
  kern<<<(T + kRouteWarps - 1) / kRouteWarps, kRouteWarps * 32, smem, s>>>(z, ldz, correction, c_f32, live, live_limit, T, E, k, groups, keep, scale,
                                                                          idx, w, counts);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// Places the pairs of idx [T, k] in a buffer of `blocks` blocks of block_rows rows (at least T * k + min(E, T * k) * (block_rows - 1) rows) and copies
// the rows x [T, row_bytes] there.  dest [T, k]: row of every pair (-1: none); tile_group [blocks]: expert of every block (-1: unused).
// Rows of the buffer that no pair owns keep what they held.
extern "C" int lvb_moe_dispatch(const int* idx, int* counts, int T, int k, int E, int block_rows, int blocks, const void* x, void* x_pad,
                                int row_bytes, int* dest, int* tile_group, void* stream) {
  using namespace lvb;
  using namespace lvb::experts;
  if (T <= 0 || k <= 0 || E <= 0 || E > kMaxExperts || block_rows <= 0 || row_bytes <= 0 || (row_bytes & 1)) return kErrBadArg;
  if (static_cast<long long>(blocks) * block_rows < static_cast<long long>(T) * k + static_cast<long long>(E < T * k ? E : T * k) * (block_rows - 1))
    return kErrBadArg;
  const int pairs = T * k;
  const int vec = (row_bytes & 15) == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(x_pad)) & 15) == 0;
  int grid = (pairs + 7) / 8;
  if (grid > 8 * num_sms()) grid = 8 * num_sms();
  dispatch_kernel<<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(idx, counts, counts + E, pairs, k, E, block_rows, blocks,
                                                                          reinterpret_cast<const uint8_t*>(x), reinterpret_cast<uint8_t*>(x_pad),
                                                                          row_bytes, vec, dest, tile_group);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

extern "C" int lvb_moe_combine(const void* y, int y_f32, const int* dest, const float* w, int T, int k, int dim, float* out, void* stream) {
  using namespace lvb;
  using namespace lvb::experts;
  if (T <= 0 || k <= 0 || dim <= 0) return kErrBadArg;
  const int vec = !y_f32 && (dim & 7) == 0 && ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int per = vec ? 8 : 1;
  const int threads = dim / per >= 256 ? 256 : dim / per >= 128 ? 128 : 64;
  int gy = (dim / per + threads - 1) / threads;  // a token's columns over several CTAs when there are few tokens
  if (gy < 1) gy = 1;
  if (static_cast<long long>(T) * gy > 16LL * num_sms()) gy = 1;
  combine_kernel<<<dim3(T, gy), threads, 0, reinterpret_cast<cudaStream_t>(stream)>>>(y, y_f32, dest, w, k, dim, out, vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// tile_group [Tp / 64]; A [Tp, K], B [groups, N, K], C [Tp, N], all contiguous and of one type.
extern "C" int lvb_grouped_fma(const void* A, const void* B, void* C, const int* tile_group, int Tp, int N, int K, int sq_relu, int is_f32,
                               void* stream) {
  using namespace lvb;
  using namespace lvb::experts;
  if (Tp <= 0 || Tp % kTile != 0 || Tp / kTile > 65535 || N <= 0 || K <= 0) return kErrBadArg;
  const dim3 grid((N + kTile - 1) / kTile, Tp / kTile);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (is_f32)
    grouped_fma_kernel<float><<<grid, 256, 0, s>>>(reinterpret_cast<const float*>(A), reinterpret_cast<const float*>(B),
                                                   reinterpret_cast<float*>(C), tile_group, N, K, sq_relu);
  else
    grouped_fma_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(reinterpret_cast<const __nv_bfloat16*>(A), reinterpret_cast<const __nv_bfloat16*>(B),
                                                           reinterpret_cast<__nv_bfloat16*>(C), tile_group, N, K, sq_relu);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
