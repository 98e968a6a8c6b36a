// What happens to the projections of an attention layer before attention reads them, in one pass over the packed rows of a step: rotary
// positions, per-head score temperatures, mixing of values with an earlier layer's, normalisation of a compressed key/value row,
// and the write into the paged cache.  One CTA per packed row; angles, norms and mixing are 32-bit arithmetic (this file is built
// without fast-math), storage is bf16 or fp32.
#include "common.cuh"

namespace lvb {
namespace prep {

constexpr int kThreads = 128;

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// Eight consecutive elements, 16-byte aligned (32 bytes of fp32).
template <typename T> struct Vec8;
template <> struct Vec8<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* f) {
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&w);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 a = __bfloat1622float2(h[i]);
      f[2 * i] = a.x;
      f[2 * i + 1] = a.y;
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* f) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  }
};
template <> struct Vec8<float> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
  }
};

struct Rotation {
  const float* inv_freq;  // [dims / 2]; null: no rotation
  int dims;               // rotated dimensions, the first ones of a head
  int interleaved;        // pair i is (2i, 2i + 1), else (i, i + dims / 2)
  float pos_scale, magnitude;
};

// cos and sin of the row's angles into shared memory [dims / 2] each
__device__ __forceinline__ void fill_angles(const Rotation& r, int pos, float* s_cos, float* s_sin) {
  for (int i = threadIdx.x; i < r.dims / 2; i += kThreads) {
    const float a = (static_cast<float>(pos) * r.pos_scale) * r.inv_freq[i];
    float sn, cs;
    sincosf(a, &sn, &cs);
    s_cos[i] = cs * r.magnitude;
    s_sin[i] = sn * r.magnitude;
  }
}

// Rotate (and scale) `heads` rows of `size` elements at src, writing to dst and, when given, to dst2; the head strides are in
// elements, and at dst2 `maps2` heads lie side by side within one stride.  Elements past r.dims pass (scaled).  head_scale: optional factor per head.  `vec`: sizes and strides are multiples
// of 8, pointers aligned and pairs fall into whole groups of 8.
template <typename T>
__device__ __forceinline__ void rotate_heads(const T* src, long long src_stride, T* dst, long long dst_stride, T* dst2, long long dst2_stride,
                                             int maps2, int heads, int size, const Rotation& r, const float* s_cos, const float* s_sin,
                                             const void* head_scale, int scale_f32, bool vec) {
  auto factor = [&](int h) -> float {
    if (head_scale == nullptr) return 1.f;
    return scale_f32 ? reinterpret_cast<const float*>(head_scale)[h] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(head_scale)[h]);
  };
  const int dims = r.inv_freq != nullptr ? r.dims : 0, half = dims / 2;
  auto second = [&](int h) { return dst2 + (maps2 == 1 ? h * dst2_stride : h / maps2 * dst2_stride + h % maps2 * size); };
  if (vec) {
    // units of 8 elements: half / 8 pair units of two groups each (or dims / 8 units of interleaved pairs), then the rest
    const int turn = r.interleaved ? dims / 8 : half / 8, units = turn + (size - dims) / 8;
    for (int i = threadIdx.x; i < heads * units; i += kThreads) {
      const int h = i / units, u = i - h * units;
      const float f = factor(h);
      const T* s = src + h * src_stride;
      T* d = dst + h * dst_stride;
      T* d2 = dst2 != nullptr ? second(h) : nullptr;
      float a[8];
      if (u < turn && !r.interleaved) {
        float b[8], x[8], y[8];
        const int c = u * 8;
        Vec8<T>::load(s + c, a);
        Vec8<T>::load(s + c + half, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          x[j] = (a[j] * s_cos[c + j] - b[j] * s_sin[c + j]) * f;
          y[j] = (b[j] * s_cos[c + j] + a[j] * s_sin[c + j]) * f;
        }
        Vec8<T>::store(d + c, x);
        Vec8<T>::store(d + c + half, y);
        if (d2 != nullptr) {
          Vec8<T>::store(d2 + c, x);
          Vec8<T>::store(d2 + c + half, y);
        }
        continue;
      }
      const int c = u < turn ? u * 8 : dims + (u - turn) * 8;
      Vec8<T>::load(s + c, a);
      if (u < turn) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float cs = s_cos[u * 4 + j], sn = s_sin[u * 4 + j], lo = a[2 * j], hi = a[2 * j + 1];
          a[2 * j] = lo * cs - hi * sn;
          a[2 * j + 1] = hi * cs + lo * sn;
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= f;
      Vec8<T>::store(d + c, a);
      if (d2 != nullptr) Vec8<T>::store(d2 + c, a);
    }
    return;
  }
  const int units = half + size - dims;  // a pair, or one element of the rest
  for (int i = threadIdx.x; i < heads * units; i += kThreads) {
    const int h = i / units, u = i - h * units;
    const float f = factor(h);
    const T* s = src + h * src_stride;
    if (u < half) {
      const int lo = r.interleaved ? 2 * u : u, hi = r.interleaved ? 2 * u + 1 : u + half;
      const float a = to_f<T>(s[lo]), b = to_f<T>(s[hi]);
      const T x = from_f<T>((a * s_cos[u] - b * s_sin[u]) * f), y = from_f<T>((b * s_cos[u] + a * s_sin[u]) * f);
      dst[h * dst_stride + lo] = x;
      dst[h * dst_stride + hi] = y;
      if (dst2 != nullptr) {
        second(h)[lo] = x;
        second(h)[hi] = y;
      }
    } else {
      const int c = dims + u - half;
      const T x = from_f<T>(to_f<T>(s[c]) * f);
      dst[h * dst_stride + c] = x;
      if (dst2 != nullptr) second(h)[c] = x;
    }
  }
}

struct QkvParams {
  void *q, *k, *v;          // rows with strides ldq, ldk, ldv; heads packed inside a row; updated in place
  const void* v_first;      // optional rows of an earlier layer's values: v <- (1 - mix) v + mix v_first
  const void* mix;          // one number
  const void* q_head_scale; // optional [H]
  void* kv_pages;           // [slots, KV, maps * dk + dv]
  const int *pos, *dests;
  int H, KV, maps, dk, dv;  // maps: keys per KV head; k has KV * maps heads
  long long ldq, ldk, ldv, ldf, slots;
  Rotation rot;
  int small_f32;            // type of mix and q_head_scale
  int vec;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) qkv_prep_kernel(QkvParams p) {
  extern __shared__ float s_angles[];
  const int half = p.rot.inv_freq != nullptr ? p.rot.dims / 2 : 0;
  float* s_cos = s_angles;
  float* s_sin = s_angles + half;
  const int t = blockIdx.x;
  if (half > 0) {
    fill_angles(p.rot, p.pos[t], s_cos, s_sin);
    __syncthreads();
  }
  const long long dest = p.dests[t];
  const bool live = dest >= 0 && dest < p.slots;
  const int keys = p.maps * p.dk, per = keys + p.dv;
  T* cache = live ? reinterpret_cast<T*>(p.kv_pages) + dest * p.KV * per : nullptr;
  T* q = reinterpret_cast<T*>(p.q) + t * p.ldq;
  T* k = reinterpret_cast<T*>(p.k) + t * p.ldk;
  T* v = reinterpret_cast<T*>(p.v) + t * p.ldv;
  if (half > 0 || p.q_head_scale != nullptr) {
    rotate_heads<T>(q, p.dk, q, p.dk, static_cast<T*>(nullptr), 0, 1, p.H, p.dk, p.rot, s_cos, s_sin, p.q_head_scale, p.small_f32, p.vec != 0);
  }
  if (half > 0 || live) rotate_heads<T>(k, p.dk, k, p.dk, cache, per, p.maps, p.KV * p.maps, p.dk, p.rot, s_cos, s_sin, nullptr, 0, p.vec != 0);
  const T* first = p.v_first != nullptr ? reinterpret_cast<const T*>(p.v_first) + t * p.ldf : nullptr;
  float lam = 0.f;
  if (first != nullptr) lam = p.small_f32 ? *reinterpret_cast<const float*>(p.mix) : __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(p.mix));
  if (first == nullptr && cache == nullptr) return;
  if (p.vec) {
    for (int i = threadIdx.x; i < p.KV * p.dv / 8; i += kThreads) {
      const int e = i * 8, h = e / p.dv, c = e - h * p.dv;
      float a[8];
      Vec8<T>::load(v + e, a);
      if (first != nullptr) {
        float b[8];
        Vec8<T>::load(first + e, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] = (1.f - lam) * a[j] + lam * b[j];
        Vec8<T>::store(v + e, a);
      }
      if (cache != nullptr) Vec8<T>::store(cache + h * per + keys + c, a);
    }
    return;
  }
  for (int e = threadIdx.x; e < p.KV * p.dv; e += kThreads) {
    const int h = e / p.dv, c = e - h * p.dv;
    float a = to_f<T>(v[e]);
    if (first != nullptr) {
      a = (1.f - lam) * a + lam * to_f<T>(first[e]);
      v[e] = from_f<T>(a);
    }
    if (cache != nullptr) cache[h * per + keys + c] = from_f<T>(a);
  }
}

struct LatentParams {
  const void* down;   // rows [rank + rot] (stride ldd): the compressed row and the shared key part
  const void* norm_w; // [rank]
  void* latent;       // [T, rank + rot]: normed, rotated
  void* kv_pages;     // [slots, rank + rot]
  const void* q_rot;  // row t, head h at q_rot + t * ldq + h * q_head: rot elements
  void* q_out;        // ditto with ldo, o_head (may be q_rot itself)
  const int *pos, *dests;
  int H, rank, rotd;
  long long ldd, ldq, q_head, ldo, o_head, slots;
  float eps;
  Rotation rot;
  int w_f32, vec_c, vec_q;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) latent_prep_kernel(LatentParams p) {
  extern __shared__ float s_angles[];
  __shared__ float s_red[kThreads / 32];
  float* s_cos = s_angles;
  float* s_sin = s_angles + p.rot.dims / 2;
  const int t = blockIdx.x;
  fill_angles(p.rot, p.pos[t], s_cos, s_sin);
  if (p.down == nullptr) {  // the queries only
    __syncthreads();
    rotate_heads<T>(reinterpret_cast<const T*>(p.q_rot) + t * p.ldq, p.q_head, reinterpret_cast<T*>(p.q_out) + t * p.ldo, p.o_head,
                    static_cast<T*>(nullptr), 0, 1, p.H, p.rotd, p.rot, s_cos, s_sin, nullptr, 0, p.vec_q != 0);
    return;
  }
  const long long dest = p.dests[t];
  const int width = p.rank + p.rotd;
  T* cache = dest >= 0 && dest < p.slots ? reinterpret_cast<T*>(p.kv_pages) + dest * width : nullptr;
  const T* down = reinterpret_cast<const T*>(p.down) + t * p.ldd;
  T* latent = reinterpret_cast<T*>(p.latent) + static_cast<long long>(t) * width;
  float ss = 0.f;
  if (p.vec_c) {
    for (int c = threadIdx.x * 8; c < p.rank; c += kThreads * 8) {
      float a[8];
      Vec8<T>::load(down + c, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(a[j], a[j], ss);
    }
  } else {
    for (int c = threadIdx.x; c < p.rank; c += kThreads) {
      const float a = to_f<T>(down[c]);
      ss = fmaf(a, a, ss);
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = ss;
  __syncthreads();  // also: the angles are in place
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) ss += s_red[i];
  const float r = 1.f / sqrtf(ss / static_cast<float>(p.rank) + p.eps);
  auto weight = [&](int c) -> float {
    return p.w_f32 ? reinterpret_cast<const float*>(p.norm_w)[c] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.norm_w)[c]);
  };
  if (p.vec_c) {
    for (int c = threadIdx.x * 8; c < p.rank; c += kThreads * 8) {
      float a[8];
      Vec8<T>::load(down + c, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= r * weight(c + j);
      Vec8<T>::store(latent + c, a);
      if (cache != nullptr) Vec8<T>::store(cache + c, a);
    }
  } else {
    for (int c = threadIdx.x; c < p.rank; c += kThreads) {
      const T a = from_f<T>(to_f<T>(down[c]) * (r * weight(c)));
      latent[c] = a;
      if (cache != nullptr) cache[c] = a;
    }
  }
  rotate_heads<T>(down + p.rank, 0, latent + p.rank, 0, cache != nullptr ? cache + p.rank : nullptr, 0, 1, 1, p.rotd, p.rot, s_cos, s_sin, nullptr, 0,
                  p.vec_c != 0 && p.vec_q != 0);
  rotate_heads<T>(reinterpret_cast<const T*>(p.q_rot) + t * p.ldq, p.q_head, reinterpret_cast<T*>(p.q_out) + t * p.ldo, p.o_head,
                  static_cast<T*>(nullptr), 0, 1, p.H, p.rotd, p.rot, s_cos, s_sin, nullptr, 0, p.vec_q != 0);
}

// latent_prep without a rotated part: the norm and the cache write, a warp per row, the row in registers.  latent may be null.
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_norm_kernel(LatentParams p, int rows) {
  constexpr int kKeep = 4;  // groups of 8 columns per lane in registers
  const int t = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= rows) return;
  const long long dest = p.dests != nullptr ? p.dests[t] : -1;
  T* cache = dest >= 0 && dest < p.slots ? reinterpret_cast<T*>(p.kv_pages) + dest * p.rank : nullptr;
  const T* down = reinterpret_cast<const T*>(p.down) + t * p.ldd;
  T* latent = p.latent != nullptr ? reinterpret_cast<T*>(p.latent) + static_cast<long long>(t) * p.rank : nullptr;
  auto weight = [&](int c) -> float {
    return p.w_f32 ? reinterpret_cast<const float*>(p.norm_w)[c] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.norm_w)[c]);
  };
  auto scale = [&](float ss) { return 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.rank) + p.eps); };
  float ss = 0.f;
  if (p.vec_c && p.rank <= kKeep * 256) {
    float a[kKeep][8];
#pragma unroll
    for (int n = 0; n < kKeep; ++n) {
      const int c = n * 256 + lane * 8;
      if (c < p.rank) Vec8<T>::load(down + c, a[n]);
      else
#pragma unroll
        for (int j = 0; j < 8; ++j) a[n][j] = 0.f;
    }
#pragma unroll
    for (int n = 0; n < kKeep; ++n)
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(a[n][j], a[n][j], ss);
    const float r = scale(ss);
#pragma unroll
    for (int n = 0; n < kKeep; ++n) {
      const int c = n * 256 + lane * 8;
      if (c >= p.rank) continue;
#pragma unroll
      for (int j = 0; j < 8; ++j) a[n][j] *= r * weight(c + j);
      if (latent != nullptr) Vec8<T>::store(latent + c, a[n]);
      if (cache != nullptr) Vec8<T>::store(cache + c, a[n]);
    }
    return;
  }
  if (p.vec_c) {  // the second read comes from L1
    for (int c = lane * 8; c < p.rank; c += 256) {
      float a[8];
      Vec8<T>::load(down + c, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(a[j], a[j], ss);
    }
    const float r = scale(ss);
    for (int c = lane * 8; c < p.rank; c += 256) {
      float a[8];
      Vec8<T>::load(down + c, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= r * weight(c + j);
      if (latent != nullptr) Vec8<T>::store(latent + c, a);
      if (cache != nullptr) Vec8<T>::store(cache + c, a);
    }
    return;
  }
  for (int c = lane; c < p.rank; c += 32) {
    const float a = to_f<T>(down[c]);
    ss = fmaf(a, a, ss);
  }
  const float r = scale(ss);
  for (int c = lane; c < p.rank; c += 32) {
    const T a = from_f<T>(to_f<T>(down[c]) * (r * weight(c)));
    if (latent != nullptr) latent[c] = a;
    if (cache != nullptr) cache[c] = a;
  }
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// whether a rotation falls into whole groups of 8 elements
inline bool groups_of_8(const float* inv_freq, int dims, int interleaved) {
  return inv_freq == nullptr || (interleaved ? (dims & 7) == 0 : (dims & 15) == 0);
}

}  // namespace prep
}  // namespace lvb

// Rows of q [T, H, dk], k [T, KV * maps, dk], v [T, KV, dv] (row strides ldq, ldk, ldv), in place:
//   q, k: the first rot_dims dimensions of each head rotated by pos[t] * pos_scale * inv_freq[i] (pairs as `interleaved` says; inv_freq
//         null: no rotation), q multiplied by q_head_scale[h] when given;
//   v:    (1 - mix) v + mix v_first[t] when v_first is given;
// and k, v written to flat slots dests[t] of kv_pages [slots, KV, maps * dk + dv] (out-of-range slots are skipped).  is_f32: type of the rows and the
// cache; small_f32: type of mix and q_head_scale.
extern "C" int lvb_qkv_prep(void* q, void* k, void* v, const void* v_first, const void* mix, const void* q_head_scale, void* kv_pages,
                            const int* pos, const int* dests, int T, int H, int KV, int maps, int dk, int dv, long long ldq, long long ldk,
                            long long ldv, long long ldf, long long slots, const float* inv_freq, int rot_dims, int interleaved,
                            float pos_scale, float magnitude, int is_f32, int small_f32, void* stream) {
  using namespace lvb;
  using namespace lvb::prep;
  if (T <= 0) return kErrOk;
  if (H <= 0 || KV <= 0 || maps <= 0 || dk <= 0 || dv <= 0 || rot_dims < 0 || rot_dims > dk || (rot_dims & 1)) return kErrBadArg;
  if (inv_freq != nullptr && (rot_dims == 0 || pos == nullptr)) return kErrBadArg;
  if (v_first != nullptr && mix == nullptr) return kErrBadArg;
  if (rot_dims > 4096) return kErrTooLarge;
  QkvParams p;
  p.q = q; p.k = k; p.v = v; p.v_first = v_first; p.mix = mix; p.q_head_scale = q_head_scale; p.kv_pages = kv_pages; p.pos = pos; p.dests = dests;
  p.H = H; p.KV = KV; p.maps = maps; p.dk = dk; p.dv = dv; p.ldq = ldq; p.ldk = ldk; p.ldv = ldv; p.ldf = ldf; p.slots = slots;
  p.rot = Rotation{inv_freq, inv_freq != nullptr ? rot_dims : 0, interleaved, pos_scale, magnitude};
  p.small_f32 = small_f32;
  p.vec = ((dk | dv | ldq | ldk | ldv) & 7) == 0 && (v_first == nullptr || ((ldf & 7) == 0 && aligned16(v_first))) && aligned16(q) && aligned16(k) &&
          aligned16(v) && aligned16(kv_pages) && groups_of_8(inv_freq, p.rot.dims, interleaved);
  const size_t smem = static_cast<size_t>(p.rot.dims) * 4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (is_f32) qkv_prep_kernel<float><<<T, kThreads, smem, s>>>(p);
  else qkv_prep_kernel<__nv_bfloat16><<<T, kThreads, smem, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// Latent attention.  Row t of down (stride ldd) holds `rank` compressed dimensions and a key part of rot_dims dimensions shared by the
// heads.  latent[t] = [RMS norm of the former with weight norm_w, the latter rotated], also written to slot dests[t] of kv_pages [slots,
// rank + rot_dims]; head h's rotated query part goes from q_rot + t * ldq + h * q_head to q_out + t * ldo + h * o_head.  rot_dims 0: the norm and
// the cache write only; latent may be null then, or dests (no cache write).  down null: the rotation of the queries only.
extern "C" int lvb_latent_prep(const void* down, const void* norm_w, void* latent, void* kv_pages, const void* q_rot, void* q_out, const int* pos,
                               const int* dests, int T, int H, int rank, int rot_dims, long long ldd, long long ldq, long long q_head,
                               long long ldo, long long o_head, long long slots, float eps, const float* inv_freq, int interleaved,
                               float pos_scale, float magnitude, int is_f32, int w_f32, void* stream) {
  using namespace lvb;
  using namespace lvb::prep;
  if (T <= 0) return kErrOk;
  if (H <= 0 || rot_dims < 0 || (rot_dims & 1)) return kErrBadArg;
  if (down == nullptr ? rot_dims == 0 : rank <= 0 || (rot_dims > 0 && (latent == nullptr || dests == nullptr)) || (latent == nullptr && dests == nullptr))
    return kErrBadArg;
  if (rot_dims > 0 && (inv_freq == nullptr || pos == nullptr)) return kErrBadArg;
  if (rot_dims > 4096) return kErrTooLarge;
  LatentParams p;
  p.down = down; p.norm_w = norm_w; p.latent = latent; p.kv_pages = kv_pages; p.q_rot = q_rot; p.q_out = q_out; p.pos = pos; p.dests = dests;
  p.H = H; p.rank = rank; p.rotd = rot_dims; p.ldd = ldd; p.ldq = ldq; p.q_head = q_head; p.ldo = ldo; p.o_head = o_head; p.slots = slots;
  p.eps = eps;
  p.rot = Rotation{inv_freq, rot_dims, interleaved, pos_scale, magnitude};
  p.w_f32 = w_f32;
  p.vec_c = ((rank | rot_dims | ldd) & 7) == 0 && aligned16(down) && aligned16(latent) && aligned16(kv_pages);
  p.vec_q = ((rot_dims | ldq | q_head | ldo | o_head) & 7) == 0 && aligned16(q_rot) && aligned16(q_out) && groups_of_8(inv_freq, rot_dims, interleaved);
  const size_t smem = static_cast<size_t>(rot_dims) * 4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (rot_dims == 0) {
    const int per = kThreads / 32;
    if (is_f32) latent_norm_kernel<float><<<(T + per - 1) / per, kThreads, 0, s>>>(p, T);
    else latent_norm_kernel<__nv_bfloat16><<<(T + per - 1) / per, kThreads, 0, s>>>(p, T);
  } else if (is_f32) latent_prep_kernel<float><<<T, kThreads, smem, s>>>(p);
  else latent_prep_kernel<__nv_bfloat16><<<T, kThreads, smem, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
