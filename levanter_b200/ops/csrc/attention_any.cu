// Paged attention and cache writes without restrictions on the element type or the sizes: fp32 serving, and bf16 models whose
// head sizes the tensor-core kernels do not take (not a multiple of 8, above 256, more than 16 query heads per KV head).
//
// Same semantics as lvb_paged_attention_general (paged_attention.cu): packed query rows, pages, an optional chunk size or window, an
// optional output gate and the difference of two score maps; and of lvb_paged_latent (paged_latent.cu), where a key's first columns are
// its value and a sink per head may join the softmax denominator.  Everything is fp32 arithmetic whatever the storage type (this file is
// built without fast-math).  One CTA per (query row, query head or map of it) walks the visible keys in blocks: a key per thread for the
// scores, an online softmax over the block, then an output column per thread for P V.  Maps leave their results in fp32 for a second kernel.
#include "common.cuh"

namespace lvb {
namespace any {

constexpr int kThreads = 128;

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

template <typename T>
__global__ void kv_write_kernel(T* __restrict__ kv_pages, const T* __restrict__ k, const T* __restrict__ v, const int* __restrict__ dests,
                                int KV, int dk, int dv, long long ldk, long long ldv, long long total_slots) {
  const int t = blockIdx.x;
  const long long dest = dests[t];
  if (dest < 0 || dest >= total_slots) return;  // padding token
  const int per = dk + dv;
  T* out = kv_pages + dest * KV * per;
  for (int i = threadIdx.x; i < KV * per; i += blockDim.x) {
    const int h = i / per, c = i - h * per;
    out[i] = c < dk ? k[t * ldk + static_cast<long long>(h) * dk + c] : v[t * ldv + static_cast<long long>(h) * dv + (c - dk)];
  }
}

// 16-byte form of kv_write_kernel (bf16; sizes and strides multiples of 8)
__global__ void kv_write_vec_kernel(uint4* __restrict__ kv_pages, const uint4* __restrict__ k, const uint4* __restrict__ v,
                                    const int* __restrict__ dests, int KV, int dk8, int dv8, long long ldk8, long long ldv8,
                                    long long total_slots) {
  const int t = blockIdx.x;
  const long long dest = dests[t];
  if (dest < 0 || dest >= total_slots) return;
  const int per = dk8 + dv8;
  uint4* out = kv_pages + dest * KV * per;
  for (int i = threadIdx.x; i < KV * per; i += blockDim.x) {
    const int h = i / per, c = i - h * per;
    out[i] = c < dk8 ? k[t * ldk8 + h * dk8 + c] : v[t * ldv8 + h * dv8 + (c - dk8)];
  }
}

struct Params {
  const void* q;
  const void* kv_pages;  // [num_pages, page_size, KV, row]
  const int* kv_lens;
  const int* page_indices;
  const int* cu_q_lens;
  const int* num_seqs;
  const void* gate;
  const float* sink;     // optional [H]
  void* out;
  float* scratch;        // [T, H, dv] fp32: the maps' results
  int T, H, KV, dk, dv, S, pages_per_seq, page_size, num_pages, chunk, window;
  int row, v_at;         // elements of a KV head's row, and where in it the value starts
  long long ldq, ldg;
  float scale, soft_cap;
  int gate_per_head;     // the gate has one number per head instead of one per element
  const float* weight;   // with two maps (H counts both of every head): o = a1 - weight a2, then diff_scale * o / sqrt(mean(o^2) + eps)
  float diff_scale, eps;
};

// the sigmoid of the gate of element d of head h
template <typename T>
__device__ __forceinline__ float gate_factor(const Params& p, int t, int h, int d) {
  if (p.gate == nullptr) return 1.f;
  const long long at = p.gate_per_head ? h : static_cast<long long>(h) * p.dv + d;
  return 1.f / (1.f + expf(-to_f<T>(reinterpret_cast<const T*>(p.gate)[t * p.ldg + at])));
}

__device__ __forceinline__ float block_reduce(float v, float* s_red, bool is_max) {
  v = is_max ? warp_max(v) : warp_sum(v);
  if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = s_red[0];
  for (int w = 1; w < kThreads / 32; ++w) r = is_max ? fmaxf(r, s_red[w]) : r + s_red[w];
  __syncthreads();
  return r;
}

template <typename T>
__global__ void __launch_bounds__(kThreads) attention_any_kernel(Params p) {
  extern __shared__ float smem[];
  float* s_q = smem;                                   // [dk]
  float* s_o = s_q + p.dk;                             // [dv]
  float* s_p = s_o + p.dv;                             // [kThreads]
  int* s_slot = reinterpret_cast<int*>(s_p + kThreads);  // [kThreads]
  float* s_red = reinterpret_cast<float*>(s_slot + kThreads);
  const int t = blockIdx.x, h = blockIdx.y;
  const int kvh = h / (p.H / p.KV);
  const int k_at = p.weight != nullptr ? (h & 1) * p.dk : 0;  // where in a KV head's row this row's key starts
  const long long out_at = (static_cast<long long>(t) * p.H + h) * p.dv;
  auto store = [&](int d, float v) {
    if (p.weight != nullptr) p.scratch[out_at + d] = v;
    else reinterpret_cast<T*>(p.out)[out_at + d] = from_f<T>(v);
  };

  // which sequence owns row t, and its position in it
  int n = p.num_seqs[0];
  n = n < p.S ? n : p.S;
  int ctx = 0, seq = 0;
  if (n > 0 && t < p.cu_q_lens[n]) {
    while (seq < n && p.cu_q_lens[seq + 1] <= t) ++seq;
    const int kl = p.kv_lens[seq];
    if (kl > 0 && kl <= p.pages_per_seq * p.page_size) ctx = kl - p.cu_q_lens[seq + 1] + t + 1;
  }
  if (ctx <= 0) {
    for (int d = threadIdx.x; d < p.dv; d += kThreads) store(d, 0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.ldq + static_cast<long long>(h) * p.dk;
  for (int d = threadIdx.x; d < p.dk; d += kThreads) s_q[d] = to_f<T>(q[d]);
  for (int d = threadIdx.x; d < p.dv; d += kThreads) s_o[d] = 0.f;
  int lo = p.chunk > 0 ? ctx - 1 - (ctx - 1) % p.chunk : 0;
  if (p.window > 0) lo = max(lo, ctx - p.window);
  const long long per = p.row;
  const T* pages = reinterpret_cast<const T*>(p.kv_pages);
  float m = -INFINITY, l = 0.f;
  for (int k0 = lo; k0 < ctx; k0 += kThreads) {
    const int key = k0 + threadIdx.x;
    int slot = -1;
    if (key < ctx) {
      const int page = p.page_indices[seq * p.pages_per_seq + key / p.page_size];
      if (page >= 0 && page < p.num_pages) slot = page * p.page_size + key % p.page_size;
    }
    __syncthreads();  // s_q / s_o written; the previous block's s_p and s_slot have been read
    float s = -INFINITY;
    if (slot >= 0) {
      const T* kr = pages + (static_cast<long long>(slot) * p.KV + kvh) * per + k_at;
      float acc = 0.f;
      for (int d = 0; d < p.dk; ++d) acc = fmaf(s_q[d], to_f<T>(kr[d]), acc);
      s = acc * p.scale;
      if (p.soft_cap > 0.f) s = p.soft_cap * tanhf(s / p.soft_cap);
    }
    const float m_new = fmaxf(m, block_reduce(s, s_red, true));
    const float e = (s == -INFINITY) ? 0.f : expf(s - m_new);
    const float alpha = (m == -INFINITY) ? 0.f : expf(m - m_new);
    s_p[threadIdx.x] = e;
    s_slot[threadIdx.x] = slot;
    l = l * alpha + block_reduce(e, s_red, false);
    m = m_new;
    const int nk = min(kThreads, ctx - k0);
    for (int d = threadIdx.x; d < p.dv; d += kThreads) {
      float acc = s_o[d] * alpha;
      for (int i = 0; i < nk; ++i) {
        const int sl = s_slot[i];
        if (sl >= 0) acc = fmaf(s_p[i], to_f<T>(pages[(static_cast<long long>(sl) * p.KV + kvh) * per + p.v_at + d]), acc);
      }
      s_o[d] = acc;
    }
  }
  float shrink = 1.f;
  if (p.sink != nullptr) {  // one more column of the softmax, whose value is zero
    const float m_new = fmaxf(m, p.sink[h]);
    shrink = expf(m - m_new);
    l = l * shrink + expf(p.sink[h] - m_new);
  }
  const float inv = l > 0.f ? shrink / l : 0.f;
  for (int d = threadIdx.x; d < p.dv; d += kThreads) store(d, p.weight != nullptr ? s_o[d] * inv : s_o[d] * inv * gate_factor<T>(p, t, h, d));
}

// One CTA per (query row, head): the two maps' results to the head's output.
template <typename T>
__global__ void __launch_bounds__(kThreads) difference_kernel(Params p) {
  __shared__ float s_red[kThreads / 32];
  const int t = blockIdx.x, h = blockIdx.y;
  const float* a1 = p.scratch + (static_cast<long long>(t) * p.H + 2 * h) * p.dv;
  const float* a2 = a1 + p.dv;
  const float lam = *p.weight;
  float ss = 0.f;
  for (int d = threadIdx.x; d < p.dv; d += kThreads) {
    const float o = a1[d] - lam * a2[d];
    ss = fmaf(o, o, ss);
  }
  ss = block_reduce(ss, s_red, false);
  const float r = p.diff_scale / sqrtf(ss / static_cast<float>(p.dv) + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + (static_cast<long long>(t) * (p.H / 2) + h) * p.dv;
  for (int d = threadIdx.x; d < p.dv; d += kThreads) out[d] = from_f<T>((a1[d] - lam * a2[d]) * r * gate_factor<T>(p, t, h, d));
}

}  // namespace any
}  // namespace lvb

// Scatter k (row t, head h at k + t * ldk + h * dk) and v to flat slots dests[t] of kv_pages [slots, KV, dk + dv]; out-of-range slots are
// skipped.  is_f32: element type of all three.
extern "C" int lvb_kv_page_write_general(void* kv_pages, const void* k, const void* v, const int* dests, int T, int KV, int dk, int dv,
                                         long long ldk, long long ldv, long long total_slots, int is_f32, void* stream) {
  using namespace lvb;
  using namespace lvb::any;
  if (T <= 0) return kErrOk;
  if (KV <= 0 || dk <= 0 || dv <= 0) return kErrBadArg;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const uintptr_t mis = (reinterpret_cast<uintptr_t>(kv_pages) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15;
  if (is_f32) {
    kv_write_kernel<float><<<T, 128, 0, s>>>(reinterpret_cast<float*>(kv_pages), reinterpret_cast<const float*>(k),
                                             reinterpret_cast<const float*>(v), dests, KV, dk, dv, ldk, ldv, total_slots);
  } else if (mis == 0 && ((dk | dv | ldk | ldv) & 7) == 0) {
    kv_write_vec_kernel<<<T, 128, 0, s>>>(reinterpret_cast<uint4*>(kv_pages), reinterpret_cast<const uint4*>(k),
                                          reinterpret_cast<const uint4*>(v), dests, KV, dk / 8, dv / 8, ldk / 8, ldv / 8, total_slots);
  } else {
    kv_write_kernel<__nv_bfloat16><<<T, 128, 0, s>>>(reinterpret_cast<__nv_bfloat16*>(kv_pages), reinterpret_cast<const __nv_bfloat16*>(k),
                                                     reinterpret_cast<const __nv_bfloat16*>(v), dests, KV, dk, dv, ldk, ldv, total_slots);
  }
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// window > 0: a query sees itself and the window - 1 positions before it.  shared: a KV head's row holds dk elements only and its first dv are
// the value (dv <= dk).  sink: optional [H] fp32.  gate: [T, heads * dv], or [T, heads] with gate_per_head.  weight: one number on the device;
// rows 2h and 2h + 1 of q are then the maps of head h, a KV head's row holds two keys and a value, out is [T, H / 2, dv] and scratch fp32
// [T, H, dv].
extern "C" int lvb_attention_any(const void* q, const void* kv_pages, const int* kv_lens, const int* page_indices, const int* cu_q_lens,
                                 const int* num_seqs, const void* gate, const float* sink, void* out, float* scratch, int T, int H, int KV, int dk,
                                 int dv, long long ldq, long long ldg, int gate_per_head, int S, int pages_per_seq, int page_size,
                                 int num_pages, int chunk, int window, int shared, float scale, float soft_cap, const float* weight,
                                 float diff_scale, float eps, int is_f32, void* stream) {
  using namespace lvb;
  using namespace lvb::any;
  if (T <= 0) return kErrOk;
  if (H <= 0 || KV <= 0 || H % KV != 0 || dk <= 0 || dv <= 0 || S <= 0 || chunk < 0 || window < 0) return kErrBadArg;
  if (shared && (dv > dk || weight != nullptr)) return kErrBadArg;
  if (weight != nullptr && ((H / KV) % 2 != 0 || scratch == nullptr || sink != nullptr)) return kErrBadArg;
  const size_t smem = (static_cast<size_t>(dk) + dv + 2 * kThreads + kThreads / 32) * 4;
  if (smem > 48 * 1024) return kErrTooLarge;
  const int keys = weight != nullptr ? 2 * dk : dk;
  Params p{q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, gate, sink, out, scratch, T, H, KV, dk, dv, S, pages_per_seq, page_size, num_pages,
           chunk, window, shared ? dk : keys + dv, shared ? 0 : keys, ldq, ldg, scale, soft_cap, gate_per_head, weight, diff_scale, eps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (is_f32) attention_any_kernel<float><<<dim3(T, H), kThreads, smem, s>>>(p);
  else attention_any_kernel<__nv_bfloat16><<<dim3(T, H), kThreads, smem, s>>>(p);
  if (weight != nullptr && cudaGetLastError() == cudaSuccess) {
    if (is_f32) difference_kernel<float><<<dim3(T, H / 2), kThreads, 0, s>>>(p);
    else difference_kernel<__nv_bfloat16><<<dim3(T, H / 2), kThreads, 0, s>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
