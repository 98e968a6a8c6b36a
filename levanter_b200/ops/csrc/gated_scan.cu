// The minimal gated recurrence of minGRU layers over packed rows, with a state per sequence slot:
//   z = sigmoid(zl), c = u + 1/2 for u >= 0 and sigmoid(u) below, S <- (1 - z) S + z c, out = S * silu(g).
// All arithmetic and the state are 32-bit (this file is built without fast-math; the gates come straight from the projections'
// accumulators).  A sequence whose first packed row is at position 0 starts from zero, any other from its slot's state; the state
// after the last row goes back to the slot.  Sequence boundaries, lengths and slots are read from device arrays.
//
// The recurrence is linear in S, so the wide kernel cuts time as well: a CTA owns 32 channels of one sequence and walks it in tiles of
// kGroups * kRows rows.  A thread composes the kRows steps of its channel into one affine map, the maps of the groups before it
// are applied to the tile's incoming state, and the steps are then replayed from there; the next tile's rows are already on
// their way into registers.  The narrow kernel (decode rounds: about a row per sequence) is one thread per channel.
#include "common.cuh"

namespace lvb {
namespace gscan {

constexpr int kGroups = 16;
constexpr int kRows = 4;
constexpr int kChannels = 32;
constexpr int kTile = kGroups * kRows;

struct Params {
  const float *z, *u, *g;  // [T, width] each, row stride ld
  void* out;               // [T, width]
  float* state;            // [slots, width]
  const int *slot_ids, *kv_lens, *cu_q_lens, *num_seqs;
  long long ld;
  int T, width, S, slots;
};

__device__ __forceinline__ void store1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void store1(float* p, float v) { *p = v; }

// sigmoid(x) and 1 - sigmoid(x) without cancellation
__device__ __forceinline__ void sigmoid2(float x, float& s, float& rest) {
  const float e = expf(-fabsf(x));
  const float r = __fdividef(1.f, 1.f + e);
  s = x >= 0.f ? r : e * r;
  rest = x >= 0.f ? e * r : r;
}

__device__ __forceinline__ void step_of(float zl, float u, float& a, float& b) {
  float z;
  sigmoid2(zl, z, a);
  float lo, rest;
  sigmoid2(fminf(u, 0.f), lo, rest);
  b = z * (u >= 0.f ? u + 0.5f : lo);
}

__device__ __forceinline__ float silu(float g) {
  float s, rest;
  sigmoid2(g, s, rest);
  return g * s;
}

// Rows of sequence i, and whether it continues from its slot.  False: nothing to do.
__device__ __forceinline__ bool sequence(const Params& p, int i, int& r0, int& r1, int& slot, bool& from_state) {
  int n = p.num_seqs[0];
  n = n < p.S ? n : p.S;
  if (i >= n) return false;
  r0 = p.cu_q_lens[i];
  r1 = p.cu_q_lens[i + 1];
  r0 = r0 < 0 ? 0 : r0;
  r1 = r1 < p.T ? r1 : p.T;
  slot = p.slot_ids[i];
  from_state = p.kv_lens[i] > r1 - r0;
  return r1 > r0 && slot >= 0 && slot < p.slots;
}

// Padding rows come after the last sequence: zeros.
template <typename T>
__device__ __forceinline__ void zero_padding(const Params& p, int c, int row0, int row_step) {
  int n = p.num_seqs[0];
  n = n < p.S ? n : p.S;
  int r = n > 0 ? p.cu_q_lens[n] : 0;
  if (c >= p.width) return;
  for (r += row0; r < p.T; r += row_step) store1(reinterpret_cast<T*>(p.out) + static_cast<long long>(r) * p.width + c, 0.f);
}

template <typename T>
__global__ void __launch_bounds__(128) narrow_kernel(Params p) {
  const int c = blockIdx.x * 128 + threadIdx.x, i = blockIdx.y;
  if (i == p.S) return zero_padding<T>(p, c, 0, 1);
  int r0, r1, slot;
  bool from_state;
  if (!sequence(p, i, r0, r1, slot, from_state) || c >= p.width) return;
  float* st = p.state + static_cast<long long>(slot) * p.width + c;
  float s = from_state ? *st : 0.f;
  for (int r = r0; r < r1; ++r) {
    const long long at = r * p.ld + c;
    float a, b;
    step_of(p.z[at], p.u[at], a, b);
    s = a * s + b;
    store1(reinterpret_cast<T*>(p.out) + static_cast<long long>(r) * p.width + c, s * silu(p.g[at]));
  }
  *st = s;
}

template <typename T>
__global__ void __launch_bounds__(kGroups * kChannels, 2) wide_kernel(Params p) {
  __shared__ float s_a[2][kGroups][kChannels], s_b[2][kGroups][kChannels];
  __shared__ float s_carry[2][kChannels];
  const int lane = threadIdx.x & 31, grp = threadIdx.x >> 5;
  const int c = blockIdx.x * kChannels + lane, i = blockIdx.y;
  if (i == p.S) return zero_padding<T>(p, c, grp, kGroups);
  int r0, r1, slot;
  bool from_state;
  if (!sequence(p, i, r0, r1, slot, from_state)) return;
  const bool in = c < p.width;
  float* st = p.state + static_cast<long long>(slot) * p.width + c;
  if (grp == 0) s_carry[0][lane] = from_state && in ? *st : 0.f;
  float z[kRows], u[kRows], g[kRows];
  auto load = [&](int base) {
#pragma unroll
    for (int j = 0; j < kRows; ++j) {
      const int r = base + grp * kRows + j;
      const bool ok = in && r < r1;
      const long long at = r * p.ld + c;
      z[j] = ok ? p.z[at] : 0.f;
      u[j] = ok ? p.u[at] : 0.f;
      g[j] = ok ? p.g[at] : 0.f;
    }
  };
  load(r0);
  int buf = 0;
  for (int base = r0; base < r1; base += kTile, buf ^= 1) {
    float a[kRows], b[kRows], w[kRows];
    float ca = 1.f, cb = 0.f;
#pragma unroll
    for (int j = 0; j < kRows; ++j) {
      step_of(z[j], u[j], a[j], b[j]);
      if (base + grp * kRows + j >= r1) {  // past the end: the identity, so that the last state survives
        a[j] = 1.f;
        b[j] = 0.f;
      }
      cb = a[j] * cb + b[j];
      ca *= a[j];
      w[j] = silu(g[j]);
    }
    s_a[buf][grp][lane] = ca;
    s_b[buf][grp][lane] = cb;
    if (base + kTile < r1) load(base + kTile);
    __syncthreads();
    float s = s_carry[buf][lane];
    for (int k = 0; k < grp; ++k) s = s_a[buf][k][lane] * s + s_b[buf][k][lane];
#pragma unroll
    for (int j = 0; j < kRows; ++j) {
      const int r = base + grp * kRows + j;
      s = a[j] * s + b[j];
      if (in && r < r1) store1(reinterpret_cast<T*>(p.out) + static_cast<long long>(r) * p.width + c, s * w[j]);
    }
    if (grp == kGroups - 1) {
      s_carry[buf ^ 1][lane] = s;  // read after the next tile's barrier
      if (base + kTile >= r1 && in) *st = s;
    }
  }
}

}  // namespace gscan
}  // namespace lvb

// z, u, g: fp32 [T, width], row stride ld.  out [T, width] bf16 or fp32 (out_f32).  state fp32 [slots, width], row slot_ids[i] for the i-th of
// num_seqs[0] <= S packed sequences (rows cu_q_lens[i] .. cu_q_lens[i + 1], the last at position kv_lens[i] - 1).  Rows past the last sequence
// come out as zeros.  long_rows: sequences of many rows are expected (a hint, not a condition).
extern "C" int lvb_min_gru_scan(const float* z, const float* u, const float* g, void* out, float* state, const int* slot_ids, const int* kv_lens,
                                const int* cu_q_lens, const int* num_seqs, int T, int width, long long ld, int S, int slots, int out_f32,
                                int long_rows, void* stream) {
  using namespace lvb;
  using namespace lvb::gscan;
  if (T <= 0) return kErrOk;
  if (width <= 0 || S <= 0 || slots <= 0 || ld < width) return kErrBadArg;
  if (S >= 65535) return kErrTooLarge;
  Params p{z, u, g, out, state, slot_ids, kv_lens, cu_q_lens, num_seqs, ld, T, width, S, slots};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (long_rows) {
    const dim3 grid((width + kChannels - 1) / kChannels, S + 1);
    if (out_f32) wide_kernel<float><<<grid, kGroups * kChannels, 0, s>>>(p);
    else wide_kernel<__nv_bfloat16><<<grid, kGroups * kChannels, 0, s>>>(p);
  } else {
    const dim3 grid((width + 127) / 128, S + 1);
    if (out_f32) narrow_kernel<float><<<grid, 128, 0, s>>>(p);
    else narrow_kernel<__nv_bfloat16><<<grid, 128, 0, s>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
