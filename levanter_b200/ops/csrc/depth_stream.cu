// Between the blocks of a model that keeps what every layer has made of the residual stream: the weighted sum over depth that the next block
// starts from, its RMS norm in groups, and the token shift that mixes a normed row with the one before it.  One kernel does all three;
// each step can be left out.  Everything is 32-bit arithmetic (this file is built without fast-math).
//
// A CTA walks a few consecutive packed rows with the normed row before the present one in registers, so the shift reads nothing
// twice but for the row before its first.  The first row of a sequence looks back at the normed row that its slot holds (or at zeros, at
// position 0), and the CTA of that row also leaves the sequence's last normed row in the slot: one CTA reads and then writes the
// slot, whatever the number of rows.
#include "row_groups.cuh"

namespace lvb {
namespace depth {

struct Params {
  const float* hist;        // [planes][T][dim], `plane` elements apart
  long long plane;
  int planes;
  const void* coef;         // [planes]; null: the one plane as it is
  float* out;               // optional [T, dim]: the sum
  const long long* rows;    // optional gather (no shift, no out)
  const void *w, *mu;       // [dim] each; mu null: no shift
  int w_f32;
  float* state;             // [slots, dim]
  const int *slot_ids, *kv_lens, *cu_q_lens, *num_seqs;
  int S, slots;
  void* y;
  int y_f32, T, dim, part, per;
  float eps;
};

template <int kN, int kVec, int kThreads, bool kShift>
__global__ void __launch_bounds__(kThreads, kThreads <= 512 ? 3 : 1) depth_kernel(Params p) {
  using Row = rowg::Row<kN, kVec>;
  extern __shared__ float smem[];
  __shared__ int s_seq;
  const typename Row::Groups groups(p.dim, p.part);
  const int scratch = kN * blockDim.x + p.dim / p.part;
  float* s_coef = smem + 2 * scratch;
  for (int j = threadIdx.x; j < p.planes; j += blockDim.x) s_coef[j] = p.coef != nullptr ? rowg::ld1(p.coef, p.w_f32, j) : 1.f;
  const int r0 = blockIdx.x * p.per, r1 = min(r0 + p.per, p.T);
  int n_seq = 0;
  if constexpr (kShift) {
    if (threadIdx.x == 0) s_seq = -1;
    __syncthreads();
    n_seq = min(p.num_seqs[0], p.S);
    for (int i = threadIdx.x; i < n_seq; i += blockDim.x)
      if (p.cu_q_lens[i] <= r0 && r0 < p.cu_q_lens[i + 1]) s_seq = i;
  }
  __syncthreads();
  int turn = 0;
  // the normed row r; store: also its sum
  auto row_at = [&](int r, bool store, Row& x) {
    const size_t src = static_cast<size_t>(p.rows != nullptr ? p.rows[r] : r) * p.dim;
#pragma unroll
    for (int n = 0; n < kN; ++n)
#pragma unroll
      for (int e = 0; e < kVec; ++e) x.a[n][e] = 0.f;
#pragma unroll 2
    for (int j = 0; j < p.planes; ++j) {
      const float c = s_coef[j];
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        const int col = Row::column(n);
        if (col >= p.dim) continue;
        float v[kVec];
        rowg::ld_unit<kVec>(p.hist + j * p.plane, 1, src + col, v);
#pragma unroll
        for (int e = 0; e < kVec; ++e) x.a[n][e] = fmaf(c, v[e], x.a[n][e]);
      }
    }
    if (store && p.out != nullptr) {
#pragma unroll
      for (int n = 0; n < kN; ++n)
        if (Row::column(n) < p.dim) rowg::st_unit<kVec>(p.out, 1, src + Row::column(n), x.a[n]);
    }
    x.normalize(groups, p.eps, smem + turn * scratch);
    turn ^= 1;
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      if (Row::column(n) >= p.dim) continue;
      float g[kVec];
      rowg::ld_unit<kVec>(p.w, p.w_f32, Row::column(n), g);
#pragma unroll
      for (int e = 0; e < kVec; ++e) x.a[n][e] *= g[e];
    }
  };
  Row h;
  if constexpr (!kShift) {
    for (int r = r0; r < r1; ++r) {
      row_at(r, true, h);
#pragma unroll
      for (int n = 0; n < kN; ++n)
        if (Row::column(n) < p.dim) rowg::st_unit<kVec>(p.y, p.y_f32, static_cast<size_t>(r) * p.dim + Row::column(n), h.a[n]);
    }
  } else {
    Row before;
    auto clear = [&] {
#pragma unroll
      for (int n = 0; n < kN; ++n)
#pragma unroll
        for (int e = 0; e < kVec; ++e) before.a[n][e] = 0.f;
    };
    auto leave = [&](float* at, const Row& x) {
#pragma unroll
      for (int n = 0; n < kN; ++n)
        if (Row::column(n) < p.dim) rowg::st_unit<kVec>(at, 1, Row::column(n), x.a[n]);
    };
    clear();
    int seq = s_seq, first = 0, end = 0;
    float* slot = nullptr;
    auto enter = [&](int i) {  // rows [first, end) of sequence i, and its slot's row
      first = p.cu_q_lens[i];
      end = min(p.cu_q_lens[i + 1], p.T);
      const int s = p.slot_ids[i];
      slot = s >= 0 && s < p.slots ? p.state + static_cast<size_t>(s) * p.dim : nullptr;
    };
    if (seq >= 0) {
      enter(seq);
      if (first < r0) row_at(r0 - 1, false, before);
    }
    for (int r = r0; r < r1; ++r) {
      while (seq >= 0 && r >= end) {
        ++seq;
        if (seq >= n_seq) seq = -1;  // padding from here on
        else enter(seq);
      }
      if (seq < 0 || r == first) {
        clear();
        if (seq >= 0 && slot != nullptr && p.kv_lens[seq] > end - first) {
#pragma unroll
          for (int n = 0; n < kN; ++n)
            if (Row::column(n) < p.dim) rowg::ld_unit<kVec>(slot, 1, Row::column(n), before.a[n]);
        }
      }
      row_at(r, true, h);
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        const int col = Row::column(n);
        if (col >= p.dim) continue;
        float m[kVec], v[kVec];
        rowg::ld_unit<kVec>(p.mu, p.w_f32, col, m);
#pragma unroll
        for (int e = 0; e < kVec; ++e) {
          v[e] = fmaf(before.a[n][e] - h.a[n][e], m[e], h.a[n][e]);
          before.a[n][e] = h.a[n][e];
        }
        rowg::st_unit<kVec>(p.y, p.y_f32, static_cast<size_t>(r) * p.dim + col, v);
      }
      if (seq < 0 || first < r0 || slot == nullptr) continue;
      if (r == end - 1) leave(slot, h);
      else if (r == r1 - 1) {  // the sequence goes on beyond this CTA
        row_at(end - 1, false, h);
        leave(slot, h);
      }
    }
  }
}

template <int kN, int kVec, int kThreads>
int launch(const Params& p, int threads, cudaStream_t s) {
  const size_t smem = (2 * rowg::Row<kN, kVec>::scratch_floats(threads, p.dim / p.part) + p.planes) * 4;
  if (smem > 200 * 1024) return kErrTooLarge;
  auto kern = p.mu != nullptr ? depth_kernel<kN, kVec, kThreads, true> : depth_kernel<kN, kVec, kThreads, false>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return kErrCuda;
  kern<<<(p.T + p.per - 1) / p.per, threads, smem, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

}  // namespace depth
}  // namespace lvb

// x[r] = sum over j of coef[j] * hist[j][r] (planes of fp32 [.., dim], `plane` elements apart; coef null: the one plane itself), to out when given;
// h[r] = x[r] with every group of dim / groups elements divided by its root mean square, times w; y[r] = h[r] + (h[r - 1] - h[r]) * mu, or h[r]
// without mu.  The row before a sequence's first packed row (cu_q_lens, the last at position kv_lens - 1) is row slot_ids[i] of state, or zeros when
// the sequence starts here; its last h replaces it.  Rows of no sequence shift from zeros.  T: rows of y; rows: int64 [T] source rows (in range;
// without mu and out).  coef, w and mu have one type (w_f32).  The row before another is formed again where a CTA's rows begin, so out must not
// be one of the planes when there is a shift.
extern "C" int lvb_depth_stream(const float* hist, long long plane, int planes, const void* coef, float* out, const long long* rows, const void* w,
                                const void* mu, int w_f32, float* state, const int* slot_ids, const int* kv_lens, const int* cu_q_lens,
                                const int* num_seqs, int S, int slots, void* y, int y_f32, int T, int dim, int groups, float eps, void* stream) {
  using namespace lvb;
  using namespace lvb::depth;
  if (T <= 0) return kErrOk;
  if (dim <= 0 || groups <= 0 || dim % groups != 0 || planes <= 0 || (coef == nullptr && planes != 1)) return kErrBadArg;
  if (mu != nullptr && (rows != nullptr || state == nullptr || S <= 0 || slots <= 0)) return kErrBadArg;
  if (rows != nullptr && out != nullptr) return kErrBadArg;
  if (planes > 4096) return kErrTooLarge;
  const int part = dim / groups;
  const int mis = static_cast<int>((reinterpret_cast<uintptr_t>(hist) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(w) |
                                    reinterpret_cast<uintptr_t>(mu) | reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(y)) & 15);
  const int vec = (part & 3) == 0 && (plane & 3) == 0 && mis == 0 ? 4 : 1;
  // rows per CTA: with a shift about one wave of CTAs, and at least a few rows, since the one before the first is formed twice
  int per = mu != nullptr ? T / (num_sms() * 6) : 1;
  if (mu != nullptr && per < 4) per = T / num_sms() < 4 ? T / num_sms() : 4;
  per = per < 1 ? 1 : per > 32 ? 32 : per;
  int n, threads;
  if (!rowg::shape_for(dim, vec, (T + per - 1) / per < 2 * num_sms(), n, threads)) return kErrTooLarge;
  Params p{hist, plane, planes, coef, out, rows, w, mu, w_f32, state, slot_ids, kv_lens, cu_q_lens, num_seqs, S, slots, y, y_f32, T, dim, part, per, eps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (vec == 4) {
    if (n == 1) return threads <= 256 ? launch<1, 4, 256>(p, threads, s) : launch<1, 4, 1024>(p, threads, s);
    return n == 2 ? launch<2, 4, 512>(p, threads, s) : n == 4 ? launch<4, 4, 1024>(p, threads, s) : kErrTooLarge;
  }
  if (n == 1) return launch<1, 1, 1024>(p, threads, s);
  return n == 2 ? launch<2, 1, 512>(p, threads, s) : n == 4 ? launch<4, 1, 1024>(p, threads, s) : launch<16, 1, 1024>(p, threads, s);
}
