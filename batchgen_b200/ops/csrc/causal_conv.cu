// Causal depthwise convolution over time with per-sequence history, and the rotary tables of a step.
//
//   causal_conv   y_t[c] = sum_j w[j][c] x_(t - taps + 1 + j)[c]; out = x + y (operand type) or silu(y).  Inputs before a piece
//                 come from the sequence's stored history, zeros before its start.  A thread owns 4 channels and walks a run of
//                 tokens with the last inputs in registers; a second kernel stores the last taps - 1 inputs of every piece
//                 (pieces shorter than that shift the old ones).  One token per sequence: one kernel does both.
//   rope_table    cosines and sines of position * frequency; the turn is formed and reduced in 64 bits
#define BG_FILE_TAG 28     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace cconv {

constexpr int kThreads = 128;
constexpr int kRun = 16;        // tokens a thread walks
constexpr int kAhead = 8;       // of them loaded ahead

struct Params {
  const float* x;          // [T, ldx]
  int ldx;
  const float* w;          // [taps, C]
  float* hist;             // [slots] rows of `hist_stride`: [taps - 1, C], oldest first
  long long hist_stride;
  const int* slots;        // [nseq], < 0: no history, none kept
  const int* cu;           // [nseq + 1] or null: one token per sequence
  const int* row_seq;      // [T] (with cu)
  const int* has_initial;  // [nseq] or null
  void* out;               // [T, ldo], columns C .. cols become zero
  int ldo, T, nseq, C, cols, taps;
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ void fma4(float4& a, const float4& w, const float4& v) {
  a.x = fmaf(w.x, v.x, a.x); a.y = fmaf(w.y, v.y, a.y); a.z = fmaf(w.z, v.z, a.z); a.w = fmaf(w.w, v.w, a.w);
}
__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
template <int KIND>
__device__ __forceinline__ float4 finish(const float4& y, const float4& x) {
  if (KIND == 0) return make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w);
  return make_float4(silu(y.x), silu(y.y), silu(y.z), silu(y.w));
}

// TAPS > 0: that many taps, the window in registers; 0: p.taps, re-read from memory
template <typename OT, int KIND, int TAPS>
__global__ void __launch_bounds__(kThreads) piece_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int c = (blockIdx.x * kThreads + threadIdx.x) * 4, lo = blockIdx.y * kRun, hi = min(lo + kRun, p.T);
  if (c >= p.cols) return;
  OT* out = reinterpret_cast<OT*>(p.out) + c;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c >= p.C) {
    for (int t = lo; t < hi; ++t) store4(out + (size_t)t * p.ldo, zero);
    return;
  }
  const int taps = TAPS > 0 ? TAPS : p.taps;
  constexpr int NW = TAPS > 0 ? TAPS : 1;
  float4 w[NW], win[NW];                                          // win[j]: input of token t - TAPS + 1 + j
#pragma unroll
  for (int j = 0; j < NW; ++j) w[j] = TAPS > 0 ? ld4(p.w + (size_t)j * p.C + c) : zero;
  int seq = -1, first = 0, slot = -1;
  bool init = false;
  auto input = [&](int t) {                                       // of the current sequence; t may lie before the piece
    if (t >= first) return ld4(p.x + (size_t)t * p.ldx + c);
    const int j = t - first + taps - 1;                           // row of the history
    return init && j >= 0 ? ld4(p.hist + slot * p.hist_stride + (size_t)j * p.C + c) : zero;
  };
  for (int g = lo; g < hi; g += kAhead) {
    float4 xs[kAhead];                                            // in flight together
    int seqs[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int t = min(g + i, hi - 1);
      xs[i] = ld4(p.x + (size_t)t * p.ldx + c);
      seqs[i] = p.row_seq[t];
    }
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int t = g + i;
      if (t >= hi) break;
      if (seqs[i] != seq) {
        seq = seqs[i];
        first = p.cu[seq];
        slot = p.slots[seq];
        init = slot >= 0 && (p.has_initial == nullptr || p.has_initial[seq] != 0);
        if (TAPS > 0) {
#pragma unroll
          for (int j = 0; j < NW - 1; ++j) win[j + 1] = input(t - TAPS + 1 + j);
        }
      }
      float4 y = zero;
      if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < NW - 1; ++j) win[j] = win[j + 1];
        win[NW - 1] = xs[i];
#pragma unroll
        for (int j = 0; j < NW; ++j) fma4(y, w[j], win[j]);
      } else {
        for (int j = 0; j < taps; ++j) fma4(y, ld4(p.w + (size_t)j * p.C + c), input(t - taps + 1 + j));
      }
      store4(out + (size_t)t * p.ldo, finish<KIND>(y, xs[i]));
    }
  }
}

// the last taps - 1 inputs of every piece
__global__ void __launch_bounds__(kThreads) history_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int c = (blockIdx.x * kThreads + threadIdx.x) * 4, seq = blockIdx.y;
  if (c >= p.C) return;
  const int slot = p.slots[seq], t0 = p.cu[seq], t1 = p.cu[seq + 1], n = t1 - t0;
  if (slot < 0 || n <= 0) return;
  const bool init = p.has_initial == nullptr || p.has_initial[seq] != 0;
  float* h = p.hist + slot * p.hist_stride + c;
  for (int r = 0; r < p.taps - 1; ++r) {                          // ascending: row r + n is read before it is written
    const int t = n - (p.taps - 1) + r;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t >= 0) v = ld4(p.x + (size_t)(t0 + t) * p.ldx + c);
    else if (init) v = ld4(h + (size_t)(r + n) * p.C);
    store4(h + (size_t)r * p.C, v);
  }
}

template <typename OT, int KIND>
__global__ void __launch_bounds__(kThreads) step_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int c = (blockIdx.x * kThreads + threadIdx.x) * 4, t = blockIdx.y;
  if (c >= p.cols) return;
  OT* out = reinterpret_cast<OT*>(p.out) + (size_t)t * p.ldo + c;
  float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c >= p.C) {
    store4(out, y);
    return;
  }
  const float4 x = ld4(p.x + (size_t)t * p.ldx + c);
  const int slot = p.slots[t], last = p.taps - 1;
  if (slot >= 0) {
    const bool init = p.has_initial == nullptr || p.has_initial[t] != 0;
    float* h = p.hist + slot * p.hist_stride + c;
    for (int j = 0; j < last; ++j) {
      const float4 old = init ? ld4(h + (size_t)j * p.C) : make_float4(0.f, 0.f, 0.f, 0.f);
      fma4(y, ld4(p.w + (size_t)j * p.C + c), old);
      if (j > 0) store4(h + (size_t)(j - 1) * p.C, old);
    }
    if (last > 0) store4(h + (size_t)(last - 1) * p.C, x);
  }
  fma4(y, ld4(p.w + (size_t)last * p.C + c), x);
  store4(out, finish<KIND>(y, x));
}

__global__ void __launch_bounds__(kThreads)
rope_kernel(const int* __restrict__ lens, const double* __restrict__ turns, float* __restrict__ out, int T, int half, float mult) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int i = blockIdx.x * kThreads + threadIdx.x, t = i / half, j = i % half;
  if (t >= T) return;
  const double a = (double)(lens[t] - 1) * turns[j];
  float s, c;
  sincospif(2.0f * (float)(a - rint(a)), &s, &c);
  out[(size_t)t * 2 * half + j] = c * mult;
  out[(size_t)t * 2 * half + half + j] = s * mult;
}

template <typename OT, int KIND>
static void launch_pieces(const Params& p, dim3 grid, cudaStream_t stream) {
  switch (p.taps) {
    case 2: bg::launch_pdl(piece_kernel<OT, KIND, 2>, grid, dim3(kThreads), 0, stream, p); break;
    case 3: bg::launch_pdl(piece_kernel<OT, KIND, 3>, grid, dim3(kThreads), 0, stream, p); break;
    case 4: bg::launch_pdl(piece_kernel<OT, KIND, 4>, grid, dim3(kThreads), 0, stream, p); break;
    case 5: bg::launch_pdl(piece_kernel<OT, KIND, 5>, grid, dim3(kThreads), 0, stream, p); break;
    default: bg::launch_pdl(piece_kernel<OT, KIND, 0>, grid, dim3(kThreads), 0, stream, p); break;
  }
}

}  // namespace cconv
}  // namespace bg

extern "C" {

// dt: 0 = bf16 output, 1 = fp32; kind 0: out = x + conv(x), 1: out = silu(conv(x)).  ldx, ldo, C, cols: multiples of 4.
int bg_causal_conv(int dt, int kind, const float* x, int ldx, const float* w, float* hist, long long hist_stride, const int* slots,
                   const int* cu, const int* row_seq, const int* has_initial, void* out, int ldo, int T, int nseq, int C, int cols,
                   int taps, cudaStream_t stream) {
  using namespace bg::cconv;
  if (T <= 0 || nseq <= 0) return 0;
  if (C <= 0 || C % 4 || cols % 4 || cols < C || ldx % 4 || ldx < C || ldo % 4 || ldo < cols || taps < 1 || hist_stride % 4 ||
      slots == nullptr || (taps > 1 && hist == nullptr) || (cu != nullptr && row_seq == nullptr) || (cu == nullptr && T != nseq) ||
      nseq > 65535 || reinterpret_cast<uintptr_t>(x) % 16 || reinterpret_cast<uintptr_t>(hist) % 16)
    return -1;
  Params p;
  p.x = x; p.ldx = ldx; p.w = w; p.hist = hist; p.hist_stride = hist_stride; p.slots = slots; p.cu = cu; p.row_seq = row_seq;
  p.has_initial = has_initial; p.out = out; p.ldo = ldo; p.T = T; p.nseq = nseq; p.C = C; p.cols = cols; p.taps = taps;
  const unsigned gx = (cols / 4 + kThreads - 1) / kThreads;
  if (cu == nullptr) {
    const dim3 grid(gx, T);
    if (dt == 0 && kind == 0) bg::launch_pdl(step_kernel<__nv_bfloat16, 0>, grid, dim3(kThreads), 0, stream, p);
    else if (dt == 0) bg::launch_pdl(step_kernel<__nv_bfloat16, 1>, grid, dim3(kThreads), 0, stream, p);
    else if (kind == 0) bg::launch_pdl(step_kernel<float, 0>, grid, dim3(kThreads), 0, stream, p);
    else bg::launch_pdl(step_kernel<float, 1>, grid, dim3(kThreads), 0, stream, p);
    return cudaGetLastError() == cudaSuccess ? 0 : -2;
  }
  const dim3 grid(gx, (T + kRun - 1) / kRun);
  if (grid.y > 65535) return -1;
  if (dt == 0 && kind == 0) launch_pieces<__nv_bfloat16, 0>(p, grid, stream);
  else if (dt == 0) launch_pieces<__nv_bfloat16, 1>(p, grid, stream);
  else if (kind == 0) launch_pieces<float, 0>(p, grid, stream);
  else launch_pieces<float, 1>(p, grid, stream);
  if (taps > 1)
    bg::launch_pdl(history_kernel, dim3((C / 4 + kThreads - 1) / kThreads, nseq), dim3(kThreads), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// lens [T]: position + 1; turns [half] turns per position -> out [T, 2 * half]: cosines, then sines, times mult
int bg_rope_table(const int* lens, const double* turns, float* out, int T, int half, float mult, cudaStream_t stream) {
  using namespace bg::cconv;
  if (T <= 0 || half <= 0) return 0;
  if ((long long)T * half > 0x7fffffffll) return -1;
  bg::launch_pdl(rope_kernel, dim3((unsigned)(((long long)T * half + kThreads - 1) / kThreads)), dim3(kThreads), 0, stream, lens,
                 turns, out, T, half, mult);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(causal_conv)
