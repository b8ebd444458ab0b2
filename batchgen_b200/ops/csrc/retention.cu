// Retention: linear attention with a fixed decay per head, S' = decay S + k v^T, o = S'^T q, rotary positions on q and k
// (pairs (i, i + half), angles tabulated per token), k times k_scale after the rotation.  The kernels that move and update the
// states are in state_rule.cuh.  Also the entry point of all linear-attention recurrences.
#define BG_FILE_TAG 27     // kernel-trace ids of this file are (tag << 16) | line
#include "linear_state.h"

namespace bg {
namespace rec {

// channel c of a head whose first 2 * half channels turn; x points at the head
__device__ __forceinline__ float turned(const float* x, int c, const float* rope, int half) {
  const float a = x[c];
  if (c >= 2 * half) return a;
  const bool low = c < half;
  const float b = x[low ? c + half : c - half], co = rope[low ? c : c - half], si = rope[half + (low ? c : c - half)];
  return low ? a * co - b * si : a * co + b * si;
}

struct Retention {
  static constexpr int kVecs = 2;
  static constexpr bool kRead = false, kTwoTerms = false, kForget = false, kDen = false, kOwnV = false;
  struct Regs { float q, k, w; };
  struct Scal { float w; };
  static __device__ __forceinline__ void fetch(const Args& p, int t, int h, int c, Regs& x) {
    x.w = p.rate[h];
    if (c >= p.K) return;
    const float* rope = p.rope + (size_t)t * p.ld_rope;
    x.q = turned(p.q + (size_t)t * p.ld_q + h * p.K, c, rope, p.ld_rope / 2);
    x.k = turned(p.k + (size_t)t * p.ld_k + h * p.K, c, rope, p.ld_rope / 2);
  }
  static __device__ __forceinline__ Scal scalars(const Args&, const Regs& x, int) { return {x.w}; }
  static __device__ __forceinline__ void vectors(const Args& p, const Regs& x, const Scal&, int, int, int, float (&v)[2], float&, float&,
                                                 float&) {
    v[0] = p.k_scale * x.k;
    v[1] = p.q_scale * x.q;
  }
  static __device__ __forceinline__ Coefs coefs(const Args&, const Scal& sc, float, float, float) {
    return {0.f, 1.0f, 0.f, 0.f, 0.f, sc.w};
  }
};

// records: k | q | decay
__global__ void __launch_bounds__(256) retention_records(const Args p, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int K = p.K;
  const float* rope = p.rope + (size_t)t * p.ld_rope;
  const float* qr = p.q + (size_t)t * p.ld_q + h * K;
  const float* kr = p.k + (size_t)t * p.ld_k + h * K;
  float* out = rec + ((size_t)t * p.H + h) * rec_floats<Retention>(K, p.V);
  for (int e = lane; e < K; e += 32) {
    out[e] = p.k_scale * turned(kr, e, rope, p.ld_rope / 2);
    out[K + e] = p.q_scale * turned(qr, e, rope, p.ld_rope / 2);
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 2 * K) = make_float4(p.rate[h], 0.f, 0.f, 0.f);
}

static int retention_forward(const Args& p, cudaStream_t stream) {
  if (p.rate == nullptr || p.rep != 1 || p.ld_rope < 0 || p.ld_rope % 2 || p.ld_rope > p.K || (p.rope == nullptr) != (p.ld_rope == 0))
    return -1;
  if (p.scratch == nullptr) return launch_decode<Retention>(p, stream);
  float* o = p.scratch + (size_t)p.T * p.H * rec_floats<Retention>(p.K, p.V);
  bg::launch_pdl(retention_records, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, p.scratch);
  return launch_scan<Retention>(p, p.scratch, o, nullptr, nullptr, stream);
}

}  // namespace rec
}  // namespace bg

// rule: 0 channel_delta, 1 mlstm, 2 retention, 3 hgrn2.  -1: sizes or strides outside the kernels' contract
extern "C" int bg_recurrent_forward(const bg::rec::Args* a, cudaStream_t stream) {
  using namespace bg::rec;
  if (a->nseq <= 0 || a->T <= 0) return 0;
  if (check_args(*a) != 0) return -1;
  switch (a->rule) {
    case 0: return channel_delta_forward(*a, stream);
    case 1: return mlstm_forward(*a, stream);
    case 2: return retention_forward(*a, stream);
    case 3: return hgrn2_forward(*a, stream);
    default: return -1;
  }
}

BG_TRACE_SETTER(retention)
