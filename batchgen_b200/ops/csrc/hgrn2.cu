// HGRN2: every row of a head's state keeps the share f of itself and takes the rest from the token's value.  Per head and key channel
//
//   f  = l + (1 - l) * sigmoid(z + bias), l the channel's lower bound
//   S' = diag(f) S + (1 - f) v^T,  o = S'^T silu(q)
//
// The kernels that move and update the states are in state_rule.cuh.
#define BG_FILE_TAG 31     // kernel-trace ids of this file are (tag << 16) | line
#include "linear_state.h"

namespace bg {
namespace rec {

__device__ __forceinline__ float forget(float z, float low) { return low + (1.0f - low) * sigm(z); }

struct Hgrn2 {
  static constexpr int kVecs = 2;
  static constexpr bool kRead = false, kTwoTerms = false, kForget = true, kDen = false, kOwnV = false;
  struct Regs { float q, z, low; };
  struct Scal {};
  static __device__ __forceinline__ void fetch(const Args& p, int t, int h, int c, Regs& x) {
    if (c >= p.K) return;
    const int hc = h * p.K + c;
    x.q = p.q[(size_t)t * p.ld_q + hc];
    x.z = p.k[(size_t)t * p.ld_k + hc] + p.bias0[hc];
    x.low = p.rate[hc];
  }
  static __device__ __forceinline__ Scal scalars(const Args&, const Regs&, int) { return {}; }
  static __device__ __forceinline__ void vectors(const Args&, const Regs& x, const Scal&, int, int, int, float (&v)[2], float&, float&,
                                                 float&) {
    v[0] = forget(x.z, x.low);
    v[1] = x.q * sigm(x.q);
  }
  static __device__ __forceinline__ Coefs coefs(const Args&, const Scal&, float, float, float) {
    return {0.f, 1.0f, 0.f, 0.f, 0.f, 0.f};
  }
};

// records: f | silu(q)
__global__ void __launch_bounds__(256) hgrn2_records(const Args p, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int K = p.K;
  const float* qr = p.q + (size_t)t * p.ld_q + h * K;
  const float* zr = p.k + (size_t)t * p.ld_k + h * K;
  float* out = rec + ((size_t)t * p.H + h) * rec_floats<Hgrn2>(K, p.V);
  for (int e = lane * 4; e < K; e += 128) {
    const float4 q = *reinterpret_cast<const float4*>(qr + e), z = *reinterpret_cast<const float4*>(zr + e);
    const float4 b = *reinterpret_cast<const float4*>(p.bias0 + h * K + e), l = *reinterpret_cast<const float4*>(p.rate + h * K + e);
    *reinterpret_cast<float4*>(out + e) =
        make_float4(forget(z.x + b.x, l.x), forget(z.y + b.y, l.y), forget(z.z + b.z, l.z), forget(z.w + b.w, l.w));
    *reinterpret_cast<float4*>(out + K + e) = make_float4(q.x * sigm(q.x), q.y * sigm(q.y), q.z * sigm(q.z), q.w * sigm(q.w));
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 2 * K) = make_float4(0.f, 0.f, 0.f, 0.f);
}

int hgrn2_forward(const Args& p, cudaStream_t stream) {
  if (p.rate == nullptr || p.bias0 == nullptr || p.rep != 1 || reinterpret_cast<uintptr_t>(p.rate) % 16 || reinterpret_cast<uintptr_t>(p.bias0) % 16)
    return -1;
  if (p.scratch == nullptr) return launch_decode<Hgrn2>(p, stream);
  float* o = p.scratch + (size_t)p.T * p.H * rec_floats<Hgrn2>(p.K, p.V);
  bg::launch_pdl(hgrn2_records, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, p.scratch);
  return launch_scan<Hgrn2>(p, p.scratch, o, nullptr, nullptr, stream);
}

}  // namespace rec
}  // namespace bg

BG_TRACE_SETTER(hgrn2)
