// Gated delta rule with a decay per head and key channel (q and k already convolved):
//
//   q, k   unit vectors per head, x / sqrt(sum x^2 + ueps), q times q_scale; `rep` heads share a query / key head
//   g      = exp(-rate[h] * softplus(low + dt_bias)), b = sigmoid(beta[h])
//   S      = diag(g) S;  u = b (v - S^T k);  S = S + k u^T;  o = S^T q
//
// Both products come from one sweep of the old state: with y = (g k)^T S, S' = g S + k u^T, u = b (v - y) and
// o = (g q)^T S + (k . q) u.  The kernels that move and update the states are in state_rule.cuh.
#define BG_FILE_TAG 25     // kernel-trace ids of this file are (tag << 16) | line
#include "linear_state.h"

namespace bg {
namespace rec {

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct ChannelDelta {
  static constexpr int kVecs = 4;
  static constexpr bool kRead = true, kTwoTerms = false, kForget = false, kDen = false, kOwnV = false;
  struct Regs { float q, k, low, dtb, beta, rate; };
  struct Scal { float b; };
  static __device__ __forceinline__ void fetch(const Args& p, int t, int h, int c, Regs& x) {
    x.beta = p.beta[(size_t)t * p.ld_beta + h];
    x.rate = p.rate[h];
    if (c >= p.K) return;
    const int qc = h / p.rep * p.K + c, hc = h * p.K + c;
    x.q = p.q[(size_t)t * p.ld_q + qc];
    x.k = p.k[(size_t)t * p.ld_k + qc];
    x.low = p.low[(size_t)t * p.ld_low + hc];
    x.dtb = p.bias0[hc];
  }
  static __device__ __forceinline__ Scal scalars(const Args&, const Regs& x, int) { return {sigm(x.beta)}; }
  // raw k and q: the norms, known after the sums, scale y, o and the write
  static __device__ __forceinline__ void vectors(const Args&, const Regs& x, const Scal&, int, int, int, float (&v)[4], float& kk,
                                                 float& qq, float& qk) {
    const float g = expf(-x.rate * softplus(x.low + x.dtb));
    v[0] = g * x.k; v[1] = g; v[2] = x.k; v[3] = g * x.q;
    kk = x.k * x.k; qq = x.q * x.q; qk = x.q * x.k;
  }
  static __device__ __forceinline__ Coefs coefs(const Args& p, const Scal& sc, float kk, float qq, float qk) {
    const float rk = 1.0f / sqrtf(kk + p.ueps), rq = p.q_scale / sqrtf(qq + p.ueps);
    return {rk, rq, sc.b * qk * rk * rq, 0.f, sc.b * rk, 0.f};
  }
};

// records: g | g k | b k | g q | b (k . q), k and q normalised
// N: K <= 128 N
template <int N>
__global__ void __launch_bounds__(256) channel_records(const Args p, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int K = p.K;
  float* out = rec + ((size_t)t * p.H + h) * rec_floats<ChannelDelta>(K, p.V);
  const float* qr = p.q + (size_t)t * p.ld_q + h / p.rep * K;
  const float* kr = p.k + (size_t)t * p.ld_k + h / p.rep * K;
  const float* lr = p.low + (size_t)t * p.ld_low + h * K;
  const float b = sigm(p.beta[(size_t)t * p.ld_beta + h]), rate = p.rate[h];
  float4 q[N], k[N];
  float kk = 0.f, qq = 0.f, qk = 0.f;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int e = n * 128 + lane * 4;
    q[n] = k[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e >= K) continue;
    q[n] = *reinterpret_cast<const float4*>(qr + e);
    k[n] = *reinterpret_cast<const float4*>(kr + e);
    kk += k[n].x * k[n].x + k[n].y * k[n].y + k[n].z * k[n].z + k[n].w * k[n].w;
    qq += q[n].x * q[n].x + q[n].y * q[n].y + q[n].z * q[n].z + q[n].w * q[n].w;
    qk += q[n].x * k[n].x + q[n].y * k[n].y + q[n].z * k[n].z + q[n].w * k[n].w;
  }
  kk = warp_sum(kk); qq = warp_sum(qq); qk = warp_sum(qk);
  const float rk = 1.0f / sqrtf(kk + p.ueps), rq = p.q_scale / sqrtf(qq + p.ueps), bk = b * rk;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int e = n * 128 + lane * 4;
    if (e >= K) continue;
    const float4 l = *reinterpret_cast<const float4*>(lr + e), d = *reinterpret_cast<const float4*>(p.bias0 + h * K + e);
    const float4 g = make_float4(expf(-rate * softplus(l.x + d.x)), expf(-rate * softplus(l.y + d.y)),
                                 expf(-rate * softplus(l.z + d.z)), expf(-rate * softplus(l.w + d.w)));
    *reinterpret_cast<float4*>(out + e) = g;
    *reinterpret_cast<float4*>(out + K + e) = make_float4(g.x * k[n].x * rk, g.y * k[n].y * rk, g.z * k[n].z * rk, g.w * k[n].w * rk);
    *reinterpret_cast<float4*>(out + 2 * K + e) = make_float4(k[n].x * bk, k[n].y * bk, k[n].z * bk, k[n].w * bk);
    *reinterpret_cast<float4*>(out + 3 * K + e) = make_float4(g.x * q[n].x * rq, g.y * q[n].y * rq, g.z * q[n].z * rq, g.w * q[n].w * rq);
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 4 * K) = make_float4(qk * bk * rq, 0.f, 0.f, 0.f);
}

int channel_delta_forward(const Args& p, cudaStream_t stream) {
  if (p.low == nullptr || p.beta == nullptr || p.rate == nullptr || p.bias0 == nullptr) return -1;
  if (p.scratch == nullptr) return launch_decode<ChannelDelta>(p, stream);
  float* o = p.scratch + (size_t)p.T * p.H * rec_floats<ChannelDelta>(p.K, p.V);
  if (p.K <= 128) bg::launch_pdl(channel_records<1>, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, p.scratch);
  else if (p.K <= 256) bg::launch_pdl(channel_records<2>, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, p.scratch);
  else bg::launch_pdl(channel_records<4>, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, p.scratch);
  return launch_scan<ChannelDelta>(p, p.scratch, o, nullptr, nullptr, stream);
}

}  // namespace rec
}  // namespace bg

BG_TRACE_SETTER(channel_delta)
