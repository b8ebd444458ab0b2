// mLSTM cell (matrix memory with exponential gating).  Per head, with q times q_scale:
//
//   i  = cap tanh((gi + bi) / cap),  f = logsigmoid(cap tanh((gf + bf) / cap))
//   m' = max(f + m, i)                               running maximum, starts at 0
//   S' = exp(f + m - m') S + exp(i - m') k v^T,      n' likewise with k alone
//   o  = S'^T q / (max(|n' . q|, exp(-m')) + den_eps)
//
// Decode updates S, n and m in one kernel.  Prompts: the gates of all tokens come first (a warp per sequence and head composes
// the maps m -> max(f + m, i) over 32 tokens at a time); S and n then run through the scan of state_rule.cuh, n as one more
// value column.  Any running maximum gives the same quotient as long as S, n and exp(-m) share it, so its rounding is immaterial.
#define BG_FILE_TAG 26     // kernel-trace ids of this file are (tag << 16) | line
#include "linear_state.h"

namespace bg {
namespace rec {

__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

struct MLstm {
  static constexpr int kVecs = 2;
  static constexpr bool kRead = false, kTwoTerms = false, kForget = false, kDen = true, kOwnV = false;
  struct Regs { float q, k, gi, gf, bi, bf, n, m; };
  struct Scal { float keep, put, m; };
  static __device__ __forceinline__ void fetch(const Args& p, int t, int h, int c, Regs& x) {
    const int slot = p.slots[t];
    if (slot < 0) return;
    x.gi = p.gate_i[(size_t)t * p.ld_gi + h];
    x.gf = p.gate_f[(size_t)t * p.ld_gf + h];
    x.bi = p.bias0[h];
    x.bf = p.bias1[h];
    x.m = p.max_state[slot * p.slot_stride + h];
    if (c >= p.K) return;
    x.q = p.q[(size_t)t * p.ld_q + h * p.K + c];
    x.k = p.k[(size_t)t * p.ld_k + h * p.K + c];
    x.n = p.norm_state[slot * p.slot_stride + h * p.K + c];
  }
  static __device__ __forceinline__ Scal scalars(const Args& p, const Regs& x, int) {
    const float i = soft_cap(x.gi + x.bi, p.cap), f = log_sigmoid(soft_cap(x.gf + x.bf, p.cap));
    const float m = fmaxf(f + x.m, i);
    return {expf(f + x.m - m), expf(i - m), m};
  }
  static __device__ __forceinline__ void vectors(const Args& p, const Regs& x, const Scal& sc, int slot, int h, int c, float (&v)[2],
                                                 float& nq, float&, float&) {
    v[0] = sc.put * x.k;
    v[1] = p.q_scale * x.q;
    const float n = sc.keep * x.n + v[0];
    p.norm_state[slot * p.slot_stride + h * p.K + c] = n;
    if (c == 0) p.max_state[slot * p.slot_stride + h] = sc.m;
    nq = n * v[1];
  }
  static __device__ __forceinline__ Coefs coefs(const Args& p, const Scal& sc, float nq, float, float) {
    return {0.f, 1.0f / (fmaxf(fabsf(nq), expf(-sc.m)) + p.den_eps), 0.f, 0.f, 0.f, sc.keep};
  }
};

// gates[t, h] = (exp(f + m_(t-1) - m_t), exp(i - m_t), exp(-m_t), 0); the last m goes to the state
__global__ void __launch_bounds__(128) gates_kernel(const Args p, float4* __restrict__ gates) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int h = blockIdx.x * 4 + (threadIdx.x >> 5), seq = blockIdx.y, lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int slot = p.slots[seq];
  const int t0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int t1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  if (t1 <= t0) return;
  if (slot < 0) {
    for (int t = t0 + lane; t < t1; t += 32) gates[(size_t)t * p.H + h] = make_float4(1.f, 0.f, 1.f, 0.f);
    return;
  }
  float* ms = p.max_state + slot * p.slot_stride + h;
  float m0 = p.has_initial == nullptr || p.has_initial[seq] != 0 ? *ms : 0.f;
  const float bi = p.bias0[h], bf = p.bias1[h];
  for (int base = t0; base < t1; base += 32) {
    const int t = base + lane;
    float i = -INFINITY, f = 0.f;                                 // past the end: m stays
    if (t < t1) {
      i = soft_cap(p.gate_i[(size_t)t * p.ld_gi + h] + bi, p.cap);
      f = log_sigmoid(soft_cap(p.gate_f[(size_t)t * p.ld_gf + h] + bf, p.cap));
    }
    float F = f, I = i;                                           // this token after the ones before it: m -> max(F + m, I)
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Ip = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(Ip + F, I);
        F += Fp;
      }
    }
    const float m = fmaxf(F + m0, I);
    float before = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) before = m0;
    if (t < t1) gates[(size_t)t * p.H + h] = make_float4(expf(f + before - m), expf(i - m), expf(-m), 0.f);
    m0 = __shfl_sync(0xffffffffu, m, 31);
  }
  if (lane == 0) *ms = m0;
}

// records: exp(i - m) k | q | exp(f + m_(t-1) - m)
__global__ void __launch_bounds__(256) mlstm_records(const Args p, const float4* __restrict__ gates, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int K = p.K;
  const float4 g = gates[(size_t)t * p.H + h];
  float* out = rec + ((size_t)t * p.H + h) * rec_floats<MLstm>(K, p.V);
  for (int e = lane * 4; e < K; e += 128) {
    const float4 k = *reinterpret_cast<const float4*>(p.k + (size_t)t * p.ld_k + h * K + e);
    const float4 q = *reinterpret_cast<const float4*>(p.q + (size_t)t * p.ld_q + h * K + e);
    *reinterpret_cast<float4*>(out + e) = make_float4(g.y * k.x, g.y * k.y, g.y * k.z, g.y * k.w);
    *reinterpret_cast<float4*>(out + K + e) = make_float4(p.q_scale * q.x, p.q_scale * q.y, p.q_scale * q.z, p.q_scale * q.w);
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 2 * K) = make_float4(g.x, 0.f, 0.f, 0.f);
}

int mlstm_forward(const Args& p, cudaStream_t stream) {
  if (p.gate_i == nullptr || p.gate_f == nullptr || p.bias0 == nullptr || p.bias1 == nullptr || p.norm_state == nullptr ||
      p.max_state == nullptr || p.rep != 1 || p.cap <= 0.f)
    return -1;
  if (p.scratch == nullptr) return launch_decode<MLstm>(p, stream);
  const size_t th = (size_t)p.T * p.H;
  float4* gates = reinterpret_cast<float4*>(p.scratch);
  float* rec = p.scratch + 4 * th;
  float* o = rec + th * rec_floats<MLstm>(p.K, p.V);
  float* den = o + th * p.V;
  bg::launch_pdl(gates_kernel, dim3((p.H + 3) / 4, p.nseq), dim3(128), 0, stream, p, gates);
  bg::launch_pdl(mlstm_records, dim3(p.T, (p.H + 7) / 8), dim3(256), 0, stream, p, (const float4*)gates, rec);
  return launch_scan<MLstm>(p, rec, o, den, gates, stream);
}

}  // namespace rec
}  // namespace bg

BG_TRACE_SETTER(mlstm)
