// Generalised delta rule: a per-head matrix state with a per-channel decay and a per-channel removal rate.
//
// Per head, state S [D keys x D values] (fp32).  For each token, with unit key u = k / sqrt(sum k^2 + ueps):
//
//   w  = exp(-cdecay * sigmoid(wl + w0))          decay per key channel
//   a  = sigmoid(al + ab)                         removal rate per key channel
//   S' = diag(w) S - (a * u) (u^T S) + k v^T      both terms read the old state
//   o  = S'^T r
//   out = o / sqrt(mean(o^2) + eps) * norm * sigmoid(g)
//
// Both products of a step come from one sweep of the old state: with y = u^T S and q = (w * r)^T S,
// o = q - (r . (a * u)) y + (r . k) v.
//
// Everything that enters the recurrence is fp32; the projections arrive as fp32 GEMM outputs.  The kernels that move and
// update the states are in state_rule.cuh.
#define BG_FILE_TAG 22     // kernel-trace ids of this file are (tag << 16) | line
#include "state_rule.cuh"

namespace bg {
namespace rec {

struct GeneralDelta {
  static constexpr int kVecs = 4;
  static constexpr bool kRead = true, kTwoTerms = true, kForget = false, kDen = false, kOwnV = true;
  struct Regs { float r, k, a, w, w0, ab; };
  struct Scal {};
  static __device__ __forceinline__ void fetch(const Args& p, int t, int h, int c, Regs& x) {
    if (c >= p.K) return;
    const int hc = h * p.K + c;
    x.r = p.q[(size_t)t * p.ld_q + hc];
    x.k = p.k[(size_t)t * p.ld_k + hc];
    x.a = p.beta[(size_t)t * p.ld_beta + hc];
    x.w = p.low[(size_t)t * p.ld_low + hc];
    x.w0 = p.bias0[hc];
    x.ab = p.bias1[hc];
  }
  static __device__ __forceinline__ Scal scalars(const Args&, const Regs&, int) { return {}; }
  static __device__ __forceinline__ void vectors(const Args& p, const Regs& x, const Scal&, int, int, int, float (&v)[4], float& kk,
                                                 float& rk, float& rak) {
    const float a = sigm(x.a + x.ab), w = expf(-p.cap * sigm(x.w + x.w0));
    v[0] = x.k; v[1] = w; v[2] = a * x.k; v[3] = w * x.r;
    kk = x.k * x.k; rk = x.r * x.k; rak = x.r * a * x.k;
  }
  static __device__ __forceinline__ Coefs coefs(const Args& p, const Scal&, float kk, float rk, float rak) {
    return {1.0f / (kk + p.ueps), 1.0f, rk, rak, 0.f, 0.f};      // u u^T = k k^T / (kk + ueps)
  }
};

// records: w | u | a * u | w * r | c1, c2, 0, 0 | v * sqrt(kk + ueps), so that k v^T = u sv^T and o = q - c1 y + c2 sv
// N: K <= 128 N
template <int N>
__global__ void __launch_bounds__(256) general_records(const Args p, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int D = p.K;
  float* out = rec + ((size_t)t * p.H + h) * rec_floats<GeneralDelta>(D, D);
  float4 k[N], au[N], v[N];
  float kk = 0.f, rk = 0.f, rak = 0.f;
  auto at = [&](const float* x, int ld, int e) { return *reinterpret_cast<const float4*>(x + (size_t)t * ld + h * D + e); };
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int e = n * 128 + lane * 4;
    k[n] = au[n] = v[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e >= D) continue;
    const float4 r = at(p.q, p.ld_q, e), a4 = at(p.beta, p.ld_beta, e), l4 = at(p.low, p.ld_low, e);
    const float4 w04 = *reinterpret_cast<const float4*>(p.bias0 + h * D + e);
    const float4 ab4 = *reinterpret_cast<const float4*>(p.bias1 + h * D + e);
    k[n] = at(p.k, p.ld_k, e);
    v[n] = at(p.v, p.ld_v, e);
    float4 w;
    w.x = expf(-p.cap * sigm(l4.x + w04.x)); w.y = expf(-p.cap * sigm(l4.y + w04.y));
    w.z = expf(-p.cap * sigm(l4.z + w04.z)); w.w = expf(-p.cap * sigm(l4.w + w04.w));
    *reinterpret_cast<float4*>(out + e) = w;
    *reinterpret_cast<float4*>(out + 3 * D + e) = make_float4(w.x * r.x, w.y * r.y, w.z * r.z, w.w * r.w);
    au[n] = make_float4(sigm(a4.x + ab4.x) * k[n].x, sigm(a4.y + ab4.y) * k[n].y, sigm(a4.z + ab4.z) * k[n].z,
                        sigm(a4.w + ab4.w) * k[n].w);
    kk += k[n].x * k[n].x + k[n].y * k[n].y + k[n].z * k[n].z + k[n].w * k[n].w;
    rk += r.x * k[n].x + r.y * k[n].y + r.z * k[n].z + r.w * k[n].w;
    rak += r.x * au[n].x + r.y * au[n].y + r.z * au[n].z + r.w * au[n].w;
  }
  kk = warp_sum(kk); rk = warp_sum(rk); rak = warp_sum(rak);
  const float s = sqrtf(kk + p.ueps), inv = 1.0f / s;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int e = n * 128 + lane * 4;
    if (e >= D) continue;
    *reinterpret_cast<float4*>(out + D + e) = make_float4(k[n].x * inv, k[n].y * inv, k[n].z * inv, k[n].w * inv);
    *reinterpret_cast<float4*>(out + 2 * D + e) = make_float4(au[n].x * inv, au[n].y * inv, au[n].z * inv, au[n].w * inv);
    *reinterpret_cast<float4*>(out + 4 * D + 4 + e) = make_float4(v[n].x * s, v[n].y * s, v[n].z * s, v[n].w * s);
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 4 * D) = make_float4(rak * inv, rk * inv, 0.f, 0.f);
}

}  // namespace rec
}  // namespace bg

extern "C" {

// offs: host array of five column offsets (r, k, v, g, a).  dt: 0 = bf16 output, 1 = fp32.  D a multiple of 8, <= 512.
// T: rows of z.  `scratch` (T * H * (6 D + 4) floats: records, then the scan's outputs) selects the prompt path; null the
// decode kernel (D <= 128, one token per sequence).
int bg_delta_forward(int dt, const float* z, int ldz, const int* offs, const float* wl, int ld_wl, const float* w0,
                     const float* ab, const float* norm_w, float* state, long long slot_stride, const int* cu,
                     const int* slots, const int* has_initial, void* out, int ldo, int T, int nseq, int H, int D, int Dreal,
                     float cdecay, float ueps, float eps, float* scratch, int num_sms, int* status, cudaStream_t stream) {
  using namespace bg::rec;
  if (nseq <= 0 || T <= 0) return 0;
  Args p = {};
  p.q = z + offs[0]; p.k = z + offs[1]; p.v = z + offs[2]; p.gate = z + offs[3]; p.beta = z + offs[4];
  p.ld_q = p.ld_k = p.ld_v = p.ld_gate = p.ld_beta = ldz;
  p.low = wl; p.ld_low = ld_wl; p.bias0 = w0; p.bias1 = ab; p.norm_w = norm_w; p.state = state; p.slot_stride = slot_stride;
  p.cu = cu; p.slots = slots; p.has_initial = has_initial; p.out = out; p.ld_out = ldo; p.scratch = scratch; p.status = status;
  p.dt = dt; p.T = T; p.nseq = nseq; p.H = H; p.rep = 1; p.K = p.V = D; p.v_real = Dreal; p.num_sms = num_sms;
  p.q_scale = p.k_scale = 1.f; p.cap = cdecay; p.ueps = ueps; p.eps = eps;
  if (check_args(p) != 0 || offs[4] % 4) return -1;
  if (scratch == nullptr) return launch_decode<GeneralDelta>(p, stream);
  float* o = scratch + (size_t)T * H * rec_floats<GeneralDelta>(D, D);
  if (p.K <= 128) bg::launch_pdl(general_records<1>, dim3(T, (H + 7) / 8), dim3(256), 0, stream, p, scratch);
  else if (p.K <= 256) bg::launch_pdl(general_records<2>, dim3(T, (H + 7) / 8), dim3(256), 0, stream, p, scratch);
  else bg::launch_pdl(general_records<4>, dim3(T, (H + 7) / 8), dim3(256), 0, stream, p, scratch);
  return launch_scan<GeneralDelta>(p, scratch, o, nullptr, nullptr, stream);
}

}  // extern "C"

BG_TRACE_SETTER(delta_rule)
