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
// `delta_step_kernel` holds the whole state of one (sequence, head) in the registers of a CTA and walks the sequence's
// tokens of this step; one token (decode) is a single read and write of the state.  Everything that enters the recurrence
// is fp32; the projections arrive as fp32 GEMM outputs.
#define BG_FILE_TAG 22     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace delta {

struct Params {
  const float* z;          // [T, ldz] stacked projections of the layer input
  int ldz;
  int off_r, off_k, off_v, off_g, off_a;   // first column of each projection in z (heads x D each)
  const float* wl;         // [T, ld_wl] low-rank decay pre-activation
  int ld_wl;
  const float* w0;         // [H * D]
  const float* ab;         // [H * D]
  const float* norm_w;     // [H * D]
  float* state;            // [slots] rows of `slot_stride` floats; this layer's [H, D, D] at the pointer
  long long slot_stride;
  const int* cu;           // [nseq + 1] token ranges, or null: one token per sequence
  const int* slots;        // [nseq], < 0 skips the sequence (its output rows become zero)
  const int* has_initial;  // [nseq] or null (always continue from the slot)
  void* out;               // [T, ldo]
  int ldo;
  int H, D, Dreal;         // D: padded head width (multiple of 8); Dreal: channels of the mean
  float cdecay, ueps, eps;
};

template <typename OT> __device__ __forceinline__ void put4(OT* p, float4 v);
template <> __device__ __forceinline__ void put4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void put4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ float sigm(float x) { return 1.0f / (1.0f + expf(-x)); }

constexpr int kMaxD = 256;

// Thread (ig, jq): value columns 4 jq .. 4 jq + 3, key rows ig, ig + RG, ... (NR of them at most).
template <typename OT, int NT, int NR>
__global__ void __launch_bounds__(NT) delta_step_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = p.D, Q = D / 4, RG = NT / Q;
  const int slot = p.slots[seq];
  const int t0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int t1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  OT* out = reinterpret_cast<OT*>(p.out) + h * D;
  if (slot < 0) {
    for (int t = t0; t < t1; ++t)
      for (int j = tid; j < Q; j += NT) put4(out + (size_t)t * p.ldo + 4 * j, make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  if (t1 <= t0) return;
  __shared__ __align__(16) float sk[kMaxD], sw[kMaxD], sak[kMaxD], swr[kMaxD], sv[kMaxD];
  __shared__ float red[3][kMaxD / 32], red_o[kMaxD / 4 / 32 + 1];
  __shared__ __align__(16) float4 part_y[NT], part_q[NT];
  const int jq = tid % Q, ig = tid / Q;
  const bool active = ig < RG;
  float* Sg = p.state + slot * p.slot_stride + (size_t)h * D * D;
  float4 S[NR];
  const bool init = p.has_initial == nullptr || p.has_initial[seq] != 0;
#pragma unroll
  for (int n = 0; n < NR; ++n) {
    const int i = ig + n * RG;
    S[n] = (init && active && i < D) ? *reinterpret_cast<const float4*>(Sg + (size_t)i * D + 4 * jq)
                                     : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int hc = h * D + tid;                           // this thread's channel in the prologue of a token (tid < D)
  float w0 = 0.f, ab = 0.f;
  if (tid < D) { w0 = p.w0[hc]; ab = p.ab[hc]; }
  const int dwarps = (D + 31) / 32;
  float nr = 0.f, nk = 0.f, nv = 0.f, na = 0.f, nw = 0.f;
  auto load = [&](int t) {
    if (tid < D) {
      const float* zr = p.z + (size_t)t * p.ldz + hc;
      nr = zr[p.off_r]; nk = zr[p.off_k]; nv = zr[p.off_v]; na = zr[p.off_a];
      nw = p.wl[(size_t)t * p.ld_wl + hc];
    }
  };
  load(t0);
  for (int t = t0; t < t1; ++t) {
    if (warp < dwarps) {
      const float r = nr, k = nk;
      const float a = sigm(na + ab);
      const float w = expf(-p.cdecay * sigm(nw + w0));
      if (tid < D) {
        sk[tid] = k; sw[tid] = w; sak[tid] = a * k; swr[tid] = w * r; sv[tid] = nv;
      }
      const float s0 = warp_sum(tid < D ? k * k : 0.f), s1 = warp_sum(tid < D ? r * k : 0.f);
      const float s2 = warp_sum(tid < D ? r * a * k : 0.f);
      if (lane == 0) { red[0][warp] = s0; red[1][warp] = s1; red[2][warp] = s2; }
    }
    __syncthreads();
    if (t + 1 < t1) load(t + 1);
    float kk = 0.f, rk = 0.f, rak = 0.f;
    for (int i = 0; i < dwarps; ++i) { kk += red[0][i]; rk += red[1][i]; rak += red[2][i]; }
    const float inv2 = 1.0f / (kk + p.ueps);             // u u^T = k k^T * inv2
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f), q = y;
    if (active) {
#pragma unroll
      for (int n = 0; n < NR; ++n) {
        const int i = ig + n * RG;
        if (i < D) {
          const float k = sk[i], wr = swr[i];
          y.x = fmaf(k, S[n].x, y.x); y.y = fmaf(k, S[n].y, y.y); y.z = fmaf(k, S[n].z, y.z); y.w = fmaf(k, S[n].w, y.w);
          q.x = fmaf(wr, S[n].x, q.x); q.y = fmaf(wr, S[n].y, q.y); q.z = fmaf(wr, S[n].z, q.z); q.w = fmaf(wr, S[n].w, q.w);
        }
      }
      part_y[tid] = y;
      part_q[tid] = q;
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active) {
      y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int i = 0; i < RG; ++i) {
        const float4 v = part_y[i * Q + jq];
        y.x += v.x; y.y += v.y; y.z += v.z; y.w += v.w;
      }
      y.x *= inv2; y.y *= inv2; y.z *= inv2; y.w *= inv2;
      const float4 v = *reinterpret_cast<const float4*>(&sv[4 * jq]);
      if (ig == 0) {
        q = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int i = 0; i < RG; ++i) {
          const float4 b = part_q[i * Q + jq];
          q.x += b.x; q.y += b.y; q.z += b.z; q.w += b.w;
        }
        o.x = q.x - rak * y.x + rk * v.x; o.y = q.y - rak * y.y + rk * v.y;
        o.z = q.z - rak * y.z + rk * v.z; o.w = q.w - rak * y.w + rk * v.w;
      }
#pragma unroll
      for (int n = 0; n < NR; ++n) {
        const int i = ig + n * RG;
        if (i < D) {
          const float k = sk[i], w = sw[i], ak = sak[i];
          S[n].x = fmaf(w, S[n].x, fmaf(k, v.x, -ak * y.x)); S[n].y = fmaf(w, S[n].y, fmaf(k, v.y, -ak * y.y));
          S[n].z = fmaf(w, S[n].z, fmaf(k, v.z, -ak * y.z)); S[n].w = fmaf(w, S[n].w, fmaf(k, v.w, -ak * y.w));
        }
      }
    }
    const int owarps = (Q + 31) / 32;
    if (warp < owarps) {
      const float s = warp_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w);
      if (lane == 0) red_o[warp] = s;
    }
    __syncthreads();
    if (tid < Q) {
      float oo = 0.f;
      for (int i = 0; i < owarps; ++i) oo += red_o[i];
      const float rs = 1.0f / sqrtf(oo / (float)p.Dreal + p.eps);
      const float4 nw4 = *reinterpret_cast<const float4*>(p.norm_w + h * D + 4 * tid);
      const float4 g = *reinterpret_cast<const float4*>(p.z + (size_t)t * p.ldz + p.off_g + h * D + 4 * tid);
      put4(out + (size_t)t * p.ldo + 4 * tid,
           make_float4(o.x * rs * nw4.x * sigm(g.x), o.y * rs * nw4.y * sigm(g.y), o.z * rs * nw4.z * sigm(g.z),
                       o.w * rs * nw4.w * sigm(g.w)));
    }
  }
  if (active) {
#pragma unroll
    for (int n = 0; n < NR; ++n) {
      const int i = ig + n * RG;
      if (i < D) *reinterpret_cast<float4*>(Sg + (size_t)i * D + 4 * jq) = S[n];
    }
  }
}

template <typename OT>
static int launch_step(const Params& p, int nseq, cudaStream_t stream) {
  dim3 grid(p.H, nseq);
  if (p.D <= 32) bg::launch_pdl(delta_step_kernel<OT, 128, 2>, grid, dim3(128), 0, stream, p);
  else if (p.D <= 64) bg::launch_pdl(delta_step_kernel<OT, 256, 4>, grid, dim3(256), 0, stream, p);
  else if (p.D <= 128) bg::launch_pdl(delta_step_kernel<OT, 256, 16>, grid, dim3(256), 0, stream, p);
  else bg::launch_pdl(delta_step_kernel<OT, 1024, 16>, grid, dim3(1024), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace delta
}  // namespace bg

extern "C" {

// offs: host array of five column offsets (r, k, v, g, a).  dt: 0 = bf16 output, 1 = fp32.  D a multiple of 8, <= 256.
int bg_delta_step(int dt, const float* z, int ldz, const int* offs, const float* wl, int ld_wl, const float* w0,
                  const float* ab, const float* norm_w, float* state, long long slot_stride, const int* cu,
                  const int* slots, const int* has_initial, void* out, int ldo, int nseq, int H, int D, int Dreal,
                  float cdecay, float ueps, float eps, cudaStream_t stream) {
  using namespace bg::delta;
  if (nseq <= 0) return 0;
  if (D <= 0 || D % 8 || D > kMaxD || H <= 0 || H > 65535 || nseq > 65535 || ldz % 4 || ldo % 4 || slot_stride % 4) return -1;
  for (int i = 0; i < 5; ++i)
    if (offs[i] % 4) return -1;
  Params p;
  p.z = z; p.ldz = ldz; p.off_r = offs[0]; p.off_k = offs[1]; p.off_v = offs[2]; p.off_g = offs[3]; p.off_a = offs[4];
  p.wl = wl; p.ld_wl = ld_wl; p.w0 = w0; p.ab = ab; p.norm_w = norm_w; p.state = state; p.slot_stride = slot_stride;
  p.cu = cu; p.slots = slots; p.has_initial = has_initial; p.out = out; p.ldo = ldo; p.H = H; p.D = D; p.Dreal = Dreal;
  p.cdecay = cdecay; p.ueps = ueps; p.eps = eps;
  return dt == 0 ? launch_step<__nv_bfloat16>(p, nseq, stream) : launch_step<float>(p, nseq, stream);
}

}  // extern "C"

BG_TRACE_SETTER(delta_rule)
