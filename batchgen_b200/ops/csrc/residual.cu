// Row kernels of models with an fp32 residual stream:
//
//   residual_norm   x[t] += sum of the sublayers' fp32 outputs (dense rows and / or routed rows gathered by position),
//                   or x[t] = embed[id] * scale for the first layer; y[t] = x[t] / sqrt(mean(x^2) + eps) * w
//   sandwich_norm   the same for blocks with a norm before and after each sublayer: the sublayer's output (or half the sum of
//                   two, each RMS-normed, or the weighted rows of routed experts) passes its own norm before it joins x; optional
//                   mean subtraction and biases; the norm before may be absent; in decode the input convolution y = h + conv(h)
//                   of the next sublayer (or its token shift, a convolution of two taps) is folded in
//   hyper_norm      the same for several residual streams: every stream becomes a weighted sum of all of them plus its share of
//                   the sublayer's output; the norm reads another weighted sum
//   token_side      tanh-GELU(z) * the token's row of a table
//   glu             gated activations (tanh-GELU, SwiGLU, clamped SwiGLU with slope 1.702 and u + 1; squared ReLU without a gate), with an optional factor on
//                   the pre-activations (routing weight applied to the expert's input) and an optional sigmoid gate
//   cast_act        out = f(x), f = tanh, squared ReLU or identity: fp32 columns of a projection to the operand type of the next one
//   moe_gather      token rows -> expert-grouped rows, one block per (token, k) pair, plus the pair's routing weight
//
// Activations are fp32 in, bf16 or fp32 out (`OT`); sums, norms and gates are fp32.
#define BG_FILE_TAG 21     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace resid {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}

constexpr int kThreads = 256;
constexpr int kMaxK = 16;

struct NormParams {
  float* x;             // [T, ldx] residual stream
  int ldx;
  const long long* rows;  // [R] rows of x to normalise, or null (row i of the grid is row i of x)
  const int* ids;       // first layer: token ids (x is written, not read)
  const void* embed;    // [V, lde]
  int lde;
  float escale;
  int vocab;
  const float* add;     // dense addend [T, ld_add] or null
  int ld_add;
  const float* routed;  // rows of the routed experts [*, ld_routed] or null
  int ld_routed;
  const int* pos;       // [T, K] row of every (token, k) pair, < 0 = none
  int K;
  const float* w;       // [D] gain
  void* y;              // [R, ldy]; columns D .. ldy are zero
  int ldy;
  int D;
  float eps;
  int keep;             // write x back
};

// One block per row; thread i owns 4-wide vectors i, i + 256, ...; D is padded to a multiple of 4 in x (ldx % 4 == 0)
template <typename OT>
__global__ void __launch_bounds__(kThreads) residual_norm_kernel(const NormParams p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ float row[];
  __shared__ float red[kThreads / 32];
  __shared__ int pos_s[kMaxK];
  const int tid = threadIdx.x;
  const long long t = p.rows != nullptr ? p.rows[blockIdx.x] : (long long)blockIdx.x;
  float* xr = p.x + t * p.ldx;
  const int D = p.D, nv = (D + 3) / 4;
  if (p.routed != nullptr) {
    if (tid < p.K) pos_s[tid] = p.pos[t * p.K + tid];
    __syncthreads();
  }
  const OT* er = nullptr;
  if (p.ids != nullptr) {
    const int id = min(max(p.ids[t], 0), p.vocab - 1);
    er = reinterpret_cast<const OT*>(p.embed) + (size_t)id * p.lde;
  }
  float ss = 0.f;
  for (int v = tid; v < nv; v += kThreads) {
    const int c = v * 4;
    float4 f;
    if (er != nullptr) {
      f.x = to_f(er[c]) * p.escale;
      f.y = c + 1 < D ? to_f(er[c + 1]) * p.escale : 0.f;
      f.z = c + 2 < D ? to_f(er[c + 2]) * p.escale : 0.f;
      f.w = c + 3 < D ? to_f(er[c + 3]) * p.escale : 0.f;
    } else {
      f = *reinterpret_cast<const float4*>(xr + c);
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.add != nullptr) s = *reinterpret_cast<const float4*>(p.add + t * p.ld_add + c);
      if (p.routed != nullptr) {
        for (int k = 0; k < p.K; ++k) {
          const int r = pos_s[k];
          if (r < 0) continue;
          const float4 a = *reinterpret_cast<const float4*>(p.routed + (size_t)r * p.ld_routed + c);
          s.x += a.x; s.y += a.y; s.z += a.z; s.w += a.w;
        }
      }
      f.x += s.x;
      f.y = c + 1 < D ? f.y + s.y : 0.f;
      f.z = c + 2 < D ? f.z + s.z : 0.f;
      f.w = c + 3 < D ? f.w + s.w : 0.f;
    }
    if (p.keep) *reinterpret_cast<float4*>(xr + c) = f;
    *reinterpret_cast<float4*>(row + c) = f;
    ss += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) tot += red[i];
  const float rstd = 1.0f / sqrtf(tot / (float)D + p.eps);
  OT* yr = reinterpret_cast<OT*>(p.y) + (size_t)blockIdx.x * p.ldy;
  for (int v = tid; v < p.ldy / 4; v += kThreads) {
    const int c = v * 4;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D) {
      o.x = row[c] * rstd * p.w[c];
      if (c + 1 < D) o.y = row[c + 1] * rstd * p.w[c + 1];
      if (c + 2 < D) o.z = row[c + 2] * rstd * p.w[c + 2];
      if (c + 3 < D) o.w = row[c + 3] * rstd * p.w[c + 3];
    }
    store4(yr + c, o);
  }
}

struct SandwichParams {
  float* x;               // [T, ldx] residual stream
  int ldx;
  const long long* rows;  // [R] rows of x, or null
  const int* ids;         // first layer: token ids (x is written, not read)
  const void* embed;      // [V, lde]
  int lde;
  float escale;
  int vocab;
  const float *a, *b;     // the sublayer's output(s) [T, ld], or null
  int lda, ldb;
  const float *wa, *wb;   // with b: weights of the outputs' RMS norms
  const float* routed;    // instead of a: rows of the routed experts [*, ld_routed], or null
  int ld_routed;
  const int* pos;         // [T, K] row of every (token, k) pair, < 0 = none
  const float* route_w;   // [T, K] factors of those rows
  int K;
  const float *w1, *b1;   // norm of the output; b1 may be null
  int center1;
  const float *w2, *b2;   // norm of x; w2 null: x itself
  int center2;
  void* y;                // [R, ldy], or null: only x
  int ldy, raw;           // raw: y is fp32 and ends at D rounded up to 4
  const float* cw;        // [taps, D4] input convolution, or null
  float* hist;            // [slots, (taps - 1) * D4] rows of `hist_stride`
  long long hist_stride;
  const int* slots;
  int taps;
  int D;
  float eps;
  int keep;
};

constexpr int kMaxWarps = kThreads / 32;

struct Moments { float n, mean, m2; };      // of a warp's elements: count, mean, sum of squared deviations from that mean

// One block of up to 256 threads per row; thread i owns the 4-wide vectors i, i + blockDim, ... (NV of them) in registers.  All
// loads of the row are issued before any is used.  A norm's mean and variance meet in one barrier: every warp takes both of its
// own elements first, then the warps' moments are put together.  Columns D .. D4 hold zeros (weights and biases are zero there).
template <typename OT, int NV>
__global__ void __launch_bounds__(kThreads) sandwich_norm_kernel(const SandwichParams p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  __shared__ float red[2][kMaxWarps];
  __shared__ Moments part[2][kMaxWarps];
  __shared__ int pos_s[kMaxK];
  __shared__ float rw[kMaxK];
  const int tid = threadIdx.x, NT = blockDim.x, warps = NT >> 5;
  const long long t = p.rows != nullptr ? p.rows[blockIdx.x] : (long long)blockIdx.x;
  float* xr = p.x + t * p.ldx;
  const int D = p.D, nv = (D + 3) / 4;
  const float inv_d = 1.0f / (float)D;
  float4 f[NV], s[NV], u[NV];
  auto each = [&](auto fn) {
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int v = tid + n * NT;
      if (v < nv) fn(n, v * 4);
    }
  };
  auto ld4 = [](const float* q, int c) { return *reinterpret_cast<const float4*>(q + c); };
  auto dot = [](const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
  auto mask = [&](float4& v, int c) {                              // zero past D
    if (c + 4 > D) {
      if (c + 1 >= D) v.y = 0.f;
      if (c + 2 >= D) v.z = 0.f;
      v.w = 0.f;
    }
  };
  float warp_n = 0.f;
  each([&](int, int c) { warp_n += (float)min(4, D - c); });
  warp_n = warp_sum(warp_n);
  const float inv_n = warp_n > 0.f ? 1.0f / warp_n : 0.f;
  // mean and 1 / sqrt(variance + eps) of the vectors in v (mean 0 without centring)
  auto moments = [&](float4 (&v)[NV], int center, Moments* out, float& mean, float& rstd) {
    float own = 0.f, m2 = 0.f;
    if (center) {
      each([&](int n, int) { own += (v[n].x + v[n].y) + (v[n].z + v[n].w); });
      own = warp_sum(own) * inv_n;
    }
    each([&](int n, int c) {
      float4 d = make_float4(v[n].x - own, v[n].y - own, v[n].z - own, v[n].w - own);
      mask(d, c);
      m2 += dot(d);
    });
    m2 = warp_sum(m2);
    if ((tid & 31) == 0) out[tid >> 5] = {warp_n, own, m2};
    __syncthreads();
    mean = 0.f;
    if (center) {
      for (int i = 0; i < warps; ++i) mean += out[i].n * out[i].mean;
      mean *= inv_d;
    }
    m2 = 0.f;
    for (int i = 0; i < warps; ++i) {
      const float d = out[i].mean - mean;
      m2 += out[i].m2 + out[i].n * d * d;
    }
    rstd = 1.0f / sqrtf(m2 * inv_d + p.eps);
  };
  auto norm4 = [&](const float4& v, float mean, float rstd, const float* w, const float* b, int c) {
    const float4 g = ld4(w, c);
    float4 o = make_float4((v.x - mean) * rstd * g.x, (v.y - mean) * rstd * g.y, (v.z - mean) * rstd * g.z, (v.w - mean) * rstd * g.w);
    if (b != nullptr) {
      const float4 a = ld4(b, c);
      o.x += a.x; o.y += a.y; o.z += a.z; o.w += a.w;
    }
    return o;
  };
  if (p.ids != nullptr) {
    const int id = min(max(p.ids[t], 0), p.vocab - 1);
    const OT* er = reinterpret_cast<const OT*>(p.embed) + (size_t)id * p.lde;
    each([&](int n, int c) {
      f[n].x = to_f(er[c]) * p.escale;
      f[n].y = c + 1 < D ? to_f(er[c + 1]) * p.escale : 0.f;
      f[n].z = c + 2 < D ? to_f(er[c + 2]) * p.escale : 0.f;
      f[n].w = c + 3 < D ? to_f(er[c + 3]) * p.escale : 0.f;
    });
  } else {
    each([&](int n, int c) { f[n] = ld4(xr, c); });
  }
  if (p.a != nullptr || p.routed != nullptr) {
    if (p.routed != nullptr) {
      if (tid < p.K) {
        pos_s[tid] = p.pos[t * p.K + tid];
        rw[tid] = p.route_w[t * p.K + tid];
      }
      __syncthreads();
      each([&](int n, int) { s[n] = make_float4(0.f, 0.f, 0.f, 0.f); });
      for (int k0 = 0; k0 < p.K; k0 += 4) {                          // four rows' loads at a time
        each([&](int n, int c) {
          float4 a[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int r = k0 + k < p.K ? pos_s[k0 + k] : -1;
            a[k] = r >= 0 ? ld4(p.routed + (size_t)r * p.ld_routed, c) : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float g = k0 + k < p.K ? rw[k0 + k] : 0.f;
            s[n].x = fmaf(g, a[k].x, s[n].x); s[n].y = fmaf(g, a[k].y, s[n].y);
            s[n].z = fmaf(g, a[k].z, s[n].z); s[n].w = fmaf(g, a[k].w, s[n].w);
          }
        });
      }
    } else {
      const float* ar = p.a + t * p.lda;
      each([&](int n, int c) { s[n] = ld4(ar, c); });
    }
    if (p.b != nullptr) {
      const float* br = p.b + t * p.ldb;
      each([&](int n, int c) { u[n] = ld4(br, c); });
      float sa = 0.f, sb = 0.f;
      each([&](int n, int c) {
        mask(s[n], c);
        mask(u[n], c);
        sa += dot(s[n]);
        sb += dot(u[n]);
      });
      sa = warp_sum(sa);
      sb = warp_sum(sb);
      if ((tid & 31) == 0) { red[0][tid >> 5] = sa; red[1][tid >> 5] = sb; }
      __syncthreads();
      float ta = 0.f, tb = 0.f;
      for (int i = 0; i < warps; ++i) { ta += red[0][i]; tb += red[1][i]; }
      const float ra = 0.5f / sqrtf(ta * inv_d + p.eps), rb = 0.5f / sqrtf(tb * inv_d + p.eps);
      each([&](int n, int c) {
        const float4 ga = ld4(p.wa, c), gb = ld4(p.wb, c);
        s[n] = make_float4(s[n].x * ra * ga.x + u[n].x * rb * gb.x, s[n].y * ra * ga.y + u[n].y * rb * gb.y,
                           s[n].z * ra * ga.z + u[n].z * rb * gb.z, s[n].w * ra * ga.w + u[n].w * rb * gb.w);
      });
    } else {
      each([&](int n, int c) { mask(s[n], c); });
    }
    float mean, rstd;
    moments(s, p.center1, part[0], mean, rstd);
    each([&](int n, int c) {
      const float4 o = norm4(s[n], mean, rstd, p.w1, p.b1, c);
      mask(f[n], c);
      f[n].x += o.x; f[n].y += o.y; f[n].z += o.z; f[n].w += o.w;
    });
  } else {
    each([&](int n, int c) { mask(f[n], c); });
  }
  if (p.keep) each([&](int n, int c) { *reinterpret_cast<float4*>(xr + c) = f[n]; });
  if (p.y == nullptr) return;
  float mean, rstd;
  if (p.w2 != nullptr) moments(f, p.center2, part[1], mean, rstd);
  OT* yr = reinterpret_cast<OT*>(p.y) + (size_t)blockIdx.x * p.ldy;
  float* hr = reinterpret_cast<float*>(p.y) + (size_t)blockIdx.x * p.ldy;
  const int slot = p.cw != nullptr ? p.slots[blockIdx.x] : -1;
  const int D4 = nv * 4;
  each([&](int n, int c) {
    float4 h = p.w2 != nullptr ? norm4(f[n], mean, rstd, p.w2, p.b2, c) : f[n];
    if (p.cw != nullptr) {                                         // y = h + conv(h); the stored inputs move up by one
      const float4 in = h;
      auto tap = [&](int j, const float4& v) {
        const float4 w = ld4(p.cw + (size_t)j * D4, c);
        h.x = fmaf(w.x, v.x, h.x); h.y = fmaf(w.y, v.y, h.y); h.z = fmaf(w.z, v.z, h.z); h.w = fmaf(w.w, v.w, h.w);
      };
      if (slot >= 0) {
        float* hs = p.hist + slot * p.hist_stride + c;
        for (int j = 0; j + 1 < p.taps; ++j) {
          const float4 old = *reinterpret_cast<const float4*>(hs + (size_t)j * D4);
          tap(j, old);
          if (j > 0) *reinterpret_cast<float4*>(hs + (size_t)(j - 1) * D4) = old;
        }
        if (p.taps > 1) *reinterpret_cast<float4*>(hs + (size_t)(p.taps - 2) * D4) = in;
      }
      tap(p.taps - 1, in);
    }
    if (p.raw) store4(hr + c, h);
    else store4(yr + c, h);
  });
  if (!p.raw)
    for (int c = D4 + tid * 4; c < p.ldy; c += NT * 4) store4(yr + c, make_float4(0.f, 0.f, 0.f, 0.f));
}

struct HyperParams {
  float* x;               // [T, S, D4] residual streams
  const long long* rows;  // [R] rows of x, or null
  const int* ids;         // first layer: token ids (every stream is written, none read)
  const void* embed;      // [V, lde]
  int lde;
  float escale;
  int vocab;
  const float* mix;       // [S, S] (from, to), or null: the streams stay
  const float* share;     // [S] factors of the sublayer's output
  const float* add;       // dense part of the output [T, ld_add], or null
  int ld_add;
  const float* bias;      // [D4] added to the output, or null
  const float* routed;    // rows of the routed experts [*, ld_routed], or null
  int ld_routed;
  const int* pos;         // [T, K] row of every (token, k) pair, < 0 = none
  const float* route_w;   // [T, K] factors of those rows
  int K;
  const float* read;      // [S] factors of the streams in what the norm reads, or null: all 1
  const float* w;         // [D4] gain
  void* y;                // [R, ldy]; columns D .. ldy are zero
  int ldy;
  int D, S;
  float eps;
  int keep;               // write the streams back
};

constexpr int kMaxStreams = 16;
constexpr int kHyperThreads = 640;

// One block per row; thread i owns the 4-wide vectors i, i + blockDim, ... of every stream.  SM: streams, or an upper bound of them
// (above 4).  What the norm reads waits in shared memory for its root mean square.
template <typename OT, int SM>
__global__ void __launch_bounds__(SM <= 4 ? kHyperThreads : kThreads) hyper_norm_kernel(const HyperParams p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ float row[];
  __shared__ float red[kHyperThreads / 32];
  __shared__ float mix[SM * SM], share[SM], read[SM], rw[kMaxK];
  __shared__ int pos_s[kMaxK];
  const int tid = threadIdx.x, NT = blockDim.x, S = SM <= 4 ? SM : p.S;
  const long long t = p.rows != nullptr ? p.rows[blockIdx.x] : (long long)blockIdx.x;
  const int D = p.D, nv = (D + 3) / 4, D4 = nv * 4;
  float* xr = p.x + t * S * D4;
  const bool pending = p.mix != nullptr;
  for (int i = tid; i < SM * SM; i += NT) mix[i] = pending && i / SM < S && i % SM < S ? p.mix[i / SM * S + i % SM] : 0.f;
  if (tid < SM) {
    share[tid] = pending && tid < S ? p.share[tid] : 0.f;
    read[tid] = tid >= S ? 0.f : p.read != nullptr ? p.read[tid] : 1.0f;
  }
  if (p.routed != nullptr && tid < p.K) {
    pos_s[tid] = p.pos[t * p.K + tid];
    rw[tid] = p.route_w[t * p.K + tid];
  }
  __syncthreads();
  const OT* er = nullptr;
  if (p.ids != nullptr) {
    const int id = min(max(p.ids[t], 0), p.vocab - 1);
    er = reinterpret_cast<const OT*>(p.embed) + (size_t)id * p.lde;
  }
  float ss = 0.f;
  for (int v = tid; v < nv; v += NT) {
    const int c = v * 4;
    float4 f[SM];
    if (er != nullptr) {
      float4 e;
      e.x = to_f(er[c]) * p.escale;
      e.y = c + 1 < D ? to_f(er[c + 1]) * p.escale : 0.f;
      e.z = c + 2 < D ? to_f(er[c + 2]) * p.escale : 0.f;
      e.w = c + 3 < D ? to_f(er[c + 3]) * p.escale : 0.f;
#pragma unroll
      for (int s = 0; s < SM; ++s) f[s] = e;
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        f[s] = s < S ? *reinterpret_cast<const float4*>(xr + (size_t)s * D4 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (pending) {
      float4 o = p.add != nullptr ? *reinterpret_cast<const float4*>(p.add + t * p.ld_add + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.bias != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(p.bias + c);
        o.x += b.x; o.y += b.y; o.z += b.z; o.w += b.w;
      }
      if (p.routed != nullptr) {
        for (int k0 = 0; k0 < p.K; k0 += 4) {            // four rows' loads at a time
          float4 a[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int r = k0 + k < p.K ? pos_s[k0 + k] : -1;
            a[k] = r >= 0 ? *reinterpret_cast<const float4*>(p.routed + (size_t)r * p.ld_routed + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float g = k0 + k < p.K ? rw[k0 + k] : 0.f;
            o.x = fmaf(g, a[k].x, o.x); o.y = fmaf(g, a[k].y, o.y); o.z = fmaf(g, a[k].z, o.z); o.w = fmaf(g, a[k].w, o.w);
          }
        }
      }
      if (c + 1 >= D) o.y = 0.f;
      if (c + 2 >= D) o.z = 0.f;
      if (c + 3 >= D) o.w = 0.f;
      float4 n[SM];
#pragma unroll
      for (int u = 0; u < SM; ++u) {
        const float g = share[u];
        n[u] = make_float4(g * o.x, g * o.y, g * o.z, g * o.w);
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          const float m = mix[s * SM + u];
          n[u].x = fmaf(m, f[s].x, n[u].x); n[u].y = fmaf(m, f[s].y, n[u].y);
          n[u].z = fmaf(m, f[s].z, n[u].z); n[u].w = fmaf(m, f[s].w, n[u].w);
        }
      }
#pragma unroll
      for (int s = 0; s < SM; ++s) f[s] = n[s];
    }
    float4 h = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < SM; ++s) {
      const float g = read[s];
      h.x = fmaf(g, f[s].x, h.x); h.y = fmaf(g, f[s].y, h.y); h.z = fmaf(g, f[s].z, h.z); h.w = fmaf(g, f[s].w, h.w);
      if (p.keep && s < S) *reinterpret_cast<float4*>(xr + (size_t)s * D4 + c) = f[s];
    }
    *reinterpret_cast<float4*>(row + c) = h;
    ss += h.x * h.x + h.y * h.y + h.z * h.z + h.w * h.w;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < NT / 32; ++i) tot += red[i];
  const float rstd = 1.0f / sqrtf(tot / (float)D + p.eps);
  OT* yr = reinterpret_cast<OT*>(p.y) + (size_t)blockIdx.x * p.ldy;
  for (int v = tid; v < p.ldy / 4; v += NT) {
    const int c = v * 4;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D) {                                        // gains and the row are zero from D to D4
      const float4 h = *reinterpret_cast<const float4*>(row + c), g = *reinterpret_cast<const float4*>(p.w + c);
      o = make_float4(h.x * rstd * g.x, h.y * rstd * g.y, h.z * rstd * g.z, h.w * rstd * g.w);
    }
    store4(yr + c, o);
  }
}

__device__ __forceinline__ float sigmoid_acc(float x) { return 1.0f / (1.0f + expf(-x)); }

template <int KIND>
__device__ __forceinline__ float glu_one(float g, float u, float limit) {
  if (KIND == 0) {                                     // tanh-GELU(g) * u
    const float t = tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g));
    return 0.5f * g * (1.0f + t) * u;
  }
  if (KIND == 2) return g * sigmoid_acc(g) * u;        // SiLU(g) * u
  if (KIND == 3) {                                     // squared ReLU, no gate
    g = fmaxf(g, 0.f);
    return g * g;
  }
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_acc(1.702f * g) * (u + 1.0f);
}

// out[r, c] = act(s * z[r, g0 + c], s * z[r, u0 + c]) * sigmoid(gate[r]); s = row_scale[r], or 1.  Columns F .. Fo of the
// output are zero.
template <typename OT, int KIND>
__global__ void __launch_bounds__(kThreads)
glu_kernel(const float* __restrict__ z, int ldz, int u_off, OT* __restrict__ out, int ldo, int F, int Fo, float limit,
           const float* __restrict__ row_scale, const float* __restrict__ gate, int ld_gate,
           const int* __restrict__ total_rows) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int r = blockIdx.x;
  if (total_rows != nullptr && r >= *total_rows) return;
  const int c = (blockIdx.y * kThreads + threadIdx.x) * 4;
  if (c >= Fo) return;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < F) {                                          // F % 4 == 0
    const float s = row_scale != nullptr ? row_scale[r] : 1.0f;
    const float m = gate != nullptr ? sigmoid_acc(gate[(size_t)r * ld_gate]) : 1.0f;
    const float* zr = z + (size_t)r * ldz + c;
    const float4 g = *reinterpret_cast<const float4*>(zr);
    const float4 u = KIND == 3 ? g : *reinterpret_cast<const float4*>(zr + u_off);
    o.x = glu_one<KIND>(g.x * s, u.x * s, limit) * m;
    o.y = glu_one<KIND>(g.y * s, u.y * s, limit) * m;
    o.z = glu_one<KIND>(g.z * s, u.z * s, limit) * m;
    o.w = glu_one<KIND>(g.w * s, u.w * s, limit) * m;
  }
  store4(out + (size_t)r * ldo + c, o);
}

// out[t, c] = tanh-GELU(z[t, c]) * table[ids[t], c], zero for c >= n
template <typename OT>
__global__ void __launch_bounds__(kThreads)
token_side_kernel(const float* __restrict__ z, int ldz, const OT* __restrict__ table, long long ldt, const int* __restrict__ ids, int vocab,
                  OT* __restrict__ out, int ldo, int T, int n) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int i = blockIdx.x * kThreads + threadIdx.x;
  const int t = i / ldo, c = i % ldo;
  if (t >= T) return;
  float v = 0.f;
  if (c < n) v = glu_one<0>(z[(size_t)t * ldz + c], to_f(table[min(max(ids[t], 0), vocab - 1) * ldt + c]), 0.f);
  out[(size_t)t * ldo + c] = from_f<OT>(v);
}

template <typename OT, int KIND>
__global__ void __launch_bounds__(kThreads)
cast_act_kernel(const float* __restrict__ x, int ldx, OT* __restrict__ out, int ldo, int T, int N) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int i = blockIdx.x * kThreads + threadIdx.x;
  const int t = i / ldo, c = i % ldo;
  if (t >= T) return;
  float v = 0.f;
  if (c < N) {
    v = x[(size_t)t * ldx + c];
    if (KIND == 1) v = tanhf(v);
    if (KIND == 2) { v = fmaxf(v, 0.f); v *= v; }
  }
  out[(size_t)t * ldo + c] = from_f<OT>(v);
}

// one block per (token, k) pair: xs[pos[pair]] = x[token], ws[pos[pair]] = w[pair]
template <typename OT>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const OT* __restrict__ x, int ldx, const int* __restrict__ pos, const float* __restrict__ w,
                  OT* __restrict__ xs, float* __restrict__ ws, int K, int bytes) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int pair = blockIdx.x;
  const int r = pos[pair];
  if (r < 0) return;
  if (threadIdx.x == 0) ws[r] = w[pair];
  const uint4* src = reinterpret_cast<const uint4*>(x + (size_t)(pair / K) * ldx);
  uint4* dst = reinterpret_cast<uint4*>(xs + (size_t)r * ldx);
  for (int i = threadIdx.x; i < bytes / 16; i += blockDim.x) dst[i] = src[i];
}

}  // namespace resid
}  // namespace bg

extern "C" {

// dt: 0 = bf16, 1 = fp32 (embedding table and output).  ldx, ldy, ld_add, ld_routed: multiples of 4 with ld >= D rounded
// up to 4; R rows.
int bg_residual_norm(int dt, float* x, int ldx, const long long* rows, const int* ids, const void* embed, int lde,
                     float escale, int vocab, const float* add, int ld_add, const float* routed, int ld_routed,
                     const int* pos, int K, const float* w, void* y, int ldy, int R, int D, float eps, int keep,
                     cudaStream_t stream) {
  using namespace bg::resid;
  if (R <= 0) return 0;
  const int D4 = (D + 3) / 4 * 4;
  if (D <= 0 || D4 > 49152 / 4 || ldx % 4 || ldx < D4 || ldy % 4 || ldy < D4 || (add != nullptr && (ld_add % 4 || ld_add < D4)) ||
      (routed != nullptr && (ld_routed % 4 || ld_routed < D4 || K <= 0 || K > kMaxK || pos == nullptr)) ||
      (ids != nullptr && (embed == nullptr || vocab <= 0)))
    return -1;
  NormParams p;
  p.x = x; p.ldx = ldx; p.rows = rows; p.ids = ids; p.embed = embed; p.lde = lde; p.escale = escale; p.vocab = vocab;
  p.add = add; p.ld_add = ld_add; p.routed = routed; p.ld_routed = ld_routed; p.pos = pos; p.K = K;
  p.w = w; p.y = y; p.ldy = ldy; p.D = D; p.eps = eps; p.keep = keep;
  const size_t smem = (size_t)D4 * sizeof(float);
  if (dt == 0) bg::launch_pdl(residual_norm_kernel<__nv_bfloat16>, dim3(R), dim3(kThreads), smem, stream, p);
  else bg::launch_pdl(residual_norm_kernel<float>, dim3(R), dim3(kThreads), smem, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// dt: 0 = bf16, 1 = fp32 (embedding table and output).  Leading dimensions: multiples of 4, at least D rounded up to 4; vectors
// of the norms hold that many floats.  D <= 16384.  a and routed null: nothing joins x; ids: x = embed[ids] * escale; w2 null: no
// norm of x; y null: only x is written.
int bg_sandwich_norm(int dt, float* x, int ldx, const long long* rows, const int* ids, const void* embed, int lde, float escale,
                     int vocab, const float* a, int lda, const float* b, int ldb, const float* wa, const float* wb, const float* routed,
                     int ld_routed, const int* pos, const float* route_w, int K, const float* w1, const float* b1, int center1, const float* w2, const float* b2, int center2, void* y, int ldy, int raw,
                     const float* cw, float* hist, long long hist_stride, const int* slots, int taps, int R, int D, float eps,
                     int keep, cudaStream_t stream) {
  using namespace bg::resid;
  if (R <= 0) return 0;
  const int D4 = (D + 3) / 4 * 4;
  if (D <= 0 || D > 16384 || ldx % 4 || ldx < D4 || ldy % 4 || ldy < D4 || (raw && ldy != D4) || (y == nullptr && cw != nullptr) ||
      (a != nullptr && (lda % 4 || lda < D4 || w1 == nullptr || routed != nullptr)) ||
      (routed != nullptr && (ld_routed % 4 || ld_routed < D4 || K <= 0 || K > kMaxK || pos == nullptr || route_w == nullptr || w1 == nullptr)) ||
      (b != nullptr && (a == nullptr || ldb % 4 || ldb < D4 || wa == nullptr || wb == nullptr)) ||
      (ids != nullptr && (embed == nullptr || vocab <= 0)) ||
      (cw != nullptr && (slots == nullptr || taps < 1 || (taps > 1 && hist == nullptr) || hist_stride % 4 || rows != nullptr)))
    return -1;
  SandwichParams p;
  p.x = x; p.ldx = ldx; p.rows = rows; p.ids = ids; p.embed = embed; p.lde = lde; p.escale = escale; p.vocab = vocab;
  p.a = a; p.b = b; p.lda = lda; p.ldb = ldb; p.wa = wa; p.wb = wb; p.routed = routed; p.ld_routed = ld_routed; p.pos = pos;
  p.route_w = route_w; p.K = K; p.w1 = w1; p.b1 = b1; p.center1 = center1;
  p.w2 = w2; p.b2 = b2; p.center2 = center2; p.y = y; p.ldy = ldy; p.raw = raw; p.cw = cw; p.hist = hist;
  p.hist_stride = hist_stride; p.slots = slots; p.taps = taps; p.D = D; p.eps = eps; p.keep = keep;
  const int nv = D4 / 4;
#define BG_SANDWICH(NV)                                                                                             \
  do {                                                                                                              \
    const dim3 block(((nv + NV - 1) / NV + 31) / 32 * 32);                                                          \
    if (dt == 0) bg::launch_pdl(sandwich_norm_kernel<__nv_bfloat16, NV>, dim3(R), block, 0, stream, p);             \
    else bg::launch_pdl(sandwich_norm_kernel<float, NV>, dim3(R), block, 0, stream, p);                             \
  } while (0)
  switch ((nv + kThreads - 1) / kThreads) {
    case 1: BG_SANDWICH(1); break;
    case 2: BG_SANDWICH(2); break;
    case 3: BG_SANDWICH(3); break;
    case 4: BG_SANDWICH(4); break;
    case 5:
    case 6: BG_SANDWICH(6); break;
    case 7:
    case 8: BG_SANDWICH(8); break;
    default: BG_SANDWICH(16); break;
  }
#undef BG_SANDWICH
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// x [T, S, D4] (D4 = D rounded up to 4); the other leading dimensions: multiples of 4, at least D4; bias and w hold D4 floats.
// D4 <= 8192, S <= 16.  mix null: nothing joins the streams; ids: every stream = embed[ids] * escale.
int bg_hyper_norm(int dt, float* x, const long long* rows, const int* ids, const void* embed, int lde, float escale, int vocab,
                  const float* mix, const float* share, const float* add, int ld_add, const float* bias, const float* routed,
                  int ld_routed, const int* pos, const float* route_w, int K, const float* read, const float* w, void* y, int ldy,
                  int R, int D, int S, float eps, int keep, cudaStream_t stream) {
  using namespace bg::resid;
  if (R <= 0) return 0;
  const int D4 = (D + 3) / 4 * 4;
  if (D <= 0 || D4 > 8192 || S <= 0 || S > kMaxStreams || ldy % 4 || ldy < D4 || (add != nullptr && (ld_add % 4 || ld_add < D4)) ||
      (routed != nullptr && (ld_routed % 4 || ld_routed < D4 || K <= 0 || K > kMaxK || pos == nullptr || route_w == nullptr)) ||
      (ids != nullptr && (embed == nullptr || vocab <= 0)) || (mix != nullptr && share == nullptr) ||
      (mix == nullptr && (add != nullptr || routed != nullptr || bias != nullptr)))
    return -1;
  HyperParams p;
  p.x = x; p.rows = rows; p.ids = ids; p.embed = embed; p.lde = lde; p.escale = escale; p.vocab = vocab; p.mix = mix;
  p.share = share; p.add = add; p.ld_add = ld_add; p.bias = bias; p.routed = routed; p.ld_routed = ld_routed; p.pos = pos;
  p.route_w = route_w; p.K = K; p.read = read; p.w = w; p.y = y; p.ldy = ldy; p.D = D; p.S = S; p.eps = eps; p.keep = keep;
  // few rows: as many threads as vectors, so that a row's loads fly together
  const int most = R <= 296 && S <= 4 ? kHyperThreads : kThreads;
  const int nv = D4 / 4, per = (nv + most - 1) / most;
  const dim3 block(((nv + per - 1) / per + 31) / 32 * 32);
  const size_t smem = (size_t)D4 * sizeof(float);
#define BG_HYPER(SM)                                                                                              \
  do {                                                                                                            \
    if (dt == 0) bg::launch_pdl(hyper_norm_kernel<__nv_bfloat16, SM>, dim3(R), block, smem, stream, p);            \
    else bg::launch_pdl(hyper_norm_kernel<float, SM>, dim3(R), block, smem, stream, p);                            \
  } while (0)
  if (S == 1) BG_HYPER(1);
  else if (S == 2) BG_HYPER(2);
  else if (S == 3) BG_HYPER(3);
  else if (S == 4) BG_HYPER(4);
  else if (S <= 8) BG_HYPER(8);
  else BG_HYPER(16);
#undef BG_HYPER
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// kind 0 tanh-GELU, 1 clamped SwiGLU, 2 SwiGLU, 3 squared ReLU (no up column).  z points at the first gate column, the up column of a gate column is u_off further.
int bg_glu(int dt, int kind, const float* z, int ldz, int u_off, void* out, int ldo, int R, int F, int Fo, float limit,
           const float* row_scale, const float* gate, int ld_gate, const int* total_rows, cudaStream_t stream) {
  using namespace bg::resid;
  if (R <= 0 || Fo <= 0) return 0;
  if (F % 4 || Fo % 4 || F > Fo || ldz % 4 || u_off % 4 || ldo % 4 || ldo < Fo) return -1;
  const dim3 grid(R, (Fo / 4 + kThreads - 1) / kThreads);
#define BG_GLU(OT, KIND)                                                                                      \
  bg::launch_pdl(glu_kernel<OT, KIND>, grid, dim3(kThreads), 0, stream, z, ldz, u_off, reinterpret_cast<OT*>(out), ldo, F, \
                 Fo, limit, row_scale, gate, ld_gate, total_rows)
  if (dt == 0 && kind == 0) BG_GLU(__nv_bfloat16, 0);
  else if (dt == 0 && kind == 1) BG_GLU(__nv_bfloat16, 1);
  else if (dt == 0 && kind == 2) BG_GLU(__nv_bfloat16, 2);
  else if (dt == 0) BG_GLU(__nv_bfloat16, 3);
  else if (kind == 0) BG_GLU(float, 0);
  else if (kind == 1) BG_GLU(float, 1);
  else if (kind == 2) BG_GLU(float, 2);
  else BG_GLU(float, 3);
#undef BG_GLU
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// z [T, ldz] fp32, table rows of ldt elements (the first n count), ids [T] -> out [T, ldo]
int bg_token_side(int dt, const float* z, int ldz, const void* table, long long ldt, const int* ids, int vocab, void* out, int ldo, int T,
                  int n, cudaStream_t stream) {
  using namespace bg::resid;
  if (T <= 0 || ldo <= 0) return 0;
  if (n < 0 || n > ldo || n > ldz || n > ldt || vocab <= 0 || (long long)T * ldo > 0x7fffffffll) return -1;
  const dim3 grid((unsigned)(((long long)T * ldo + kThreads - 1) / kThreads));
  if (dt == 0)
    bg::launch_pdl(token_side_kernel<__nv_bfloat16>, grid, dim3(kThreads), 0, stream, z, ldz, reinterpret_cast<const __nv_bfloat16*>(table),
                   ldt, ids, vocab, reinterpret_cast<__nv_bfloat16*>(out), ldo, T, n);
  else
    bg::launch_pdl(token_side_kernel<float>, grid, dim3(kThreads), 0, stream, z, ldz, reinterpret_cast<const float*>(table), ldt, ids, vocab,
                   reinterpret_cast<float*>(out), ldo, T, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// out [T, ldo] = f(x[:, :N]) with zero columns N .. ldo; kind 0 identity, 1 tanh, 2 squared ReLU
int bg_cast_act(int dt, int kind, const float* x, int ldx, void* out, int ldo, int T, int N, cudaStream_t stream) {
  using namespace bg::resid;
  if (T <= 0 || ldo <= 0) return 0;
  if (N > ldo || (long long)T * ldo > 0x7fffffffll) return -1;
  const dim3 grid((unsigned)(((long long)T * ldo + kThreads - 1) / kThreads));
#define BG_CAST(OT, KIND) \
  bg::launch_pdl(cast_act_kernel<OT, KIND>, grid, dim3(kThreads), 0, stream, x, ldx, reinterpret_cast<OT*>(out), ldo, T, N)
  if (dt == 0 && kind == 0) BG_CAST(__nv_bfloat16, 0);
  else if (dt == 0 && kind == 1) BG_CAST(__nv_bfloat16, 1);
  else if (dt == 0) BG_CAST(__nv_bfloat16, 2);
  else if (kind == 0) BG_CAST(float, 0);
  else if (kind == 1) BG_CAST(float, 1);
  else BG_CAST(float, 2);
#undef BG_CAST
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// x [T, ldx] rows of ldx elements -> xs [*, ldx]; ldx * element size a multiple of 16 bytes
int bg_moe_gather(int dt, const void* x, int ldx, const int* pos, const float* w, void* xs, float* ws, int T, int K,
                  cudaStream_t stream) {
  using namespace bg::resid;
  if (T <= 0) return 0;
  const int bytes = ldx * (dt == 0 ? 2 : 4);
  if (bytes % 16 || K <= 0) return -1;
  if (dt == 0)
    bg::launch_pdl(moe_gather_kernel<__nv_bfloat16>, dim3(T * K), dim3(128), 0, stream,
                   reinterpret_cast<const __nv_bfloat16*>(x), ldx, pos, w, reinterpret_cast<__nv_bfloat16*>(xs), ws, K, bytes);
  else
    bg::launch_pdl(moe_gather_kernel<float>, dim3(T * K), dim3(128), 0, stream, reinterpret_cast<const float*>(x), ldx, pos,
                   w, reinterpret_cast<float*>(xs), ws, K, bytes);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(residual)
