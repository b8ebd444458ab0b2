// Row kernels of models with an fp32 residual stream and parallel blocks (mixer and feed-forward read one norm):
//
//   residual_norm   x[t] += sum of the sublayers' fp32 outputs (dense rows and / or routed rows gathered by position),
//                   or x[t] = embed[id] * scale for the first layer; y[t] = x[t] / sqrt(mean(x^2) + eps) * w
//   glu             gated activations (tanh-GELU, clamped SwiGLU with slope 1.702 and u + 1), with an optional factor on
//                   the pre-activations (routing weight applied to the expert's input) and an optional sigmoid gate
//   cast_act        out = f(x), f = tanh or identity: fp32 columns of a projection to the operand type of the next one
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

__device__ __forceinline__ float sigmoid_acc(float x) { return 1.0f / (1.0f + expf(-x)); }

template <int KIND>
__device__ __forceinline__ float glu_one(float g, float u, float limit) {
  if (KIND == 0) {                                     // tanh-GELU(g) * u
    const float t = tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g));
    return 0.5f * g * (1.0f + t) * u;
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
    const float4 u = *reinterpret_cast<const float4*>(zr + u_off);
    o.x = glu_one<KIND>(g.x * s, u.x * s, limit) * m;
    o.y = glu_one<KIND>(g.y * s, u.y * s, limit) * m;
    o.z = glu_one<KIND>(g.z * s, u.z * s, limit) * m;
    o.w = glu_one<KIND>(g.w * s, u.w * s, limit) * m;
  }
  store4(out + (size_t)r * ldo + c, o);
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

// kind 0 tanh-GELU, 1 clamped SwiGLU.  z points at the first gate column, the up column of a gate column is u_off further.
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
  else if (dt == 0) BG_GLU(__nv_bfloat16, 1);
  else if (kind == 0) BG_GLU(float, 0);
  else BG_GLU(float, 1);
#undef BG_GLU
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// out [T, ldo] = f(x[:, :N]) with zero columns N .. ldo; kind 0 identity, 1 tanh
int bg_cast_act(int dt, int kind, const float* x, int ldx, void* out, int ldo, int T, int N, cudaStream_t stream) {
  using namespace bg::resid;
  if (T <= 0 || ldo <= 0) return 0;
  if (N > ldo || (long long)T * ldo > 0x7fffffffll) return -1;
  const dim3 grid((unsigned)(((long long)T * ldo + kThreads - 1) / kThreads));
#define BG_CAST(OT, KIND) \
  bg::launch_pdl(cast_act_kernel<OT, KIND>, grid, dim3(kThreads), 0, stream, x, ldx, reinterpret_cast<OT*>(out), ldo, T, N)
  if (dt == 0 && kind == 0) BG_CAST(__nv_bfloat16, 0);
  else if (dt == 0) BG_CAST(__nv_bfloat16, 1);
  else if (kind == 0) BG_CAST(float, 0);
  else BG_CAST(float, 1);
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
