// What a step does to attention heads between their projections and the scores, in one kernel: bias, RMS norm per query and key
// head, rotary positions; keys and values go to the paged cache, queries back to their columns (fp32, for the row kernel) and / or
// into the bf16 operand of the prompt kernel, times scale * log2(e).
//
// A warp takes one head of one token.  Norms and rotations are fp32; channels past the real width stay zero (zero weights and
// biases).  Pairs that turn together: (i, i + half), or (2 i, 2 i + 1) when interleaved.
#define BG_FILE_TAG 30     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace heads {

constexpr int kWarps = 8;
constexpr int kMaxWidth = 1024;

struct Params {
  float* z;               // [T, ld]: H query heads of dp, G key heads of dp, G value heads of dvp
  int ld;
  const float* bias;      // [H dp + row] or null
  const float *wq, *wk;   // [dp] gains of the heads' norms, or null (no norm)
  float eps, inv_d;       // 1 / real head width
  const float* rope;      // [T, 2 * half] cosines, then sines, or null
  int half, interleaved;
  const long long* slots; // [T] cache slots, < 0: not written
  void* cache;            // [pages, page, row]
  long long page_stride;
  int page, row;
  int write_q;            // queries go back to z
  __nv_bfloat16* qf;      // [T, H, kc] or null
  int kc;
  float q_scale;
  int H, G, dp, dvp;
};

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 biased(const float* z, const float* b, int c) {
  float4 v = ld4(z + c);
  if (b != nullptr) {
    const float4 a = ld4(b + c);
    v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
  }
  return v;
}

template <typename KT>
__global__ void __launch_bounds__(kWarps * 32) prep_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, u = blockIdx.y * kWarps + warp;
  if (u >= p.H + 2 * p.G) return;
  const bool query = u < p.H;
  const long long slot = query ? -1 : p.slots[t];
  if (!query && slot < 0) return;
  KT* dst = query ? nullptr : reinterpret_cast<KT*>(p.cache) + (slot / p.page) * p.page_stride + (slot % p.page) * p.row;
  const int qk = (p.H + p.G) * p.dp;
  if (u >= p.H + p.G) {                                          // a value head: bias only
    const int g = u - p.H - p.G;
    const float* z = p.z + (size_t)t * p.ld + qk + g * p.dvp;
    const float* b = p.bias != nullptr ? p.bias + qk + g * p.dvp : nullptr;
    for (int c = lane * 4; c < p.dvp; c += 128) put4(dst + p.G * p.dp + g * p.dvp + c, biased(z, b, c));
    return;
  }
  float* z = p.z + (size_t)t * p.ld + u * p.dp;
  const float* b = p.bias != nullptr ? p.bias + u * p.dp : nullptr;
  const float* w = query ? p.wq : p.wk;
  float* head = sm + warp * p.dp;
  float ss = 0.f;
  for (int c = lane * 4; c < p.dp; c += 128) {
    const float4 v = biased(z, b, c);
    put4(head + c, v);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  if (w != nullptr) {
    const float rstd = 1.0f / sqrtf(warp_sum(ss) * p.inv_d + p.eps);
    for (int c = lane * 4; c < p.dp; c += 128) {
      const float4 v = ld4(head + c), g = ld4(w + c);
      put4(head + c, make_float4(v.x * rstd * g.x, v.y * rstd * g.y, v.z * rstd * g.z, v.w * rstd * g.w));
    }
  }
  __syncwarp();
  const float* cs = p.rope != nullptr ? p.rope + (size_t)t * 2 * p.half : nullptr;
  auto turned = [&](int c) -> float4 {                           // channels c .. c + 3
    float4 v = ld4(head + c);
    if (cs == nullptr || c >= 2 * p.half) return v;
    float* x = &v.x;
    if (p.interleaved) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int i = (c + j) >> 1;
        if (i < p.half) {
          const float a = x[j], d = x[j + 1], co = cs[i], si = cs[p.half + i];
          x[j] = a * co - d * si;
          x[j + 1] = d * co + a * si;
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int e = c + j;
        if (e < 2 * p.half) {
          const bool low = e < p.half;
          const int i = low ? e : e - p.half;
          const float other = head[low ? e + p.half : i], co = cs[i], si = cs[p.half + i];
          x[j] = low ? x[j] * co - other * si : x[j] * co + other * si;
        }
      }
    }
    return v;
  };
  if (!query) {
    KT* k = dst + (u - p.H) * p.dp;
    for (int c = lane * 4; c < p.dp; c += 128) put4(k + c, turned(c));
    return;
  }
  __nv_bfloat16* qf = p.qf != nullptr ? p.qf + ((size_t)t * p.H + u) * p.kc : nullptr;
  for (int c = lane * 4; c < p.dp; c += 128) {
    const float4 v = turned(c);
    if (p.write_q) put4(z + c, v);
    if (qf != nullptr) put4(qf + c, make_float4(v.x * p.q_scale, v.y * p.q_scale, v.z * p.q_scale, v.w * p.q_scale));
  }
  if (qf != nullptr)
    for (int c = p.dp + lane * 4; c < p.kc; c += 128) put4(qf + c, make_float4(0.f, 0.f, 0.f, 0.f));
}

}  // namespace heads
}  // namespace bg

extern "C" {

// dt: 0 = bf16 cache, 1 = fp32.  z: T rows of ld floats, the heads' columns first; row = G (dp + dvp); d: real width of query and
// key heads (for the norms).  qf [T, H, kc] bf16 or null.
int bg_head_prep(int dt, float* z, int ld, const float* bias, const float* wq, const float* wk, float eps, int d, const float* rope,
                 int half, int interleaved, const long long* slots, void* cache, long long page_stride, int page, int row, int write_q,
                 void* qf, int kc, float scale, int T, int H, int G, int dp, int dvp, cudaStream_t stream) {
  using namespace bg::heads;
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || dp <= 0 || dp % 8 || dp > kMaxWidth || d <= 0 || d > dp || dvp <= 0 || dvp % 8 || row != G * (dp + dvp) ||
      ld % 4 || ld < H * dp + row || page <= 0 || page_stride % 8 || (rope != nullptr && (half <= 0 || 2 * half > dp)) ||
      (qf != nullptr && (kc < dp || kc % 8)) || (wq == nullptr) != (wk == nullptr) || reinterpret_cast<uintptr_t>(z) % 16)
    return -1;
  Params p;
  p.z = z; p.ld = ld; p.bias = bias; p.wq = wq; p.wk = wk; p.eps = eps; p.inv_d = 1.0f / (float)d; p.rope = rope; p.half = half;
  p.interleaved = interleaved; p.slots = slots; p.cache = cache; p.page_stride = page_stride; p.page = page; p.row = row;
  p.write_q = write_q; p.qf = reinterpret_cast<__nv_bfloat16*>(qf); p.kc = kc; p.q_scale = scale * 1.4426950408889634f;
  p.H = H; p.G = G; p.dp = dp; p.dvp = dvp;
  const dim3 grid(T, (H + 2 * G + kWarps - 1) / kWarps), block(kWarps * 32);
  if (grid.y > 65535) return -1;
  const size_t smem = (size_t)kWarps * dp * sizeof(float);
  if (dt == 0) bg::launch_pdl(prep_kernel<__nv_bfloat16>, grid, block, smem, stream, p);
  else bg::launch_pdl(prep_kernel<float>, grid, block, smem, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(head_prep)
