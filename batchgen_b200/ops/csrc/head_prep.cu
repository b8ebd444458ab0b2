// What a step does to attention heads between their projections and the scores, in one kernel: bias, RMS norm per query and key
// head (or over all query heads and over all key heads at once), rotary positions; keys and values go to the paged cache, queries back to their columns (fp32, for the row kernel) and / or
// into the bf16 operand of the prompt kernel, times scale * log2(e).
//
// A warp takes kHeads heads of one token, with norms over all heads a block takes the token; all loads are issued before any is used.
// Norms and rotations are fp32; channels past the real width stay zero (zero weights and
// biases).  Pairs that turn together: (i, i + half), or (2 i, 2 i + 1) when interleaved.
#define BG_FILE_TAG 30     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace heads {

constexpr int kWarps = 8;
constexpr int kHeads = 2;      // of a warp: u and u + kWarps
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
  int page, shift, row;   // tokens per page = 2^shift, elements per token
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

// NV: 4-wide vectors of a head in a lane's registers (widths up to 128 NV)
template <typename KT, int NV, bool INTER>
__global__ void __launch_bounds__(kWarps * 32) prep_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, units = p.H + 2 * p.G, qk = (p.H + p.G) * p.dp;
  const float* zr = p.z + (size_t)t * p.ld;
  const float* cs = p.rope != nullptr ? p.rope + (size_t)t * 2 * p.half : nullptr;
  const long long slot = p.slots[t];
  float4 v[kHeads][NV];
  int off[kHeads], width[kHeads];                                 // first column, 0 = no head
#pragma unroll
  for (int i = 0; i < kHeads; ++i) {
    const int u = blockIdx.y * kWarps * kHeads + i * kWarps + warp, g = u - p.H - p.G;
    off[i] = g < 0 ? u * p.dp : qk + g * p.dvp;
    width[i] = u >= units || (u >= p.H && slot < 0) ? 0 : g < 0 ? p.dp : p.dvp;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int c = lane * 4 + n * 128;
      v[i][n] = c < width[i] ? ld4(zr + off[i] + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  KT* dst = reinterpret_cast<KT*>(p.cache) + (slot >> p.shift) * p.page_stride + (int)(slot & (p.page - 1)) * (long long)p.row;
#pragma unroll
  for (int i = 0; i < kHeads; ++i) {
    if (width[i] == 0) continue;                                  // the same for all lanes of the warp
    const int u = blockIdx.y * kWarps * kHeads + i * kWarps + warp;
    const bool query = u < p.H, value = u >= p.H + p.G;
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int c = lane * 4 + n * 128;
      if (c < width[i] && p.bias != nullptr) {
        const float4 a = ld4(p.bias + off[i] + c);
        v[i][n].x += a.x; v[i][n].y += a.y; v[i][n].z += a.z; v[i][n].w += a.w;
      }
      ss += v[i][n].x * v[i][n].x + v[i][n].y * v[i][n].y + v[i][n].z * v[i][n].z + v[i][n].w * v[i][n].w;
    }
    if (value) {
#pragma unroll
      for (int n = 0; n < NV; ++n)
        if (lane * 4 + n * 128 < p.dvp) put4(dst + off[i] - p.H * p.dp + lane * 4 + n * 128, v[i][n]);
      continue;
    }
    const float* w = query ? p.wq : p.wk;
    if (w != nullptr) {
      const float rstd = 1.0f / sqrtf(warp_sum(ss) * p.inv_d + p.eps);
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int c = lane * 4 + n * 128;
        if (c < p.dp) {
          const float4 g = ld4(w + c);
          v[i][n] = make_float4(v[i][n].x * rstd * g.x, v[i][n].y * rstd * g.y, v[i][n].z * rstd * g.z, v[i][n].w * rstd * g.w);
        }
      }
    }
    float* head = sm + warp * p.dp;                               // (i, i + half): the partner may sit in another lane
    if (cs != nullptr && !INTER) {
      __syncwarp();
#pragma unroll
      for (int n = 0; n < NV; ++n)
        if (lane * 4 + n * 128 < p.dp) put4(head + lane * 4 + n * 128, v[i][n]);
      __syncwarp();
    }
    __nv_bfloat16* qf = query && p.qf != nullptr ? p.qf + ((size_t)t * p.H + u) * p.kc : nullptr;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int c = lane * 4 + n * 128;
      if (c >= p.dp) continue;
      float* x = &v[i][n].x;
      if (cs != nullptr) {
        if (INTER) {
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            const int k = (c + j) >> 1;
            if (k < p.half) {
              const float a = x[j], d = x[j + 1], co = cs[k], si = cs[p.half + k];
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
              const int k = low ? e : e - p.half;
              const float other = head[low ? e + p.half : k], co = cs[k], si = cs[p.half + k];
              x[j] = low ? x[j] * co - other * si : x[j] * co + other * si;
            }
          }
        }
      }
      if (!query) {
        put4(dst + off[i] - p.H * p.dp + c, v[i][n]);
        continue;
      }
      if (p.write_q) put4(p.z + (size_t)t * p.ld + off[i] + c, v[i][n]);
      if (qf != nullptr) put4(qf + c, make_float4(x[0] * p.q_scale, x[1] * p.q_scale, x[2] * p.q_scale, x[3] * p.q_scale));
    }
    if (qf != nullptr)
      for (int c = p.dp + lane * 4; c < p.kc; c += 128) put4(qf + c, make_float4(0.f, 0.f, 0.f, 0.f));
  }
}

// Norms over all heads: a block takes a token, NV vectors of 4 columns a thread; wq [H dp], wk [G dp].  With rotary positions the normed
// queries and keys wait in shared memory for their partners.
constexpr int kWholeThreads = 512;
template <typename KT, int NV>
__global__ void __launch_bounds__(kWholeThreads) whole_kernel(const Params p, float inv_q, float inv_k) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[2][kWholeThreads / 32];
  const int tid = threadIdx.x, t = blockIdx.x, NT = blockDim.x;
  const int nq = p.H * p.dp, nk = nq + p.G * p.dp, n = nq + p.row;
  float* zr = p.z + (size_t)t * p.ld;
  const float* cs = p.rope != nullptr ? p.rope + (size_t)t * 2 * p.half : nullptr;
  const long long slot = p.slots[t];
  float4 v[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * NT) * 4;
    v[i] = c < n ? ld4(zr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * NT) * 4;
    if (c < n && p.bias != nullptr) {
      const float4 a = ld4(p.bias + c);
      v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
    }
    const float ss = v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    if (c < nq) sq += ss;
    else if (c < nk) sk += ss;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
  }
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int i = 0; i < NT / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float rq = 1.0f / sqrtf(sq * inv_q + p.eps), rk = 1.0f / sqrtf(sk * inv_k + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * NT) * 4;
    if (c >= nk) continue;
    const float4 g = ld4(c < nq ? p.wq + c : p.wk + c - nq);
    const float r = c < nq ? rq : rk;
    v[i] = make_float4(v[i].x * r * g.x, v[i].y * r * g.y, v[i].z * r * g.z, v[i].w * r * g.w);
    if (cs != nullptr) put4(sm + c, v[i]);
  }
  if (cs != nullptr) __syncthreads();
  KT* dst = reinterpret_cast<KT*>(p.cache) + (slot >> p.shift) * p.page_stride + (int)(slot & (p.page - 1)) * (long long)p.row;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * NT) * 4;
    if (c >= n) continue;
    const int h = c / p.dp, e = c - h * p.dp;                        // dp % 8 == 0: the four channels share a head
    float* x = &v[i].x;
    if (cs != nullptr && c < nk) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int f = e + j;
        if (f >= 2 * p.half) continue;
        const bool first = p.interleaved ? (f & 1) == 0 : f < p.half;
        const int k = p.interleaved ? f >> 1 : first ? f : f - p.half;
        const int other = p.interleaved ? f ^ 1 : first ? f + p.half : k;
        const float a = sm[c + j], b = sm[h * p.dp + other], co = cs[k], si = cs[p.half + k];
        x[j] = first ? a * co - b * si : a * co + b * si;
      }
    }
    if (c >= nq) {
      if (slot >= 0) put4(dst + c - nq, v[i]);
      continue;
    }
    if (p.write_q) put4(zr + c, v[i]);
    if (p.qf != nullptr) {
      __nv_bfloat16* qf = p.qf + ((size_t)t * p.H + h) * p.kc;
      put4(qf + e, make_float4(x[0] * p.q_scale, x[1] * p.q_scale, x[2] * p.q_scale, x[3] * p.q_scale));
      if (e + 4 == p.dp)
        for (int k = p.dp; k < p.kc; k += 4) put4(qf + k, make_float4(0.f, 0.f, 0.f, 0.f));
    }
  }
}

template <typename KT>
static int launch_whole(const Params& p, int T, float inv_q, float inv_k, cudaStream_t stream) {
  const int vecs = (p.H * p.dp + p.row) / 4;
  const size_t smem = p.rope != nullptr ? (size_t)(p.H + p.G) * p.dp * sizeof(float) : 0;
  if (vecs > 16 * kWholeThreads || smem > 200 * 1024) return -3;
#define BG_WHOLE(NV)                                                                                       \
  do {                                                                                                     \
    static DeviceOnce once;                                                                                \
    auto kern = whole_kernel<KT, NV>;                                                                      \
    if (smem > 40 * 1024 && !ensure_dynamic_smem(kern, 200 * 1024, once)) return -4;                       \
    const dim3 block(((vecs + NV - 1) / NV + 31) / 32 * 32);                                               \
    bg::launch_pdl(kern, dim3(T), block, smem, stream, p, inv_q, inv_k);                                   \
  } while (0)
  if (vecs <= kWholeThreads) BG_WHOLE(1);
  else if (vecs <= 2 * kWholeThreads) BG_WHOLE(2);
  else if (vecs <= 4 * kWholeThreads) BG_WHOLE(4);
  else if (vecs <= 8 * kWholeThreads) BG_WHOLE(8);
  else BG_WHOLE(16);
#undef BG_WHOLE
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename KT, int NV>
static void launch(const Params& p, dim3 grid, size_t smem, cudaStream_t stream) {
  if (p.interleaved) bg::launch_pdl(prep_kernel<KT, NV, true>, grid, dim3(kWarps * 32), 0, stream, p);
  else bg::launch_pdl(prep_kernel<KT, NV, false>, grid, dim3(kWarps * 32), smem, stream, p);
}
template <typename KT>
static void launch(const Params& p, dim3 grid, size_t smem, cudaStream_t stream) {
  const int w = p.dp > p.dvp ? p.dp : p.dvp;
  if (w <= 128) launch<KT, 1>(p, grid, smem, stream);
  else if (w <= 256) launch<KT, 2>(p, grid, smem, stream);
  else if (w <= 512) launch<KT, 4>(p, grid, smem, stream);
  else launch<KT, 8>(p, grid, smem, stream);
}

}  // namespace heads
}  // namespace bg

extern "C" {

// dt: 0 = bf16 cache, 1 = fp32.  page: a power of two.  z: T rows of ld floats, the heads' columns first; row = G (dp + dvp); d: real width of query and
// key heads (for the norms).  whole: wq [H dp], wk [G dp], one norm over all query heads and one over all key heads.  qf [T, H, kc] bf16
// or null.  -3: more heads than a block takes.
int bg_head_prep(int dt, float* z, int ld, const float* bias, const float* wq, const float* wk, int whole, float eps, int d, const float* rope,
                 int half, int interleaved, const long long* slots, void* cache, long long page_stride, int page, int row, int write_q,
                 void* qf, int kc, float scale, int T, int H, int G, int dp, int dvp, cudaStream_t stream) {
  using namespace bg::heads;
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || dp <= 0 || dp % 8 || dp > kMaxWidth || d <= 0 || d > dp || dvp <= 0 || dvp % 8 || dvp > kMaxWidth || row != G * (dp + dvp) ||
      ld % 4 || ld < H * dp + row || page <= 0 || (page & (page - 1)) || page_stride % 8 || (rope != nullptr && (half <= 0 || 2 * half > dp)) ||
      (qf != nullptr && (kc < dp || kc % 8)) || (wq == nullptr) != (wk == nullptr) || reinterpret_cast<uintptr_t>(z) % 16)
    return -1;
  Params p;
  p.z = z; p.ld = ld; p.bias = bias; p.wq = wq; p.wk = wk; p.eps = eps; p.inv_d = 1.0f / (float)d; p.rope = rope; p.half = half;
  p.interleaved = interleaved; p.slots = slots; p.cache = cache; p.page_stride = page_stride; p.page = page; p.row = row;
  p.write_q = write_q; p.qf = reinterpret_cast<__nv_bfloat16*>(qf); p.kc = kc; p.q_scale = scale * 1.4426950408889634f;
  for (p.shift = 0; (1 << p.shift) < page; ++p.shift) {}
  p.H = H; p.G = G; p.dp = dp; p.dvp = dvp;
  if (whole && wq != nullptr) {
    const float inv_q = 1.0f / ((float)H * (float)d), inv_k = 1.0f / ((float)G * (float)d);
    return dt == 0 ? launch_whole<__nv_bfloat16>(p, T, inv_q, inv_k, stream) : launch_whole<float>(p, T, inv_q, inv_k, stream);
  }
  const dim3 grid(T, (H + 2 * G + kWarps * kHeads - 1) / (kWarps * kHeads));
  if (grid.y > 65535) return -1;
  const size_t smem = (size_t)kWarps * dp * sizeof(float);
  if (dt == 0) launch<__nv_bfloat16>(p, grid, smem, stream);
  else launch<float>(p, grid, smem, stream);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(head_prep)
