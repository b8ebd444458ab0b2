// Row kernels around attention over a cached latent (its scores: latent_rows.cuh, talking_attn.cu, gqa_prefill.cu):
//
//   latent_prep     the projections of a token: RMS norm of the query latent into the operand of the query projection; RMS norm of the
//                   cached latent and rotation of the key part all heads share, both into the token's cache row
//   latent_query    projected queries of a decode row: rotated part into its columns of the latent-space query, the rest into the operand
//                   of the product with the key projection
//   latent_gather   pages of cached rows one after the other, the operand of the product that expands them to keys and values
//
// Norms and rotations are fp32.  Rotary pairs are (i, i + half); a query head is laid out as [rotated | rest], a cache row as
// [latent | rotated], each part padded with zero channels to a multiple of 8.
#define BG_FILE_TAG 32     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace lat {

constexpr int kThreads = 256;

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ float dot4(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 turned4(const float* x, int c, const float* rope, int half) {
  float4 o;
  float* y = &o.x;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int e = c + j;
    const float a = x[e];
    if (e >= 2 * half) { y[j] = a; continue; }
    const bool low = e < half;
    const int k = low ? e : e - half;
    const float b = x[low ? e + half : k], co = rope[k], si = rope[half + k];
    y[j] = low ? a * co - b * si : a * co + b * si;
  }
  return o;
}

struct Prep {
  const float *zq, *zc, *zr;       // columns of a token's projections; zc, zr null: nothing is cached
  int ld;
  const float *wq, *wc;            // gains, zero past the real widths
  int q_rank, rank, half;          // real widths (half: rotary pairs)
  int q_pad, rank_p, rot_p;        // as stored: operand row, latent and rotated part of a cache row
  const float* rope;               // [T, 2 half]
  void* out;                       // [T, q_pad]
  const long long* slots;
  void* cache;
  long long page_stride;
  int page, row;
  float eps;
};

template <typename OT>
__global__ void __launch_bounds__(kThreads) prep_kernel(const Prep p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  __shared__ float red[2][kThreads / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const float* zq = p.zq + (size_t)t * p.ld;
  const long long slot = p.zc != nullptr ? p.slots[t] : -1;
  const float* zc = p.zc + (size_t)t * p.ld;
  float sq = 0.f, sc = 0.f;
  for (int c = tid * 4; c < p.q_rank; c += kThreads * 4) sq += dot4(ld4(zq + c));          // columns past the real width are zero
  if (slot >= 0)
    for (int c = tid * 4; c < p.rank; c += kThreads * 4) sc += dot4(ld4(zc + c));
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sc; }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) { sq += red[0][i]; sc += red[1][i]; }
  const float rq = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps);
  OT* out = reinterpret_cast<OT*>(p.out) + (size_t)t * p.q_pad;
  for (int c = tid * 4; c < p.q_pad; c += kThreads * 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < p.q_rank) {
      const float4 x = ld4(zq + c), g = ld4(p.wq + c);
      v = make_float4(x.x * rq * g.x, x.y * rq * g.y, x.z * rq * g.z, x.w * rq * g.w);
    }
    put4(out + c, v);
  }
  if (slot < 0) return;
  const float rc = 1.0f / sqrtf(sc / (float)p.rank + p.eps);
  OT* dst = reinterpret_cast<OT*>(p.cache) + (slot / p.page) * p.page_stride + (slot % p.page) * p.row;
  for (int c = tid * 4; c < p.rank_p; c += kThreads * 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < p.rank) {
      const float4 x = ld4(zc + c), g = ld4(p.wc + c);
      v = make_float4(x.x * rc * g.x, x.y * rc * g.y, x.z * rc * g.z, x.w * rc * g.w);
    }
    put4(dst + c, v);
  }
  const float* zr = p.zr + (size_t)t * p.ld;
  for (int c = tid * 4; c < p.rot_p; c += kThreads * 4)
    put4(dst + p.rank_p + c, c < 2 * p.half ? turned4(zr, c, p.rope + (size_t)t * 2 * p.half, p.half) : make_float4(0.f, 0.f, 0.f, 0.f));
}

// q [*, ldq] fp32 heads of [rot_p | dim_p] -> rest [R, H, dim_p], qa [R, H, row] (columns rank_p .. row)
template <typename OT>
__global__ void __launch_bounds__(kThreads)
query_kernel(const float* __restrict__ q, int ldq, const int* __restrict__ row_ids, const float* __restrict__ rope, int half,
             OT* __restrict__ rest, OT* __restrict__ qa, int H, int rot_p, int dim_p, int rank_p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int r = blockIdx.x, t = row_ids != nullptr ? row_ids[r] : r, hw = rot_p + dim_p, row = rank_p + rot_p;
  const int i = (blockIdx.y * kThreads + threadIdx.x) * 4;
  if (i >= H * hw) return;
  const int h = i / hw, c = i % hw;                                  // every width is a multiple of 8
  const float* head = q + (size_t)t * ldq + h * hw;
  if (c < rot_p) put4(qa + ((size_t)r * H + h) * row + rank_p + c, turned4(head, c, rope + (size_t)t * 2 * half, half));
  else put4(rest + ((size_t)r * H + h) * dim_p + c - rot_p, ld4(head + c));
}

// pages [n, 2]: (block-table row, page of the sequence); out [n, page, cols]: cached rows, zero columns row .. cols
__global__ void __launch_bounds__(kThreads)
gather_kernel(const uint4* __restrict__ cache, long long page_vecs, const int* __restrict__ block_table, int bt_stride,
              const int* __restrict__ pages, uint4* __restrict__ out, int page, int row_vecs, int col_vecs) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int i = blockIdx.x;
  const uint4* src = cache + (long long)block_table[(size_t)pages[2 * i] * bt_stride + pages[2 * i + 1]] * page_vecs;
  uint4* dst = out + (size_t)i * page * col_vecs;
  for (int k = blockIdx.y * kThreads + threadIdx.x; k < page * col_vecs; k += kThreads * gridDim.y) {
    const int t = k / col_vecs, c = k % col_vecs;
    dst[k] = c < row_vecs ? src[(size_t)t * row_vecs + c] : make_uint4(0, 0, 0, 0);
  }
}

}  // namespace lat
}  // namespace bg

extern "C" {

// dt: 0 = bf16 operand and cache, 1 = fp32.  z columns start on multiples of 4 and are zero between a part's real width and the next
// multiple of 8; gains are zero there too.  zc null: only the query latent.  q_pad >= q_rank rounded up to 4, a multiple of 8.
int bg_latent_prep(int dt, const float* zq, const float* zc, const float* zr, int ld, const float* wq, const float* wc, int q_rank, int rank,
                   int half, int q_pad, int rank_p, int rot_p, const float* rope, void* out, const long long* slots, void* cache,
                   long long page_stride, int page, int row, float eps, int T, cudaStream_t stream) {
  using namespace bg::lat;
  if (T <= 0) return 0;
  auto off = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 != 0; };
  if (q_rank <= 0 || q_pad % 8 || q_pad < (q_rank + 3) / 4 * 4 || ld % 4 || off(zq) || off(wq)) return -1;
  if (zc != nullptr && (rank <= 0 || rank_p % 8 || rank_p < rank || half <= 0 || rot_p % 8 || rot_p < 2 * half || row != rank_p + rot_p || off(zc) ||
                        off(zr) || off(wc) || zr == nullptr || wc == nullptr || rope == nullptr || slots == nullptr || page <= 0 || page_stride % 8))
    return -1;
  Prep p;
  p.zq = zq; p.zc = zc; p.zr = zr; p.ld = ld; p.wq = wq; p.wc = wc; p.q_rank = q_rank; p.rank = rank; p.half = half; p.q_pad = q_pad;
  p.rank_p = rank_p; p.rot_p = rot_p; p.rope = rope; p.out = out; p.slots = slots; p.cache = cache; p.page_stride = page_stride;
  p.page = page; p.row = row; p.eps = eps;
  if (dt == 0) bg::launch_pdl(prep_kernel<__nv_bfloat16>, dim3(T), dim3(kThreads), 0, stream, p);
  else bg::launch_pdl(prep_kernel<float>, dim3(T), dim3(kThreads), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// q [*, ldq] fp32, R rows (row_ids, or rows 0 .. R); rope [*, 2 half] by the same row
int bg_latent_query(int dt, const float* q, int ldq, const int* row_ids, const float* rope, int half, void* rest, void* qa, int R, int H,
                    int rot_p, int dim_p, int rank_p, cudaStream_t stream) {
  using namespace bg::lat;
  if (R <= 0) return 0;
  if (H <= 0 || rot_p % 8 || dim_p % 8 || rank_p % 8 || half <= 0 || 2 * half > rot_p || ldq % 4 || ldq < H * (rot_p + dim_p) || rope == nullptr) return -1;
  const dim3 grid(R, (H * (rot_p + dim_p) / 4 + kThreads - 1) / kThreads);
  if (grid.y > 65535) return -1;
  if (dt == 0)
    bg::launch_pdl(query_kernel<__nv_bfloat16>, grid, dim3(kThreads), 0, stream, q, ldq, row_ids, rope, half,
                   reinterpret_cast<__nv_bfloat16*>(rest), reinterpret_cast<__nv_bfloat16*>(qa), H, rot_p, dim_p, rank_p);
  else
    bg::launch_pdl(query_kernel<float>, grid, dim3(kThreads), 0, stream, q, ldq, row_ids, rope, half, reinterpret_cast<float*>(rest),
                   reinterpret_cast<float*>(qa), H, rot_p, dim_p, rank_p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// bf16 cache [*, page, row] with page_stride elements between pages -> out [n, page, cols]; row, cols, page_stride: multiples of 8
int bg_latent_gather(const void* cache, long long page_stride, const int* block_table, int bt_stride, const int* pages, int n, void* out,
                     int page, int row, int cols, cudaStream_t stream) {
  using namespace bg::lat;
  if (n <= 0) return 0;
  if (row <= 0 || row % 8 || cols % 8 || cols < row || page <= 0 || page_stride % 8) return -1;
  bg::launch_pdl(gather_kernel, dim3(n, 4), dim3(kThreads), 0, stream, reinterpret_cast<const uint4*>(cache), page_stride / 8, block_table,
                 bt_stride, pages, reinterpret_cast<uint4*>(out), page, row / 8, cols / 8);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(latent_attn)
