// Decode attention in latent space over a paged bf16 cache, included by talking_attn.cu (same parameters, same merge of key
// ranges).  All heads share a token's cached row: the keys are the whole row (latent, then rotated part), the values its first dvp
// columns.  A CTA takes up to 32 heads of one query row and a range of keys, so a row is read once for all of them.
//
//   s[h, j] = scale * qb[h, :] . row_j      o[h] = sum_j softmax(s)[h, j] row_j[0 : dvp]
//
// Tiles of 32 keys come through a ring of bulk copies, a cached row each (rows lie 16 bytes further apart in shared memory, so that
// fragments hit different banks).  Sixteen warps share a tile: for the scores a warp takes an eighth of the channels and half of the
// keys (its queries stay in registers, every key byte is read from shared memory once for all heads), the eighths meet in shared
// memory, sixteen threads a head take the online softmax, and for the values a warp owns a sixteenth of the columns.  The scores of
// tile t + 1 and the values of tile t are multiplied between the same two barriers.  A few dozen heads would leave most of a 128-row
// tcgen05 shape idle, so the products are mma m16n8k16.
#pragma once

namespace bg {
namespace talk {
namespace latent {

constexpr int kWarpsL = 16, kTileL = 32, kStagesL = 4;
constexpr int kParts = kWarpsL / 2;             // shares of the channels
constexpr int kPartRow = kTileL + 8;            // floats of a head's partial scores: rows of a fragment hit different banks
constexpr int kProbBytes = kTileL * 2 + 16;     // bytes of a head's probabilities

__host__ __device__ inline int row_bytes(int row) { return (row + 15) / 16 * 32 + 16; }
__host__ __device__ inline int ring_bytes(int row) { return kStagesL * kTileL * row_bytes(row); }
__host__ __device__ inline int shared_bytes(int row, int mt) {
  return ring_bytes(row) + 16 * mt * (kParts * kPartRow * 4 + kProbBytes + 4 + 8);
}

__device__ __forceinline__ void bulk_row(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes),
               "r"(smem_u32(bar))
               : "memory");
}

// MT: 16-head tiles; KQ: upper bound of the 16-wide steps in a share of the channels; NV: 8-wide value tiles of a warp (even)
template <int MT, int KQ, int NV>
__global__ void __launch_bounds__(kWarpsL * 32, 1) latent_rows_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) char sm_raw[];
  __shared__ uint64_t full[kStagesL];
  __shared__ int abort_s;
  volatile int* abort_flag = &abort_s;
  using plain::ldsm4;
  using plain::ldsm4t;
  using plain::mma16816;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = p.row, dvp = p.dvp, rb = row_bytes(row);
  const int r = blockIdx.x, split = blockIdx.z, h0 = blockIdx.y * 16 * MT, nh = min(16 * MT, p.H - h0);
  const int L = p.lens[r];
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)r * p.ldo + h0 * dvp;
  if (L <= 0) {
    if (p.n_splits == 1)
      for (int i = tid; i < nh * dvp / 4; i += kWarpsL * 32) put4(out + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;                                                        // (a split row without a query is zeroed by the merge)
  }
  char* ring = sm_raw;
  float* part = reinterpret_cast<float*>(sm_raw + ring_bytes(row));                    // [kParts][16 MT][kPartRow]
  char* prob = reinterpret_cast<char*>(part + kParts * 16 * MT * kPartRow);                 // [16 MT] rows of kProbBytes
  float* alpha = reinterpret_cast<float*>(prob + 16 * MT * kProbBytes);                // [16 MT]
  float2* ml = reinterpret_cast<float2*>(alpha + 16 * MT);                             // [16 MT] maximum, sum
  const uint32_t ring_u = smem_u32(ring), prob_u = smem_u32(prob);
  const int first = p.window > 0 ? max(0, L - p.window) : 0;
  const int t_lo = first / kTileL, n_t = (L + kTileL - 1) / kTileL - t_lo;
  const int my_lo = t_lo + (int)(((long long)n_t * split) / p.n_splits);
  const int my_hi = t_lo + (int)(((long long)n_t * (split + 1)) / p.n_splits);
  const int n = my_hi - my_lo;
  const int* bt = p.block_table + (size_t)(p.row_seq != nullptr ? p.row_seq[r] : r) * p.bt_stride;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  // warp 0 copies: a lane a key.  Keys that are not seen are another copy of a seen one, with a score of minus infinity
  auto key_row = [&](int i) {
    const int pos = max(first, min((my_lo + i) * kTileL + lane, L - 1));
    return cache + (long long)bt[pos / p.page] * p.page_stride + (long long)(pos % p.page) * row;
  };
  auto fetch = [&](int i, const __nv_bfloat16* src) {
    uint64_t* bar = &full[i % kStagesL];
    if (lane == 0) mbar_expect_tx(bar, kTileL * row * 2);
    __syncwarp();
    bulk_row(ring_u + ((i % kStagesL) * kTileL + lane) * rb, src, row * 2, bar);
  };
  if (tid == 0) {
    for (int k = 0; k < kStagesL; ++k) mbar_init(&full[k], 1);
    abort_s = 0;
    mbar_fence_init();
  }
  __syncthreads();
  const __nv_bfloat16* ahead = cache;
  if (warp == 0) {
    for (int k = 0; k < kStagesL - 1 && k < n; ++k) fetch(k, key_row(k));
    ahead = key_row(kStagesL - 1);
  }
  if (row % 16)                                                    // the last 8 channels of a step past the row meet zero queries
    for (int i = tid; i < kStagesL * kTileL; i += kWarpsL * 32) *reinterpret_cast<uint4*>(ring + (size_t)i * rb + row * 2) = make_uint4(0, 0, 0, 0);
  // queries of this warp's share of the channels
  const int ksteps = (row + 15) / 16, per = (ksteps + kParts - 1) / kParts, kq = warp & (kParts - 1), khalf = warp / kParts;
  const int k_lo = kq * per, k_n = max(0, min(per, ksteps - k_lo));
  uint32_t qa[MT][KQ][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int k = 0; k < KQ; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int h = m * 16 + (lane >> 2) + (j & 1) * 8, c = (k_lo + k) * 16 + (lane & 3) * 2 + (j >> 1) * 8;
        qa[m][k][j] = k < k_n && h < nh && c < row
            ? *reinterpret_cast<const uint32_t*>(p.qb + ((size_t)r * p.H + h0 + h) * row + c) : 0u;
      }
  float o[MT][NV][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int v = 0; v < NV; ++v) o[m][v][0] = o[m][v][1] = o[m][v][2] = o[m][v][3] = 0.f;
  const int v0 = warp * NV * 8;                                    // first value column of the warp
  const int sh = tid >> 4, sj = (tid & 15) * 2;                    // softmax: head, first of 2 keys
  float run_m = -INFINITY, run_l = 0.f;                            // of head sh; run_l: this thread's keys only
  if (row % 16) __syncthreads();
  for (int i = 0; i <= n; ++i) {
    if (i < n) {                                                   // partial scores of tile i
      mbar_wait(&full[i % kStagesL], (i / kStagesL) & 1, abort_flag, kTimeoutMma);      // (after a time-out the loop runs out without waiting)
      float s[MT][2][4] = {};
      const uint32_t ka = ring_u + ((i % kStagesL) * kTileL + khalf * 16 + (lane >> 4) * 8 + (lane & 7)) * rb + ((lane >> 3) & 1) * 16 + k_lo * 32;
#pragma unroll
      for (int k = 0; k < KQ; ++k)
        if (k < k_n) {
          uint32_t kf[4];
          ldsm4(kf, ka + k * 32);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma16816(s[m][0], qa[m][k], kf[0], kf[1]);
            mma16816(s[m][1], qa[m][k], kf[2], kf[3]);
          }
        }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
          for (int g = 0; g < 2; ++g)
            *reinterpret_cast<float2*>(part + ((size_t)kq * 16 * MT + m * 16 + g * 8 + (lane >> 2)) * kPartRow + khalf * 16 + b * 8 + (lane & 3) * 2) =
                make_float2(s[m][b][2 * g], s[m][b][2 * g + 1]);
    }
    if (i > 0) {                                                   // values of tile i - 1
      const uint32_t va = ring_u + (((i - 1) % kStagesL) * kTileL + (lane & 15)) * rb + (lane >> 4) * 16 + v0 * 2;
      uint32_t pa[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = alpha[m * 16 + (lane >> 2)], a1 = alpha[m * 16 + 8 + (lane >> 2)];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int v = 0; v < NV; ++v) { o[m][v][0] *= a0; o[m][v][1] *= a0; o[m][v][2] *= a1; o[m][v][3] *= a1; }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) ldsm4(pa[m][k], prob_u + (m * 16 + (lane & 15)) * kProbBytes + (k * 16 + (lane >> 4) * 8) * 2);
      }
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int v = 0; v < NV; v += 2)
          if (v0 + v * 8 < dvp) {
            uint32_t vf[4];
            ldsm4t(vf, va + k * 16 * rb + v * 16);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma16816(o[m][v], pa[m][k], vf[0], vf[1]);
              mma16816(o[m][v + 1], pa[m][k], vf[2], vf[3]);
            }
          }
    }
    __syncthreads();                                               // scores are there; tile i - 1 and its probabilities are done with
    if (warp == 0 && i + kStagesL - 1 < n) {
      if (!__any_sync(0xffffffffu, abort_s != 0)) fetch(i + kStagesL - 1, ahead);
      ahead = key_row(i + kStagesL);
    }
    if (i < n && sh < 16 * MT) {
      float2 s = make_float2(0.f, 0.f);
#pragma unroll
      for (int q = 0; q < kParts; ++q) {
        const float2 x = *reinterpret_cast<const float2*>(part + ((size_t)q * 16 * MT + sh) * kPartRow + sj);
        s.x += x.x; s.y += x.y;
      }
      const int pos = (my_lo + i) * kTileL + sj;
      s.x = pos >= first && pos < L ? s.x * p.scale_log2 : -INFINITY;
      s.y = pos + 1 >= first && pos + 1 < L ? s.y * p.scale_log2 : -INFINITY;
      float mt = fmaxf(s.x, s.y);
#pragma unroll
      for (int b = 1; b < 16; b <<= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, b));
      const float mn = fmaxf(run_m, mt), sub = mn == -INFINITY ? 0.f : mn, al = exp2f(run_m - sub);
      run_m = mn;
      const __nv_bfloat162 e = __floats2bfloat162_rn(exp2f(s.x - sub), exp2f(s.y - sub));
      run_l = run_l * al + (__low2float(e) + __high2float(e));
      *reinterpret_cast<__nv_bfloat162*>(prob + sh * kProbBytes + sj * 2) = e;
      if ((tid & 15) == 0) alpha[sh] = al;
    }
    __syncthreads();                                               // the probabilities are there
  }
  if (tid == 0 && abort_s != 0) {
    for (uint32_t k = 0; k < (1u << 16); ++k) __nanosleep(20);     // bounded grace period for copies in flight
    if (p.status != nullptr) atomicMax(p.status, abort_s);
  }
  if (sh < 16 * MT) {
#pragma unroll
    for (int b = 1; b < 16; b <<= 1) run_l += __shfl_xor_sync(0xffffffffu, run_l, b);
    if ((tid & 15) == 0) ml[sh] = make_float2(run_m, run_l);
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int g = 0; g < 2; ++g) {
      const int head = m * 16 + g * 8 + (lane >> 2), h = h0 + head;
      if (head >= nh) continue;
      const float2 x = ml[head];
      const float inv = p.n_splits == 1 ? p.out_scale / (x.y + (p.sink ? exp2f(sink_score(p, h) - x.x) : 0.f)) : 1.f;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = v0 + v * 8 + (lane & 3) * 2;
        if (c >= dvp) continue;
        if (p.n_splits == 1)
          *reinterpret_cast<__nv_bfloat162*>(out + head * dvp + c) = __floats2bfloat162_rn(o[m][v][2 * g] * inv, o[m][v][2 * g + 1] * inv);
        else
          *reinterpret_cast<float2*>(p.part_o + (((size_t)r * p.n_splits + split) * p.H + h) * dvp + c) = make_float2(o[m][v][2 * g], o[m][v][2 * g + 1]);
      }
      if (p.n_splits > 1 && warp == 0 && (lane & 3) == 0)
        *reinterpret_cast<float2*>(p.part_ml + (((size_t)r * p.n_splits + split) * p.H + h) * 2) = x;
    }
}

template <int MT, int KQ, int NV>
static int launch_as(const Params& p, int R, cudaStream_t stream) {
  static DeviceOnce once;
  auto kern = latent_rows_kernel<MT, KQ, NV>;
  if (!ensure_dynamic_smem(kern, shared_bytes(16 * kParts * KQ, MT), once)) return -4;
  bg::launch_pdl(kern, dim3(R, (p.H + 16 * MT - 1) / (16 * MT), p.n_splits), dim3(kWarpsL * 32), shared_bytes(p.row, MT), stream, p);
  if (p.n_splits > 1) bg::launch_pdl(merge_kernel<__nv_bfloat16>, dim3(R, p.H), dim3(64), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int KQ, int NV>
static int launch_heads(const Params& p, int R, cudaStream_t stream) {
  return p.H > 16 ? launch_as<2, KQ, NV>(p, R, stream) : launch_as<1, KQ, NV>(p, R, stream);
}

}  // namespace latent
}  // namespace talk
}  // namespace bg

extern "C" {

// qb [R, H, row] bf16; cache rows of `row` elements whose first dvp are the values; lens [R] = position + 1 (0: zero output); out
// [R, ldo] bf16, heads of dvp.  row <= 640, dvp <= 512, both multiples of 8.
int bg_latent_rows(const void* qb, const void* cache, long long page_stride, int page, int row, const int* block_table, int bt_stride,
                   const int* row_seq, const int* lens, void* out, int ldo, float* part_o, float* part_ml, int R, int H, int dvp, int window,
                   const float* sinks, float scale, int n_splits, int* status, cudaStream_t stream) {
  using namespace bg::talk;
  if (R <= 0) return 0;
  if (H <= 0 || H > 65535 || row <= 0 || row % 8 || row > 640 || dvp <= 0 || dvp % 8 || dvp > 512 || dvp > row || page <= 0 || page_stride % 8 || reinterpret_cast<uintptr_t>(cache) % 16 ||
      ldo % 8 || ldo < H * dvp || window < 0 || n_splits < 1 || n_splits > 65535 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return -1;
  Params p = {};
  p.qb = reinterpret_cast<const __nv_bfloat16*>(qb); p.cache = cache; p.page_stride = page_stride; p.page = page; p.row = row;
  p.block_table = block_table; p.bt_stride = bt_stride; p.row_seq = row_seq; p.lens = lens; p.out = out; p.ldo = ldo; p.part_o = part_o;
  p.part_ml = part_ml; p.H = H; p.G = 1; p.dp = row; p.dvp = dvp; p.window = window; p.sink = sinks != nullptr; p.sinks = sinks;
  p.n_splits = n_splits; p.scale_log2 = scale * kLog2e; p.out_scale = 1.0f; p.gate_cols = 1;
  p.status = status;
  if (row <= 384 && dvp <= 256) return latent::launch_heads<3, 2>(p, R, stream);
  return latent::launch_heads<5, 4>(p, R, stream);
}

}  // extern "C"
