// Decode attention in latent space over a paged bf16 cache, included by talking_attn.cu (same merge of key ranges).  All heads share a
// token's cached row: the keys are the whole row (latent, then rotated part), the values its first dvp columns.  A CTA takes up to 32
// heads of one query row and a range of keys, so a row is read once for all of them.
//
//   s[h, j] = scale * qb[h, :] . row_j      o[h] = sum_j softmax(s)[h, j] row_j[0 : dvp]
//
// Tiles of 32 keys come through a ring by TMA (3-D map: column, token of the page, page; 128-byte swizzle, columns past the row arrive
// as zeros), issued by a warp of its own: between the multiplying warps' barriers its some hundred cycles a tile would count.  Eight warps share a tile: for the scores a warp takes every fourth 16-wide
// step of the channels and half of the keys (its queries stay in registers, every key byte is read from shared memory once for all heads), the quarters meet in shared memory, eight
// threads a head take the online softmax, and for the values a warp owns an eighth of the columns.  The scores of tile t + 1 and the
// values of tile t are multiplied between the same two barriers.  A few dozen heads would leave most of a 128-row tcgen05 shape idle, so
// the products are mma m16n8k16.  All waits are bounded (common.cuh).
#pragma once

namespace bg {
namespace talk {
namespace latent {

constexpr int kWarpsL = 8, kTileL = 32, kStagesL = 4;
constexpr int kThreadsL = (kWarpsL + 4) * 32;   // eight multiplying warps, a warpgroup of which one thread brings the tiles
constexpr int kRegsMul = 232, kRegsLoad = 40;   // registers a thread of each where the launch's share is too few (kSplit)
constexpr int kParts = kWarpsL / 2;             // shares of the channels
constexpr int kPartRow = kTileL + 8;            // floats of a head's partial scores: rows of a fragment hit different banks
constexpr int kProbBytes = kTileL * 2 + 16;     // bytes of a head's probabilities
constexpr int kChunkL = kTileL * 128;           // bytes of 64 columns of a tile

__host__ __device__ inline int ring_bytes(int row) { return kStagesL * ((row + 63) / 64) * kChunkL; }
__host__ __device__ inline int shared_bytes(int row, int mt) {
  return 1024 + ring_bytes(row) + 16 * mt * (kParts * kPartRow * 4 + kProbBytes + 4 + 8);
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ void sync_mul() { asm volatile("bar.sync 1, %0;" ::"n"(kWarpsL * 32) : "memory"); }

// MT: 16-head tiles; KQ: upper bound of the 16-wide steps in a share of the channels; NV: 8-wide value tiles of a warp (even); EXACT:
// rows of 64 KQ channels, values of 64 NV
template <int MT, int KQ, int NV, bool EXACT>
__global__ void __launch_bounds__(kThreadsL, 1) latent_rows_kernel(const __grid_constant__ CUtensorMap tm, const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(1024) char sm_raw[];
  constexpr bool kSplit = MT == 2 && KQ >= 9;                      // 12 warps start with up to 168 registers a thread
  __shared__ uint64_t full[kStagesL], empty[kStagesL];
  __shared__ int abort_s;
  volatile int* abort_flag = &abort_s;
  using plain::ldsm4;
  using plain::ldsm4t;
  using plain::mma16816;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = p.row, dvp = p.dvp, chunks = (row + 63) / 64, stage_bytes = chunks * kChunkL;
  const int r = blockIdx.x, split = blockIdx.z, h0 = blockIdx.y * 16 * MT, nh = min(16 * MT, p.H - h0);
  const int L = p.lens[r];
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)r * p.ldo + h0 * dvp;
  if (L <= 0) {
    if (p.n_splits == 1)
      for (int i = tid; i < nh * dvp / 4; i += kThreadsL) put4(out + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;                                                        // (a split row without a query is zeroed by the merge)
  }
  char* ring = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(sm_raw) + 1023) & ~uintptr_t(1023));
  float* part = reinterpret_cast<float*>(ring + kStagesL * stage_bytes);               // [kParts][16 MT][kPartRow]
  char* prob = reinterpret_cast<char*>(part + kParts * 16 * MT * kPartRow);            // [16 MT] rows of kProbBytes
  float* alpha = reinterpret_cast<float*>(prob + 16 * MT * kProbBytes);                // [16 MT]
  float2* ml = reinterpret_cast<float2*>(alpha + 16 * MT);                             // [16 MT] maximum, sum
  const uint32_t ring_u = smem_u32(ring), prob_u = smem_u32(prob);
  const int first = p.window > 0 ? max(0, L - p.window) : 0;
  const int t_lo = first / kTileL, n_t = (L + kTileL - 1) / kTileL - t_lo;
  const int my_lo = t_lo + (int)(((long long)n_t * split) / p.n_splits);
  const int my_hi = t_lo + (int)(((long long)n_t * (split + 1)) / p.n_splits);
  const int n = my_hi - my_lo;
  if (tid == 0) {
    for (int k = 0; k < kStagesL; ++k) { mbar_init(&full[k], 1); mbar_init(&empty[k], 1); }
    abort_s = 0;
    mbar_fence_init();
  }
  __syncthreads();
  if (warp >= kWarpsL) {
    // ------------------------------------------------------------ producer (one thread)
    if constexpr (kSplit) asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kRegsLoad));
    if (warp != kWarpsL || !elect_one()) return;
    tma_prefetch_desc(&tm);
    const int* bt = p.block_table + (size_t)(p.row_seq != nullptr ? p.row_seq[r] : r) * p.bt_stride;
    const int box = min(p.page, kTileL), boxes = kTileL / box, last_page = (L - 1) / p.page;      // page: a power of two >= 16
    // tokens of a tile that lie past the sequence's last page are another copy of that page's (their scores are not seen)
    int page0 = 0, page1 = 0;
    auto look_up = [&](int i) {
      page0 = bt[min((my_lo + i) * kTileL / p.page, last_page)];
      if (boxes > 1) page1 = bt[min(((my_lo + i) * kTileL + box) / p.page, last_page)];
    };
    bool ok = true;
    look_up(0);
    for (int i = 0; i < n; ++i) {
      const int s = i % kStagesL, tok = ((my_lo + i) * kTileL) & (p.page - 1), a = page0, b = page1;
      look_up(i + 1);
      if (!mbar_wait(&empty[s], ((i / kStagesL) & 1) ^ 1, abort_flag, kTimeoutProducer)) { ok = false; break; }
      mbar_expect_tx(&full[s], stage_bytes);
      for (int c = 0; c < chunks; ++c) {
        char* dst = ring + s * stage_bytes + c * kChunkL;
        tma_load_3d(dst, &tm, &full[s], c * 64, tok, a);
        if (boxes > 1) tma_load_3d(dst + box * 128, &tm, &full[s], c * 64, 0, b);
      }
    }
    for (int i = max(0, n - kStagesL); ok && i < n; ++i)           // leave only when every tile has landed and been read
      ok = mbar_wait(&empty[i % kStagesL], (i / kStagesL) & 1, abort_flag, kTimeoutProducer);
    if (!ok) {
      for (uint32_t k = 0; k < (1u << 16); ++k) __nanosleep(20);   // bounded grace period for copies in flight
      if (p.status != nullptr) atomicMax(p.status, abort_s);
    }
    return;
  }
  if constexpr (kSplit) asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kRegsMul));
  // queries of the steps 4 k + kq of the channels
  const int ksteps = (row + 15) / 16, kq = warp & (kParts - 1), khalf = warp / kParts, swz = lane & 7;
  const int k_n = max(0, (ksteps - kq + kParts - 1) / kParts);
  const uint32_t ko = (khalf * 16 + (lane >> 4) * 8 + (lane & 7)) * 128 + (((kq * 2 + ((lane >> 3) & 1)) ^ swz) << 4);
  uint32_t qa[MT][KQ][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int k = 0; k < KQ; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int h = m * 16 + (lane >> 2) + (j & 1) * 8, c = (k * kParts + kq) * 16 + (lane & 3) * 2 + (j >> 1) * 8;
        qa[m][k][j] = k < k_n && h < nh && c < row
            ? *reinterpret_cast<const uint32_t*>(p.qb + ((size_t)r * p.H + h0 + h) * row + c) : 0u;
      }
  float o[MT][NV][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int v = 0; v < NV; ++v) o[m][v][0] = o[m][v][1] = o[m][v][2] = o[m][v][3] = 0.f;
  const int v0 = warp * NV * 8;                                    // first value column of the warp
  const uint32_t vo = (warp * NV / 8) * kChunkL + (lane & 15) * 128 + ((((warp * NV) & 7) ^ (lane >> 4) ^ swz) << 4);
  const int sh = tid >> 3, sj = (tid & 7) * 4;                     // softmax: head, first of 4 keys
  float run_m = -INFINITY, run_l = 0.f;                            // of head sh; run_l: this thread's keys only
  for (int i = 0; i <= n; ++i) {
    if (i < n) {                                                   // partial scores of tile i
      // (after a time-out the loop runs out without waiting)
      if (!mbar_try_wait(&full[i % kStagesL], (i / kStagesL) & 1)) mbar_wait(&full[i % kStagesL], (i / kStagesL) & 1, abort_flag, kTimeoutMma);
      const uint32_t ks = ring_u + (i % kStagesL) * stage_bytes;
      float s[MT][2][4] = {};
#pragma unroll
      for (int k = 0; k < KQ; ++k)
        if (EXACT || k < k_n) {
          uint32_t kf[4];
          ldsm4(kf, ks + ko + k * kChunkL);
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
      const uint32_t vs = ring_u + ((i - 1) % kStagesL) * stage_bytes;
      uint32_t pa[MT][2][4];
      float a[MT][2];
      bool scaled = false;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        a[m][0] = alpha[m * 16 + (lane >> 2)];
        a[m][1] = alpha[m * 16 + 8 + (lane >> 2)];
        scaled = scaled || a[m][0] != 1.f || a[m][1] != 1.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) ldsm4(pa[m][k], prob_u + (m * 16 + (lane & 15)) * kProbBytes + (k * 16 + (lane >> 4) * 8) * 2);
      }
      if (__any_sync(0xffffffffu, scaled)) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int v = 0; v < NV; ++v) { o[m][v][0] *= a[m][0]; o[m][v][1] *= a[m][0]; o[m][v][2] *= a[m][1]; o[m][v][3] *= a[m][1]; }
      }
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int v = 0; v < NV; v += 2)
          if (EXACT || v0 + v * 8 < dvp) {
            uint32_t vf[4];
            ldsm4t(vf, ((vs + vo) ^ (v << 4)) + k * 16 * 128);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma16816(o[m][v], pa[m][k], vf[0], vf[1]);
              mma16816(o[m][v + 1], pa[m][k], vf[2], vf[3]);
            }
          }
    }
    sync_mul();                                                   // scores are there; tile i - 1 and its probabilities are done with
    if (tid == 0 && i > 0) mbar_arrive(&empty[(i - 1) % kStagesL]);
    if (i < n && sh < 16 * MT) {
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int q = 0; q < kParts; ++q) {
        const float4 x = *reinterpret_cast<const float4*>(part + ((size_t)q * 16 * MT + sh) * kPartRow + sj);
        s.x += x.x; s.y += x.y; s.z += x.z; s.w += x.w;
      }
      const int k0 = (my_lo + i) * kTileL, pos = k0 + sj;
      s.x *= p.scale_log2; s.y *= p.scale_log2; s.z *= p.scale_log2; s.w *= p.scale_log2;
      if (k0 < first || k0 + kTileL > L) {                         // a tile at an edge
        if (pos < first || pos >= L) s.x = -INFINITY;
        if (pos + 1 < first || pos + 1 >= L) s.y = -INFINITY;
        if (pos + 2 < first || pos + 2 >= L) s.z = -INFINITY;
        if (pos + 3 < first || pos + 3 >= L) s.w = -INFINITY;
      }
      float mt = fmaxf(fmaxf(s.x, s.y), fmaxf(s.z, s.w));
#pragma unroll
      for (int b = 1; b < 8; b <<= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, b));
      // the maximum moves only when it grows by more than 2^8: the accumulators are rarely scaled
      const float mn = mt > run_m + 8.f ? mt : run_m, sub = mn == -INFINITY ? 0.f : mn, al = mn == run_m ? 1.f : ex2(run_m - sub);
      run_m = mn;
      __align__(8) __nv_bfloat162 e[2] = {__floats2bfloat162_rn(ex2(s.x - sub), ex2(s.y - sub)),
                                          __floats2bfloat162_rn(ex2(s.z - sub), ex2(s.w - sub))};
      run_l = run_l * al + (__low2float(e[0]) + __high2float(e[0])) + (__low2float(e[1]) + __high2float(e[1]));
      *reinterpret_cast<uint2*>(prob + sh * kProbBytes + sj * 2) = *reinterpret_cast<const uint2*>(e);
      if ((tid & 7) == 0) alpha[sh] = al;
    }
    sync_mul();                                                   // the probabilities are there
  }
  if (sh < 16 * MT) {
#pragma unroll
    for (int b = 1; b < 8; b <<= 1) run_l += __shfl_xor_sync(0xffffffffu, run_l, b);
    if ((tid & 7) == 0) ml[sh] = make_float2(run_m, run_l);
  }
  sync_mul();      
  if (tid == 0 && abort_s != 0 && p.status != nullptr) atomicMax(p.status, abort_s);
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

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// cache [n_pages, page, row]: boxes of 64 columns x min(page, 32) tokens
static int make_map(CUtensorMap* m, const void* cache, long long page_stride, int n_pages, int page, int row) {
  static EncodeTiledFn fn = nullptr;
  if (fn == nullptr) {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult found;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess)
      return -1;
    fn = reinterpret_cast<EncodeTiledFn>(sym);
  }
  cuuint64_t dims[3] = {(cuuint64_t)row, (cuuint64_t)page, (cuuint64_t)n_pages};
  cuuint64_t strides[2] = {(cuuint64_t)row * 2, (cuuint64_t)page_stride * 2};
  cuuint32_t box[3] = {64, (cuuint32_t)(page < kTileL ? page : kTileL), 1}, step[3] = {1, 1, 1};
  return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(cache), dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -2;
}

template <int MT, int KQ, int NV, bool EXACT>
static int launch_sized(const CUtensorMap& tm, const Params& p, int R, cudaStream_t stream) {
  static DeviceOnce once;
  auto kern = latent_rows_kernel<MT, KQ, NV, EXACT>;
  if (!ensure_dynamic_smem(kern, shared_bytes(16 * kParts * KQ, MT), once)) return -4;
  if (MT == 2 && KQ >= 9) {                                        // the warpgroups' shares have to fit what the launch brings
    static int regs = 0;
    cudaFuncAttributes a;
    if (regs == 0) regs = cudaFuncGetAttributes(&a, kern) == cudaSuccess ? a.numRegs : -1;
    if (regs * (kWarpsL + 4) < kRegsMul * kWarpsL + kRegsLoad * 4) return -5;
  }
  bg::launch_pdl(kern, dim3(R, (p.H + 16 * MT - 1) / (16 * MT), p.n_splits), dim3(kThreadsL), shared_bytes(p.row, MT), stream, tm, p);
  if (p.n_splits > 1) bg::launch_pdl(merge_kernel<__nv_bfloat16>, dim3(R, p.H), dim3(64), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int MT, int KQ, int NV>
static int launch_as(const CUtensorMap& tm, const Params& p, int R, cudaStream_t stream) {
  if (KQ == 9 && p.row == 64 * KQ && p.dvp == 64 * NV) return launch_sized<MT, KQ, NV, KQ == 9>(tm, p, R, stream);
  return launch_sized<MT, KQ, NV, false>(tm, p, R, stream);
}
template <int KQ, int NV>
static int launch_heads(const CUtensorMap& tm, const Params& p, int R, cudaStream_t stream) {
  return p.H > 16 ? launch_as<2, KQ, NV>(tm, p, R, stream) : launch_as<1, KQ, NV>(tm, p, R, stream);
}

}  // namespace latent
}  // namespace talk
}  // namespace bg

extern "C" {

// qb [R, H, row] bf16; cache [n_pages, page, row] bf16 with page_stride elements between pages, a row's first dvp are the values; lens [R]
// = position + 1 (0: zero output); out [R, ldo] bf16, heads of dvp.  row <= 640, dvp <= 512, both multiples of 8; page: a power of two
// >= 16.
int bg_latent_rows(const void* qb, const void* cache, long long page_stride, int n_pages, int page, int row, const int* block_table,
                   int bt_stride, const int* row_seq, const int* lens, void* out, int ldo, float* part_o, float* part_ml, int R, int H, int dvp,
                   int window, const float* sinks, float scale, int n_splits, int* status, cudaStream_t stream) {
  using namespace bg::talk;
  if (R <= 0) return 0;
  if (H <= 0 || H > 65535 || row <= 0 || row % 8 || row > 640 || dvp <= 0 || dvp % 8 || dvp > 512 || dvp > row || page < 16 || (page & (page - 1)) ||
      n_pages <= 0 || page_stride % 8 || reinterpret_cast<uintptr_t>(cache) % 16 || ldo % 8 || ldo < H * dvp || window < 0 || n_splits < 1 ||
      n_splits > 65535 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return -1;
  Params p = {};
  p.qb = reinterpret_cast<const __nv_bfloat16*>(qb); p.cache = cache; p.page_stride = page_stride; p.page = page; p.row = row;
  p.block_table = block_table; p.bt_stride = bt_stride; p.row_seq = row_seq; p.lens = lens; p.out = out; p.ldo = ldo; p.part_o = part_o;
  p.part_ml = part_ml; p.H = H; p.G = 1; p.dp = row; p.dvp = dvp; p.window = window; p.sink = sinks != nullptr; p.sinks = sinks;
  p.n_splits = n_splits; p.scale_log2 = scale * kLog2e; p.out_scale = 1.0f; p.gate_cols = 1; p.status = status;
  CUtensorMap tm;
  if (latent::make_map(&tm, cache, page_stride, n_pages, page, row) != 0) return -10;
  if (row <= 192 && dvp <= 128) return latent::launch_heads<3, 2>(tm, p, R, stream);
  if (row <= 384 && dvp <= 256) return latent::launch_heads<6, 4>(tm, p, R, stream);
  if (row <= 576) return latent::launch_heads<9, 8>(tm, p, R, stream);
  return latent::launch_heads<10, 8>(tm, p, R, stream);
}

}  // extern "C"
