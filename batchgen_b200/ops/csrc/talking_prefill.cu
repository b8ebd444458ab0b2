// Prefill attention with mixed heads ("talking heads"), chunked visibility and a zero-score sink, on tcgen05.
//
// Mixing couples the heads at every (query, key) pair: s[h] = scale * sum_g talk[h, g] (q[g] . k[kv(g)]).  Grouping the sum
// by key head c turns it into one longer dot product,
//
//   s[h] = q'[h] . [k_0 | k_1 | .. | k_(G-1)],   q'[h, c, :] = scale * sum_(g of c) talk[h, g] q[g, :]
//
// so a first kernel mixes the *queries* (in fp32, one rounding to bf16, with log2(e) folded in) and the attention itself
// is ordinary flash attention whose keys are a cached token's whole key block (width G * dp) and whose values are head
// kv(h)'s.  The mixed scores leave the tensor core in fp32.
//
// One CTA = (tile of 128 queries of one sequence, head h).  M = 128 queries on the TMEM lanes, key tiles of 128:
//   S (2 x 128 columns, double buffered) = Q' . K^T, both operands streamed in 64-wide K blocks through a TMA ring
//   O (dv columns) += P . V,  P written by the softmax threads as a swizzled K-major tile, V read N-major
// K and V come straight from the paged cache by TMA (3-D map: column, token of the page, page).  A thread owns a query row:
// no cross-thread reduction; O is rescaled only when the running maximum grew by more than 2^8.
//
// Roles (192 threads): warp 0 TMA producer, warp 1 MMA issuer + TMEM owner, warps 2..5 softmax / epilogue.  All waits are
// bounded (common.cuh).
#define BG_FILE_TAG 24     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace talkpre {

constexpr int BM = 128, BN = 128;
constexpr int kMaxStages = 5;                              // K-block stages: five with up to 128 value columns, else four
constexpr int kThreads = 192;
constexpr int kMaxBoxes = BN / 16;                         // pages of 16 tokens and more
constexpr int kABytes = BM * 128, kBBytes = BN * 128;      // one 64-wide bf16 K block of each operand
constexpr int kPBytes = 2 * BM * 128;
constexpr int kTmemCols = 512;                             // S: 2 x 128, O: up to 256

struct Work {
  int q_row0;    // first query row of the tile (rows of Q' and out)
  int n_q;       // queries in the tile (<= 128)
  int seq;       // block-table row
  int pos0;      // position of the first query in its sequence
};

struct Params {
  const Work* work;
  const int* block_table;
  int bt_stride, bt_cols;
  int page, box_rows;            // tokens per page, rows of one TMA box (min(page, 64))
  int KB;                        // 64-wide blocks of the contraction
  int v_col0, dvp, dv64, rep;    // first value column of a cache row, head widths, heads per key head
  int chunk, sink;
  __nv_bfloat16* out;
  int ldo;
  int row_shift;                 // rows of Q' = rows of out - row_shift
  int* status;
};

struct Shared {
  uint64_t full[kMaxStages], empty[kMaxStages];
  uint64_t v_full, v_empty;
  uint64_t s_full[2];
  uint64_t p_full, o_done;
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ uint64_t desc_mn_sw128(uint32_t addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>(lbo >> 4) << 16;
  d |= static_cast<uint64_t>(sbo >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ uint32_t idesc_bf16(int M, int N, int b_mn_major) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(b_mn_major) << 16) |
         (static_cast<uint32_t>(N >> 3) << 17) | (static_cast<uint32_t>(M >> 4) << 24);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ bool vote_any_128(bool v) {      // barrier over the 128 softmax threads, OR of a flag
  uint32_t r;
  asm volatile(
      "{\n"
      ".reg .pred p, q;\n"
      "setp.ne.u32 q, %1, 0;\n"
      "bar.red.or.pred p, 2, 128, q;\n"
      "selp.u32 %0, 1, 0, p;\n"
      "}\n"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v))
      : "memory");
  return r != 0;
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, %21, %22, %23, %24, "
      "%25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]),
      "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]),
      "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]), "r"(v[26]),
      "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
      : "memory");
}

template <int kStages>
__global__ void __launch_bounds__(kThreads, 1)
attn_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* a_buf = smem;
  uint8_t* b_buf = a_buf + kStages * kABytes;
  uint8_t* v_buf = b_buf + kStages * kBBytes;
  uint8_t* p_buf = v_buf + (p.dv64 / 64) * BN * 128;
  Shared& ss = *reinterpret_cast<Shared*>(p_buf + kPBytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  volatile int* abort_flag = &ss.abort_flag;
  const Work w = p.work[blockIdx.x];
  const int h = blockIdx.y;
  const int last = w.pos0 + w.n_q - 1;
  const int first = p.chunk > 0 ? w.pos0 - w.pos0 % p.chunk : 0;
  const int k0 = first - first % p.box_rows;                     // first key of tile 0: starts on a box of a page
  const int n_tiles = (last + 1 - k0 + BN - 1) / BN;
  const int v_tile_bytes = (p.dv64 / 64) * BN * 128;

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) { mbar_init(&ss.full[s], 1); mbar_init(&ss.empty[s], 1); }
    for (int s = 0; s < 2; ++s) mbar_init(&ss.s_full[s], 1);
    mbar_init(&ss.v_full, 1);
    mbar_init(&ss.v_empty, 1);
    mbar_init(&ss.p_full, 128);
    mbar_init(&ss.o_done, 1);
    ss.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&ss.tmem_base, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = ss.tmem_base;

  if (warp == 0) {
    // ------------------------------------------------------------ TMA producer
    if (elect_one()) {
      tma_prefetch_desc(&tm_q);
      tma_prefetch_desc(&tm_kv);
      const int* bt = p.block_table + (size_t)w.seq * p.bt_stride;
      const int boxes = BN / p.box_rows;
      uint32_t it = 0;
      bool ok = true;
      // box b of tile t: tokens k0 + t * BN + b * box_rows ..; past the table's end the last page is read (masked keys).
      // Page numbers of a tile are looked up once, one tile ahead of their use.
      const int shift = 31 - __clz(p.page);
      int old[kMaxBoxes], pg[kMaxBoxes] = {}, nxt[kMaxBoxes] = {};
      auto look_up = [&](int t) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b)
          if (b < boxes) nxt[b] = bt[min((k0 + t * BN + b * p.box_rows) >> shift, p.bt_cols - 1)];
      };
      const int vcol = p.v_col0 + (h / p.rep) * p.dvp;
      auto load_v = [&](int t) -> bool {                           // values of tile t, whose pages are in `old`
        if (!mbar_wait(&ss.v_empty, (t & 1) ^ 1, abort_flag, kTimeoutProducer)) return false;
        mbar_expect_tx(&ss.v_full, v_tile_bytes);
        for (int c = 0; c < p.dv64 / 64; ++c)
#pragma unroll
          for (int b = 0; b < kMaxBoxes; ++b)
            if (b < boxes)
              tma_load_3d(v_buf + (c * BN + b * p.box_rows) * 128, &tm_kv, &ss.v_full, vcol + c * 64,
                          (k0 + t * BN + b * p.box_rows) & (p.page - 1), old[b]);
        return true;
      };
      look_up(0);
      // the MMA warp takes S(0), S(1), PV(0), S(2), PV(1), ..: values follow the next tile's keys
      for (int t = 0; ok && t < n_tiles; ++t) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b) { old[b] = pg[b]; pg[b] = nxt[b]; }
        if (t + 1 < n_tiles) look_up(t + 1);
        const int pos = k0 + t * BN;
        for (int kb = 0; kb < p.KB; ++kb, ++it) {
          const int s = it % kStages;
          if (!mbar_wait(&ss.empty[s], ((it / kStages) & 1) ^ 1, abort_flag, kTimeoutProducer)) { ok = false; break; }
          mbar_expect_tx(&ss.full[s], kABytes + kBBytes);
          tma_load_2d(a_buf + s * kABytes, &tm_q, &ss.full[s], (h * p.KB + kb) * 64, w.q_row0 - p.row_shift);
#pragma unroll
          for (int b = 0; b < kMaxBoxes; ++b)
            if (b < boxes)
              tma_load_3d(b_buf + s * kBBytes + b * p.box_rows * 128, &tm_kv, &ss.full[s], kb * 64,
                          (pos + b * p.box_rows) & (p.page - 1), pg[b]);
        }
        if (ok && t > 0) ok = load_v(t - 1);
      }
      if (ok && n_tiles > 0) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b) old[b] = pg[b];
        ok = load_v(n_tiles - 1);
      }
      if (ok) {
        // leave only when every copy has landed and been consumed
        const uint32_t n = it < (uint32_t)kStages ? it : (uint32_t)kStages;
        for (uint32_t j = it - n; j < it; ++j)
          if (!mbar_wait(&ss.empty[j % kStages], (j / kStages) & 1, abort_flag, kTimeoutProducer)) break;
        if (n_tiles > 0) mbar_wait(&ss.v_empty, (n_tiles - 1) & 1, abort_flag, kTimeoutProducer);
      } else {
        for (uint32_t i = 0; i < (1u << 16); ++i) __nanosleep(20);   // bounded grace period for copies in flight
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      const uint32_t idesc_s = idesc_bf16(BM, BN, 0);
      const uint32_t idesc_pv = idesc_bf16(BM, p.dv64, 1);
      const uint32_t tm_o = tmem_base + 2 * BN;
      uint32_t it = 0;
      bool ok = true;
      auto issue_s = [&](int t) -> bool {
        const uint32_t tm_s = tmem_base + (t & 1) * BN;
        for (int kb = 0; kb < p.KB; ++kb, ++it) {
          const int s = it % kStages;
          if (!mbar_wait(&ss.full[s], (it / kStages) & 1, abort_flag, kTimeoutMma)) return false;
          tc_fence_after();
          const uint64_t adesc = make_smem_desc_sw128(smem_u32(a_buf + s * kABytes));
          const uint64_t bdesc = make_smem_desc_sw128(smem_u32(b_buf + s * kBBytes));
#pragma unroll
          for (int k = 0; k < 4; ++k) mma_f16(tm_s, adesc + 2 * k, bdesc + 2 * k, idesc_s, (kb | k) ? 1u : 0u);
          tc_commit(&ss.empty[s]);
        }
        tc_commit(&ss.s_full[t & 1]);
        return true;
      };
      if (n_tiles > 0) ok = issue_s(0);
      for (int t = 0; ok && t < n_tiles; ++t) {
        // S of tile t + 1 goes into the buffer that the softmax of tile t - 1 has left (its P was handed over before PV(t-1))
        if (t + 1 < n_tiles && !issue_s(t + 1)) { ok = false; break; }
        if (!mbar_wait(&ss.v_full, t & 1, abort_flag, kTimeoutMma)) { ok = false; break; }
        if (!mbar_wait(&ss.p_full, t & 1, abort_flag, kTimeoutMma)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_base = smem_u32(v_buf);
#pragma unroll
        for (int j = 0; j < BN / 16; ++j) {
          const uint64_t pdesc = make_smem_desc_sw128(smem_u32(p_buf + (j / 4) * BM * 128)) + 2 * (j % 4);
          mma_f16(tm_o, pdesc, desc_mn_sw128(v_base + j * 2048, BN * 128, 1024), idesc_pv, (t > 0 || j > 0) ? 1u : 0u);
        }
        tc_commit(&ss.v_empty);
        tc_commit(&ss.o_done);
      }
    }
  } else {
    // ------------------------------------------------------------ softmax / correction / epilogue: thread = query row
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t tm_o = tmem_base + 2 * BN + lane_addr;
    const int pos = w.pos0 + r;
    const bool live = r < w.n_q;
    const int vis_lo = live ? (p.chunk > 0 ? pos - pos % p.chunk : 0) - k0 : 0;     // keys [vis_lo, vis_hi) from k0
    const int vis_hi = live ? pos + 1 - k0 : 0;
    float m_run = -INFINITY, l_run = 0.f;
    uint8_t* prow = p_buf + (r >> 3) * 1024 + (r & 7) * 128;
    bool ok = true;
    for (int t = 0; ok && t < n_tiles; ++t) {
      if (vote_any_128(!mbar_wait(&ss.s_full[t & 1], (t >> 1) & 1, abort_flag, kTimeoutEpilogue))) { ok = false; break; }
      tc_fence_after();
      const uint32_t tm_s = tmem_base + lane_addr + (t & 1) * BN;
      const int lo = vis_lo - t * BN, hi = vis_hi - t * BN;
      float mt = -INFINITY;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t sv[32];
        tmem_ld_32x32(tm_s + c * 32, sv);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const int k = c * 32 + j;
          mt = fmaxf(mt, (k >= lo && k < hi) ? __uint_as_float(sv[j]) : -INFINITY);
        }
      }
      const bool grow = mt > m_run + 8.f;
      const float m_new = grow ? mt : m_run;
      const float alpha = (grow && m_run != -INFINITY) ? ex2(m_run - m_new) : 1.f;
      // PV(t - 1) done: O may be rescaled and P overwritten
      if (t > 0 && vote_any_128(!mbar_wait(&ss.o_done, (t - 1) & 1, abort_flag, kTimeoutEpilogue))) { ok = false; break; }
      tc_fence_after();
      if (t > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
        for (int c = 0; c < p.dv64 / 32; ++c) {
          uint32_t ov[32];
          tmem_ld_32x32(tm_o + c * 32, ov);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) ov[j] = __float_as_uint(__uint_as_float(ov[j]) * alpha);
          tmem_st32(tm_o + c * 32, ov);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      }
      float lsum = 0.f;
      const float neg_m = (m_new == -INFINITY) ? 0.f : -m_new;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t sv[32];
        tmem_ld_32x32(tm_s + c * 32, sv);
        tmem_ld_wait();
#pragma unroll
        for (int q8 = 0; q8 < 4; ++q8) {
          __align__(16) __nv_bfloat162 o[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int k = c * 32 + q8 * 8 + 2 * q;
            const float p0 = (k >= lo && k < hi) ? ex2(__uint_as_float(sv[q8 * 8 + 2 * q]) + neg_m) : 0.f;
            const float p1 = (k + 1 >= lo && k + 1 < hi) ? ex2(__uint_as_float(sv[q8 * 8 + 2 * q + 1]) + neg_m) : 0.f;
            o[q] = __floats2bfloat162_rn(p0, p1);
            lsum += __low2float(o[q]) + __high2float(o[q]);
          }
          const int ch = (c & 1) * 4 + q8;                     // 16-byte piece of the row inside its 64-key block
          *reinterpret_cast<uint4*>(prow + (c >> 1) * BM * 128 + ((ch ^ (r & 7)) << 4)) = *reinterpret_cast<const uint4*>(o);
        }
      }
      l_run = l_run * alpha + lsum;
      m_run = m_new;
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      tc_fence_before();
      mbar_arrive(&ss.p_full);
    }
    if (ok && n_tiles > 0) ok = !vote_any_128(!mbar_wait(&ss.o_done, (n_tiles - 1) & 1, abort_flag, kTimeoutEpilogue));
    if (ok) {
      tc_fence_after();
      if (p.sink && live) l_run += exp2f(-m_run);
      const float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
      __nv_bfloat16* orow = p.out + (size_t)(w.q_row0 + r) * p.ldo + h * p.dvp;
#pragma unroll 1
      for (int c = 0; c < p.dv64 / 32; ++c) {
        uint32_t ov[32];
        tmem_ld_32x32(tm_o + c * 32, ov);
        tmem_ld_wait();
        if (live) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (c * 32 + j < p.dvp) {                          // dvp is a multiple of 8
              __align__(16) __nv_bfloat162 o[4];
#pragma unroll
              for (int q = 0; q < 4; ++q)
                o[q] = __floats2bfloat162_rn(__uint_as_float(ov[j + 2 * q]) * inv, __uint_as_float(ov[j + 2 * q + 1]) * inv);
              *reinterpret_cast<uint4*>(orow + c * 32 + j) = *reinterpret_cast<const uint4*>(o);
            }
          }
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem_base, kTmemCols);
  if (threadIdx.x == 0 && ss.abort_flag != 0 && p.status != nullptr) atomicMax(p.status, ss.abort_flag);
}

// q' of one token: q'[h, c * dp + e] = f * sum_(i < rep) talk[h, c * rep + i] q[c * rep + i, e]; columns G * dp .. kc are zero.
// A thread owns 4 columns (c, e .. e + 3) and walks the heads.
constexpr int kFoldThreads = 256;
template <int REP>
__global__ void __launch_bounds__(kFoldThreads)
fold_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ talk, __nv_bfloat16* __restrict__ out, int H,
            int G, int dp, int kc, float f) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ float ts[];                                // talk [H][H]
  const int rep = REP > 0 ? REP : H / G;
  for (int i = threadIdx.x; i < H * H; i += kFoldThreads)
    ts[i] = talk != nullptr ? talk[i] * f : (i / H == i % H ? f : 0.f);
  __syncthreads();
  const float* qr = q + (size_t)blockIdx.x * ldq;
  __nv_bfloat16* orow = out + (size_t)blockIdx.x * H * kc;
  for (int col = threadIdx.x * 4; col < kc; col += kFoldThreads * 4) {
    const bool ok = col < G * dp;
    const int c = ok ? col / dp : 0, e = ok ? col % dp : 0;
    float4 qv[REP > 0 ? REP : 1];
    if (REP > 0) {
#pragma unroll
      for (int i = 0; i < (REP > 0 ? REP : 1); ++i)
        qv[i] = ok ? *reinterpret_cast<const float4*>(qr + (c * rep + i) * dp + e) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int h = 0; h < H; ++h) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      const float* tr = ts + h * H + c * rep;
      if (REP > 0) {
#pragma unroll
        for (int i = 0; i < (REP > 0 ? REP : 1); ++i) {
          const float w = tr[i];
          a.x = fmaf(w, qv[i].x, a.x); a.y = fmaf(w, qv[i].y, a.y); a.z = fmaf(w, qv[i].z, a.z); a.w = fmaf(w, qv[i].w, a.w);
        }
      } else if (ok) {
        for (int i = 0; i < rep; ++i) {
          const float w = tr[i];
          const float4 v = *reinterpret_cast<const float4*>(qr + (c * rep + i) * dp + e);
          a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
        }
      }
      __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(a.x, a.y), __floats2bfloat162_rn(a.z, a.w)};
      *reinterpret_cast<uint2*>(orow + (size_t)h * kc + col) = *reinterpret_cast<const uint2*>(o);
    }
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeTiledFn get_encode() {
  static EncodeTiledFn fn = nullptr;
  if (fn == nullptr) {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres) == cudaSuccess &&
        qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(sym);
  }
  return fn;
}
static int encode(CUtensorMap* m, int rank, const void* base, const cuuint64_t* dims, const cuuint64_t* strides,
                  const cuuint32_t* box) {
  EncodeTiledFn enc = get_encode();
  if (enc == nullptr) return -1;
  cuuint32_t es[3] = {1, 1, 1};
  return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), dims, strides, box, es,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -2;
}

}  // namespace talkpre
}  // namespace bg

extern "C" {

// Mixed queries of R rows: q fp32 [R, ldq] -> out bf16 [R, H, kc] (kc = G * dp rounded up to 64), times scale * log2(e).
int bg_talk_fold(const float* q, int ldq, const float* talk, void* out, int R, int H, int G, int dp, int kc, float scale,
                 cudaStream_t stream) {
  using namespace bg::talkpre;
  if (R <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dp % 8 || kc % 64 || kc < G * dp || ldq % 4 || H * H * 4 > 227 * 1024) return -1;
  const float f = scale * 1.4426950408889634f;
  const size_t smem = (size_t)H * H * sizeof(float);
  auto O = reinterpret_cast<__nv_bfloat16*>(out);
#define BG_FOLD(REP)                                                                                           \
  do {                                                                                                         \
    static bg::DeviceOnce once;                                                                                \
    if (!bg::ensure_dynamic_smem(fold_kernel<REP>, 227 * 1024, once)) return -4;                               \
    bg::launch_pdl(fold_kernel<REP>, dim3(R), dim3(kFoldThreads), smem, stream, q, ldq, talk, O, H, G, dp, kc, f); \
  } while (0)
  switch (H / G) {
    case 1: BG_FOLD(1); break;
    case 2: BG_FOLD(2); break;
    case 4: BG_FOLD(4); break;
    case 8: BG_FOLD(8); break;
    default: BG_FOLD(0); break;
  }
#undef BG_FOLD
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// qf [R, H, kc] bf16 mixed queries of rows row_shift .. row_shift + R of the step; cache [pages, page, row] bf16 with
// `page_stride` elements between pages; work: n_work x 4 ints (q_row0, n_q, block-table row, position of the first query),
// q_row0 counted in rows of the step; out [T, ldo] bf16.  page: a power of two >= 16; dvp <= 256.
int bg_talk_prefill(const void* qf, const void* cache, long long page_stride, int n_pages, int page, int row,
                    const int* block_table, int bt_stride, int bt_cols, const int* work, int n_work, int R, int row_shift,
                    void* out, int ldo, int H, int G, int dp, int dvp, int kc, int chunk, int sink, int* status,
                    cudaStream_t stream) {
  using namespace bg::talkpre;
  if (n_work <= 0) return 0;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || dp % 8 || dvp % 8 || dvp > 256 || kc % 64 || kc < G * dp || page < 16 ||
      (page & (page - 1)) || row != G * (dp + dvp) || page_stride % 8 || ldo % 8 || bt_cols <= 0)
    return -1;
  const int box_rows = page < 64 ? page : 64;
  CUtensorMap tq, tk;
  {
    cuuint64_t dims[2] = {(cuuint64_t)H * kc, (cuuint64_t)R};
    cuuint64_t strides[1] = {(cuuint64_t)H * kc * 2};
    cuuint32_t box[2] = {64, BM};
    if (encode(&tq, 2, qf, dims, strides, box) != 0) return -10;
  }
  {
    cuuint64_t dims[3] = {(cuuint64_t)row, (cuuint64_t)page, (cuuint64_t)n_pages};
    cuuint64_t strides[2] = {(cuuint64_t)row * 2, (cuuint64_t)page_stride * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)box_rows, 1};
    if (encode(&tk, 3, cache, dims, strides, box) != 0) return -11;
  }
  Params p;
  p.work = reinterpret_cast<const Work*>(work);
  p.block_table = block_table; p.bt_stride = bt_stride; p.bt_cols = bt_cols; p.page = page; p.box_rows = box_rows;
  p.KB = kc / 64; p.v_col0 = G * dp; p.dvp = dvp; p.dv64 = (dvp + 63) / 64 * 64; p.rep = H / G; p.chunk = chunk;
  p.sink = sink; p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.row_shift = row_shift; p.status = status;
  const int stages = p.dv64 <= 128 ? 5 : 4;
  const size_t smem = stages * (kABytes + kBBytes) + (p.dv64 / 64) * BN * 128 + kPBytes + sizeof(Shared) + 1024;
  static bg::DeviceOnce once4, once5;
  constexpr size_t kSmemMax = 227 * 1024;
  if (!bg::ensure_dynamic_smem(attn_kernel<4>, kSmemMax, once4) || !bg::ensure_dynamic_smem(attn_kernel<5>, kSmemMax, once5))
    return -13;
  if (stages == 5) attn_kernel<5><<<dim3(n_work, H), kThreads, smem, stream>>>(tq, tk, p);
  else attn_kernel<4><<<dim3(n_work, H), kThreads, smem, stream>>>(tq, tk, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -14;
}

}  // extern "C"

BG_TRACE_SETTER(talking_prefill)
