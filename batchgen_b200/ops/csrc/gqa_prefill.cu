// Prompt attention of grouped-query heads over a paged K/V cache, on tcgen05: causal, optionally with chunked visibility or a
// sliding window that keeps a sequence's first keys, a sink (score zero or one per head), rotary queries and a sigmoid gate per head
// or per element on the output.
//
//   S[q, k] = Q[q, :] . K[k, kv(h)]      (M = 128 queries, N = 64 keys; Q resident, K streamed, both K-major)
//   O[q, :] += P[q, k] . V[k, kv(h)]     (V read N-major, P written by the softmax threads as a swizzled K-major tile)
//
// A first kernel turns the queries, folds scale * log2(e) in and rounds them once to bf16.  One CTA = (tile of 128 queries of
// one sequence, head).  K and V come straight from the paged cache by TMA (3-D map: column, token of the page, page) through a
// ring each, so a key tile is free again as soon as its scores are done; a head's last 64-wide block may reach into the next
// head's columns, which meet zeros of the query (keys) or are not stored (values).  A thread owns a query row (TMEM lane): no
// cross-thread reduction; O is rescaled only when the running maximum grew by more than 2^8.  S of tile t + 1 is issued before
// P.V of tile t, and with head widths up to 128 two CTAs share an SM, so one's softmax runs under the other's products.
//
// Roles (192 threads): warp 0 TMA producer, warp 1 MMA issuer + TMEM owner, warps 2..5 softmax / epilogue.  All waits are
// bounded (common.cuh).
#define BG_FILE_TAG 29     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace gqapre {

constexpr int BM = 128, BN = 64;
constexpr int kMaxStages = 4;
constexpr int kThreads = 192;
constexpr int kMaxBoxes = BN / 16;                         // pages of 16 tokens and more
constexpr int kBlockBytes = BN * 128;                      // one 64-wide bf16 block of a key or value tile
constexpr int kQBlockBytes = BM * 128;
constexpr int kPBytes = BM * 128;
constexpr int kSmemTwo = 113 * 1024;                       // what a CTA may take so that two fit an SM

struct Work {
  int q_row0;    // first query row of the tile (rows of out)
  int n_q;       // queries in the tile (<= 128)
  int seq;       // block-table row
  int pos0;      // position of the first query in its sequence
};

struct Params {
  const Work* work;
  const int* block_table;
  int bt_stride, bt_cols;
  int page, box_rows;            // tokens per page, rows of one TMA box (min(page, 64))
  int KB, VB;                    // 64-wide blocks of a key / value head
  int stages, tmem_cols;
  int dp, dvp, v_col0, rep;      // head widths, first value column of a cache row, heads per key head
  int chunk, window, keep, sink;  // keys seen: from the query's chunk, within the window, and the first `keep`
  float out_scale;
  __nv_bfloat16* out;
  int ldo;
  const float* gate;             // [T, ld_gate] or null: out[h] *= sigmoid(gate[h]), or per element
  int ld_gate, gate_cols;        // columns of a head: 1 or dvp
  const float* sinks;            // [H] scores of the sink, or null: zero
  int staged;                    // gates per element: rows leave through shared memory, a warp a row at a time
  int row_shift;                 // rows of Q = rows of out - row_shift
  int smem_bytes;
  int* status;
};

struct Shared {
  uint64_t q_full;
  uint64_t k_full[kMaxStages], k_empty[kMaxStages], v_full[kMaxStages], v_empty[kMaxStages];
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
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t* v) {
  tmem_ld_32x32(taddr, *reinterpret_cast<uint32_t(*)[32]>(v));
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

// shared memory: Q [KB] | K [stages][KB] | V [stages][VB] | P, all on 1,024-byte boundaries, then Shared
__host__ __device__ inline int tile_bytes(int KB, int VB, int stages) {
  return KB * kQBlockBytes + stages * (KB + VB) * kBlockBytes + kPBytes;
}

__global__ void __launch_bounds__(kThreads, 2)
attn_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_buf = smem;
  uint8_t* k_buf = q_buf + p.KB * kQBlockBytes;
  uint8_t* v_buf = k_buf + p.stages * p.KB * kBlockBytes;
  uint8_t* p_buf = v_buf + p.stages * p.VB * kBlockBytes;
  Shared& ss = *reinterpret_cast<Shared*>(p_buf + kPBytes);
  if (reinterpret_cast<uint8_t*>(&ss + 1) > smem_raw + p.smem_bytes) {      // a base that is off its boundary leaves no room
    if (threadIdx.x == 0 && p.status != nullptr) atomicMax(p.status, (int)kBadArgument);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  volatile int* abort_flag = &ss.abort_flag;
  const Work w = p.work[blockIdx.y];
  const int h = blockIdx.x;
  const int last = w.pos0 + w.n_q - 1;
  int first = p.chunk > 0 ? w.pos0 - w.pos0 % p.chunk : 0;
  if (p.window > 0) first = max(first, w.pos0 + 1 - p.window);
  int k0 = first - first % p.box_rows;                           // first key of the tiles: starts on a box of a page
  if (p.keep > k0) k0 = 0;
  const int n_keep = k0 > 0 ? (p.keep + BN - 1) / BN : 0;        // kept keys that end before k0 have tiles of their own
  const int n_tiles = n_keep + (last + 1 - k0 + BN - 1) / BN;
  auto first_key = [&](int t) { return t < n_keep ? t * BN : k0 + (t - n_keep) * BN; };
  const int ST = p.stages;

  if (threadIdx.x == 0) {
    mbar_init(&ss.q_full, 1);
    for (int s = 0; s < kMaxStages; ++s) {
      mbar_init(&ss.k_full[s], 1); mbar_init(&ss.k_empty[s], 1);
      mbar_init(&ss.v_full[s], 1); mbar_init(&ss.v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) mbar_init(&ss.s_full[s], 1);
    mbar_init(&ss.p_full, 128);
    mbar_init(&ss.o_done, 1);
    ss.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&ss.tmem_base, p.tmem_cols);
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
      const int boxes = BN / p.box_rows, shift = 31 - __clz(p.page);
      const int kcol = (h / p.rep) * p.dp, vcol = p.v_col0 + (h / p.rep) * p.dvp;
      // box b of tile t: tokens first_key(t) + b * box_rows ..; past the table's end the last page is read (masked keys).
      // Page numbers of a tile are looked up once, one tile ahead of their use.
      int old[kMaxBoxes], pg[kMaxBoxes] = {}, nxt[kMaxBoxes] = {};
      auto look_up = [&](int t) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b)
          if (b < boxes) nxt[b] = bt[min((first_key(t) + b * p.box_rows) >> shift, p.bt_cols - 1)];
      };
      auto load = [&](uint8_t* dst, uint64_t* full, int blocks, int col, int t, const int (&pages)[kMaxBoxes]) {
        mbar_expect_tx(full, blocks * kBlockBytes);
        for (int c = 0; c < blocks; ++c)
#pragma unroll
          for (int b = 0; b < kMaxBoxes; ++b)
            if (b < boxes)
              tma_load_3d(dst + c * kBlockBytes + b * p.box_rows * 128, &tm_kv, full, col + c * 64,
                          (first_key(t) + b * p.box_rows) & (p.page - 1), pages[b]);
      };
      auto load_v = [&](int t) -> bool {                           // values of tile t, whose pages are in `old`
        const int s = t % ST;
        if (!mbar_wait(&ss.v_empty[s], ((t / ST) & 1) ^ 1, abort_flag, kTimeoutProducer)) return false;
        load(v_buf + s * p.VB * kBlockBytes, &ss.v_full[s], p.VB, vcol, t, old);
        return true;
      };
      bool ok = true;
      look_up(0);
      mbar_expect_tx(&ss.q_full, p.KB * kQBlockBytes);
      for (int c = 0; c < p.KB; ++c)
        tma_load_2d(q_buf + c * kQBlockBytes, &tm_q, &ss.q_full, (h * p.KB + c) * 64, w.q_row0 - p.row_shift);
      // the MMA warp takes S(0), S(1), PV(0), S(2), PV(1), ..: values follow the next tile's keys
      for (int t = 0; ok && t < n_tiles; ++t) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b) { old[b] = pg[b]; pg[b] = nxt[b]; }
        if (t + 1 < n_tiles) look_up(t + 1);
        const int s = t % ST;
        ok = mbar_wait(&ss.k_empty[s], ((t / ST) & 1) ^ 1, abort_flag, kTimeoutProducer);
        if (ok) load(k_buf + s * p.KB * kBlockBytes, &ss.k_full[s], p.KB, kcol, t, pg);
        if (ok && t > 0) ok = load_v(t - 1);
      }
      if (ok && n_tiles > 0) {
#pragma unroll
        for (int b = 0; b < kMaxBoxes; ++b) old[b] = pg[b];
        ok = load_v(n_tiles - 1);
      }
      if (ok) {
        // leave only when every copy has landed and been consumed
        const int n = min(n_tiles, ST);
        for (int j = n_tiles - n; j < n_tiles; ++j) {
          if (!mbar_wait(&ss.k_empty[j % ST], (j / ST) & 1, abort_flag, kTimeoutProducer)) break;
          if (!mbar_wait(&ss.v_empty[j % ST], (j / ST) & 1, abort_flag, kTimeoutProducer)) break;
        }
        if (n_tiles <= 0) mbar_wait(&ss.q_full, 0, abort_flag, kTimeoutProducer);
      } else {
        for (uint32_t i = 0; i < (1u << 16); ++i) __nanosleep(20);   // bounded grace period for copies in flight
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      const uint32_t idesc_s = idesc_bf16(BM, BN, 0), idesc_pv = idesc_bf16(BM, p.VB * 64, 1);
      const uint32_t tm_o = tmem_base + 2 * BN;
      bool ok = mbar_wait(&ss.q_full, 0, abort_flag, kTimeoutMma);
      auto issue_s = [&](int t) -> bool {
        const int s = t % ST;
        if (!mbar_wait(&ss.k_full[s], (t / ST) & 1, abort_flag, kTimeoutMma)) return false;
        tc_fence_after();
        const uint32_t tm_s = tmem_base + (t & 1) * BN;
        for (int c = 0; c < p.KB; ++c) {
          const uint64_t adesc = make_smem_desc_sw128(smem_u32(q_buf + c * kQBlockBytes));
          const uint64_t bdesc = make_smem_desc_sw128(smem_u32(k_buf + (s * p.KB + c) * kBlockBytes));
#pragma unroll
          for (int k = 0; k < 4; ++k) mma_f16(tm_s, adesc + 2 * k, bdesc + 2 * k, idesc_s, (c | k) ? 1u : 0u);
        }
        tc_commit(&ss.k_empty[s]);
        tc_commit(&ss.s_full[t & 1]);
        return true;
      };
      if (ok && n_tiles > 0) ok = issue_s(0);
      for (int t = 0; ok && t < n_tiles; ++t) {
        // S of tile t + 1 goes into the buffer that the softmax of tile t - 1 has left (its P was handed over before PV(t-1))
        if (t + 1 < n_tiles && !issue_s(t + 1)) { ok = false; break; }
        const int s = t % ST;
        if (!mbar_wait(&ss.v_full[s], (t / ST) & 1, abort_flag, kTimeoutMma)) { ok = false; break; }
        if (!mbar_wait(&ss.p_full, t & 1, abort_flag, kTimeoutMma)) { ok = false; break; }
        tc_fence_after();
        const uint64_t pdesc = make_smem_desc_sw128(smem_u32(p_buf));
        const uint32_t v_base = smem_u32(v_buf + s * p.VB * kBlockBytes);
#pragma unroll
        for (int j = 0; j < BN / 16; ++j)
          mma_f16(tm_o, pdesc + 2 * j, desc_mn_sw128(v_base + j * 2048, kBlockBytes, 1024), idesc_pv, (t > 0 || j > 0) ? 1u : 0u);
        tc_commit(&ss.v_empty[s]);
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
    int vis_lo = p.chunk > 0 ? pos - pos % p.chunk : 0;            // keys [vis_lo, pos] and those before `keep`
    if (p.window > 0) vis_lo = max(vis_lo, pos + 1 - p.window);
    float m_run = -INFINITY, l_run = 0.f;
    uint8_t* prow = p_buf + (r >> 3) * 1024 + (r & 7) * 128;
    bool ok = true;
    for (int t = 0; ok && t < n_tiles; ++t) {
      if (vote_any_128(!mbar_wait(&ss.s_full[t & 1], (t >> 1) & 1, abort_flag, kTimeoutEpilogue))) { ok = false; break; }
      tc_fence_after();
      uint32_t sv[BN];
      tmem_ld32(tmem_base + lane_addr + (t & 1) * BN, sv);
      tmem_ld32(tmem_base + lane_addr + (t & 1) * BN + 32, sv + 32);
      tmem_ld_wait();
      const int kt = first_key(t);
      const bool kept = t < n_keep;
      const int lo = kept ? 0 : vis_lo - kt, hi = !live ? 0 : kept ? p.keep - kt : pos + 1 - kt;
      const int below = n_keep > 0 ? 0 : p.keep - kt;              // kept keys among this tile's
      if (!__all_sync(0xffffffffu, (lo <= 0 || below >= BN) && hi >= BN)) {
#pragma unroll
        for (int j = 0; j < BN; ++j)
          if ((j < lo && j >= below) || j >= hi) sv[j] = 0xff800000u;              // minus infinity
      }
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < BN; ++j) m4[j & 3] = fmaxf(m4[j & 3], __uint_as_float(sv[j]));
      const float mt = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      const bool grow = mt > m_run + 8.f;
      const float m_new = grow ? mt : m_run;
      const float alpha = (grow && m_run != -INFINITY) ? ex2(m_run - m_new) : 1.f;
      const float neg_m = (m_new == -INFINITY) ? 0.f : -m_new;
      float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < BN; j += 2) {
        const __nv_bfloat162 o = __floats2bfloat162_rn(ex2(__uint_as_float(sv[j]) + neg_m), ex2(__uint_as_float(sv[j + 1]) + neg_m));
        l4[(j >> 1) & 3] += __low2float(o) + __high2float(o);
        sv[j >> 1] = *reinterpret_cast<const uint32_t*>(&o);
      }
      // PV(t - 1) done: O may be rescaled and P overwritten
      if (t > 0 && vote_any_128(!mbar_wait(&ss.o_done, (t - 1) & 1, abort_flag, kTimeoutEpilogue))) { ok = false; break; }
      tc_fence_after();
      if (t > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
        for (int c = 0; c < p.VB * 2; ++c) {
          uint32_t ov[32];
          tmem_ld_32x32(tm_o + c * 32, ov);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) ov[j] = __float_as_uint(__uint_as_float(ov[j]) * alpha);
          tmem_st32(tm_o + c * 32, ov);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      }
#pragma unroll
      for (int c = 0; c < BN / 8; ++c)
        *reinterpret_cast<uint4*>(prow + ((c ^ (r & 7)) << 4)) = make_uint4(sv[4 * c], sv[4 * c + 1], sv[4 * c + 2], sv[4 * c + 3]);
      l_run = l_run * alpha + (l4[0] + l4[1]) + (l4[2] + l4[3]);
      m_run = m_new;
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      tc_fence_before();
      mbar_arrive(&ss.p_full);
    }
    if (ok && n_tiles > 0) ok = !vote_any_128(!mbar_wait(&ss.o_done, (n_tiles - 1) & 1, abort_flag, kTimeoutEpilogue));
    if (ok) {
      tc_fence_after();
      if (p.sink && live) l_run += exp2f((p.sinks != nullptr ? p.sinks[h] * 1.4426950408889634f : 0.f) - m_run);
      float inv = l_run > 0.f ? p.out_scale / l_run : 0.f;
      const float* gate = p.gate != nullptr ? p.gate + (size_t)(w.q_row0 + r) * p.ld_gate + h * p.gate_cols : nullptr;
      const bool each = gate != nullptr && p.gate_cols > 1;
      if (gate != nullptr && !each && live) inv *= 1.0f / (1.0f + expf(-gate[0]));
      __nv_bfloat16* orow = p.out + (size_t)(w.q_row0 + r) * p.ldo + h * p.dvp;
      if (p.staged) {                                          // the tiles are done with: their memory takes fp32 rows of this warp
        const int W = p.VB * 64;                               // row r: 16-byte chunks c at c ^ (r & 7)
        float* stage = reinterpret_cast<float*>(smem);
#pragma unroll 1
        for (int c = 0; c < p.VB * 2; ++c) {
          uint32_t ov[32];
          tmem_ld_32x32(tm_o + c * 32, ov);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 8; ++j)
            *reinterpret_cast<float4*>(stage + r * W + (((c * 8 + j) ^ (r & 7)) << 2)) =
                make_float4(__uint_as_float(ov[4 * j]) * inv, __uint_as_float(ov[4 * j + 1]) * inv, __uint_as_float(ov[4 * j + 2]) * inv,
                            __uint_as_float(ov[4 * j + 3]) * inv);
        }
        __syncwarp();
        const int rows = min(32, w.n_q - quad * 32), c4 = p.dvp / 4;
        const size_t row0 = (size_t)w.q_row0 + quad * 32;
        for (int ch = lane; ch < c4; ch += 32) {
          for (int i0 = 0; i0 < rows; i0 += 8) {               // eight rows' gates in flight
            float4 g[8];
#pragma unroll
            for (int i = 0; i < 8; ++i)
              g[i] = *reinterpret_cast<const float4*>(p.gate + (row0 + min(i0 + i, rows - 1)) * p.ld_gate + h * p.dvp + ch * 4);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              if (i0 + i >= rows) break;
              const int sr = quad * 32 + i0 + i;
              const float4 o = *reinterpret_cast<const float4*>(stage + sr * W + ((ch ^ (sr & 7)) << 2));
              __align__(8) __nv_bfloat162 y[2] = {__floats2bfloat162_rn(o.x / (1.0f + expf(-g[i].x)), o.y / (1.0f + expf(-g[i].y))),
                                                  __floats2bfloat162_rn(o.z / (1.0f + expf(-g[i].z)), o.w / (1.0f + expf(-g[i].w)))};
              *reinterpret_cast<uint2*>(p.out + (row0 + i0 + i) * p.ldo + h * p.dvp + ch * 4) = *reinterpret_cast<const uint2*>(y);
            }
          }
        }
      }
#pragma unroll 1
      for (int c = 0; c < (p.staged ? 0 : p.VB * 2); ++c) {
        uint32_t ov[32];
        tmem_ld_32x32(tm_o + c * 32, ov);
        tmem_ld_wait();
        if (live) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (c * 32 + j < p.dvp) {                          // dvp is a multiple of 8
              __align__(16) __nv_bfloat162 o[4];
              if (each) {
#pragma unroll
                for (int q = 0; q < 8; q += 4) {
                  const float4 g = *reinterpret_cast<const float4*>(gate + c * 32 + j + q);
                  ov[j + q] = __float_as_uint(__uint_as_float(ov[j + q]) / (1.0f + expf(-g.x)));
                  ov[j + q + 1] = __float_as_uint(__uint_as_float(ov[j + q + 1]) / (1.0f + expf(-g.y)));
                  ov[j + q + 2] = __float_as_uint(__uint_as_float(ov[j + q + 2]) / (1.0f + expf(-g.z)));
                  ov[j + q + 3] = __float_as_uint(__uint_as_float(ov[j + q + 3]) / (1.0f + expf(-g.w)));
                }
              }
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
  if (warp == 1) tmem_dealloc(tmem_base, p.tmem_cols);
  if (threadIdx.x == 0 && ss.abort_flag != 0 && p.status != nullptr) atomicMax(p.status, ss.abort_flag);
}

// out[h] = f * q[h], turned by the token's row of `rope` ([T, 2 * half], or null); columns dp .. kc are zero
constexpr int kTurnThreads = 256;
__global__ void __launch_bounds__(kTurnThreads)
turn_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ rope, int half, __nv_bfloat16* __restrict__ out, int H,
            int dp, int kc, float f) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const float* qr = q + (size_t)blockIdx.x * ldq;
  const float* rr = rope + (size_t)blockIdx.x * 2 * half;
  __nv_bfloat16* orow = out + (size_t)blockIdx.x * H * kc;
  for (int i = threadIdx.x * 4; i < H * kc; i += kTurnThreads * 4) {
    const int h = i / kc, e = i % kc;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e < dp) {                                              // dp % 8 == 0
      const float* head = qr + h * dp;
      v = *reinterpret_cast<const float4*>(head + e);
      float* x = &v.x;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = e + j;
        if (rope != nullptr && c < 2 * half) {
          const bool low = c < half;
          const int k = low ? c : c - half;
          const float b = head[low ? c + half : k], co = rr[k], si = rr[half + k];
          x[j] = low ? x[j] * co - b * si : x[j] * co + b * si;
        }
      }
    }
    __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x * f, v.y * f), __floats2bfloat162_rn(v.z * f, v.w * f)};
    *reinterpret_cast<uint2*>(orow + i) = *reinterpret_cast<const uint2*>(o);
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

}  // namespace gqapre
}  // namespace bg

extern "C" {

// Queries of R rows: q fp32 [R, ldq], rope [R, 2 * half] or null -> out bf16 [R, H, kc] (kc = dp rounded up to
// 64), times scale * log2(e).
int bg_gqa_prompt_queries(const float* q, int ldq, const float* rope, int half, void* out, int R, int H, int dp, int kc, float scale,
                 cudaStream_t stream) {
  using namespace bg::gqapre;
  if (R <= 0) return 0;
  if (H <= 0 || dp <= 0 || dp % 8 || kc % 64 || kc < dp || ldq % 4 || (rope != nullptr && (half <= 0 || 2 * half > dp))) return -1;
  bg::launch_pdl(turn_kernel, dim3(R), dim3(kTurnThreads), 0, stream, q, ldq, rope, half, reinterpret_cast<__nv_bfloat16*>(out), H,
                 dp, kc, scale * 1.4426950408889634f);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// qf [R, H, kc] bf16 queries (bg_gqa_prompt_queries) of rows row_shift .. row_shift + R of the step; cache [pages, page, row]
// bf16 with `page_stride` elements between pages; work: n_work x 4 ints (q_row0, n_q, block-table row, position of the first
// query), q_row0 counted in rows of the step; gate [T, ld_gate] fp32 or null; out [T, ldo] bf16.  page: a power of two >= 16;
// dp, dvp <= 256, multiples of 8.
int bg_gqa_prompt(const void* qf, const void* cache, long long page_stride, int n_pages, int page, int row, const int* block_table,
                  int bt_stride, int bt_cols, const int* work, int n_work, int R, int row_shift, void* out, int ldo, int H, int G,
                  int dp, int dvp, int kc, int chunk, int sink, int window, int keep, float out_scale, const float* gate, int ld_gate, int gate_cols, const float* sinks,
                  int* status, cudaStream_t stream) {
  using namespace bg::gqapre;
  if (n_work <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dp <= 0 || dp % 8 || dp > 256 || dvp <= 0 || dvp % 8 || dvp > 256 || kc != (dp + 63) / 64 * 64 ||
      page < 16 || (page & (page - 1)) || row != G * (dp + dvp) || page_stride % 8 || ldo % 8 || bt_cols <= 0 || n_work > 65535 || window < 0 || keep < 0 ||
      (gate != nullptr && gate_cols != 1 && (gate_cols != dvp || ld_gate % 4 || reinterpret_cast<uintptr_t>(gate) % 16)))
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
  p.KB = kc / 64; p.VB = (dvp + 63) / 64; p.dp = dp; p.dvp = dvp; p.v_col0 = G * dp; p.rep = H / G; p.chunk = chunk; p.sink = sink;
  p.window = window; p.keep = keep; p.out_scale = out_scale;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.gate = gate; p.ld_gate = ld_gate; p.gate_cols = gate_cols; p.sinks = sinks; p.row_shift = row_shift;
  p.status = status;
  // two CTAs an SM when two stages and half of TMEM are enough, otherwise one with as many stages as fit
  const bool two = p.VB <= 2 && tile_bytes(p.KB, p.VB, 2) + (int)sizeof(Shared) <= kSmemTwo;
  const int room = (two ? kSmemTwo : 226 * 1024) - (int)sizeof(Shared);
  p.stages = 2;
  while (p.stages < kMaxStages && tile_bytes(p.KB, p.VB, p.stages + 1) <= room) ++p.stages;
  p.staged = gate != nullptr && gate_cols > 1 && tile_bytes(p.KB, p.VB, p.stages) >= BM * p.VB * 256;
  p.tmem_cols = two ? 256 : 512;
  p.smem_bytes = two ? kSmemTwo : 227 * 1024;
  static bg::DeviceOnce once;
  if (!bg::ensure_dynamic_smem(attn_kernel, 227 * 1024, once)) return -13;
  attn_kernel<<<dim3(H, n_work), kThreads, p.smem_bytes, stream>>>(tq, tk, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -14;
}

}  // extern "C"

BG_TRACE_SETTER(gqa_prefill)
