// Grouped-query attention over a paged K/V cache with mixed heads ("talking heads"), chunked visibility and a zero-score
// sink, one query row per CTA (decode, short pieces of prompts, and the fp32 form).
//
//   s[h, j]  = scale * sum_g talk[h, g] (q[g] . k[kv(g), j])        g over all query heads, kv(g) = g / (H / G)
//   seen     = j <= position and (j >= first or j < keep), first = position - position % chunk (chunk 0: first = 0), with a
//              window not before position - window + 1
//   p[h, j]  = exp(s[h, j]) / (exp(sink[h]) + sum exp(s[h, :]))      (the sink's term only with a sink; without numbers of its own it is 1)
//   o[h]     = sum_j p[h, j] v[kv(h), j], times out_scale, times sigmoid(gate[h]) (or a gate per element) when there is a gate
//
// Without a mixing matrix a head keeps its own score (bf16 heads up to 128 wide then run on gqa_rows.cuh instead).  Queries (on load) and keys (on the way to the cache) may carry rotary
// positions: channel i turns with channel i + half.  Mixing couples all heads at a key, so a CTA takes all heads of its row.
// Keys go in tiles of 32 (a lane per key); a
// tile's steps are: raw scores (each warp takes key heads, whose K rows it stages through its own shared-memory buffer;
// the next tile's rows are fetched while the rest of this tile runs), mixing and online softmax (a warp owns blocks of 4
// heads, all 32 keys in its lanes), P.V (a thread owns 4 value columns of up to 4 heads that share a value head, so V is
// read once).  With `n_splits` > 1 the key range is split over CTAs and merged by a second kernel.
//
// The cache row of a token holds the keys of all G heads (dp each), then the values (dvp each); dp and dvp are the head
// widths padded to multiples of 8 with zero channels.  The values may also be the first columns of the keys (a cached latent).
#define BG_FILE_TAG 23     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace talk {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int NT = 32;          // keys per tile

struct Params {
  const float* q;               // [T, ldq]: H heads x dp
  int ldq;
  const float* talk;            // [H, H] or null (no mixing)
  const void* cache;            // [pages, page, row]
  long long page_stride;        // elements between pages
  int page, row;                // tokens per page, elements per token
  const int* block_table;       // [*, bt_stride]
  int bt_stride;
  const int* row_seq;           // [R] block-table row of each query row, or null (identity)
  const int* row_ids;           // [R] row of q / out of each query row, or null (identity)
  const int* lens;              // [T] position + 1 of each row of q; 0 = no query (zero output)
  void* out;                    // [T, ldo]: H heads x dvp
  int ldo;
  float* part_o;                // [R, n_splits, H * dvp]
  float* part_ml;               // [R, n_splits, H, 2]
  int H, G, dp, dvp, chunk, window, keep, sink, n_splits;
  int k_warps;                  // warps with a K buffer (all of them unless heads are very wide)
  float scale_log2, out_scale;
  const float* rope;            // [T, 2 * half] cosines, then sines, or null
  int half;
  const float* gate;            // [T, ld_gate] or null
  int ld_gate, gate_cols;       // columns of a head: 1 or dvp
  const float* sinks;           // [H] or null: all zero
  int v_col0;                   // first value column of a cache row
  const __nv_bfloat16* qb;      // latent_rows.cuh: [R, H, row] queries
  int* status;
};

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 a = __bfloat1622float2(v[i]); f[2 * i] = a.x; f[2 * i + 1] = a.y; }
}
__device__ __forceinline__ float sigm(float x) { return 1.0f / (1.0f + expf(-x)); }
constexpr float kLog2e = 1.4426950408889634f;
// the sink's score of head h, in the scores' base-2 units
__device__ __forceinline__ float sink_score(const Params& p, int h) { return p.sinks != nullptr ? p.sinks[h] * kLog2e : 0.f; }
// times the gate of columns c .. c + 3 of head h
__device__ __forceinline__ float4 gated4(const Params& p, int t, int h, int c, float4 v) {
  if (p.gate == nullptr) return v;
  const float* g = p.gate + (size_t)t * p.ld_gate + h * p.gate_cols;
  if (p.gate_cols == 1) {
    const float f = sigm(g[0]);
    return make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
  }
  const float4 f = *reinterpret_cast<const float4*>(g + c);
  return make_float4(v.x * sigm(f.x), v.y * sigm(f.y), v.z * sigm(f.z), v.w * sigm(f.w));
}
// channel e of a head whose first 2 * half channels turn
__device__ __forceinline__ float turned(const float* x, int e, const float* rope, int half) {
  const float a = x[e];
  if (e >= 2 * half) return a;
  const bool low = e < half;
  const int i = low ? e : e - half;
  const float b = x[low ? e + half : i], c = rope[i], s = rope[half + i];
  return low ? a * c - b * s : a * c + b * s;
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait0() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// shared memory, in floats: q [H dp] | talk^T [H][Hp] (mixed heads only) | raw scores [H][NT] | probabilities [Hp][NT] |
// m, l, a [Hp] each |
// key offsets [NT] (long long), then the K buffers (one per warp), reused for the last reduction
__host__ __device__ inline int pad4(int x) { return (x + 3) / 4 * 4; }
__host__ __device__ inline size_t smem_floats(int H, int dp, bool mixed) {
  const int Hp = pad4(H);
  return (size_t)pad4(H * dp) + (mixed ? (size_t)H * Hp : 0) + (size_t)H * NT + (size_t)Hp * NT + 3 * (size_t)Hp + 2 * NT;
}
template <typename KT>
__host__ __device__ inline size_t kbuf_bytes(int dp) { return (size_t)NT * (dp * sizeof(KT) + 16); }

template <typename KT, int NI, bool MIX>
__global__ void __launch_bounds__(kThreads) rows_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.H, G = p.G, dp = p.dp, dvp = p.dvp, rep = H / G, Hp = pad4(H);
  float* q_s = sm;
  float* tt = q_s + pad4(H * dp);
  float* raw = tt + (MIX ? H * Hp : 0);
  float* pr = raw + H * NT;
  float* m_s = pr + Hp * NT;
  float* l_s = m_s + Hp;
  float* a_s = l_s + Hp;
  long long* koff = reinterpret_cast<long long*>(a_s + Hp);     // 16-byte aligned: every part is a multiple of 4 floats
  char* kb_all = reinterpret_cast<char*>(koff + NT);
  const int r = blockIdx.x, split = blockIdx.y;
  const int t = p.row_ids != nullptr ? p.row_ids[r] : r;
  const int L = p.lens[t];
  KT* out = reinterpret_cast<KT*>(p.out) + (size_t)t * p.ldo;
  if (L <= 0) {
    if (p.n_splits == 1)
      for (int i = tid; i < H * dvp / 4; i += kThreads) put4(out + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;                                                       // (a split row without a query is zeroed by the merge)
  }
  const float* qr = p.q + (size_t)t * p.ldq;
  if (p.rope == nullptr) {
    for (int i = tid; i < H * dp / 4; i += kThreads) reinterpret_cast<float4*>(q_s)[i] = reinterpret_cast<const float4*>(qr)[i];
  } else {
    const float* rope = p.rope + (size_t)t * 2 * p.half;
    for (int i = tid; i < H * dp; i += kThreads) q_s[i] = turned(qr + i / dp * dp, i % dp, rope, p.half);
  }
  if (MIX) {
    for (int i = tid; i < H * Hp; i += kThreads) {
      const int g = i / Hp, h = i % Hp;
      tt[i] = h < H ? p.talk[h * H + g] * p.scale_log2 : 0.f;
    }
  }
  for (int i = tid; i < Hp; i += kThreads) { m_s[i] = -INFINITY; l_s[i] = 0.f; }
  int first = p.chunk > 0 ? (L - 1) - (L - 1) % p.chunk : 0;
  if (p.window > 0) first = max(first, L - p.window);
  // kept first keys that end before the tile of `first` have tiles of their own, ahead of the others
  int t_lo = first / NT, n_keep = 0;
  if (p.keep > t_lo * NT) t_lo = 0;
  else n_keep = (p.keep + NT - 1) / NT;
  const int n_t = n_keep + (L + NT - 1) / NT - t_lo, past_keep = t_lo - n_keep;
  const int my_lo = (int)(((long long)n_t * split) / p.n_splits);
  const int my_hi = (int)(((long long)n_t * (split + 1)) / p.n_splits);
  const int* bt = p.block_table + (size_t)(p.row_seq != nullptr ? p.row_seq[r] : r) * p.bt_stride;
  const KT* cache = reinterpret_cast<const KT*>(p.cache);

  const int hg_n = (rep + 3) / 4;                                 // groups of up to 4 heads per key head
  const int units = G * hg_n;
  const int krow = dp * (int)sizeof(KT) + 16;                     // bytes of a staged K row
  char* kb = kb_all + (size_t)warp * kbuf_bytes<KT>(dp);
  auto key_offset = [&](int tile) -> long long {                  // element offset of this lane's key, < 0 = not seen
    const int pos = (tile < n_keep ? tile : tile + past_keep) * NT + lane;
    if (pos >= L || (pos < first && pos >= p.keep)) return -1;
    return (long long)bt[pos / p.page] * p.page_stride + (long long)(pos % p.page) * p.row;
  };
  auto fetch = [&](int unit, long long off) {                     // K rows of unit's key head -> this warp's buffer
    const int c = unit / hg_n, vec = dp * (int)sizeof(KT) / 16;    // 16-byte pieces of a K row; NT * vec % 32 == 0
    const int step_k = 32 / vec, step_c = 32 % vec;
    int kr = lane / vec, cc = lane % vec;
    for (int i = 0; i < vec; ++i) {
      const long long o = __shfl_sync(0xffffffffu, off, kr);
      if (o >= 0) cp16(kb + kr * krow + cc * 16, reinterpret_cast<const char*>(cache + o + c * dp) + cc * 16);
      kr += step_k;
      cc += step_c;
      if (cc >= vec) { cc -= vec; ++kr; }
    }
    cp_commit();
  };
  // P.V: item = (value head c, group of 4 heads, 4 columns); KG groups of threads take alternate keys
  const int cols = dvp / 4, items = G * hg_n * cols;
  const int KG = items >= kThreads ? 1 : kThreads / items;
  const int kg = items >= kThreads ? 0 : tid / items, item0 = items >= kThreads ? tid : tid % items;
  float2 acc[NI][4][2];
#pragma unroll
  for (int n = 0; n < NI; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i][0] = acc[n][i][1] = make_float2(0.f, 0.f);

  long long off = my_lo < my_hi ? key_offset(my_lo) : -1;
  if (my_lo < my_hi && warp < p.k_warps && warp < units) fetch(warp, off);
  __syncthreads();                                                 // q_s, tt, m_s, l_s
  for (int tile = my_lo; tile < my_hi; ++tile) {
    const long long off_now = off;
    if (warp == 0) koff[lane] = off_now;
    off = tile + 1 < my_hi ? key_offset(tile + 1) : -1;
    for (int u = warp < p.k_warps ? warp : units; u < units; u += p.k_warps) {
      cp_wait0();
      __syncwarp();
      const int c = u / hg_n, h0 = c * rep + (u % hg_n) * 4, nh = min(4, rep - (u % hg_n) * 4);
      float2 s[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) s[i] = make_float2(0.f, 0.f);
      const KT* kr = reinterpret_cast<const KT*>(kb + lane * krow);
      const float* qh[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) qh[i] = q_s + (h0 + min(i, nh - 1)) * dp;
#pragma unroll 2
      for (int e = 0; e < dp; e += 8) {
        float k[8], qv[8];
        load8(kr + e, k);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          load8(qh[i] + e, qv);
#pragma unroll
          for (int j = 0; j < 8; j += 2)                           // packed FMAs (fma.rn.f32x2)
            s[i] = __ffma2_rn(make_float2(qv[j], qv[j + 1]), make_float2(k[j], k[j + 1]), s[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (i < nh) raw[(h0 + i) * NT + lane] = s[i].x + s[i].y;
      __syncwarp();
      if (u + p.k_warps < units) fetch(u + p.k_warps, off_now);
      else if (tile + 1 < my_hi) fetch(warp, off);                 // next tile's rows fly during the rest of this tile
    }
    __syncthreads();
    // mixing + online softmax
    for (int hb = warp; hb < Hp / 4; hb += kWarps) {
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (MIX) {
#pragma unroll 4
        for (int g = 0; g < H; ++g) {
          const float sg = raw[g * NT + lane];
          const float4 w = *reinterpret_cast<const float4*>(tt + g * Hp + hb * 4);
          v[0] = fmaf(w.x, sg, v[0]); v[1] = fmaf(w.y, sg, v[1]); v[2] = fmaf(w.z, sg, v[2]); v[3] = fmaf(w.w, sg, v[3]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (hb * 4 + i < H) v[i] = raw[(hb * 4 + i) * NT + lane] * p.scale_log2;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int h = hb * 4 + i;
        const float x = off_now >= 0 ? v[i] : -INFINITY;
        const float mo = m_s[h], mn = fmaxf(mo, warp_max(x));
        const float e = mn == -INFINITY ? 0.f : exp2f(x - mn);
        const float sum = warp_sum(e);
        pr[h * NT + lane] = e;
        __syncwarp();
        if (lane == 0) {
          const float al = mn == -INFINITY ? 1.f : exp2f(mo - mn);
          a_s[h] = al;
          m_s[h] = mn;
          l_s[h] = l_s[h] * al + sum;
        }
      }
    }
    __syncthreads();
    // O = O * alpha + P . V, four keys at a time (unseen keys have p = 0 and are not read)
    if (kg < KG) {
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        const int it = item0 + n * kThreads;
        if (it < items) {
          const int u = it / cols, cc = it % cols, c = u / hg_n;
          const int h0 = c * rep + (u % hg_n) * 4, nh = min(4, rep - (u % hg_n) * 4);
          const KT* vb = cache + (size_t)p.v_col0 + (size_t)c * dvp + cc * 4;
          const float* ph[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int h = h0 + min(i, nh - 1);
            ph[i] = pr + h * NT;
            const float al = a_s[h];
            acc[n][i][0].x *= al; acc[n][i][0].y *= al; acc[n][i][1].x *= al; acc[n][i][1].y *= al;
          }
#pragma unroll 2
          for (int j = 4 * kg; j < NT; j += 4 * KG) {
            float4 v[4], w[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
              const long long o = koff[j + x];
              v[x] = o >= 0 ? load4(vb + o) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) w[i] = *reinterpret_cast<const float4*>(ph[i] + j);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
              const float2 lo = make_float2(v[x].x, v[x].y), hi = make_float2(v[x].z, v[x].w);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float f = x == 0 ? w[i].x : x == 1 ? w[i].y : x == 2 ? w[i].z : w[i].w;
                acc[n][i][0] = __ffma2_rn(make_float2(f, f), lo, acc[n][i][0]);
                acc[n][i][1] = __ffma2_rn(make_float2(f, f), hi, acc[n][i][1]);
              }
            }
          }
        }
      }
    }
    __syncthreads();                                               // koff, pr and raw are free again
  }
  // sum over the key groups (only when all items fit one pass: NI == 1)
  float* red = reinterpret_cast<float*>(kb_all);
  if (KG > 1) {
    cp_wait0();
    __syncthreads();
    if (kg > 0 && kg < KG) {
#pragma unroll
      for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(red + ((size_t)i * kThreads + tid) * 4) =
          make_float4(acc[0][i][0].x, acc[0][i][0].y, acc[0][i][1].x, acc[0][i][1].y);
    }
    __syncthreads();
    if (kg == 0) {
      for (int k = 1; k < KG; ++k) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 v = *reinterpret_cast<const float4*>(red + ((size_t)i * kThreads + k * items + tid) * 4);
          acc[0][i][0].x += v.x; acc[0][i][0].y += v.y; acc[0][i][1].x += v.z; acc[0][i][1].y += v.w;
        }
      }
    }
  }
  if (kg == 0) {
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int it = item0 + n * kThreads;
      if (it < items) {
        const int u = it / cols, cc = it % cols, c = u / hg_n;
        const int h0 = c * rep + (u % hg_n) * 4, nh = min(4, rep - (u % hg_n) * 4);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (i >= nh) break;
          const int h = h0 + i, col = h * dvp + cc * 4;
          const float4 v = make_float4(acc[n][i][0].x, acc[n][i][0].y, acc[n][i][1].x, acc[n][i][1].y);
          if (p.n_splits == 1) {
            const float inv = p.out_scale / (l_s[h] + (p.sink ? exp2f(sink_score(p, h) - m_s[h]) : 0.f));
            put4(out + col, gated4(p, t, h, cc * 4, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv)));
          } else {
            *reinterpret_cast<float4*>(p.part_o + ((size_t)r * p.n_splits + split) * H * dvp + col) = v;
          }
        }
      }
    }
  }
  if (p.n_splits > 1)
    for (int h = tid; h < H; h += kThreads) {
      float* ml = p.part_ml + (((size_t)r * p.n_splits + split) * H + h) * 2;
      ml[0] = m_s[h];
      ml[1] = l_s[h];
    }
}

// one block per (row, head)
template <typename KT>
__global__ void merge_kernel(const Params p) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int r = blockIdx.x, h = blockIdx.y, S = p.n_splits;
  const int t = p.row_ids != nullptr ? p.row_ids[r] : r;
  KT* out = reinterpret_cast<KT*>(p.out) + (size_t)t * p.ldo + h * p.dvp;
  if (p.lens[t] <= 0) {
    for (int i = threadIdx.x; i < p.dvp / 4; i += blockDim.x) put4(out + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  const float* ml = p.part_ml + (size_t)r * S * p.H * 2 + h * 2;
  const float sink = p.sink ? sink_score(p, h) : -INFINITY;
  float m = sink;
  for (int s = 0; s < S; ++s) m = fmaxf(m, ml[(size_t)s * p.H * 2]);
  float l = p.sink ? exp2f(sink - m) : 0.f;
  for (int s = 0; s < S; ++s) {
    const float ms = ml[(size_t)s * p.H * 2];
    if (ms != -INFINITY) l += ml[(size_t)s * p.H * 2 + 1] * exp2f(ms - m);
  }
  const float inv = p.out_scale / l;
  for (int i = threadIdx.x; i < p.dvp / 4; i += blockDim.x) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < S; ++s) {
      const float ms = ml[(size_t)s * p.H * 2];
      if (ms == -INFINITY) continue;
      const float f = exp2f(ms - m);
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + ((size_t)r * S + s) * p.H * p.dvp + h * p.dvp + 4 * i);
      a.x += f * v.x; a.y += f * v.y; a.z += f * v.z; a.w += f * v.w;
    }
    put4(out + 4 * i, gated4(p, t, h, 4 * i, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv)));
  }
}

// cache[slot[t]] = kv[t] (fp32 projection columns: keys of all G heads of dp channels, then values), the keys turned by the
// token's row of `rope` when there is one; slot < 0 writes nothing
template <typename KT>
__global__ void __launch_bounds__(128)
kv_write_kernel(const float* __restrict__ kv, int ld, const long long* __restrict__ slots, KT* __restrict__ cache,
                long long page_stride, int page, int row, const float* __restrict__ rope, int half, int G, int dp) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const long long slot = slots[blockIdx.x];
  if (slot < 0) return;
  KT* dst = cache + (slot / page) * page_stride + (slot % page) * row;
  const float* src = kv + (size_t)blockIdx.x * ld;
  const float* rr = rope + (size_t)blockIdx.x * 2 * half;
  for (int i = threadIdx.x; i < row / 4; i += blockDim.x) {
    const int c = 4 * i;
    float4 v = *reinterpret_cast<const float4*>(src + c);
    if (rope != nullptr && c < G * dp && c % dp < 2 * half) {       // dp % 8 == 0: the four channels share a head
      const float* head = src + c / dp * dp;
      const int e = c % dp;
      v = make_float4(turned(head, e, rr, half), turned(head, e + 1, rr, half), turned(head, e + 2, rr, half),
                      turned(head, e + 3, rr, half));
    }
    put4(dst + c, v);
  }
}

template <typename KT, int NI, bool MIX>
static int launch_rows_as(Params p, int R, cudaStream_t stream) {
  const size_t fixed = smem_floats(p.H, p.dp, MIX) * sizeof(float), one = kbuf_bytes<KT>(p.dp), most = 227 * 1024;
  const size_t red = (size_t)kThreads * 16 * sizeof(float);
  for (p.k_warps = kWarps; p.k_warps > 1 && fixed + p.k_warps * one > most; --p.k_warps) {}
  const size_t smem = fixed + (p.k_warps * one < red ? red : p.k_warps * one);
  if (smem > most) return -3;
  static DeviceOnce once;
  auto kern = rows_kernel<KT, NI, MIX>;
  if (!ensure_dynamic_smem(kern, 227 * 1024, once)) return -4;
  bg::launch_pdl(kern, dim3(R, p.n_splits), dim3(kThreads), smem, stream, p);
  if (p.n_splits > 1) bg::launch_pdl(merge_kernel<KT>, dim3(R, p.H), dim3(64), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <typename KT, int NI>
static int launch_rows(const Params& p, int R, cudaStream_t stream) {
  return p.talk != nullptr ? launch_rows_as<KT, NI, true>(p, R, stream) : launch_rows_as<KT, NI, false>(p, R, stream);
}

}  // namespace talk
}  // namespace bg

#include "gqa_rows.cuh"
#include "latent_rows.cuh"

extern "C" {

// dt: 0 = bf16 cache and output, 1 = fp32.  -1: sizes out of contract; -3: heads x width need more shared memory than a CTA has.
int bg_talk_rows(int dt, const float* q, int ldq, const float* talk, const void* cache, long long page_stride, int page,
                 int row, const int* block_table, int bt_stride, const int* row_seq, const int* row_ids, const int* lens,
                 void* out, int ldo, float* part_o, float* part_ml, int R, int H, int G, int dp, int dvp, int chunk,
                 int window, int keep, int sink, float scale, float out_scale, int n_splits, const float* rope, int half, const float* gate, int ld_gate, int gate_cols,
                 const float* sinks, int v_col0, cudaStream_t stream) {
  using namespace bg::talk;
  if (R <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dp <= 0 || dp % 8 || dvp <= 0 || dvp % 8 || row < G * dp || v_col0 < 0 || v_col0 % 8 || row < v_col0 + G * dvp || row % 8 || page <= 0 ||
      page_stride % 8 || ldq % 4 || ldo % 4 || (rope != nullptr && (half <= 0 || 2 * half > dp)) || n_splits < 1 || n_splits > 65535 || H > 65535 ||
      window < 0 || keep < 0 || (gate != nullptr && gate_cols != 1 && (gate_cols != dvp || ld_gate % 4 || reinterpret_cast<uintptr_t>(gate) % 16)) ||
      (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return -1;
  Params p;
  p.q = q; p.ldq = ldq; p.talk = talk; p.cache = cache; p.page_stride = page_stride; p.page = page; p.row = row;
  p.block_table = block_table; p.bt_stride = bt_stride; p.row_seq = row_seq; p.row_ids = row_ids; p.lens = lens;
  p.out = out; p.ldo = ldo; p.part_o = part_o; p.part_ml = part_ml; p.H = H; p.G = G; p.dp = dp; p.dvp = dvp;
  p.chunk = chunk; p.window = window; p.keep = keep; p.out_scale = out_scale; p.sink = sink; p.n_splits = n_splits; p.scale_log2 = scale * 1.4426950408889634f;
  p.rope = rope; p.half = half; p.gate = gate; p.ld_gate = ld_gate; p.gate_cols = gate_cols; p.sinks = sinks;
  p.v_col0 = v_col0; p.qb = nullptr; p.status = nullptr;
  const int items = G * ((H / G + 3) / 4) * (dvp / 4);
  const int ni = (items + kThreads - 1) / kThreads;
  if (ni > 8 && !(dt == 0 && plain::supported(p))) return -1;
  if (dt == 0) {
    if (plain::supported(p)) return plain::launch(p, R, stream);
    if (ni == 1) return launch_rows<__nv_bfloat16, 1>(p, R, stream);
    if (ni == 2) return launch_rows<__nv_bfloat16, 2>(p, R, stream);
    if (ni <= 4) return launch_rows<__nv_bfloat16, 4>(p, R, stream);
    return launch_rows<__nv_bfloat16, 8>(p, R, stream);
  }
  if (ni == 1) return launch_rows<float, 1>(p, R, stream);
  if (ni == 2) return launch_rows<float, 2>(p, R, stream);
  if (ni <= 4) return launch_rows<float, 4>(p, R, stream);
  return launch_rows<float, 8>(p, R, stream);
}

int bg_talk_kv_write(int dt, const float* kv, int ld, const long long* slots, void* cache, long long page_stride, int page,
                     int row, int T, const float* rope, int half, int G, int dp, cudaStream_t stream) {
  using namespace bg::talk;
  if (T <= 0) return 0;
  if (row % 8 || ld % 4 || ld < row || page <= 0 || page_stride % 8) return -1;
  if (rope != nullptr && (half <= 0 || dp % 8 || 2 * half > dp || G * dp > row)) return -1;
  if (dp <= 0) dp = row;
  if (dt == 0)
    bg::launch_pdl(kv_write_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, stream, kv, ld, slots,
                   reinterpret_cast<__nv_bfloat16*>(cache), page_stride, page, row, rope, half, G, dp);
  else
    bg::launch_pdl(kv_write_kernel<float>, dim3(T), dim3(128), 0, stream, kv, ld, slots, reinterpret_cast<float*>(cache),
                   page_stride, page, row, rope, half, G, dp);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"

BG_TRACE_SETTER(talking_attn)
