// Decode attention of plain grouped-query heads over a bf16 cache, included by talking_attn.cu (same parameters, same merge of
// key ranges).  A CTA takes one query row, up to 16 heads of one key head and a range of keys; its warps take alternate tiles of
// 16 keys and never meet until the end.
//
// Per tile a warp has K and V rows brought into its own ring by cp.async, multiplies its 16 query rows (bf16, scale * log2(e)
// folded in before the rounding) with the keys on the tensor cores (mma m16n8k16: with a handful of heads per key head the 128-row
// tcgen05 shapes would be idle rows), takes the online softmax in registers and feeds the probabilities straight into P.V.
// Memory-bound by design: every key and value byte is read once per key head.
#pragma once

namespace bg {
namespace talk {
namespace plain {

constexpr int kRowWarps = 4, kTile = 16, kStages = 3;
constexpr int kMaxWidth = 128;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes from src, or zeros (nothing is read then)
__device__ __forceinline__ void cp16_or_zero(uint32_t dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(real ? 16 : 0) : "memory");
}
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// bytes of a staged key / value row: whole 16-wide steps, plus 16 so that eight rows start in different banks
__host__ __device__ inline int row_bytes(int w) { return (w + 15) / 16 * 32 + 16; }
__host__ __device__ inline int stage_bytes(int dp, int dvp) { return kTile * (row_bytes(dp) + row_bytes(dvp)); }
__host__ __device__ inline int shared_bytes(int dp, int dvp, int heads) {
  const int ring = kRowWarps * kStages * stage_bytes(dp, dvp), red = kRowWarps * heads * dvp * 4;
  return 16 * row_bytes(dp) + kRowWarps * 16 * 8 + (ring > red ? ring : red);
}

// KD, VD: upper bounds of the 16-wide steps of a key / value head; HI: more than 8 heads in the CTA
template <int KD, int VD, bool HI>
__global__ void __launch_bounds__(kRowWarps * 32, 2) gqa_rows_kernel(const Params p, int groups) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(16) char sm_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.H, G = p.G, dp = p.dp, dvp = p.dvp, rep = H / G;
  const int r = blockIdx.x, split = blockIdx.z, c = blockIdx.y / groups, h0 = c * rep + blockIdx.y % groups * 16;
  const int nh = min(16, (c + 1) * rep - h0);                      // heads h0 .. h0 + nh of key head c
  const int t = p.row_ids != nullptr ? p.row_ids[r] : r;
  const int L = p.lens[t];
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)t * p.ldo + h0 * dvp;
  if (L <= 0) {
    if (p.n_splits == 1)
      for (int i = tid; i < nh * dvp / 4; i += kRowWarps * 32) put4(out + 4 * i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;                                                        // (a split row without a query is zeroed by the merge)
  }
  const int kb = row_bytes(dp), vb = row_bytes(dvp), sb = stage_bytes(dp, dvp);
  char* q_s = sm_raw;
  float2* ml_s = reinterpret_cast<float2*>(q_s + 16 * kb);         // [warps][16]
  char* ring_all = reinterpret_cast<char*>(ml_s + kRowWarps * 16);
  char* ring = ring_all + warp * kStages * sb;
  const uint32_t ring_u = smem_u32(ring);
  int first = p.chunk > 0 ? (L - 1) - (L - 1) % p.chunk : 0;
  if (p.window > 0) first = max(first, L - p.window);
  int t_lo = first / kTile, n_keep = 0;                            // as in rows_kernel
  if (p.keep > t_lo * kTile) t_lo = 0;
  else n_keep = (p.keep + kTile - 1) / kTile;
  const int n_t = n_keep + (L + kTile - 1) / kTile - t_lo, past_keep = t_lo - n_keep;
  const int my_lo = (int)(((long long)n_t * split) / p.n_splits) + warp;
  const int my_hi = (int)(((long long)n_t * (split + 1)) / p.n_splits);
  const int* bt = p.block_table + (size_t)(p.row_seq != nullptr ? p.row_seq[r] : r) * p.bt_stride;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  auto first_pos = [&](int tile) { return (tile < n_keep ? tile : tile + past_keep) * kTile; };
  auto seen = [&](int pos) { return pos < L && (pos >= first || pos < p.keep); };
  auto key_offset = [&](int tile) -> long long {                   // of key lane % 16 of the tile; < 0: not seen
    if (tile >= my_hi) return -1;
    const int pos = first_pos(tile) + (lane & 15);
    return seen(pos) ? (long long)bt[pos / p.page] * p.page_stride + (long long)(pos % p.page) * p.row : -1;
  };
  auto copy_rows = [&](uint32_t dst, int stride, int w, const __nv_bfloat16* src, long long off) {
    const int vec = w / 8, step_r = 32 / vec, step_c = 32 % vec;   // 16-byte pieces of a row
    int kr = lane / vec, cc = lane % vec;
    for (int i = 0; i < kTile * vec; i += 32) {
      const long long o = __shfl_sync(0xffffffffu, off, kr & 15);
      if (kr < kTile) cp16_or_zero(dst + kr * stride + cc * 16, src + (o >= 0 ? o + cc * 8 : 0), o >= 0);
      kr += step_r;
      cc += step_c;
      if (cc >= vec) { cc -= vec; ++kr; }
    }
  };
  auto fetch = [&](int tile, int slot, long long off) {
    if (tile < my_hi) {
      copy_rows(ring_u + slot * sb, kb, dp, cache + c * dp, off);
      copy_rows(ring_u + slot * sb + kTile * kb, vb, dvp, cache + (size_t)p.v_col0 + (size_t)c * dvp, off);
    }
    cp_commit();                                                   // an empty group keeps the count of groups in step
  };
  const int ksteps = (dp + 15) / 16, vsteps = (dvp + 15) / 16;
  float o[2 * VD][4];
#pragma unroll
  for (int n = 0; n < 2 * VD; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};          // rows lane / 4 and lane / 4 + 8; l: this lane's keys only
  if (dp % 16 || dvp % 16)                                         // channels past the widths meet zeros of the query, or are not stored
    for (int i = lane; i < kStages * sb / 16; i += 32) reinterpret_cast<uint4*>(ring)[i] = make_uint4(0, 0, 0, 0);
  __syncwarp();
  int ahead = my_lo;
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s, ahead += kRowWarps) fetch(ahead, s, key_offset(ahead));
  long long off = key_offset(ahead);
  // queries -> bf16 rows, zero past the width and past the last head
  for (int i = tid; i < 16 * kb / 16; i += kRowWarps * 32) {
    const int h = i * 16 / kb, e = i * 16 % kb / 2;                // 8 channels
    __align__(16) __nv_bfloat162 v[4] = {};
    if (h < nh && e < dp) {
      const float* x = p.q + (size_t)t * p.ldq + (h0 + h) * dp;
      float f[8];
      load8(x + e, f);
      if (p.rope != nullptr) {
        const float* rope = p.rope + (size_t)t * 2 * p.half;
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = turned(x, e + j, rope, p.half);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = __floats2bfloat162_rn(f[2 * j] * p.scale_log2, f[2 * j + 1] * p.scale_log2);
    }
    *reinterpret_cast<uint4*>(q_s + i * 16) = *reinterpret_cast<const uint4*>(v);
  }
  __syncthreads();                                                 // q_s
  uint32_t qa[KD][4];
#pragma unroll
  for (int k = 0; k < KD; ++k)
    if (k < ksteps) ldsm4(qa[k], smem_u32(q_s) + (lane & 15) * kb + (k * 16 + (lane >> 4) * 8) * 2);
  int slot = 0, free_slot = kStages - 1;
  for (int tile = my_lo; tile < my_hi; tile += kRowWarps) {
    cp_wait<kStages - 2>();
    __syncwarp();
    fetch(ahead, free_slot, off);
    ahead += kRowWarps;
    off = key_offset(ahead);
    const uint32_t ks = ring_u + slot * sb, vs = ks + kTile * kb;
    float s[2][4] = {}, s2[2][4] = {};
    const uint32_t ka = ks + ((lane >> 4) * 8 + (lane & 7)) * kb + ((lane >> 3) & 1) * 16;
    uint32_t kf[KD][4];                                            // all of a tile's keys first, then the products
#pragma unroll
    for (int k = 0; k < KD; ++k)
      if (k < ksteps) ldsm4(kf[k], ka + k * 32);
#pragma unroll
    for (int k = 0; k < KD; ++k)
      if (k < ksteps) {
        mma16816(k & 1 ? s2[0] : s[0], qa[k], kf[k][0], kf[k][1]);
        mma16816(k & 1 ? s2[1] : s[1], qa[k], kf[k][2], kf[k][3]);
      }
    const int pos = first_pos(tile) + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
#pragma unroll
      for (int j = 0; j < 4; ++j) s[n][j] += s2[n][j];
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (!seen(pos + n * 8 + j)) s[n][j] = s[n][2 + j] = -INFINITY;
    }
    uint32_t pa[4] = {0, 0, 0, 0};
    float al[2] = {1.f, 1.f};
#pragma unroll
    for (int i = 0; i < (HI ? 2 : 1); ++i) {
      float mt = fmaxf(fmaxf(s[0][2 * i], s[0][2 * i + 1]), fmaxf(s[1][2 * i], s[1][2 * i + 1]));
      mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 1));
      mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 2));
      const float mn = fmaxf(m[i], mt), sub = mn == -INFINITY ? 0.f : mn;
      al[i] = exp2f(m[i] - sub);
      m[i] = mn;
      const __nv_bfloat162 lo = __floats2bfloat162_rn(exp2f(s[0][2 * i] - sub), exp2f(s[0][2 * i + 1] - sub));
      const __nv_bfloat162 hi = __floats2bfloat162_rn(exp2f(s[1][2 * i] - sub), exp2f(s[1][2 * i + 1] - sub));
      l[i] = l[i] * al[i] + (__low2float(lo) + __high2float(lo)) + (__low2float(hi) + __high2float(hi));
      pa[i] = *reinterpret_cast<const uint32_t*>(&lo);
      pa[2 + i] = *reinterpret_cast<const uint32_t*>(&hi);
    }
    if (__any_sync(0xffffffffu, al[0] != 1.f || al[1] != 1.f)) {
#pragma unroll
      for (int n = 0; n < 2 * VD; ++n) { o[n][0] *= al[0]; o[n][1] *= al[0]; o[n][2] *= al[1]; o[n][3] *= al[1]; }
    }
    const uint32_t va = vs + (lane & 15) * vb + (lane >> 4) * 16;
#pragma unroll
    for (int n0 = 0; n0 < VD; n0 += 4) {
      uint32_t vf[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
        if (n0 + n < vsteps) ldsm4t(vf[n], va + (n0 + n) * 32);
#pragma unroll
      for (int n = 0; n < 4; ++n)
        if (n0 + n < vsteps) {
          mma16816(o[2 * (n0 + n)], pa, vf[n][0], vf[n][1]);
          mma16816(o[2 * (n0 + n) + 1], pa, vf[n][2], vf[n][3]);
        }
    }
    slot = slot + 1 == kStages ? 0 : slot + 1;
    free_slot = free_slot + 1 == kStages ? 0 : free_slot + 1;
  }
  cp_wait<0>();
  // the warps' sums meet: row i of a warp counts with 2^(m_i - m)
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    if ((lane & 3) == 0) ml_s[warp * 16 + i * 8 + (lane >> 2)] = make_float2(m[i], l[i]);
  }
  __syncthreads();                                                 // every ring is free
  float* red = reinterpret_cast<float*>(ring_all);                 // [warps][nh][dvp]
#pragma unroll
  for (int i = 0; i < (HI ? 2 : 1); ++i) {
    const int row = i * 8 + (lane >> 2);
    if (row < nh) {
#pragma unroll
      for (int n = 0; n < 2 * VD; ++n) {
        const int col = n * 8 + (lane & 3) * 2;
        if (col < dvp)
          *reinterpret_cast<float2*>(red + ((size_t)warp * nh + row) * dvp + col) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < nh * dvp / 4; i += kRowWarps * 32) {
    const int row = 4 * i / dvp, col = 4 * i % dvp, h = h0 + row;
    float mm = -INFINITY, ll = 0.f;
#pragma unroll
    for (int w = 0; w < kRowWarps; ++w) mm = fmaxf(mm, ml_s[w * 16 + row].x);
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kRowWarps; ++w) {
      const float2 x = ml_s[w * 16 + row];
      const float f = x.x == -INFINITY ? 0.f : exp2f(x.x - mm);
      const float4 v = *reinterpret_cast<const float4*>(red + ((size_t)w * nh + row) * dvp + col);
      ll += f * x.y;
      a.x += f * v.x; a.y += f * v.y; a.z += f * v.z; a.w += f * v.w;
    }
    if (p.n_splits == 1) {
      const float inv = p.out_scale / (ll + (p.sink ? exp2f(sink_score(p, h) - mm) : 0.f));
      put4(out + 4 * i, gated4(p, t, h, col, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv)));
    } else {
      *reinterpret_cast<float4*>(p.part_o + (((size_t)r * p.n_splits + split) * H + h) * dvp + col) = a;
      if (col == 0) *reinterpret_cast<float2*>(p.part_ml + (((size_t)r * p.n_splits + split) * H + h) * 2) = make_float2(mm, ll);
    }
  }
}

template <int KD, int VD, bool HI>
static int launch_as(const Params& p, int R, int groups, cudaStream_t stream) {
  const size_t smem = shared_bytes(p.dp, p.dvp, min(16, p.H / p.G));
  static DeviceOnce once;
  auto kern = gqa_rows_kernel<KD, VD, HI>;
  if (!ensure_dynamic_smem(kern, shared_bytes(16 * KD, 16 * VD, 16), once)) return -4;
  bg::launch_pdl(kern, dim3(R, p.G * groups, p.n_splits), dim3(kRowWarps * 32), smem, stream, p, groups);
  if (p.n_splits > 1) bg::launch_pdl(merge_kernel<__nv_bfloat16>, dim3(R, p.H), dim3(64), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int KD, int VD>
static int launch_heads(const Params& p, int R, int groups, cudaStream_t stream) {
  return p.H / p.G > 8 ? launch_as<KD, VD, true>(p, R, groups, stream) : launch_as<KD, VD, false>(p, R, groups, stream);
}
static bool supported(const Params& p) {
  const int groups = (p.H / p.G + 15) / 16;
  return p.talk == nullptr && p.v_col0 == p.G * p.dp && p.dp <= kMaxWidth && p.dvp <= kMaxWidth && (long long)p.G * groups <= 65535;
}
static int launch(const Params& p, int R, cudaStream_t stream) {
  const int groups = (p.H / p.G + 15) / 16;
  if (p.dp <= 64 && p.dvp <= 64) return launch_heads<4, 4>(p, R, groups, stream);
  return launch_heads<8, 8>(p, R, groups, stream);
}

}  // namespace plain
}  // namespace talk
}  // namespace bg
