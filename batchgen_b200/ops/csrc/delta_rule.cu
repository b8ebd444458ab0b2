// Generalised delta rule: a per-head matrix state with a per-channel decay and a per-channel removal rate.
//
// Per head, state S [D keys x D values] (fp32).  For each token, with unit key u = k / sqrt(sum k^2 + ueps):
//
//   w  = exp(-cdecay * sigmoid(wl + w0))          decay per key channel
//   a  = sigmoid(al + ab)                         removal rate per key channel
//   S' = diag(w) S - (a * u) (u^T S) + k v^T      both terms read the old state
//   o  = S'^T r
//   out = o / sqrt(mean(o^2) + eps) * norm * sigmoid(g)
//
// Both products of a step come from one sweep of the old state: with y = u^T S and q = (w * r)^T S,
// o = q - (r . (a * u)) y + (r . k) v.
//
// Decode (`decode_kernel`, D <= 128): a token is one read and write of the state with everything else fused around it.
//
// Prompts (`prep` -> `scan` -> `finish`): a value column of S evolves on its own once w, u, a * u and w * r are known, so the
// scan splits a head's columns over CTAs of 32 columns and needs no barrier inside a token (16 lanes share a column, four
// shuffles sum their rows; packed fp32 FMAs).  `prep` computes the per-token vectors for all tokens in parallel and `finish`
// applies the output norm and gate, which need whole heads.
//
// Everything that enters the recurrence is fp32; the projections arrive as fp32 GEMM outputs.
#define BG_FILE_TAG 22     // kernel-trace ids of this file are (tag << 16) | line
#include "common.cuh"

namespace bg {
namespace delta {

struct Params {
  const float* z;          // [T, ldz] stacked projections of the layer input
  int ldz;
  int off_r, off_k, off_v, off_g, off_a;   // first column of each projection in z (heads x D each)
  const float* wl;         // [T, ld_wl] low-rank decay pre-activation
  int ld_wl;
  const float* w0;         // [H * D]
  const float* ab;         // [H * D]
  const float* norm_w;     // [H * D]
  float* state;            // [slots] rows of `slot_stride` floats; this layer's [H, D, D] at the pointer
  long long slot_stride;
  const int* cu;           // [nseq + 1] token ranges, or null: one token per sequence
  const int* slots;        // [nseq], < 0 skips the sequence (its output rows become zero)
  const int* has_initial;  // [nseq] or null (always continue from the slot)
  void* out;               // [T, ldo]
  int ldo;
  int H, D, Dreal;         // D: padded head width (multiple of 8); Dreal: channels of the mean
  float cdecay, ueps, eps;
};

template <typename OT> __device__ __forceinline__ void put4(OT* p, float4 v);
template <> __device__ __forceinline__ void put4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void put4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ float sigm(float x) { return 1.0f / (1.0f + expf(-x)); }

constexpr int kMaxD = 256;

// Decode, one token per sequence, persistent over (sequence, head) items.  A head's state is one contiguous block of
// D * D * 4 bytes.  A producer thread brings blocks into a ring of three shared-memory buffers with bulk copies and takes
// them back the same way; two groups of four warps work on alternate items in place, so one group's barriers and reductions
// hide behind the other's arithmetic and the SM always has loads and stores in flight.
//
// A warp owns 32 value columns: lane (rg, jq) has columns 4 jq .. 4 jq + 3 of them and the key rows rg * NR .. + NR - 1
// (two shuffles sum the four row groups), so a group needs two barriers per item: vectors ready, output norm.
constexpr int kBufs = 3;

__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void bulk_store(void* dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(smem_u32(src)), "r"(bytes)
               : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

__device__ __forceinline__ void group_sync(int group) { asm volatile("bar.sync %0, 128;" ::"r"(group + 1) : "memory"); }
__device__ __forceinline__ float4 xor_sum(float4 v, int mask) {
  v.x += __shfl_xor_sync(0xffffffffu, v.x, mask); v.y += __shfl_xor_sync(0xffffffffu, v.y, mask);
  v.z += __shfl_xor_sync(0xffffffffu, v.z, mask); v.w += __shfl_xor_sync(0xffffffffu, v.w, mask);
  return v;
}

template <typename OT, int NR>
__global__ void __launch_bounds__(288) decode_kernel(const Params p, int items, int* status) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(128) float ring[];                // kBufs x D * D
  __shared__ uint64_t full[kBufs], done[kBufs];
  __shared__ int abort_s;
  __shared__ __align__(16) float vec[2][4][4 * NR];             // per group: k, w, a * k, w * r (zero past D)
  __shared__ __align__(16) float sv[2][128];
  __shared__ float red[2][3][4], red_o[2][4];
  const int tid = threadIdx.x, lane = tid & 31;
  const int D = p.D, H = p.H, DD = D * D, Q = D / 4;
  volatile int* abort_flag = &abort_s;
  if (tid == 0) {
    for (int s = 0; s < kBufs; ++s) { mbar_init(&full[s], 1); mbar_init(&done[s], 1); }
    abort_s = 0;
    mbar_fence_init();
  }
  for (int i = tid; i < 2 * 4 * 4 * NR; i += 288) (&vec[0][0][0])[i] = 0.f;
  __syncthreads();
  if (tid >= 256) {
    // ------------------------------------------------------------ producer (one thread): item k lives in buffer k % kBufs
    if (tid != 256) return;
    const uint32_t bytes = (uint32_t)DD * 4;
    auto next_live = [&](int item) {
      while (item < items && p.slots[item / H] < 0) item += gridDim.x;
      return item;
    };
    auto block_of = [&](int item) { return p.state + p.slots[item / H] * p.slot_stride + (size_t)(item % H) * DD; };
    int ahead = next_live(blockIdx.x);
    auto load = [&](int k) {
      if (ahead >= items) return;
      mbar_expect_tx(&full[k % kBufs], bytes);
      bulk_load(ring + (size_t)(k % kBufs) * DD, block_of(ahead), bytes, &full[k % kBufs]);
      ahead = next_live(ahead + gridDim.x);
    };
    for (int k = 0; k < kBufs; ++k) load(k);
    int k = 0;
    for (int item = next_live(blockIdx.x); item < items; item = next_live(item + gridDim.x), ++k) {
      if (!mbar_wait(&done[k % kBufs], (k / kBufs) & 1, abort_flag, kTimeoutProducer)) break;
      bulk_store(block_of(item), ring + (size_t)(k % kBufs) * DD, bytes);
      asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
      load(k + kBufs);
    }
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    if (abort_s != 0) {
      for (uint32_t i = 0; i < (1u << 16); ++i) __nanosleep(20);     // bounded grace period for copies in flight
      if (status != nullptr) atomicMax(status, abort_s);
    }
    return;
  }
  // -------------------------------------------------------------- two groups of 128 threads
  const int group = tid >> 7, gt = tid & 127, gw = gt >> 5, jq = lane & 7, rg = lane >> 3;
  const int quad = gw * 8 + jq, dwarps = (D + 31) / 32;
  const bool col_ok = quad < Q;
  float nr = 0.f, nk = 0.f, nv = 0.f, na = 0.f, nw = 0.f, nw0 = 0.f, nab = 0.f;
  auto fetch = [&](int item) {
    if (item < items && gt < D) {
      const int hc = (item % H) * D + gt;
      const float* zr = p.z + (size_t)(item / H) * p.ldz + hc;
      nr = zr[p.off_r]; nk = zr[p.off_k]; nv = zr[p.off_v]; na = zr[p.off_a];
      nw = p.wl[(size_t)(item / H) * p.ld_wl + hc];
      nw0 = p.w0[hc];
      nab = p.ab[hc];
    }
  };
  int fetched = blockIdx.x + group * gridDim.x, k = 0;          // k: live items so far; the group takes those with k % 2 == group
  fetch(fetched);
  int slot_next = blockIdx.x < items ? p.slots[blockIdx.x / H] : -1;
  for (int item = blockIdx.x; item < items; item += gridDim.x) {
    const int slot = slot_next;
    slot_next = item + (int)gridDim.x < items ? p.slots[(item + gridDim.x) / H] : -1;
    const int t = item / H, h = item % H;
    OT* out = reinterpret_cast<OT*>(p.out) + (size_t)t * p.ldo + h * D;
    if (slot < 0) {
      if (group == 0 && gt < Q) put4(out + 4 * gt, make_float4(0.f, 0.f, 0.f, 0.f));
      continue;
    }
    const int buf = k % kBufs, phase = (k / kBufs) & 1;
    if ((k++ & 1) != group) continue;
    if (fetched != item) fetch(item);                            // rows without a slot shifted the turns
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f), nw4 = g;
    if (col_ok && rg == 0) {
      g = *reinterpret_cast<const float4*>(p.z + (size_t)t * p.ldz + p.off_g + h * D + 4 * quad);
      nw4 = *reinterpret_cast<const float4*>(p.norm_w + h * D + 4 * quad);
    }
    float (*v4)[4 * NR] = vec[group];
    if (gw < dwarps) {
      const float r = nr, kc = nk;
      const float a = sigm(na + nab);
      const float w = expf(-p.cdecay * sigm(nw + nw0));
      const bool in = gt < D;
      if (in) {
        v4[0][gt] = kc; v4[1][gt] = w; v4[2][gt] = a * kc; v4[3][gt] = w * r;
        sv[group][gt] = nv;
      }
      float s0 = in ? kc * kc : 0.f, s1 = in ? r * kc : 0.f, s2 = in ? r * a * kc : 0.f;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        s0 += __shfl_xor_sync(0xffffffffu, s0, o);
        s1 += __shfl_xor_sync(0xffffffffu, s1, o);
        s2 += __shfl_xor_sync(0xffffffffu, s2, o);
      }
      if (lane == 0) { red[group][0][gw] = s0; red[group][1][gw] = s1; red[group][2][gw] = s2; }
    }
    fetched = item + 2 * (int)gridDim.x;
    fetch(fetched);
    group_sync(group);
    const bool ok = mbar_wait(&full[buf], phase, abort_flag, kTimeoutMma);
    float kk = 0.f, rk = 0.f, rak = 0.f;
    for (int i = 0; i < dwarps; ++i) { kk += red[group][0][i]; rk += red[group][1][i]; rak += red[group][2][i]; }
    const float inv2 = 1.0f / (kk + p.ueps);                    // u u^T = k k^T * inv2
    float* Sb = ring + (size_t)buf * DD + (size_t)rg * NR * D + 4 * quad;
    float2 y[2], q[2];
    y[0] = y[1] = q[0] = q[1] = make_float2(0.f, 0.f);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    const int rows = min(NR, max(D - rg * NR, 0));
    const bool whole = D == 4 * NR;                              // every lane has all its rows: no guards
    auto read_row = [&](int m, float kf, float rf) {
      const float4 s = *reinterpret_cast<const float4*>(Sb + m * D);
      const float2 s0 = make_float2(s.x, s.y), s1 = make_float2(s.z, s.w), k2 = make_float2(kf, kf), r2 = make_float2(rf, rf);
      y[0] = __ffma2_rn(k2, s0, y[0]); y[1] = __ffma2_rn(k2, s1, y[1]);
      q[0] = __ffma2_rn(r2, s0, q[0]); q[1] = __ffma2_rn(r2, s1, q[1]);
    };
    if (ok && col_ok) {
      const float* kv = &v4[0][rg * NR];
      const float* rv = &v4[3][rg * NR];
      if (whole) {
#pragma unroll
        for (int m = 0; m < NR; m += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kv + m), r4 = *reinterpret_cast<const float4*>(rv + m);
          read_row(m, k4.x, r4.x); read_row(m + 1, k4.y, r4.y); read_row(m + 2, k4.z, r4.z); read_row(m + 3, k4.w, r4.w);
        }
      } else {
        for (int m = 0; m < rows; ++m) read_row(m, kv[m], rv[m]);
      }
    }
    float4 ys = make_float4(y[0].x, y[0].y, y[1].x, y[1].y), qs = make_float4(q[0].x, q[0].y, q[1].x, q[1].y);
    ys = xor_sum(xor_sum(ys, 8), 16);
    qs = xor_sum(xor_sum(qs, 8), 16);
    if (ok && col_ok) {
      ys.x *= inv2; ys.y *= inv2; ys.z *= inv2; ys.w *= inv2;
      const float4 v = *reinterpret_cast<const float4*>(&sv[group][4 * quad]);
      o.x = qs.x - rak * ys.x + rk * v.x; o.y = qs.y - rak * ys.y + rk * v.y;
      o.z = qs.z - rak * ys.z + rk * v.z; o.w = qs.w - rak * ys.w + rk * v.w;
      const float2 ny0 = make_float2(-ys.x, -ys.y), ny1 = make_float2(-ys.z, -ys.w);
      const float2 v0 = make_float2(v.x, v.y), v1 = make_float2(v.z, v.w);
      auto next_row = [&](const float4& s, float kf, float wf, float af) {
        const float2 k2 = make_float2(kf, kf), w2 = make_float2(wf, wf), a2 = make_float2(af, af);
        const float2 n0 = __ffma2_rn(w2, make_float2(s.x, s.y), __ffma2_rn(k2, v0, __fmul2_rn(a2, ny0)));
        const float2 n1 = __ffma2_rn(w2, make_float2(s.z, s.w), __ffma2_rn(k2, v1, __fmul2_rn(a2, ny1)));
        return make_float4(n0.x, n0.y, n1.x, n1.y);
      };
      const float* kv = &v4[0][rg * NR];
      const float* wv = &v4[1][rg * NR];
      const float* av = &v4[2][rg * NR];
      if (whole) {
#pragma unroll
        for (int m = 0; m < NR; m += 8) {                        // eight rows in flight: loads first, then stores
          float4 s[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) s[j] = *reinterpret_cast<const float4*>(Sb + (m + j) * D);
#pragma unroll
          for (int j = 0; j < 8; j += 4) {
            const float4 k4 = *reinterpret_cast<const float4*>(kv + m + j), w4 = *reinterpret_cast<const float4*>(wv + m + j);
            const float4 a4 = *reinterpret_cast<const float4*>(av + m + j);
            s[j] = next_row(s[j], k4.x, w4.x, a4.x);
            s[j + 1] = next_row(s[j + 1], k4.y, w4.y, a4.y);
            s[j + 2] = next_row(s[j + 2], k4.z, w4.z, a4.z);
            s[j + 3] = next_row(s[j + 3], k4.w, w4.w, a4.w);
          }
#pragma unroll
          for (int j = 0; j < 8; ++j) *reinterpret_cast<float4*>(Sb + (m + j) * D) = s[j];
        }
      } else {
        for (int m = 0; m < rows; ++m)
          *reinterpret_cast<float4*>(Sb + m * D) = next_row(*reinterpret_cast<const float4*>(Sb + m * D), kv[m], wv[m], av[m]);
      }
    }
    const float so = warp_sum(rg == 0 ? o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w : 0.f);
    if (lane == 0) red_o[group][gw] = so;
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    group_sync(group);
    if (abort_s != 0) break;
    if (gt == 0) mbar_arrive(&done[buf]);
    if (col_ok && rg == 0) {
      const float oo = red_o[group][0] + red_o[group][1] + red_o[group][2] + red_o[group][3];
      const float rs = 1.0f / sqrtf(oo / (float)p.Dreal + p.eps);
      put4(out + 4 * quad, make_float4(o.x * rs * nw4.x * sigm(g.x), o.y * rs * nw4.y * sigm(g.y),
                                       o.z * rs * nw4.z * sigm(g.z), o.w * rs * nw4.w * sigm(g.w)));
    }
  }
}

// ---------------------------------------------------------------- prompts
// Record of a (token, head): w [D] | u [D] | a * u [D] | w * r [D] | sv [D] | c1, c2, 0, 0, with sv = v * sqrt(kk + ueps),
// so that k v^T = u sv^T, and o = q - c1 y + c2 sv.
__host__ __device__ inline int rec_floats(int D) { return 5 * D + 4; }

__global__ void __launch_bounds__(256) prep_kernel(const Params p, float* __restrict__ rec) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int D = p.D;
  const float* zr = p.z + (size_t)t * p.ldz + h * D;
  const float* wlr = p.wl + (size_t)t * p.ld_wl + h * D;
  float* out = rec + ((size_t)t * p.H + h) * rec_floats(D);
  float4 k[2], au[2], v[2];
  float kk = 0.f, rk = 0.f, rak = 0.f;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int e = n * 128 + lane * 4;
    k[n] = au[n] = v[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e >= D) continue;
    const float4 r = *reinterpret_cast<const float4*>(zr + p.off_r + e), a4 = *reinterpret_cast<const float4*>(zr + p.off_a + e);
    const float4 l4 = *reinterpret_cast<const float4*>(wlr + e), w04 = *reinterpret_cast<const float4*>(p.w0 + h * D + e);
    const float4 ab4 = *reinterpret_cast<const float4*>(p.ab + h * D + e);
    k[n] = *reinterpret_cast<const float4*>(zr + p.off_k + e);
    v[n] = *reinterpret_cast<const float4*>(zr + p.off_v + e);
    float4 w;
    w.x = expf(-p.cdecay * sigm(l4.x + w04.x)); w.y = expf(-p.cdecay * sigm(l4.y + w04.y));
    w.z = expf(-p.cdecay * sigm(l4.z + w04.z)); w.w = expf(-p.cdecay * sigm(l4.w + w04.w));
    *reinterpret_cast<float4*>(out + e) = w;
    *reinterpret_cast<float4*>(out + 3 * D + e) = make_float4(w.x * r.x, w.y * r.y, w.z * r.z, w.w * r.w);
    au[n] = make_float4(sigm(a4.x + ab4.x) * k[n].x, sigm(a4.y + ab4.y) * k[n].y, sigm(a4.z + ab4.z) * k[n].z,
                        sigm(a4.w + ab4.w) * k[n].w);
    kk += k[n].x * k[n].x + k[n].y * k[n].y + k[n].z * k[n].z + k[n].w * k[n].w;
    rk += r.x * k[n].x + r.y * k[n].y + r.z * k[n].z + r.w * k[n].w;
    rak += r.x * au[n].x + r.y * au[n].y + r.z * au[n].z + r.w * au[n].w;
  }
  kk = warp_sum(kk); rk = warp_sum(rk); rak = warp_sum(rak);
  const float s = sqrtf(kk + p.ueps), inv = 1.0f / s;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int e = n * 128 + lane * 4;
    if (e >= D) continue;
    *reinterpret_cast<float4*>(out + D + e) = make_float4(k[n].x * inv, k[n].y * inv, k[n].z * inv, k[n].w * inv);
    *reinterpret_cast<float4*>(out + 2 * D + e) = make_float4(au[n].x * inv, au[n].y * inv, au[n].z * inv, au[n].w * inv);
    *reinterpret_cast<float4*>(out + 4 * D + e) = make_float4(v[n].x * s, v[n].y * s, v[n].z * s, v[n].w * s);
  }
  if (lane == 0) *reinterpret_cast<float4*>(out + 5 * D) = make_float4(rak * inv, rk * inv, 0.f, 0.f);
}

constexpr int kScanCols = 32;      // value columns of a CTA
constexpr int kScanGroup = 8;      // tokens per staged group

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// A lane holds R key rows x C value columns of the state; 16 lanes share a column: lane (cg, lr) of a warp has columns
// cg * C .. + C - 1 of the warp's 2 C columns and rows 64 n + 4 lr .. + 3 (n < R / 4, lr < 16; D <= 16 R).  Few rows and many
// columns a lane keep the shared-memory reads of the vectors, the scan's limit, small; the row sums of a column meet in four
// shuffles.  C = 4 reads the vectors once per 8 columns (many sequences); C = 2 spreads a head over twice the warps (few).
// Shared memory of a token: w | u | au | wr (16 R floats each, zero past D) | c1 c2 . . | sv of the CTA's 32 columns.
template <int R, int C>
__global__ void __launch_bounds__(32 * kScanCols / (2 * C))
scan_kernel(const Params p, const float* __restrict__ rec, float* __restrict__ o_out) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  constexpr int kWarps = kScanCols / (2 * C), NT = 32 * kWarps;
  constexpr int V = 16 * R, TOK = 4 * V + 4 + kScanCols;
  extern __shared__ __align__(16) float sm[];
  const int split = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane & 15, cg = lane >> 4;
  const int D = p.D, H = p.H;
  const int slot = p.slots[seq];
  const int t0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int t1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  if (t1 <= t0) return;
  const int c0 = split * kScanCols, lc = (warp * 2 + cg) * C, col = c0 + lc;      // D % 8 == 0: all C columns in or out
  const bool col_ok = col < D;
  if (slot < 0) {
    for (int i = tid; i < (t1 - t0) * kScanCols; i += NT)
      if (c0 + i % kScanCols < D) o_out[((size_t)(t0 + i / kScanCols) * H + h) * D + c0 + i % kScanCols] = 0.f;
    return;
  }
  for (int i = tid; i < 2 * kScanGroup * TOK; i += NT) sm[i] = 0.f;               // zero padding of the vectors, once
  __syncthreads();
  const int q16 = D / 4, cols16 = min(kScanCols, D - c0) / 4;                     // 16-byte pieces of a vector / of sv
  auto fetch = [&](int g0, int buf) {                                             // tokens g0 .. of the group -> buffer
    const int n = min(kScanGroup, t1 - g0);
    for (int tt = warp; tt < n; tt += kWarps) {
      const float* src = rec + ((size_t)(g0 + tt) * H + h) * rec_floats(D);
      float* dst = sm + (buf * kScanGroup + tt) * TOK;
#pragma unroll
      for (int v = 0; v < 4; ++v)
        for (int j = lane; j < q16; j += 32) cp16(dst + v * V + j * 4, src + v * D + j * 4);
      if (lane < cols16) cp16(dst + 4 * V + 4 + lane * 4, src + 4 * D + c0 + lane * 4);
      else if (lane == 31) cp16(dst + 4 * V, src + 5 * D);
    }
    // a short last group is filled up with tokens that leave the state alone: w = 1, everything else 0
    for (int tt = n + warp; tt < kScanGroup; tt += kWarps) {
      float* dst = sm + (buf * kScanGroup + tt) * TOK;
      for (int j = lane; j < TOK; j += 32) dst[j] = j < V ? 1.f : 0.f;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(t0, 0);
  float* Sg = p.state + slot * p.slot_stride + (size_t)h * D * D + col;
  const bool init = p.has_initial == nullptr || p.has_initial[seq] != 0;
  float2 S[C][R / 2];                                                             // rows in pairs
#pragma unroll
  for (int n = 0; n < R / 4; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = 64 * n + 4 * lr + j;
      const bool in = init && col_ok && i < D;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float v = in ? Sg[(size_t)i * D + c] : 0.f;
        if (j & 1) S[c][2 * n + j / 2].y = v;
        else S[c][2 * n + j / 2].x = v;
      }
    }
  int buf = 0;
  for (int g0 = t0; g0 < t1; g0 += kScanGroup, buf ^= 1) {
    if (g0 + kScanGroup < t1) {
      fetch(g0 + kScanGroup, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    // this lane's share of the group's outputs: its rows' part of q, lane 0 of a column adds -c1 y + c2 sv
    float part[kScanGroup][C];
    const float* base = sm + buf * kScanGroup * TOK;
#pragma unroll
    for (int tt = 0; tt < kScanGroup; ++tt) {
      const float* tok = base + tt * TOK;
      const float4* w4 = reinterpret_cast<const float4*>(tok) + lr;
      const float4* u4 = w4 + V / 4;
      const float4* a4 = u4 + V / 4;
      const float4* r4 = a4 + V / 4;
      float2 y0[C], y1[C], q[C];
      float4 u[R / 4];
#pragma unroll
      for (int c = 0; c < C; ++c) y0[c] = y1[c] = q[c] = make_float2(0.f, 0.f);
#pragma unroll
      for (int n = 0; n < R / 4; ++n) {
        u[n] = u4[16 * n];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          y0[c] = __ffma2_rn(make_float2(u[n].x, u[n].y), S[c][2 * n], y0[c]);
          y1[c] = __ffma2_rn(make_float2(u[n].z, u[n].w), S[c][2 * n + 1], y1[c]);
        }
      }
      float ys[C];
#pragma unroll
      for (int c = 0; c < C; ++c) ys[c] = (y0[c].x + y0[c].y) + (y1[c].x + y1[c].y);
#pragma unroll
      for (int o = 1; o < 16; o <<= 1)
#pragma unroll
        for (int c = 0; c < C; ++c) ys[c] += __shfl_xor_sync(0xffffffffu, ys[c], o);
      const float2 cc = *reinterpret_cast<const float2*>(tok + 4 * V);
      float2 sv[C], ny[C];
#pragma unroll
      for (int c = 0; c < C; c += 2) {
        const float2 s = *reinterpret_cast<const float2*>(tok + 4 * V + 4 + lc + c);
        sv[c] = make_float2(s.x, s.x);
        sv[c + 1] = make_float2(s.y, s.y);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) ny[c] = make_float2(-ys[c], -ys[c]);
#pragma unroll
      for (int n = 0; n < R / 4; ++n) {
        const float4 w = w4[16 * n], a = a4[16 * n], r = r4[16 * n];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          q[c] = __ffma2_rn(make_float2(r.x, r.y), S[c][2 * n], q[c]);
          q[c] = __ffma2_rn(make_float2(r.z, r.w), S[c][2 * n + 1], q[c]);
          S[c][2 * n] = __ffma2_rn(make_float2(a.x, a.y), ny[c],
                                   __ffma2_rn(make_float2(u[n].x, u[n].y), sv[c], __fmul2_rn(make_float2(w.x, w.y), S[c][2 * n])));
          S[c][2 * n + 1] = __ffma2_rn(make_float2(a.z, a.w), ny[c],
                                       __ffma2_rn(make_float2(u[n].z, u[n].w), sv[c], __fmul2_rn(make_float2(w.z, w.w), S[c][2 * n + 1])));
        }
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        part[tt][c] = q[c].x + q[c].y;
        if (lr == 0) part[tt][c] += fmaf(cc.y, sv[c].x, -cc.x * ys[c]);
      }
    }
    // sum over the 16 lanes of a column, handing half of the tokens to the partner at every step: lanes lr and lr + 8 end
    // with token lr
#pragma unroll
    for (int half = 4, bit = 4; half >= 1; half >>= 1, bit >>= 1)
#pragma unroll
      for (int tt = 0; tt < half; ++tt)
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const bool up = lr & bit;
          const float mine = up ? part[tt + half][c] : part[tt][c], give = up ? part[tt][c] : part[tt + half][c];
          part[tt][c] = mine + __shfl_xor_sync(0xffffffffu, give, bit);
        }
#pragma unroll
    for (int c = 0; c < C; ++c) part[0][c] += __shfl_xor_sync(0xffffffffu, part[0][c], 8);
    if (lr < 8 && g0 + lr < t1 && col_ok) {
      float* dst = o_out + ((size_t)(g0 + lr) * H + h) * D + col;
#pragma unroll
      for (int c = 0; c < C; c += 2) *reinterpret_cast<float2*>(dst + c) = make_float2(part[0][c], part[0][c + 1]);
    }
    __syncthreads();
  }
  if (col_ok) {
#pragma unroll
    for (int n = 0; n < R / 4; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = 64 * n + 4 * lr + j;
        if (i < D) {
#pragma unroll
          for (int c = 0; c < C; ++c) Sg[(size_t)i * D + c] = (j & 1) ? S[c][2 * n + j / 2].y : S[c][2 * n + j / 2].x;
        }
      }
  }
}

// out[t, h] = o / sqrt(mean(o^2) + eps) * norm * sigmoid(g); a warp per (token, head)
template <typename OT>
__global__ void __launch_bounds__(256) finish_kernel(const Params p, const float* __restrict__ o_in) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int D = p.D;
  const float* o = o_in + ((size_t)t * p.H + h) * D;
  float4 v[2];
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int e = n * 128 + lane * 4;
    v[n] = e < D ? *reinterpret_cast<const float4*>(o + e) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
  }
  const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)p.Dreal + p.eps);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int e = n * 128 + lane * 4;
    if (e >= D) continue;
    const float4 g = *reinterpret_cast<const float4*>(p.z + (size_t)t * p.ldz + p.off_g + h * D + e);
    const float4 nw = *reinterpret_cast<const float4*>(p.norm_w + h * D + e);
    put4(reinterpret_cast<OT*>(p.out) + (size_t)t * p.ldo + h * D + e,
         make_float4(v[n].x * rs * nw.x * sigm(g.x), v[n].y * rs * nw.y * sigm(g.y), v[n].z * rs * nw.z * sigm(g.z),
                     v[n].w * rs * nw.w * sigm(g.w)));
  }
}

template <int R, int C>
static int launch_scan_as(const Params& p, const float* rec, float* o, int nseq, cudaStream_t stream) {
  const size_t smem = (size_t)2 * kScanGroup * (64 * R + 4 + kScanCols) * sizeof(float);
  static DeviceOnce once;
  auto kern = scan_kernel<R, C>;
  if (!ensure_dynamic_smem(kern, smem, once)) return -4;
  dim3 grid((p.D + kScanCols - 1) / kScanCols, p.H, nseq);
  bg::launch_pdl(kern, grid, dim3(32 * kScanCols / (2 * C)), smem, stream, p, rec, o);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int R>
static int launch_scan(const Params& p, const float* rec, float* o, int nseq, cudaStream_t stream) {
  const long long ctas = (long long)((p.D + kScanCols - 1) / kScanCols) * p.H * nseq;
  return ctas <= 296 ? launch_scan_as<R, 2>(p, rec, o, nseq, stream) : launch_scan_as<R, 4>(p, rec, o, nseq, stream);
}

template <typename OT>
static int launch_prompt(const Params& p, float* rec, float* o, int T, int nseq, cudaStream_t stream) {
  const dim3 grid(T, (p.H + 7) / 8);
  bg::launch_pdl(prep_kernel, grid, dim3(256), 0, stream, p, rec);
  int rc;
  if (p.D <= 64) rc = launch_scan<4>(p, rec, o, nseq, stream);
  else if (p.D <= 128) rc = launch_scan<8>(p, rec, o, nseq, stream);
  else if (p.D <= 192) rc = launch_scan<12>(p, rec, o, nseq, stream);
  else rc = launch_scan<16>(p, rec, o, nseq, stream);
  if (rc != 0) return rc;
  bg::launch_pdl(finish_kernel<OT>, grid, dim3(256), 0, stream, p, (const float*)o);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename OT, int NR>
static int launch_decode_as(const Params& p, int nseq, int num_sms, int* status, cudaStream_t stream) {
  const size_t smem = (size_t)kBufs * p.D * p.D * sizeof(float);
  static DeviceOnce once;
  auto kern = decode_kernel<OT, NR>;
  if (!ensure_dynamic_smem(kern, 3 * 128 * 128 * sizeof(float), once)) return -4;
  const int per_sm = smem > 100 * 1024 || NR > 16 ? 1 : smem > 48 * 1024 ? 2 : 3;
  const int items = nseq * p.H, most = num_sms * per_sm;
  bg::launch_pdl(kern, dim3(items < most ? items : most), dim3(288), smem, stream, p, items, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename OT>
static int launch_decode(const Params& p, int nseq, int num_sms, int* status, cudaStream_t stream) {
  if (p.D <= 32) return launch_decode_as<OT, 8>(p, nseq, num_sms, status, stream);
  if (p.D <= 64) return launch_decode_as<OT, 16>(p, nseq, num_sms, status, stream);
  return launch_decode_as<OT, 32>(p, nseq, num_sms, status, stream);
}

}  // namespace delta
}  // namespace bg

extern "C" {

// offs: host array of five column offsets (r, k, v, g, a).  dt: 0 = bf16 output, 1 = fp32.  D a multiple of 8, <= 256.
// T: rows of z.  `scratch` (T * H * (6 D + 4) floats: records, then the scan's outputs) selects the prompt path; null the decode kernel (D <= 128, one
// token per sequence).
int bg_delta_forward(int dt, const float* z, int ldz, const int* offs, const float* wl, int ld_wl, const float* w0,
                     const float* ab, const float* norm_w, float* state, long long slot_stride, const int* cu,
                     const int* slots, const int* has_initial, void* out, int ldo, int T, int nseq, int H, int D, int Dreal,
                     float cdecay, float ueps, float eps, float* scratch, int num_sms, int* status, cudaStream_t stream) {
  using namespace bg::delta;
  if (nseq <= 0 || T <= 0) return 0;
  if (D <= 0 || D % 8 || D > kMaxD || H <= 0 || H > 65535 || nseq > 65535 || ldz % 4 || ldo % 4 || ld_wl % 4 || slot_stride % 4 ||
      (scratch == nullptr && (D > 128 || cu != nullptr || num_sms <= 0)) || (cu == nullptr && T != nseq) ||
      (long long)nseq * H > 0x7fffffffll)
    return -1;
  for (int i = 0; i < 5; ++i)
    if (offs[i] % 4) return -1;
  Params p;
  p.z = z; p.ldz = ldz; p.off_r = offs[0]; p.off_k = offs[1]; p.off_v = offs[2]; p.off_g = offs[3]; p.off_a = offs[4];
  p.wl = wl; p.ld_wl = ld_wl; p.w0 = w0; p.ab = ab; p.norm_w = norm_w; p.state = state; p.slot_stride = slot_stride;
  p.cu = cu; p.slots = slots; p.has_initial = has_initial; p.out = out; p.ldo = ldo; p.H = H; p.D = D; p.Dreal = Dreal;
  p.cdecay = cdecay; p.ueps = ueps; p.eps = eps;
  if (scratch != nullptr) {
    float* o = scratch + (size_t)T * H * rec_floats(D);
    return dt == 0 ? launch_prompt<__nv_bfloat16>(p, scratch, o, T, nseq, stream)
                   : launch_prompt<float>(p, scratch, o, T, nseq, stream);
  }
  return dt == 0 ? launch_decode<__nv_bfloat16>(p, nseq, num_sms, status, stream)
                 : launch_decode<float>(p, nseq, num_sms, status, stream);
}

}  // extern "C"

BG_TRACE_SETTER(delta_rule)
