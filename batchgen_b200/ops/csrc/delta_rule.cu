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
// scan splits a head's columns over CTAs of 32 columns and needs no barrier inside a token (4 lanes share a column, two
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
// D * D * 4 bytes: bulk copies bring the next two items' blocks into a ring of three shared-memory buffers while the current
// one is worked on in place, and a bulk copy takes it back, so the SM always has loads and stores in flight.
//
// Thread (ig, jq): value columns 4 jq .. 4 jq + 3, key rows ig, ig + RG, ... (NR of them at most).
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

template <typename OT, int NT, int NR>
__global__ void __launch_bounds__(NT) decode_kernel(const Params p, int items, int* status) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(128) float ring[];                // kBufs x D * D
  __shared__ uint64_t full[kBufs];
  __shared__ int abort_s;
  __shared__ __align__(16) float sk[128], sw[128], sak[128], swr[128], sv[128];
  __shared__ float red[3][4], red_o[2];
  __shared__ __align__(16) float4 part_y[NT], part_q[NT];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = p.D, H = p.H, Q = D / 4, RG = NT / Q, DD = D * D;
  const uint32_t bytes = (uint32_t)DD * 4;
  const int jq = tid % Q, ig = tid / Q;
  const bool active = ig < RG;
  const int dwarps = (D + 31) / 32, owarps = (Q + 31) / 32;
  volatile int* abort_flag = &abort_s;
  if (tid == 0) {
    for (int s = 0; s < kBufs; ++s) mbar_init(&full[s], 1);
    abort_s = 0;
    mbar_fence_init();
  }
  __syncthreads();
  auto block_of = [&](int item) { return p.state + p.slots[item / H] * p.slot_stride + (size_t)(item % H) * DD; };
  int ahead = blockIdx.x;                                       // thread 0: next item to load (rows without a slot are skipped)
  auto load_state = [&](int stage) {
    while (ahead < items && p.slots[ahead / H] < 0) ahead += gridDim.x;
    if (ahead < items) {
      mbar_expect_tx(&full[stage], bytes);
      bulk_load(ring + (size_t)stage * DD, block_of(ahead), bytes, &full[stage]);
      ahead += gridDim.x;
    }
  };
  if (tid == 0) { load_state(0); load_state(1); }
  float nr = 0.f, nk = 0.f, nv = 0.f, na = 0.f, nw = 0.f, nw0 = 0.f, nab = 0.f;
  auto load = [&](int item) {
    if (item < items && tid < D) {
      const int t = item / H, hc = (item % H) * D + tid;
      const float* zr = p.z + (size_t)t * p.ldz + hc;
      nr = zr[p.off_r]; nk = zr[p.off_k]; nv = zr[p.off_v]; na = zr[p.off_a];
      nw = p.wl[(size_t)t * p.ld_wl + hc];
      nw0 = p.w0[hc];
      nab = p.ab[hc];
    }
  };
  load(blockIdx.x);
  int n = 0;                                                    // items worked on so far
  for (int item = blockIdx.x; item < items; item += gridDim.x) {
    const int t = item / H, h = item % H;
    OT* out = reinterpret_cast<OT*>(p.out) + (size_t)t * p.ldo + h * D;
    if (p.slots[t] < 0) {
      for (int j = tid; j < Q; j += NT) put4(out + 4 * j, make_float4(0.f, 0.f, 0.f, 0.f));
      load(item + gridDim.x);
      continue;
    }
    const int stage = n % kBufs;
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f), nw4 = g;
    if (tid < Q) {
      g = *reinterpret_cast<const float4*>(p.z + (size_t)t * p.ldz + p.off_g + h * D + 4 * tid);
      nw4 = *reinterpret_cast<const float4*>(p.norm_w + h * D + 4 * tid);
    }
    if (warp < dwarps) {
      const float r = nr, k = nk;
      const float a = sigm(na + nab);
      const float w = expf(-p.cdecay * sigm(nw + nw0));
      if (tid < D) {
        sk[tid] = k; sw[tid] = w; sak[tid] = a * k; swr[tid] = w * r; sv[tid] = nv;
      }
      const float s0 = warp_sum(tid < D ? k * k : 0.f), s1 = warp_sum(tid < D ? r * k : 0.f);
      const float s2 = warp_sum(tid < D ? r * a * k : 0.f);
      if (lane == 0) { red[0][warp] = s0; red[1][warp] = s1; red[2][warp] = s2; }
    }
    load(item + gridDim.x);
    const bool ok = mbar_wait(&full[stage], (n / kBufs) & 1, abort_flag, kTimeoutProducer);
    if (__syncthreads_or(!ok)) break;
    float kk = 0.f, rk = 0.f, rak = 0.f;
    for (int i = 0; i < dwarps; ++i) { kk += red[0][i]; rk += red[1][i]; rak += red[2][i]; }
    const float inv2 = 1.0f / (kk + p.ueps);                    // u u^T = k k^T * inv2
    float* Sb = ring + (size_t)stage * DD;
    float4 S[NR], y = make_float4(0.f, 0.f, 0.f, 0.f), q = y;
    if (active) {
#pragma unroll
      for (int m = 0; m < NR; ++m) {
        const int i = ig + m * RG;
        if (i < D) {
          S[m] = *reinterpret_cast<const float4*>(Sb + i * D + 4 * jq);
          const float k = sk[i], wr = swr[i];
          y.x = fmaf(k, S[m].x, y.x); y.y = fmaf(k, S[m].y, y.y); y.z = fmaf(k, S[m].z, y.z); y.w = fmaf(k, S[m].w, y.w);
          q.x = fmaf(wr, S[m].x, q.x); q.y = fmaf(wr, S[m].y, q.y); q.z = fmaf(wr, S[m].z, q.z); q.w = fmaf(wr, S[m].w, q.w);
        }
      }
      part_y[tid] = y;
      part_q[tid] = q;
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active) {
      y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int i = 0; i < RG; ++i) {
        const float4 v = part_y[i * Q + jq];
        y.x += v.x; y.y += v.y; y.z += v.z; y.w += v.w;
      }
      y.x *= inv2; y.y *= inv2; y.z *= inv2; y.w *= inv2;
      const float4 v = *reinterpret_cast<const float4*>(&sv[4 * jq]);
      if (ig == 0) {
        q = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int i = 0; i < RG; ++i) {
          const float4 b = part_q[i * Q + jq];
          q.x += b.x; q.y += b.y; q.z += b.z; q.w += b.w;
        }
        o.x = q.x - rak * y.x + rk * v.x; o.y = q.y - rak * y.y + rk * v.y;
        o.z = q.z - rak * y.z + rk * v.z; o.w = q.w - rak * y.w + rk * v.w;
      }
#pragma unroll
      for (int m = 0; m < NR; ++m) {
        const int i = ig + m * RG;
        if (i < D) {
          const float k = sk[i], w = sw[i], ak = sak[i];
          *reinterpret_cast<float4*>(Sb + i * D + 4 * jq) =
              make_float4(fmaf(w, S[m].x, fmaf(k, v.x, -ak * y.x)), fmaf(w, S[m].y, fmaf(k, v.y, -ak * y.y)),
                          fmaf(w, S[m].z, fmaf(k, v.z, -ak * y.z)), fmaf(w, S[m].w, fmaf(k, v.w, -ak * y.w)));
        }
      }
    }
    if (warp < owarps) {
      const float s = warp_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w);
      if (lane == 0) red_o[warp] = s;
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    __syncthreads();
    if (tid == 0) {
      bulk_store(block_of(item), Sb, bytes);
      // the block stored before this one has left its buffer: that buffer takes the item two ahead
      asm volatile("cp.async.bulk.wait_group.read 1;" ::: "memory");
      load_state((n + 2) % kBufs);
    }
    if (tid < Q) {
      float oo = 0.f;
      for (int i = 0; i < owarps; ++i) oo += red_o[i];
      const float rs = 1.0f / sqrtf(oo / (float)p.Dreal + p.eps);
      put4(out + 4 * tid, make_float4(o.x * rs * nw4.x * sigm(g.x), o.y * rs * nw4.y * sigm(g.y),
                                      o.z * rs * nw4.z * sigm(g.z), o.w * rs * nw4.w * sigm(g.w)));
    }
    ++n;
  }
  if (tid == 0) {
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    if (abort_s != 0) {
      for (uint32_t i = 0; i < (1u << 16); ++i) __nanosleep(20);     // bounded grace period for copies in flight
      if (status != nullptr) atomicMax(status, abort_s);
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

constexpr int kScanCols = 32;      // value columns of a CTA: 4 warps x 8
constexpr int kScanThreads = 128;
constexpr int kScanGroup = 8;      // tokens per staged group

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// Lane (cj, lr) of a warp: column cj of the warp's 8, rows 16 n + 4 lr .. + 3 for n < R / 4 (R rows a lane, D <= 4 R).
// Shared memory of a token: w | u | au | wr (4 R floats each, zero past D) | c1 c2 . . | sv of the CTA's 32 columns.
template <int R>
__global__ void __launch_bounds__(kScanThreads) scan_kernel(const Params p, const float* __restrict__ rec, float* __restrict__ o_out) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  constexpr int V = 4 * R, TOK = 4 * V + 4 + kScanCols;
  extern __shared__ __align__(16) float sm[];
  const int split = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane & 3, cj = lane >> 2;
  const int D = p.D, H = p.H;
  const int slot = p.slots[seq];
  const int t0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int t1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  if (t1 <= t0) return;
  const int c0 = split * kScanCols, lc = warp * 8 + cj, col = c0 + lc;
  const bool col_ok = col < D;
  if (slot < 0) {
    if (lr == 0 && col_ok)
      for (int t = t0; t < t1; ++t) o_out[((size_t)t * H + h) * D + col] = 0.f;
    return;
  }
  for (int i = tid; i < 2 * kScanGroup * TOK; i += kScanThreads) sm[i] = 0.f;     // zero padding of the vectors, once
  __syncthreads();
  const int q16 = D / 4, cols16 = min(kScanCols, D - c0) / 4;                     // 16-byte pieces of a vector / of sv
  auto fetch = [&](int g0, int buf) {                                             // tokens g0 .. of the group -> buffer
    const int n = min(kScanGroup, t1 - g0);
    for (int tt = warp; tt < n; tt += kScanThreads / 32) {
      const float* src = rec + ((size_t)(g0 + tt) * H + h) * rec_floats(D);
      float* dst = sm + (buf * kScanGroup + tt) * TOK;
#pragma unroll
      for (int v = 0; v < 4; ++v)
        for (int j = lane; j < q16; j += 32) cp16(dst + v * V + j * 4, src + v * D + j * 4);
      if (lane < cols16) cp16(dst + 4 * V + 4 + lane * 4, src + 4 * D + c0 + lane * 4);
      else if (lane == 31) cp16(dst + 4 * V, src + 5 * D);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(t0, 0);
  float* Sg = p.state + slot * p.slot_stride + (size_t)h * D * D + col;
  const bool init = p.has_initial == nullptr || p.has_initial[seq] != 0;
  float2 S[R / 2];                                                                // rows in pairs
#pragma unroll
  for (int n = 0; n < R / 4; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = 16 * n + 4 * lr + j;
      const float v = (init && col_ok && i < D) ? Sg[(size_t)i * D] : 0.f;
      if (j & 1) S[2 * n + j / 2].y = v;
      else S[2 * n + j / 2].x = v;
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
    const int n_tok = min(kScanGroup, t1 - g0);
    for (int tt = 0; tt < n_tok; ++tt) {
      const float* tok = sm + (buf * kScanGroup + tt) * TOK;
      const float4* w4 = reinterpret_cast<const float4*>(tok) + lr;
      const float4* u4 = w4 + V / 4;
      const float4* a4 = u4 + V / 4;
      const float4* r4 = a4 + V / 4;
      float2 y0 = make_float2(0.f, 0.f), y1 = y0, q0 = y0, q1 = y0;
#pragma unroll
      for (int n = 0; n < R / 4; ++n) {
        const float4 u = u4[4 * n], r = r4[4 * n];
        y0 = __ffma2_rn(make_float2(u.x, u.y), S[2 * n], y0);
        y1 = __ffma2_rn(make_float2(u.z, u.w), S[2 * n + 1], y1);
        q0 = __ffma2_rn(make_float2(r.x, r.y), S[2 * n], q0);
        q1 = __ffma2_rn(make_float2(r.z, r.w), S[2 * n + 1], q1);
      }
      float y = (y0.x + y0.y) + (y1.x + y1.y), q = (q0.x + q0.y) + (q1.x + q1.y);
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      q += __shfl_xor_sync(0xffffffffu, q, 1);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      q += __shfl_xor_sync(0xffffffffu, q, 2);
      const float sv = tok[4 * V + 4 + lc];
      const float2 c = *reinterpret_cast<const float2*>(tok + 4 * V);
      const float2 ny = make_float2(-y, -y), sv2 = make_float2(sv, sv);
#pragma unroll
      for (int n = 0; n < R / 4; ++n) {
        const float4 w = w4[4 * n], u = u4[4 * n], a = a4[4 * n];
        S[2 * n] = __ffma2_rn(make_float2(a.x, a.y), ny,
                              __ffma2_rn(make_float2(u.x, u.y), sv2, __fmul2_rn(make_float2(w.x, w.y), S[2 * n])));
        S[2 * n + 1] = __ffma2_rn(make_float2(a.z, a.w), ny,
                                  __ffma2_rn(make_float2(u.z, u.w), sv2, __fmul2_rn(make_float2(w.z, w.w), S[2 * n + 1])));
      }
      if (lr == 0 && col_ok) o_out[((size_t)(g0 + tt) * H + h) * D + col] = fmaf(c.y, sv, fmaf(-c.x, y, q));
    }
    __syncthreads();
  }
  if (col_ok) {
#pragma unroll
    for (int n = 0; n < R / 4; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = 16 * n + 4 * lr + j;
        if (i < D) Sg[(size_t)i * D] = (j & 1) ? S[2 * n + j / 2].y : S[2 * n + j / 2].x;
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

template <int R>
static int launch_scan(const Params& p, const float* rec, float* o, int nseq, cudaStream_t stream) {
  const size_t smem = (size_t)2 * kScanGroup * (16 * R + 4 + kScanCols) * sizeof(float);
  static DeviceOnce once;
  auto kern = scan_kernel<R>;
  if (!ensure_dynamic_smem(kern, smem, once)) return -4;
  dim3 grid((p.D + kScanCols - 1) / kScanCols, p.H, nseq);
  bg::launch_pdl(kern, grid, dim3(kScanThreads), smem, stream, p, rec, o);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename OT>
static int launch_prompt(const Params& p, float* rec, float* o, int T, int nseq, cudaStream_t stream) {
  const dim3 grid(T, (p.H + 7) / 8);
  bg::launch_pdl(prep_kernel, grid, dim3(256), 0, stream, p, rec);
  int rc;
  if (p.D <= 32) rc = launch_scan<8>(p, rec, o, nseq, stream);
  else if (p.D <= 48) rc = launch_scan<12>(p, rec, o, nseq, stream);
  else if (p.D <= 64) rc = launch_scan<16>(p, rec, o, nseq, stream);
  else if (p.D <= 96) rc = launch_scan<24>(p, rec, o, nseq, stream);
  else if (p.D <= 128) rc = launch_scan<32>(p, rec, o, nseq, stream);
  else if (p.D <= 192) rc = launch_scan<48>(p, rec, o, nseq, stream);
  else rc = launch_scan<64>(p, rec, o, nseq, stream);
  if (rc != 0) return rc;
  bg::launch_pdl(finish_kernel<OT>, grid, dim3(256), 0, stream, p, (const float*)o);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename OT, int NT, int NR>
static int launch_decode_as(const Params& p, int nseq, int num_sms, int* status, cudaStream_t stream) {
  const size_t smem = (size_t)kBufs * p.D * p.D * sizeof(float);
  static DeviceOnce once;
  auto kern = decode_kernel<OT, NT, NR>;
  if (!ensure_dynamic_smem(kern, 3 * 128 * 128 * sizeof(float), once)) return -4;
  const int per_sm = smem > 100 * 1024 ? 1 : smem > 48 * 1024 ? 2 : 4;
  const int items = nseq * p.H, most = num_sms * per_sm;
  bg::launch_pdl(kern, dim3(items < most ? items : most), dim3(NT), smem, stream, p, items, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename OT>
static int launch_decode(const Params& p, int nseq, int num_sms, int* status, cudaStream_t stream) {
  if (p.D <= 32) return launch_decode_as<OT, 128, 2>(p, nseq, num_sms, status, stream);
  if (p.D <= 64) return launch_decode_as<OT, 256, 4>(p, nseq, num_sms, status, stream);
  return launch_decode_as<OT, 256, 16>(p, nseq, num_sms, status, stream);
}

}  // namespace delta
}  // namespace bg

extern "C" {

// Floats of scratch per token: prompt records and the scan's outputs.
long long bg_delta_scratch_floats(int H, int D) { return (long long)H * (bg::delta::rec_floats(D) + D); }

// offs: host array of five column offsets (r, k, v, g, a).  dt: 0 = bf16 output, 1 = fp32.  D a multiple of 8, <= 256.
// T: rows of z.  `scratch` (T * bg_delta_scratch_floats floats) selects the prompt path; null the decode kernel (D <= 128, one
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
