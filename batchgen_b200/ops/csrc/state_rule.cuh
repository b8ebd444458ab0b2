// Recurrences with a matrix state per head, S [K key channels x V value channels] in fp32: the kernels that move and update
// states, with the update itself as a template parameter (`Rule`).  A rule brings
//
//   kVecs         vectors of K channels a token contributes
//   kRead         the update needs y = (read vector)^T S of the old state; otherwise the decay is one number per token
//   kForget       without kRead: the decay f is a vector over the key channels and the write vector is 1 - f (HGRN2)
//   kTwoTerms     the correction by y and the new value are written along different vectors
//   kDen          a normaliser vector is carried like one more value column with value 1 (mLSTM)
//   Regs, fetch   what a thread loads of a token ahead of its turn (thread = channel)
//   Scal, scalars what every thread of a token's group computes for itself
//   vectors       the token's vectors in shared memory, and up to three sums over the key channels
//
// Decode, one token per sequence (`decode_kernel`): states stream through a ring in shared memory, everything else of the
// token is fused around the update.  Prompts (a rule's own record kernel -> `scan_kernel` -> `finish_kernel`): a value column
// of S evolves on its own once the token vectors are known, so the scan splits a head's columns over CTAs of 32 columns and
// needs no barrier inside a token; `finish` applies the output norm and gate, which need whole heads.
#pragma once
#include "common.cuh"

namespace bg {
namespace rec {

struct Args {
  const float *q, *k, *v, *gate;   // fp32 column views of the step's projections; gate null: the output has none
  const float* low;                // [T, H * K] decay pre-activation
  const float* beta;               // write strength (channel_delta, [T, H]) or removal rate (general_delta, [T, H * K])
  const float *gate_i, *gate_f;    // mlstm: [T, H]
  const float *bias0, *bias1;      // general_delta: decay and removal offsets; channel_delta: dt_bias; mlstm: gate biases; hgrn2:
                                   // forget bias (k: its pre-activation)
  const float* rate;               // channel_delta: exp(A_log) [H]; retention: decay [H]; hgrn2: lower bounds [H * K]
  const float* rope;               // retention: [T, 2 * half] cosines, then sines
  const float* norm_w;             // [H * V] gain of the output norm
  float* state;                    // this layer's S [H, K, V] in slot 0; slots are `slot_stride` floats apart
  float* norm_state;               // mlstm: [H, K]
  float* max_state;                // mlstm: [H]
  const int* cu;                   // [nseq + 1] token ranges, or null: one token per sequence
  const int* slots;                // [nseq], < 0 skips the sequence (its output rows become zero)
  const int* has_initial;          // [nseq] or null (always continue from the slot)
  void* out;                       // [T, ld_out]
  float* scratch;                  // prompts: gates | records | scan outputs | denominators; null selects the decode kernel
  int* status;
  long long slot_stride;
  int dt, rule;                    // dt: 0 = bf16 output, 1 = fp32
  int ld_q, ld_k, ld_v, ld_gate, ld_low, ld_beta, ld_gi, ld_gf, ld_rope, ld_out;
  int T, nseq, H, rep, K, V, v_real, silu, num_sms;      // rep: heads per query / key head; v_real: channels of the mean
  float q_scale, k_scale, cap, ueps, eps, den_eps;       // cap: mlstm's soft cap, general_delta's decay scale
};

constexpr int kMaxK = 512;

template <typename OT> __device__ __forceinline__ void put4(OT* p, float4 v);
template <> __device__ __forceinline__ void put4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void put4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
}
__device__ __forceinline__ float sigm(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gate_act(float x, int silu) { return silu ? x * sigm(x) : sigm(x); }
// factors of 4 output channels; g null: no gate
__device__ __forceinline__ float4 gate4(const float* g, int silu) {
  if (g == nullptr) return make_float4(1.f, 1.f, 1.f, 1.f);
  const float4 v = *reinterpret_cast<const float4*>(g);
  return make_float4(gate_act(v.x, silu), gate_act(v.y, silu), gate_act(v.z, silu), gate_act(v.w, silu));
}
__device__ __forceinline__ float2 twice(float x) { return make_float2(x, x); }

// ---------------------------------------------------------------- decode
// One token per sequence, persistent over (sequence, head) items.  A head's state is one contiguous block of K * V * 4 bytes.
// A producer thread brings blocks into a ring of three shared-memory buffers with bulk copies and takes them back the same
// way; two groups of four warps work on alternate items in place, so one group's barriers and reductions hide behind the
// other's arithmetic and the SM always has loads and stores in flight.
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

// What a column's outputs and its next state are made of, from the token's sums (filled by `Rule::coefs`):
//   kRead:  y' = ys * y;  o = os * q + ov * v - oy * y'  (kTwoTerms)   or   u = us * (v - y'), o = os * q + ov * u
//   linear: S' = w S + k v, o = os * (q^T S')   (kForget: w and k per key channel, f and 1 - f)
struct Coefs {
  float ys, os, ov, oy, us, w;
};

// SQ: K = V = 4 NR, known when the kernel is compiled.
template <typename Rule, typename OT, int NR, bool SQ>
__global__ void __launch_bounds__(288) decode_kernel(const Args p, int items) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  extern __shared__ __align__(128) float ring[];                // kBufs x K * V
  __shared__ uint64_t full[kBufs], done[kBufs];
  __shared__ int abort_s;
  __shared__ __align__(16) float vec[2][Rule::kVecs][4 * NR];   // per group, zero past K
  __shared__ __align__(16) float sv[2][128];
  __shared__ float red[2][3][4], red_o[2][4];
  const int tid = threadIdx.x, lane = tid & 31;
  const int K = SQ ? 4 * NR : p.K, V = SQ ? 4 * NR : p.V, H = p.H, KV = K * V, Q = V / 4;
  volatile int* abort_flag = &abort_s;
  if (tid == 0) {
    for (int s = 0; s < kBufs; ++s) { mbar_init(&full[s], 1); mbar_init(&done[s], 1); }
    abort_s = 0;
    mbar_fence_init();
  }
  for (int i = tid; i < 2 * Rule::kVecs * 4 * NR; i += 288) (&vec[0][0][0])[i] = 0.f;
  __syncthreads();
  if (tid >= 256) {
    // ------------------------------------------------------------ producer (one thread): item k lives in buffer k % kBufs
    if (tid != 256) return;
    const uint32_t bytes = (uint32_t)KV * 4;
    auto next_live = [&](int item) {
      while (item < items && p.slots[item / H] < 0) item += gridDim.x;
      return item;
    };
    auto block_of = [&](int item) { return p.state + p.slots[item / H] * p.slot_stride + (size_t)(item % H) * KV; };
    int ahead = next_live(blockIdx.x);
    auto load = [&](int k) {
      if (ahead >= items) return;
      mbar_expect_tx(&full[k % kBufs], bytes);
      bulk_load(ring + (size_t)(k % kBufs) * KV, block_of(ahead), bytes, &full[k % kBufs]);
      ahead = next_live(ahead + gridDim.x);
    };
    for (int k = 0; k < kBufs; ++k) load(k);
    int k = 0;
    for (int item = next_live(blockIdx.x); item < items; item = next_live(item + gridDim.x), ++k) {
      if (!mbar_wait(&done[k % kBufs], (k / kBufs) & 1, abort_flag, kTimeoutProducer)) break;
      bulk_store(block_of(item), ring + (size_t)(k % kBufs) * KV, bytes);
      asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
      load(k + kBufs);
    }
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    if (abort_s != 0) {
      for (uint32_t i = 0; i < (1u << 16); ++i) __nanosleep(20);     // bounded grace period for copies in flight
      if (p.status != nullptr) atomicMax(p.status, abort_s);
    }
    return;
  }
  // -------------------------------------------------------------- two groups of 128 threads
  const int group = tid >> 7, gt = tid & 127, gw = gt >> 5, jq = lane & 7, rg = lane >> 3;
  const int quad = gw * 8 + jq, dwarps = (max(K, V) + 31) / 32;
  const bool col_ok = quad < Q;
  typename Rule::Regs next = {};
  float nv = 0.f;
  auto fetch = [&](int item) {
    if (item < items) {
      const int t = item / H, h = item % H;
      Rule::fetch(p, t, h, gt, next);
      if (gt < V) nv = p.v[(size_t)t * p.ld_v + h * V + gt];
    }
  };
  int fetched = blockIdx.x + group * gridDim.x, k = 0;          // k: live items so far; the group takes those with k % 2 == group
  fetch(fetched);
  int slot_next = blockIdx.x < items ? p.slots[blockIdx.x / H] : -1;
  for (int item = blockIdx.x; item < items; item += gridDim.x) {
    const int slot = slot_next;
    slot_next = item + (int)gridDim.x < items ? p.slots[(item + gridDim.x) / H] : -1;
    const int t = item / H, h = item % H;
    OT* out = reinterpret_cast<OT*>(p.out) + (size_t)t * p.ld_out + h * V;
    if (slot < 0) {
      if (group == 0 && gt < Q) put4(out + 4 * gt, make_float4(0.f, 0.f, 0.f, 0.f));
      continue;
    }
    const int buf = k % kBufs, phase = (k / kBufs) & 1;
    if ((k++ & 1) != group) continue;
    if (fetched != item) fetch(item);                            // rows without a slot shifted the turns
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f), nw4 = g;
    if (col_ok && rg == 0) {
      g = gate4(p.gate != nullptr ? p.gate + (size_t)t * p.ld_gate + h * V + 4 * quad : nullptr, p.silu);
      nw4 = *reinterpret_cast<const float4*>(p.norm_w + h * V + 4 * quad);
    }
    float (*v4)[4 * NR] = vec[group];
    const typename Rule::Regs in = next;
    const typename Rule::Scal sc = Rule::scalars(p, in, h);
    if (gw < dwarps) {
      float s0 = 0.f, s1 = 0.f, s2 = 0.f;
      if (gt < K) {
        float x[Rule::kVecs];
        Rule::vectors(p, in, sc, slot, h, gt, x, s0, s1, s2);
#pragma unroll
        for (int i = 0; i < Rule::kVecs; ++i) v4[i][gt] = x[i];
      }
      if (gt < V) sv[group][gt] = nv;
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
    float s0 = 0.f, s1 = 0.f, s2 = 0.f;
    for (int i = 0; i < dwarps; ++i) { s0 += red[group][0][i]; s1 += red[group][1][i]; s2 += red[group][2][i]; }
    const Coefs cf = Rule::coefs(p, sc, s0, s1, s2);
    float* Sb = ring + (size_t)buf * KV + (size_t)rg * NR * V + 4 * quad;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    const int rows = min(NR, max(K - rg * NR, 0));
    const bool whole = SQ || K == 4 * NR;                              // every lane has all its rows: no guards
    float2 y[2], q[2];
    y[0] = y[1] = q[0] = q[1] = make_float2(0.f, 0.f);
    if constexpr (Rule::kRead) {
      auto read_row = [&](int m, float kf, float rf) {
        const float4 s = *reinterpret_cast<const float4*>(Sb + m * V);
        const float2 sa = make_float2(s.x, s.y), sb = make_float2(s.z, s.w), k2 = twice(kf), r2 = twice(rf);
        y[0] = __ffma2_rn(k2, sa, y[0]); y[1] = __ffma2_rn(k2, sb, y[1]);
        q[0] = __ffma2_rn(r2, sa, q[0]); q[1] = __ffma2_rn(r2, sb, q[1]);
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
        ys.x *= cf.ys; ys.y *= cf.ys; ys.z *= cf.ys; ys.w *= cf.ys;
        const float4 v = *reinterpret_cast<const float4*>(&sv[group][4 * quad]);
        // S' = w S + c1 * vector0 + c2 * vector2 per column
        float2 c1a, c1b, c2a, c2b;
        if constexpr (Rule::kTwoTerms) {
          o.x = qs.x - cf.oy * ys.x + cf.ov * v.x; o.y = qs.y - cf.oy * ys.y + cf.ov * v.y;
          o.z = qs.z - cf.oy * ys.z + cf.ov * v.z; o.w = qs.w - cf.oy * ys.w + cf.ov * v.w;
          c1a = make_float2(v.x, v.y); c1b = make_float2(v.z, v.w);
          c2a = make_float2(-ys.x, -ys.y); c2b = make_float2(-ys.z, -ys.w);
        } else {
          const float4 u = make_float4(v.x - ys.x, v.y - ys.y, v.z - ys.z, v.w - ys.w);
          o.x = cf.os * qs.x + cf.ov * u.x; o.y = cf.os * qs.y + cf.ov * u.y;
          o.z = cf.os * qs.z + cf.ov * u.z; o.w = cf.os * qs.w + cf.ov * u.w;
          c1a = c1b = make_float2(0.f, 0.f);
          c2a = make_float2(cf.us * u.x, cf.us * u.y); c2b = make_float2(cf.us * u.z, cf.us * u.w);
        }
        auto next_row = [&](const float4& s, float kf, float wf, float af) {
          const float2 w2 = twice(wf), a2 = twice(af);
          float2 ta = __fmul2_rn(a2, c2a), tb = __fmul2_rn(a2, c2b);
          if constexpr (Rule::kTwoTerms) {
            const float2 k2 = twice(kf);
            ta = __ffma2_rn(k2, c1a, ta);
            tb = __ffma2_rn(k2, c1b, tb);
          }
          const float2 n0 = __ffma2_rn(w2, make_float2(s.x, s.y), ta), n1 = __ffma2_rn(w2, make_float2(s.z, s.w), tb);
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
            for (int j = 0; j < 8; ++j) s[j] = *reinterpret_cast<const float4*>(Sb + (m + j) * V);
#pragma unroll
            for (int j = 0; j < 8; j += 4) {
              const float4 k4 = Rule::kTwoTerms ? *reinterpret_cast<const float4*>(kv + m + j) : make_float4(0.f, 0.f, 0.f, 0.f);
              const float4 w4 = *reinterpret_cast<const float4*>(wv + m + j);
              const float4 a4 = *reinterpret_cast<const float4*>(av + m + j);
              s[j] = next_row(s[j], k4.x, w4.x, a4.x);
              s[j + 1] = next_row(s[j + 1], k4.y, w4.y, a4.y);
              s[j + 2] = next_row(s[j + 2], k4.z, w4.z, a4.z);
              s[j + 3] = next_row(s[j + 3], k4.w, w4.w, a4.w);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) *reinterpret_cast<float4*>(Sb + (m + j) * V) = s[j];
          }
        } else {
          for (int m = 0; m < rows; ++m)
            *reinterpret_cast<float4*>(Sb + m * V) = next_row(*reinterpret_cast<const float4*>(Sb + m * V), kv[m], wv[m], av[m]);
        }
      }
    } else {
      // one sweep: S' = w S + k v, o = q^T S'
      if (ok && col_ok) {
        const float4 v = *reinterpret_cast<const float4*>(&sv[group][4 * quad]);
        const float2 va = make_float2(v.x, v.y), vb = make_float2(v.z, v.w);
        auto step = [&](float4& s, float kf, float rf) {
          const float2 k2 = twice(Rule::kForget ? 1.0f - kf : kf), r2 = twice(rf);
          const float2 w2 = twice(Rule::kForget ? kf : cf.w);
          const float2 n0 = __ffma2_rn(w2, make_float2(s.x, s.y), __fmul2_rn(k2, va));
          const float2 n1 = __ffma2_rn(w2, make_float2(s.z, s.w), __fmul2_rn(k2, vb));
          q[0] = __ffma2_rn(r2, n0, q[0]); q[1] = __ffma2_rn(r2, n1, q[1]);
          s = make_float4(n0.x, n0.y, n1.x, n1.y);
        };
        const float* kv = &v4[0][rg * NR];
        const float* rv = &v4[1][rg * NR];
        if (whole) {
#pragma unroll
          for (int m = 0; m < NR; m += 8) {
            float4 s[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) s[j] = *reinterpret_cast<const float4*>(Sb + (m + j) * V);
#pragma unroll
            for (int j = 0; j < 8; j += 4) {
              const float4 k4 = *reinterpret_cast<const float4*>(kv + m + j), r4 = *reinterpret_cast<const float4*>(rv + m + j);
              step(s[j], k4.x, r4.x); step(s[j + 1], k4.y, r4.y); step(s[j + 2], k4.z, r4.z); step(s[j + 3], k4.w, r4.w);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) *reinterpret_cast<float4*>(Sb + (m + j) * V) = s[j];
          }
        } else {
          for (int m = 0; m < rows; ++m) {
            float4 s = *reinterpret_cast<const float4*>(Sb + m * V);
            step(s, kv[m], rv[m]);
            *reinterpret_cast<float4*>(Sb + m * V) = s;
          }
        }
      }
      const float4 qs = make_float4(q[0].x, q[0].y, q[1].x, q[1].y);
      o = xor_sum(xor_sum(qs, 8), 16);
      o.x *= cf.os; o.y *= cf.os; o.z *= cf.os; o.w *= cf.os;
    }
    const float so = warp_sum(rg == 0 ? o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w : 0.f);
    if (lane == 0) red_o[group][gw] = so;
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    group_sync(group);
    if (abort_s != 0) break;
    if (gt == 0) mbar_arrive(&done[buf]);
    if (col_ok && rg == 0) {
      const float oo = red_o[group][0] + red_o[group][1] + red_o[group][2] + red_o[group][3];
      const float rs = 1.0f / sqrtf(oo / (float)p.v_real + p.eps);
      put4(out + 4 * quad, make_float4(o.x * rs * nw4.x * g.x, o.y * rs * nw4.y * g.y, o.z * rs * nw4.z * g.z, o.w * rs * nw4.w * g.w));
    }
  }
}

// ---------------------------------------------------------------- prompts
// Record of a (token, head): the rule's kVecs vectors [K] | 4 numbers | the value vector [V] when the rule scales it (kOwnV).
//   general (kTwoTerms):  w | u | a u | w r, numbers c1 c2;  S' = w S - (a u) y + u v, y = u^T S, o = (w r)^T S - c1 y + c2 v
//   kRead:                w | read | write | w r, number c;  S' = w S + write (v - y), y = read^T S, o = (w r)^T S + c (v - y)
//   linear:               k | r, number w;                   S' = w S + k v, o = r^T S'
//   kForget:              f | r;                             S' = f S + (1 - f) v, o = r^T S'
template <typename Rule>
__host__ __device__ inline int rec_floats(int K, int V) { return Rule::kVecs * K + 4 + (Rule::kOwnV ? V : 0); }

constexpr int kScanCols = 32;      // value columns of a CTA
constexpr int kScanGroup = 8;      // tokens per staged group

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// A lane holds R key rows x C value columns of the state; 16 lanes share a column: lane (cg, lr) of a warp has columns
// cg * C .. + C - 1 of the warp's 2 C columns and rows 64 n + 4 lr .. + 3 (n < R / 4, lr < 16; K <= 16 R).  Few rows and many
// columns a lane keep the shared-memory reads of the vectors, the scan's limit, small; the row sums of a column meet in four
// shuffles.  C = 4 reads the vectors once per 8 columns (many sequences); C = 2 spreads a head over twice the warps (few).
// Shared memory of a token: kVecs vectors (16 R floats each, zero past K) | 4 numbers | v of the CTA's 32 columns.
// With a normaliser (kDen) one more CTA per head carries it as a column whose value is 1.
template <typename Rule, int R, int C>
__global__ void __launch_bounds__(32 * kScanCols / (2 * C))
scan_kernel(const Args p, const float* __restrict__ rec, float* __restrict__ o_out, float* __restrict__ den_out) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  constexpr int kWarps = kScanCols / (2 * C), NT = 32 * kWarps;
  constexpr int W = 16 * R, NUM = Rule::kVecs * W, TOK = NUM + 4 + kScanCols;
  extern __shared__ __align__(16) float sm[];
  const int split = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane & 15, cg = lane >> 4;
  const int K = p.K, V = p.V, H = p.H;
  const int slot = p.slots[seq];
  const int t0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int t1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  if (t1 <= t0) return;
  const bool den = Rule::kDen && split == (V + kScanCols - 1) / kScanCols;
  const int c0 = den ? 0 : split * kScanCols, lc = (warp * 2 + cg) * C, col = c0 + lc;   // V % 8 == 0: all C columns in or out
  const int width = den ? 1 : V;
  const bool col_ok = col < width;
  if (slot < 0) {
    for (int i = tid; i < (t1 - t0) * kScanCols; i += NT) {
      const int t = t0 + i / kScanCols, c = c0 + i % kScanCols;
      if (c < width) {
        if (den) den_out[(size_t)t * H + h] = 0.f;
        else o_out[((size_t)t * H + h) * V + c] = 0.f;
      }
    }
    return;
  }
  // zero padding of the vectors, once; the normaliser's value is 1
  for (int i = tid; i < 2 * kScanGroup * TOK; i += NT) sm[i] = den && i % TOK == NUM + 4 ? 1.f : 0.f;
  __syncthreads();
  const int q16 = K / 4, cols16 = den ? 0 : min(kScanCols, V - c0) / 4;           // 16-byte pieces of a vector / of v
  const int rf = rec_floats<Rule>(K, V);
  auto fetch = [&](int g0, int buf) {                                             // tokens g0 .. of the group -> buffer
    const int n = min(kScanGroup, t1 - g0);
    for (int tt = warp; tt < n; tt += kWarps) {
      const float* src = rec + ((size_t)(g0 + tt) * H + h) * rf;
      const float* vs = Rule::kOwnV ? src + Rule::kVecs * K + 4 : p.v + (size_t)(g0 + tt) * p.ld_v + h * V;
      float* dst = sm + (buf * kScanGroup + tt) * TOK;
#pragma unroll
      for (int v = 0; v < Rule::kVecs; ++v)
        for (int j = lane; j < q16; j += 32) cp16(dst + v * W + j * 4, src + v * K + j * 4);
      if (lane < cols16) cp16(dst + NUM + 4 + lane * 4, vs + c0 + lane * 4);
      else if (lane == 31) cp16(dst + NUM, src + Rule::kVecs * K);
    }
    // a short last group is filled up with tokens that leave the state alone: decay 1, everything else 0
    for (int tt = n + warp; tt < kScanGroup; tt += kWarps) {
      float* dst = sm + (buf * kScanGroup + tt) * TOK;
      for (int j = lane; j < TOK; j += 32) dst[j] = (Rule::kRead || Rule::kForget ? j < W : j == NUM) ? 1.f : 0.f;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(t0, 0);
  float* Sg = den ? p.norm_state + slot * p.slot_stride + (size_t)h * K
                  : p.state + slot * p.slot_stride + (size_t)h * K * V + col;
  const int row = den ? 1 : V;                                                    // floats between rows of a column
  const bool init = p.has_initial == nullptr || p.has_initial[seq] != 0;
  float2 S[C][R / 2];                                                             // rows in pairs
#pragma unroll
  for (int n = 0; n < R / 4; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = 64 * n + 4 * lr + j;
      const bool in = init && col_ok && i < K;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float v = in && (!Rule::kDen || col + c < width) ? Sg[(size_t)i * row + c] : 0.f;
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
    // this lane's share of the group's outputs: its rows' part of the product, lane 0 of a column adds the terms in v and y
    float part[kScanGroup][C];
    const float* base = sm + buf * kScanGroup * TOK;
#pragma unroll
    for (int tt = 0; tt < kScanGroup; ++tt) {
      const float* tok = base + tt * TOK;
      float2 sv[C], q[C], cc;
      auto load_values = [&]() {
        cc = *reinterpret_cast<const float2*>(tok + NUM);
#pragma unroll
        for (int c = 0; c < C; c += 2) {
          const float2 s = *reinterpret_cast<const float2*>(tok + NUM + 4 + lc + c);
          sv[c] = twice(s.x);
          sv[c + 1] = twice(s.y);
        }
      };
#pragma unroll
      for (int c = 0; c < C; ++c) q[c] = make_float2(0.f, 0.f);
      if constexpr (Rule::kRead) {
        const float4* w4 = reinterpret_cast<const float4*>(tok) + lr;
        const float4* u4 = w4 + W / 4;
        const float4* a4 = u4 + W / 4;
        const float4* r4 = a4 + W / 4;
        float2 y0[C], y1[C];
        float4 u[R / 4];
#pragma unroll
        for (int c = 0; c < C; ++c) y0[c] = y1[c] = make_float2(0.f, 0.f);
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
        load_values();
        float2 ny[C];                                            // what the write vector is multiplied by
#pragma unroll
        for (int c = 0; c < C; ++c) ny[c] = twice(Rule::kTwoTerms ? -ys[c] : sv[c].x - ys[c]);
#pragma unroll
        for (int n = 0; n < R / 4; ++n) {
          const float4 w = w4[16 * n], a = a4[16 * n], r = r4[16 * n];
#pragma unroll
          for (int c = 0; c < C; ++c) {
            q[c] = __ffma2_rn(make_float2(r.x, r.y), S[c][2 * n], q[c]);
            q[c] = __ffma2_rn(make_float2(r.z, r.w), S[c][2 * n + 1], q[c]);
            float2 s0 = __fmul2_rn(make_float2(w.x, w.y), S[c][2 * n]), s1 = __fmul2_rn(make_float2(w.z, w.w), S[c][2 * n + 1]);
            if constexpr (Rule::kTwoTerms) {
              s0 = __ffma2_rn(make_float2(u[n].x, u[n].y), sv[c], s0);
              s1 = __ffma2_rn(make_float2(u[n].z, u[n].w), sv[c], s1);
            }
            S[c][2 * n] = __ffma2_rn(make_float2(a.x, a.y), ny[c], s0);
            S[c][2 * n + 1] = __ffma2_rn(make_float2(a.z, a.w), ny[c], s1);
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          part[tt][c] = q[c].x + q[c].y;
          if (lr == 0) part[tt][c] += Rule::kTwoTerms ? fmaf(cc.y, sv[c].x, -cc.x * ys[c]) : cc.x * ny[c].x;
        }
      } else {
        const float4* k4 = reinterpret_cast<const float4*>(tok) + lr;
        const float4* r4 = k4 + W / 4;
        load_values();
        const float2 w2 = twice(cc.x);
#pragma unroll
        for (int n = 0; n < R / 4; ++n) {
          const float4 k = k4[16 * n], r = r4[16 * n];
#pragma unroll
          for (int c = 0; c < C; ++c) {
            if constexpr (Rule::kForget) {
              S[c][2 * n] = __ffma2_rn(make_float2(k.x, k.y), S[c][2 * n], __fmul2_rn(make_float2(1.0f - k.x, 1.0f - k.y), sv[c]));
              S[c][2 * n + 1] = __ffma2_rn(make_float2(k.z, k.w), S[c][2 * n + 1], __fmul2_rn(make_float2(1.0f - k.z, 1.0f - k.w), sv[c]));
            } else {
              S[c][2 * n] = __ffma2_rn(make_float2(k.x, k.y), sv[c], __fmul2_rn(w2, S[c][2 * n]));
              S[c][2 * n + 1] = __ffma2_rn(make_float2(k.z, k.w), sv[c], __fmul2_rn(w2, S[c][2 * n + 1]));
            }
            q[c] = __ffma2_rn(make_float2(r.x, r.y), S[c][2 * n], q[c]);
            q[c] = __ffma2_rn(make_float2(r.z, r.w), S[c][2 * n + 1], q[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) part[tt][c] = q[c].x + q[c].y;
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
      if (den) {
        den_out[(size_t)(g0 + lr) * H + h] = part[0][0];
      } else {
        float* dst = o_out + ((size_t)(g0 + lr) * H + h) * V + col;
#pragma unroll
        for (int c = 0; c < C; c += 2) *reinterpret_cast<float2*>(dst + c) = make_float2(part[0][c], part[0][c + 1]);
      }
    }
    __syncthreads();
  }
  if (col_ok) {
#pragma unroll
    for (int n = 0; n < R / 4; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = 64 * n + 4 * lr + j;
        if (i < K) {
#pragma unroll
          for (int c = 0; c < C; ++c)
            if (!Rule::kDen || col + c < width) Sg[(size_t)i * row + c] = (j & 1) ? S[c][2 * n + j / 2].y : S[c][2 * n + j / 2].x;
        }
      }
  }
}

// out[t, h] = o / sqrt(mean(o^2) + eps) * norm * act(gate), o first divided by max(|n . q|, exp(-m)) + den_eps with a
// normaliser; a warp per (token, head).  gates [T * H]: (., ., exp(-m), .)
template <typename OT>
__global__ void __launch_bounds__(256)
finish_kernel(const Args p, const float* __restrict__ o_in, const float* __restrict__ den, const float4* __restrict__ gates) {
  bg::pdl_prologue((BG_FILE_TAG << 16) | __LINE__);
  const int t = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= p.H) return;
  const int V = p.V;
  const size_t th = (size_t)t * p.H + h;
  const float* o = o_in + th * V;
  const float scale = den != nullptr ? 1.0f / (fmaxf(fabsf(den[th]), gates[th].z) + p.den_eps) : 1.0f;
  constexpr int kHeld = 2;                                       // vectors a lane keeps; wider heads are read twice
  float4 held[kHeld];
  float ss = 0.f;
  for (int n = 0, e = lane * 4; e < V; e += 128, ++n) {
    float4 v = *reinterpret_cast<const float4*>(o + e);
    v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
    if (n == 0) held[0] = v;
    else if (n == 1) held[1] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)p.v_real + p.eps);
  for (int n = 0, e = lane * 4; e < V; e += 128, ++n) {
    float4 v;
    if (n < kHeld) {
      v = n == 0 ? held[0] : held[1];
    } else {
      v = *reinterpret_cast<const float4*>(o + e);
      v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
    }
    const float4 g = gate4(p.gate != nullptr ? p.gate + (size_t)t * p.ld_gate + h * V + e : nullptr, p.silu);
    const float4 nw = *reinterpret_cast<const float4*>(p.norm_w + h * V + e);
    put4(reinterpret_cast<OT*>(p.out) + (size_t)t * p.ld_out + h * V + e,
         make_float4(v.x * rs * nw.x * g.x, v.y * rs * nw.y * g.y, v.z * rs * nw.z * g.z, v.w * rs * nw.w * g.w));
  }
}

// ---------------------------------------------------------------- launches
template <typename Rule, int R, int C>
static int launch_scan_as(const Args& p, const float* rec, float* o, float* den, cudaStream_t stream) {
  const size_t smem = (size_t)2 * kScanGroup * (Rule::kVecs * 16 * R + 4 + kScanCols) * sizeof(float);
  static DeviceOnce once;
  auto kern = scan_kernel<Rule, R, C>;
  if (!ensure_dynamic_smem(kern, smem, once)) return -4;
  dim3 grid((p.V + kScanCols - 1) / kScanCols + (Rule::kDen ? 1 : 0), p.H, p.nseq);
  bg::launch_pdl(kern, grid, dim3(32 * kScanCols / (2 * C)), smem, stream, p, rec, o, den);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <typename Rule, int R>
static int launch_scan_rows(const Args& p, const float* rec, float* o, float* den, cudaStream_t stream) {
  const long long ctas = (long long)((p.V + kScanCols - 1) / kScanCols) * p.H * p.nseq;
  if constexpr (R > 16) return launch_scan_as<Rule, R, 2>(p, rec, o, den, stream);       // registers
  else return ctas <= 296 ? launch_scan_as<Rule, R, 2>(p, rec, o, den, stream) : launch_scan_as<Rule, R, 4>(p, rec, o, den, stream);
}
// records, then scan and output; `rec`, `o`, `den`, `gates` are parts of the scratch
template <typename Rule>
static int launch_scan(const Args& p, const float* rec, float* o, float* den, const float4* gates, cudaStream_t stream) {
  int rc;
  if (p.K <= 64) rc = launch_scan_rows<Rule, 4>(p, rec, o, den, stream);
  else if (p.K <= 128) rc = launch_scan_rows<Rule, 8>(p, rec, o, den, stream);
  else if (p.K <= 192) rc = launch_scan_rows<Rule, 12>(p, rec, o, den, stream);
  else if (p.K <= 256) rc = launch_scan_rows<Rule, 16>(p, rec, o, den, stream);
  else rc = launch_scan_rows<Rule, 32>(p, rec, o, den, stream);
  if (rc != 0) return rc;
  const dim3 grid(p.T, (p.H + 7) / 8);
  const float* d = Rule::kDen ? den : nullptr;
  if (p.dt == 0) bg::launch_pdl(finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, p, (const float*)o, d, gates);
  else bg::launch_pdl(finish_kernel<float>, grid, dim3(256), 0, stream, p, (const float*)o, d, gates);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename Rule, typename OT, int NR, bool SQ>
static int launch_decode_sized(const Args& p, cudaStream_t stream) {
  const size_t smem = (size_t)kBufs * p.K * p.V * sizeof(float);
  static DeviceOnce once;
  auto kern = decode_kernel<Rule, OT, NR, SQ>;
  if (!ensure_dynamic_smem(kern, 3 * 128 * 128 * sizeof(float), once)) return -4;
  const int per_sm = smem > 100 * 1024 || NR > 16 ? 1 : smem > 48 * 1024 ? 2 : 3;
  const int items = p.nseq * p.H, most = p.num_sms * per_sm;
  bg::launch_pdl(kern, dim3(items < most ? items : most), dim3(288), smem, stream, p, items);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <typename Rule, typename OT, int NR>
static int launch_decode_as(const Args& p, cudaStream_t stream) {
  return p.K == 4 * NR && p.V == 4 * NR ? launch_decode_sized<Rule, OT, NR, true>(p, stream)
                                        : launch_decode_sized<Rule, OT, NR, false>(p, stream);
}
template <typename Rule, typename OT>
static int launch_decode_rows(const Args& p, cudaStream_t stream) {
  if (p.K <= 32) return launch_decode_as<Rule, OT, 8>(p, stream);
  if (p.K <= 64) return launch_decode_as<Rule, OT, 16>(p, stream);
  return launch_decode_as<Rule, OT, 32>(p, stream);
}
template <typename Rule>
static int launch_decode(const Args& p, cudaStream_t stream) {
  return p.dt == 0 ? launch_decode_rows<Rule, __nv_bfloat16>(p, stream) : launch_decode_rows<Rule, float>(p, stream);
}

// 0, or -1 when sizes or strides are outside the kernels' contract
inline int check_args(const Args& p) {
  auto off4 = [](const float* x, int ld) { return x != nullptr && (ld % 4 != 0 || reinterpret_cast<uintptr_t>(x) % 16 != 0); };
  if (p.K <= 0 || p.K % 8 || p.K > kMaxK || p.V <= 0 || p.V % 8 || p.H <= 0 || p.H > 65535 || p.nseq > 65535 || p.rep <= 0 ||
      p.H % p.rep || p.slot_stride % 4 || p.ld_out % 4 || off4(p.v, p.ld_v) || off4(p.gate, p.ld_gate) || off4(p.q, p.ld_q) ||
      off4(p.k, p.ld_k) || off4(p.low, p.ld_low) || off4(p.state, 0) || (p.cu == nullptr && p.T != p.nseq) ||
      (long long)p.nseq * p.H > 0x7fffffffll)
    return -1;
  if (p.scratch == nullptr && (p.K > 128 || p.V > 128 || p.cu != nullptr || p.has_initial != nullptr || p.num_sms <= 0)) return -1;
  return 0;
}

}  // namespace rec
}  // namespace bg
