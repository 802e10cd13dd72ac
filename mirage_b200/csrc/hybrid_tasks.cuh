// Task bodies of hybrid graphs: decoders whose layers mix softmax attention with recurrent state.
//
//   float32 residual stream      TASK_EMBED_F32, TASK_RESIDUAL_NORM
//   attention                    TASK_QKV_APPEND (rotation, unit norms, cache rows), TASK_EXT_ATTENTION (any head size,
//                                score scale, soft cap, sink)
//   recurrences                  TASK_SHORT_CONV, TASK_RGLRU (gated diagonal), TASK_MLSTM (matrix memory)
//   32-bit graphs                TASK_LINEAR_F32
//
// A recurrent layer keeps its state in float32 tensors indexed by the request's state slot, which the batching task
// hands out at admission; a request whose batch portion starts at position 0 starts from a zero state, so slots are
// reused without being cleared.  Every body walks the tokens of the batch by request (qo_indptr), whatever mixture of
// prompt portions and single decoded tokens it holds.
//
// HYB = HYB_BF16: matrix operands, the KV cache and the operands handed to projections are bf16, everything else is
// float32.  HYB = HYB_F32: those are float32 as well.
#pragma once
#include "megakernel.cuh"

namespace mpk {

template <int HYB>
struct HybElt { typedef __nv_bfloat16 T; };
template <>
struct HybElt<HYB_F32> { typedef float T; };

__device__ __forceinline__ void store_elt(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_elt(float *p, float v) { *p = v; }
__device__ __forceinline__ float bf16_at(uint64_t base, size_t i) {
  return bf16_to_f(__ldg(reinterpret_cast<const __nv_bfloat16 *>(base) + i));
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// Decay factor exp(x), x <= 0, of a recurrence that applies it once per token: near 1 the last-bit error of expf has a
// sign of its own and adds up over a long memory; 1 + expm1f(x) rounds to nearest.
__device__ __forceinline__ float decay_exp(float x) { return x > -0.35f ? 1.0f + expm1f(x) : expf(x); }
__device__ __forceinline__ float gelu_tanh_f(float x) {
  return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the 256 compute threads (slots: 8 floats of shared memory; the caller keeps two calls apart with a barrier
// or with different slots).
__device__ __forceinline__ float block_sum(float v, float *slots) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) slots[threadIdx.x >> 5] = v;
  consumer_sync();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) t += slots[w];
  return t;
}

// One request of the batch: its tokens [q0, q0 + nq), the position of the first, its cache pages and its state slot.
struct SeqView {
  int q0, nq, pos0, kv0, slot;
};
__device__ __forceinline__ SeqView seq_view(const KernelParams &P, int k) {
  const BatchMeta &M = P.meta;
  SeqView s;
  s.q0 = __ldcg(&M.qo_indptr[k]);
  s.nq = __ldcg(&M.qo_indptr[k + 1]) - s.q0;
  s.kv0 = __ldcg(&M.paged_kv_indptr[k]);
  const int pages = __ldcg(&M.paged_kv_indptr[k + 1]) - s.kv0;
  s.pos0 = (pages - 1) * P.page_size + __ldcg(&M.paged_kv_last_page_len[k]) - s.nq;
  s.slot = M.state_slots ? __ldcg(&M.state_slots[k]) : k;
  return s;
}

// Per-token view for bodies that take all tokens of the batch at once (filled by token_map, shared memory).
struct TokenRec {
  int q0;      // first token of this token's request
  int slot;    // its state slot
  int flags;   // 1 first token of the request in this batch, 2 last one, 4 the request starts at position 0
  int pad;
};
constexpr int kTokenMapBytes = kMaxLinearTokens * (int)sizeof(TokenRec);
// `qo` needs max_num_batched_requests + 1 ints of shared memory.  Ends with a barrier.
__device__ __forceinline__ void token_map(const KernelParams &P, int B, TokenRec *rec, int *qo) {
  const int mbr = P.max_num_batched_requests;
  for (int i = threadIdx.x; i <= mbr; i += kConsumerThreads) qo[i] = __ldcg(&P.meta.qo_indptr[i]);
  consumer_sync();
  for (int t = threadIdx.x; t < B; t += kConsumerThreads) {
    int lo = 0, hi = mbr - 1;   // largest k with qo[k] <= t and qo[k + 1] > t
    while (lo < hi) {
      const int mid = (lo + hi) >> 1;
      if (qo[mid + 1] <= t) lo = mid + 1; else hi = mid;
    }
    const SeqView s = seq_view(P, lo);
    rec[t].q0 = s.q0;
    rec[t].slot = s.slot;
    rec[t].flags = (t == s.q0 ? 1 : 0) | (t == s.q0 + s.nq - 1 ? 2 : 0) | (s.pos0 == 0 ? 4 : 0);
  }
  consumer_sync();
}

// ---------------------------------------------------------------------------
// float32 residual stream
// ---------------------------------------------------------------------------
__device__ __forceinline__ void run_embed_f32(const Ctx &c, const TaskDesc &d) {
  const int B = active_tokens(c.P);
  const int t0 = d.a[E_T0], t1 = min(d.a[E_T1], B), width = d.a[E_WIDTH];
  const int64_t *ids = reinterpret_cast<const int64_t *>(d.p[0]);
  float *out = reinterpret_cast<float *>(d.p[2]);
  for (int t = t0; t < t1; ++t) {
    const long long id = __ldcg(reinterpret_cast<const long long *>(&ids[t]));
    const bool in_table = id >= 0 && id < (long long)d.a[E_AUX];   // ids outside the table read as a zero row
    for (int j = threadIdx.x; j < width; j += kConsumerThreads)
      out[(size_t)t * d.a[E_LDO] + j] = in_table ? bf16_at(d.p[1], (size_t)id * d.a[E_LDI] + j) : 0.f;
  }
}

// x += norm(y) (or x += y, or nothing), then out = norm(x): one token row at a time.  VEC consecutive elements per
// thread and step; the row stays in shared memory between the passes (every element is touched by one thread only).
template <int HYB, int VEC>
__device__ __forceinline__ void residual_norm_rows(const Ctx &c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const int B = active_tokens(c.P);
  const int t0 = d.a[0], t1 = min(d.a[1], B), W = d.a[2];
  const float eps = __int_as_float(d.a[6]);
  const float off = (d.a[7] & 2) ? 1.0f : 0.0f;
  const bool has_y = d.p[1] != 0, has_post = d.p[2] != 0, has_out = d.p[3] != 0;
  float *row = reinterpret_cast<float *>(c.s.xtile);
  for (int t = t0; t < t1; ++t) {
    float *x = reinterpret_cast<float *>(d.p[0]) + (size_t)t * d.a[3];
    const float *y = reinterpret_cast<const float *>(d.p[1]) + (size_t)t * d.a[4];
    float inv = 1.f;
    if (has_y && has_post) {
      float ss = 0.f;
      for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC) {
        if (VEC == 4) {
          const float4 v = __ldcg(reinterpret_cast<const float4 *>(y + j));
          *reinterpret_cast<float4 *>(row + j) = v;
          ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        } else {
          const float v = __ldcg(y + j);
          row[j] = v;
          ss += v * v;
        }
      }
      inv = 1.0f / sqrtf(block_sum(ss, c.s.red) / (float)W + eps);
    }
    float ss = 0.f;
    for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC) {
      float xv[VEC], yv[VEC];
      if (VEC == 4) {
        *reinterpret_cast<float4 *>(xv) = __ldcg(reinterpret_cast<const float4 *>(x + j));
        if (has_y) *reinterpret_cast<float4 *>(yv) = has_post ? *reinterpret_cast<const float4 *>(row + j)
                                                              : __ldcg(reinterpret_cast<const float4 *>(y + j));
      } else {
        xv[0] = __ldcg(x + j);
        if (has_y) yv[0] = has_post ? row[j] : __ldcg(y + j);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (has_y) xv[e] += has_post ? yv[e] * inv * (off + bf16_at(d.p[2], j + e)) : yv[e];
        ss += xv[e] * xv[e];
        row[j + e] = xv[e];
        if (has_y) x[j + e] = xv[e];
      }
    }
    if (has_out) {
      const float inv2 = 1.0f / sqrtf(block_sum(ss, c.s.red + 8) / (float)W + eps);
      T *out = reinterpret_cast<T *>(d.p[4]) + (size_t)t * d.a[5];
      for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) store_elt(out + j + e, row[j + e] * inv2 * (off + bf16_at(d.p[3], j + e)));
      }
    }
    consumer_sync();   // the reduction slots are used again by the next row
  }
}
template <int HYB>
__device__ __forceinline__ void run_residual_norm(const Ctx &c, const TaskDesc &d) {
  if (((d.a[2] | d.a[3] | d.a[4]) & 3) == 0 && ((d.p[0] | d.p[1]) & 15) == 0) residual_norm_rows<HYB, 4>(c, d);
  else residual_norm_rows<HYB, 1>(c, d);
}

// ---------------------------------------------------------------------------
// linear layer in 32-bit arithmetic: one warp per weight row, eight tokens at a time
// ---------------------------------------------------------------------------
__device__ __forceinline__ void run_linear_f32(const Ctx &c, const TaskDesc &d) {
  const int B = active_tokens(c.P);
  const int n0 = d.a[0], n1 = d.a[1], K = d.a[2], act = d.a[6], TT = d.a[7];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float *xs = reinterpret_cast<float *>(c.s.xtile);   // [TT][K]
  const float *x = reinterpret_cast<const float *>(d.p[1]);
  float *out = reinterpret_cast<float *>(d.p[2]);
  for (int tb = 0; tb < B; tb += TT) {
    const int nt = min(TT, B - tb);
    if (tb > 0) consumer_sync();
    for (int t = 0; t < nt; ++t)
      for (int k = tid; k < K; k += kConsumerThreads) xs[(size_t)t * K + k] = __ldcg(x + (size_t)(tb + t) * d.a[4] + k);
    consumer_sync();
    for (int n = n0 + warp; n < n1; n += 8) {
      const size_t wrow = (size_t)n * d.a[3];
      for (int t8 = 0; t8 < nt; t8 += 8) {
        float acc[8];
        const float *xr[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          acc[u] = 0.f;
          xr[u] = xs + (size_t)min(t8 + u, nt - 1) * K;
        }
        for (int k = lane; k < K; k += 32) {
          const float w = bf16_at(d.p[0], wrow + k);
#pragma unroll
          for (int u = 0; u < 8; ++u) acc[u] = fmaf(w, xr[u][k], acc[u]);
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          float v = warp_sum(acc[u]);
          if (act == 1) { v = fmaxf(v, 0.f); v *= v; }
          if (lane == u && t8 + u < nt) out[(size_t)(tb + t8 + u) * d.a[5] + n] = v;
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------
// TASK_QKV_APPEND: one warp per (token, head).  q: rotate, normalise, store; k: rotate, normalise, store in the cache
// page of its position together with the value row.
// ---------------------------------------------------------------------------
template <int HYB>
__device__ __forceinline__ void run_qkv_append(const Ctx &c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hq = d.a[QA_HQ], hkv = d.a[QA_HKV], dim = d.a[QA_DIM], dimp = d.a[QA_DIMP], vdim = d.a[QA_VDIM], vdimp = d.a[QA_VDIMP];
  const int rot = d.a[QA_ROT], half = rot >> 1, page = d.a[QA_PAGE];
  const float eps = __int_as_float(d.a[QA_EPS]);
  const int mbr = P.max_num_batched_requests;
  const int heads = hq + hkv, first = d.a[QA_T0], tasks = d.a[QA_T1];
  for (int item = first * 8 + warp; item < B * heads; item += tasks * 8) {
    const int t = item / heads, h = item - t * heads;
    int k = 0;   // the request this token belongs to: as many requests end at or before the token
    for (int b = 0; b < mbr; b += 32) {
      const bool before = b + lane < mbr && __ldcg(&P.meta.qo_indptr[b + lane + 1]) <= t;
      const int n = __popc(__ballot_sync(0xffffffffu, before));
      k += n;
      if (n < 32) break;
    }
    const SeqView s = seq_view(P, k);
    const int pos = s.pos0 + t - s.q0;
    const bool is_q = h < hq;
    const float *src = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[QA_LDP] +
                       (is_q ? d.a[QA_QOFF] + h * dim : d.a[QA_KOFF] + (h - hq) * dim);
    const size_t trow = (size_t)min(pos, d.a[QA_ROWS] - 1) * half;
    const float *cosT = reinterpret_cast<const float *>(d.p[4]) + trow, *sinT = reinterpret_cast<const float *>(d.p[5]) + trow;
    auto rotated = [&](int i) {
      const float v = __ldcg(src + i);
      if (i >= rot) return v;
      if (i < half) return v * __ldg(cosT + i) - __ldcg(src + i + half) * __ldg(sinT + i);
      return v * __ldg(cosT + i - half) + __ldcg(src + i - half) * __ldg(sinT + i - half);
    };
    float inv = 1.f;
    if (d.a[QA_NORM]) {
      float ss = 0.f;
      for (int i = lane; i < dim; i += 32) { const float v = rotated(i); ss += v * v; }
      inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
    }
    T *dst;
    if (is_q) {
      dst = reinterpret_cast<T *>(d.p[1]) + (size_t)t * d.a[QA_LDQ] + (size_t)h * dimp;
    } else {
      const int pg = pos / page;
      const size_t cell = ((size_t)__ldcg(&P.meta.paged_kv_indices[s.kv0 + pg]) * page + (pos - pg * page)) * hkv + (h - hq);
      dst = reinterpret_cast<T *>(d.p[2]) + cell * dimp;
      T *vdst = reinterpret_cast<T *>(d.p[3]) + cell * vdimp;
      const float *vsrc = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[QA_LDP] + d.a[QA_VOFF] + (h - hq) * vdim;
      for (int i = lane; i < vdim; i += 32) store_elt(vdst + i, __ldcg(vsrc + i));
    }
    for (int i = lane; i < dim; i += 32) store_elt(dst + i, rotated(i) * inv);
  }
}

// ---------------------------------------------------------------------------
// TASK_EXT_ATTENTION: (request, kv head, chunk of the keys).  The M rows of a task are the (token, query head of the
// group) pairs, row r = token r / G, head r % G.  Chunks are merged by the last task of the (request, kv head) to
// arrive.  Scores live in base 2 (bf16) or base e (float32): exp_dom undoes the same base everywhere.
// ---------------------------------------------------------------------------
template <int HYB>
__device__ __forceinline__ float exp_dom(float x) { return HYB == HYB_F32 ? expf(x) : exp2f(x); }

// scaled, capped score in the domain's base
template <int HYB>
__device__ __forceinline__ float attn_score(float dot, float scale, float cap, float cap2) {
  float s = dot * scale;
  if (HYB == HYB_F32) return cap > 0.f ? cap * tanhf(s / cap) : s;
  // tanh(z) = 1 - 2 / (exp(2 z) + 1); cap2 = 2 log2(e) / cap
  if (cap > 0.f) s = cap * (1.0f - __fdividef(2.0f, exp2f(s * cap2) + 1.0f));
  return s * 1.4426950408889634f;
}

struct AttnOut {   // where a task's rows go
  int hq, G, head, q0, NC, chunk, n_act, vdim, ldo, ocol, srec;
  float oscale;
  bool sink;
};
// Row r with (max m, sum l); val(col) gives the unnormalised output column.  Called by one warp.
template <int HYB, class F>
__device__ __forceinline__ void attn_emit_row(const Ctx &c, const TaskDesc &d, const AttnOut &o, int r, float m, float l, F val) {
  typedef typename HybElt<HYB>::T T;
  const int lane = threadIdx.x & 31;
  const int tok = o.q0 + r / o.G, hq_idx = o.head * o.G + r % o.G;
  if (o.n_act == 1) {
    const float M = o.sink ? fmaxf(m, 0.f) : m;
    const float w = m == -INFINITY ? 0.f : exp_dom<HYB>(m - M);
    const float L = l * w + (o.sink ? exp_dom<HYB>(-M) : 0.f);
    const float f = L > 0.f ? w / L * o.oscale : 0.f;
    T *out = reinterpret_cast<T *>(d.p[3]) + (size_t)tok * o.ldo + o.ocol + (size_t)hq_idx * o.vdim;
    for (int j = lane; j < o.vdim; j += 32) store_elt(out + j, val(j) * f);
  } else {
    float *rec = c.P.attn_scratch + (((size_t)tok * o.hq + hq_idx) * o.NC + o.chunk) * o.srec;
    if (lane == 0) {
      __stcg(rec, m);
      __stcg(rec + 1, l);
    }
    for (int j = lane; j < o.vdim; j += 32) __stcg(rec + 2 + j, val(j));
  }
}

// Merge of the chunks' records by the last arriver.  NC <= 32.
template <int HYB>
__device__ __forceinline__ void attn_merge(const Ctx &c, const TaskDesc &d, const AttnOut &o, int rows) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  consumer_sync();
  if (threadIdx.x == 0) {
    unsigned int *ticket = &P.attn_tickets[d.a[XA_TICKET]];
    unsigned int old;
    asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(old) : "l"(ticket) : "memory");
    const bool last = old + 1u == (unsigned)o.n_act;
    if (last) *reinterpret_cast<volatile unsigned int *>(ticket) = 0u;
    c.s.flags[1] = last ? 1 : 0;
  }
  consumer_sync();
  if (c.s.flags[1] == 0) return;
  for (int r = warp; r < rows; r += 8) {
    const int tok = o.q0 + r / o.G, hq_idx = o.head * o.G + r % o.G;
    const float *rec = P.attn_scratch + ((size_t)tok * o.hq + hq_idx) * o.NC * o.srec;
    const bool v = lane < o.n_act;
    const float m = v ? __ldcg(rec + (size_t)lane * o.srec) : -INFINITY;
    const float l = v ? __ldcg(rec + (size_t)lane * o.srec + 1) : 0.f;
    float M = warp_max(m);
    if (o.sink) M = fmaxf(M, 0.f);
    const float w = m == -INFINITY ? 0.f : exp_dom<HYB>(m - M);
    const float L = warp_sum(l * w) + (o.sink ? exp_dom<HYB>(-M) : 0.f);
    const float f = L > 0.f ? o.oscale / L : 0.f;
    T *out = reinterpret_cast<T *>(d.p[3]) + (size_t)tok * o.ldo + o.ocol + (size_t)hq_idx * o.vdim;
    for (int j0 = 0; j0 < o.vdim; j0 += 32) {
      const int j = j0 + lane;
      float acc = 0.f;
      for (int u = 0; u < o.n_act; ++u) {
        const float wu = __shfl_sync(0xffffffffu, w, u);
        if (j < o.vdim && wu > 0.f) acc = fmaf(wu, __ldcg(rec + (size_t)u * o.srec + 2 + j), acc);
      }
      if (j < o.vdim) store_elt(out + j, acc * f);
    }
  }
}

// bf16: QK^T and PV on mma.sync.  Head sizes are padded to D columns in shared memory.  The eight warps are split over
// row tiles (16 rows), key octets and, for D = 256, halves of the output columns; the key split is combined in shared
// memory.  The probabilities enter PV as a bf16 value and a bf16 remainder, so that the weights keep 16 bits.
template <int D>
__device__ __forceinline__ void ext_attention_mma(const Ctx &c, const TaskDesc &d, const SeqView &sv, const AttnOut &ao, int k0, int k1,
                                                  int rows) {
  constexpr int ON = D < 128 ? D : 128, WN = D / ON, KEYS = D > 128 ? 32 : 64, NSUB = KEYS / 8, PITCH = D * 2 + 16;
  constexpr int WMAX = 8 / WN, MROWS = WMAX * 16, TILE = KEYS * PITCH;
  const KernelParams &P = c.P;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int G = ao.G, hkv = d.a[XA_HKV], dimp = d.a[XA_DIMP], vdimp = d.a[XA_VDIMP], page = d.a[XA_PAGE];
  const float scale = __int_as_float(d.a[XA_SCALE]), cap = __int_as_float(d.a[XA_CAP]);
  const float cap2 = cap > 0.f ? 2.0f * 1.4426950408889634f / cap : 0.f;
  const int RB = min(MROWS, ext_attention_rows(P.max_num_batched_tokens * G));
  uint8_t *qs = c.s.xtile;                // [RB][PITCH]
  uint8_t *st = qs + RB * PITCH;          // two stages of K rows, V rows
  const uint8_t *qg = reinterpret_cast<const uint8_t *>(d.p[0]);
  const uint8_t *kg = reinterpret_cast<const uint8_t *>(d.p[1]), *vg = reinterpret_cast<const uint8_t *>(d.p[2]);
  const int kp = dimp >> 3, vp = vdimp >> 3;   // 16-byte pieces of a row

  for (int rb = 0; rb < rows; rb += RB) {
    const int nrow = min(RB, rows - rb), mt = (nrow + 15) >> 4;
    const int WM = mt <= 1 ? 1 : (mt <= 2 ? 2 : (mt <= 4 ? 4 : WMAX));
    const int WK = WMAX / WM;                                      // <= NSUB
    const int wn = warp % WN, w2 = warp / WN, wm = w2 % WM, wk = w2 / WM;
    const int kend = min(k1, sv.pos0 + (rb + nrow - 1) / G + 1);   // keys past the last row's position are not needed
    if (rb > 0) consumer_sync();
    for (int i = tid; i < WM * 16 * (D / 8); i += kConsumerThreads) {
      const int r = i / (D / 8), p = i - r * (D / 8);
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nrow && p < kp) {
        const int row = rb + r;
        v = __ldcg(reinterpret_cast<const uint4 *>(qg + ((size_t)(sv.q0 + row / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + row % G) * dimp) * 2) + p);
      }
      *reinterpret_cast<uint4 *>(qs + r * PITCH + p * 16) = v;
    }
    auto issue = [&](int base, int stage) {
      for (int i = tid; i < KEYS * (D / 8); i += kConsumerThreads) {
        const int r = i / (D / 8), p = i - r * (D / 8), key = base + r;
        uint8_t *kd = st + stage * 2 * TILE + r * PITCH + p * 16, *vd = kd + TILE;
        const bool in = key < kend;
        size_t cell = 0;
        if (in) {
          const int pg = key / page;
          cell = ((size_t)__ldcg(&P.meta.paged_kv_indices[sv.kv0 + pg]) * page + (key - pg * page)) * hkv + ao.head;
        }
        // pieces outside the row or past the last key are zeros: a masked key has weight 0, and 0 x NaN would be NaN
        if (in && p < kp) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(kd)), "l"(kg + (cell * kp + p) * 16) : "memory");
        else *reinterpret_cast<uint4 *>(kd) = make_uint4(0, 0, 0, 0);
        if (in && p < vp) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(vd)), "l"(vg + (cell * vp + p) * 16) : "memory");
        else *reinterpret_cast<uint4 *>(vd) = make_uint4(0, 0, 0, 0);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float o[ON / 8][4];
#pragma unroll
    for (int i = 0; i < ON / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
    const int r_lo = rb + wm * 16 + (lane >> 2);
    const int p_lo = sv.pos0 + r_lo / G, p_hi = sv.pos0 + (r_lo + 8) / G;   // last key each row sees
    const int ntiles = kend > k0 ? (kend - k0 + KEYS - 1) / KEYS : 0;
    if (ntiles > 0) issue(k0, 0);
    for (int it = 0; it < ntiles; ++it) {
      if (it + 1 < ntiles) issue(k0 + (it + 1) * KEYS, (it + 1) & 1);
      if (it + 1 < ntiles) asm volatile("cp.async.wait_group 1;" ::: "memory");
      else asm volatile("cp.async.wait_group 0;" ::: "memory");
      consumer_sync();
      const int base = k0 + it * KEYS;
      const uint32_t kt = smem_u32(st + (it & 1) * 2 * TILE), vt = kt + TILE;
      if (wm < mt) {
        float s[NSUB][4];
#pragma unroll
        for (int j = 0; j < NSUB; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
        const uint32_t qa = smem_u32(qs) + (uint32_t)((wm * 16 + (lane & 15)) * PITCH + (lane >> 4) * 16);
#pragma unroll
        for (int kk = 0; kk < D / 32; ++kk) {
          uint32_t a0[4], a1[4];
          ldmatrix_x4(a0, qa + kk * 64u);
          ldmatrix_x4(a1, qa + kk * 64u + 32u);
#pragma unroll
          for (int j = 0; j < NSUB; ++j) {
            if ((j & (WK - 1)) == wk) {
              uint32_t b[4];
              ldmatrix_x4(b, kt + (uint32_t)((j * 8 + (lane & 7)) * PITCH + (lane >> 3) * 16) + kk * 64u);
              mma_bf16_16816(s[j], a0, b[0], b[1]);
              mma_bf16_16816(s[j], a1, b[2], b[3]);
            }
          }
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < NSUB; ++j) {
          if ((j & (WK - 1)) == wk) {
            const int key = base + j * 8 + 2 * (lane & 3);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int kpos = key + (e & 1);
              const bool ok = kpos < kend && kpos <= (e < 2 ? p_lo : p_hi);
              s[j][e] = ok ? attn_score<HYB_BF16>(s[j][e], scale, cap, cap2) : -INFINITY;
              mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
            }
          }
        }
        float corr[2], ms[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
          const float mn = fmaxf(m_run[i], mx[i]);
          ms[i] = mn == -INFINITY ? 0.f : mn;
          corr[i] = exp2f(m_run[i] - ms[i]);
          m_run[i] = mn;
          l_run[i] *= corr[i];
        }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
          for (int i = 0; i < ON / 8; ++i) {
            o[i][0] *= corr[0]; o[i][1] *= corr[0];
            o[i][2] *= corr[1]; o[i][3] *= corr[1];
          }
        }
#pragma unroll
        for (int j = 0; j < NSUB; ++j) {
          if ((j & (WK - 1)) == wk) {
            float p[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              p[e] = exp2f(s[j][e] - ms[e >> 1]);
              l_run[e >> 1] += p[e];
            }
            const uint32_t h0 = pack_bf16(p[0], p[1]), h1 = pack_bf16(p[2], p[3]);
            const uint32_t r0 = pack_bf16(p[0] - bf16_lo(h0), p[1] - bf16_hi(h0)), r1 = pack_bf16(p[2] - bf16_lo(h1), p[3] - bf16_hi(h1));
            const uint32_t va = vt + (uint32_t)((j * 8 + (lane & 7)) * PITCH + (lane >> 3) * 16 + wn * ON * 2);
#pragma unroll
            for (int vq = 0; vq < ON / 32; ++vq) {
              uint32_t b[4];
              ldmatrix_x4_trans(b, va + vq * 64u);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                mma_bf16_1688(o[4 * vq + i], h0, h1, b[i]);
                mma_bf16_1688(o[4 * vq + i], r0, r1, b[i]);
              }
            }
          }
        }
      }
      consumer_sync();   // the stage is refilled by the next trip
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
      l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
    }
    // combine the key split: records [wk][row] of (m, l, D columns) over the stages (at most MROWS of them)
    float *comb = reinterpret_cast<float *>(st);
    if (wm < mt) {
      const int r = wm * 16 + (lane >> 2);
      float *c0 = comb + (size_t)(wk * WM * 16 + r) * (D + 2), *c1 = c0 + 8 * (D + 2);
      if (wn == 0 && (lane & 3) == 0) {
        c0[0] = m_run[0]; c0[1] = l_run[0];
        c1[0] = m_run[1]; c1[1] = l_run[1];
      }
#pragma unroll
      for (int i = 0; i < ON / 8; ++i) {
        const int col = 2 + wn * ON + i * 8 + 2 * (lane & 3);
        *reinterpret_cast<float2 *>(c0 + col) = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2 *>(c1 + col) = make_float2(o[i][2], o[i][3]);
      }
    }
    consumer_sync();
    for (int r = warp; r < nrow; r += 8) {
      const float *cr = comb + (size_t)r * (D + 2);
      const size_t step = (size_t)WM * 16 * (D + 2);
      float M = -INFINITY, L = 0.f, wgt[8];
#pragma unroll
      for (int w = 0; w < 8; ++w)
        if (w < WK) M = fmaxf(M, cr[w * step]);
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        wgt[w] = 0.f;
        if (w < WK) {
          const float mw = cr[w * step];
          wgt[w] = mw == -INFINITY ? 0.f : exp2f(mw - M);
          L += cr[w * step + 1] * wgt[w];
        }
      }
      attn_emit_row<HYB_BF16>(c, d, ao, rb + r, M, L, [&](int j) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w)
          if (w < WK) v += wgt[w] * cr[w * step + 2 + j];
        return v;
      });
    }
  }
}

// 32-bit: one warp per row, 32 keys at a time (a lane per key for the scores, a lane per output column for PV)
__device__ __forceinline__ void ext_attention_f32(const Ctx &c, const TaskDesc &d, const SeqView &sv, const AttnOut &ao, int k0, int k1,
                                                  int rows) {
  constexpr int NO = 16;   // output columns per lane: value sizes up to 512
  const KernelParams &P = c.P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = ao.G, hkv = d.a[XA_HKV], dimp = d.a[XA_DIMP], vdimp = d.a[XA_VDIMP], page = d.a[XA_PAGE];
  const float scale = __int_as_float(d.a[XA_SCALE]), cap = __int_as_float(d.a[XA_CAP]);
  float *q = reinterpret_cast<float *>(c.s.xtile) + warp * dimp;
  const float *qg = reinterpret_cast<const float *>(d.p[0]);
  const float *kg = reinterpret_cast<const float *>(d.p[1]), *vg = reinterpret_cast<const float *>(d.p[2]);
  auto cell_of = [&](int key) {
    const int pg = key / page;
    return ((size_t)__ldcg(&P.meta.paged_kv_indices[sv.kv0 + pg]) * page + (key - pg * page)) * hkv + ao.head;
  };
  for (int r = warp; r < rows; r += 8) {
    const int kend = min(k1, sv.pos0 + r / G + 1);
    __syncwarp();
    for (int i = lane; i < dimp; i += 32) q[i] = __ldcg(qg + (size_t)(sv.q0 + r / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + r % G) * dimp + i);
    __syncwarp();
    float m = -INFINITY, l = 0.f, o[NO];
#pragma unroll
    for (int i = 0; i < NO; ++i) o[i] = 0.f;
    for (int kb = k0; kb < kend; kb += 32) {
      const int key = kb + lane;
      float s = -INFINITY;
      size_t cell = 0;
      if (key < kend) {
        cell = cell_of(key);
        const float4 *kr = reinterpret_cast<const float4 *>(kg + cell * dimp);
        float dot = 0.f;
        for (int i = 0; i < dimp >> 2; ++i) {
          const float4 kv = __ldcg(kr + i), qv = *reinterpret_cast<const float4 *>(q + 4 * i);
          dot += kv.x * qv.x + kv.y * qv.y + kv.z * qv.z + kv.w * qv.w;
        }
        s = attn_score<HYB_F32>(dot, scale, cap, 0.f);
      }
      const float mn = fmaxf(m, warp_max(s));
      const float corr = expf(m - mn), p = key < kend ? expf(s - mn) : 0.f;
      l = l * corr + warp_sum(p);
      m = mn;
#pragma unroll
      for (int i = 0; i < NO; ++i) o[i] *= corr;
      const int n = min(32, kend - kb);
      for (int j = 0; j < n; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
        const size_t cj = __shfl_sync(0xffffffffu, (unsigned long long)cell, j);
#pragma unroll
        for (int i = 0; i < NO; ++i)
          if (i * 32 + lane < ao.vdim) o[i] = fmaf(pj, __ldcg(vg + cj * vdimp + i * 32 + lane), o[i]);
      }
    }
    attn_emit_row<HYB_F32>(c, d, ao, r, m, l, [&](int j) {
      float v = 0.f;
#pragma unroll
      for (int i = 0; i < NO; ++i)
        if (i == (j >> 5)) v = o[i];
      return v;
    });
  }
}

template <int HYB>
__device__ __forceinline__ void run_ext_attention(const Ctx &c, const TaskDesc &d) {
  const SeqView sv = seq_view(c.P, d.a[XA_SLOT]);
  if (sv.nq <= 0) return;
  AttnOut ao;
  ao.hq = d.a[XA_HQ];
  ao.G = ao.hq / d.a[XA_HKV];
  ao.head = d.a[XA_HEAD];
  ao.q0 = sv.q0;
  ao.NC = d.a[XA_NCHUNK];
  ao.chunk = d.a[XA_CHUNK];
  ao.vdim = d.a[XA_VDIM];
  ao.ldo = d.a[XA_LDO];
  ao.ocol = d.a[XA_OCOL];
  ao.srec = d.a[XA_SREC];
  ao.oscale = __int_as_float(d.a[XA_OSCALE]);
  ao.sink = d.a[XA_SINK] != 0;
  const int len = sv.pos0 + sv.nq, rows = sv.nq * ao.G;
  const int per = max(128, ((len + ao.NC - 1) / ao.NC + 63) & ~63);   // keys of a chunk
  ao.n_act = (len + per - 1) / per;
  if (ao.chunk >= ao.n_act) return;
  const int k0 = ao.chunk * per, k1 = min(len, k0 + per);
  if (HYB == HYB_F32) {
    ext_attention_f32(c, d, sv, ao, k0, k1, rows);
  } else {
    const int w = max(d.a[XA_DIMP], d.a[XA_VDIMP]);
    if (w <= 64) ext_attention_mma<64>(c, d, sv, ao, k0, k1, rows);
    else if (w <= 128) ext_attention_mma<128>(c, d, sv, ao, k0, k1, rows);
    else ext_attention_mma<256>(c, d, sv, ao, k0, k1, rows);
  }
  if (ao.n_act > 1) attn_merge<HYB>(c, d, ao, rows);
}

// ---------------------------------------------------------------------------
// TASK_SHORT_CONV: out[t][ch] = bias[ch] + sum_j taps[ch][j] in[t - (taps - 1) + j][ch], inputs before the portion come
// from the carried state (zeros before the sequence).  A task owns a channel range of every request.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void run_short_conv(const Ctx &c, const TaskDesc &d) {
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  if (B <= 0) return;
  TokenRec *rec = reinterpret_cast<TokenRec *>(c.s.xtile);
  token_map(P, B, rec, reinterpret_cast<int *>(c.s.xtile + kTokenMapBytes));
  const int c0 = d.a[0], nc = d.a[1] - c0, C = d.a[2], taps = d.a[3], hist = taps - 1;
  const float *in = reinterpret_cast<const float *>(d.p[0]) + d.a[5];
  float *state = reinterpret_cast<float *>(d.p[4]);
  float *out = reinterpret_cast<float *>(d.p[5]);
  auto input = [&](const TokenRec &r, int t, int ch, float bias) {   // input of token t (may lie before the portion)
    if (t >= r.q0) return __ldcg(in + (size_t)t * d.a[4] + ch) + bias;
    if (r.flags & 4) return 0.f;
    return __ldcg(state + ((size_t)r.slot * hist + (hist + t - r.q0)) * C + ch);
  };
  for (int i = threadIdx.x; i < B * nc; i += kConsumerThreads) {
    const int t = i / nc, ch = c0 + i - t * nc;
    const float bias = d.p[1] ? bf16_at(d.p[1], ch) : 0.f;
    const TokenRec r = rec[t];
    float v = d.p[3] ? bf16_at(d.p[3], ch) : 0.f;
    for (int j = 0; j < taps; ++j) v = fmaf(bf16_at(d.p[2], (size_t)ch * taps + j), input(r, t - hist + j, ch, bias), v);
    if (d.a[7] == 1) v = v * sigmoid_f(v);
    out[(size_t)t * d.a[6] + ch] = v;
  }
  consumer_sync();   // the carried inputs have been read
  for (int i = threadIdx.x; i < B * nc; i += kConsumerThreads) {
    const int t = i / nc, ch = c0 + i - t * nc;
    const TokenRec r = rec[t];
    if (!(r.flags & 2)) continue;
    const float bias = d.p[1] ? bf16_at(d.p[1], ch) : 0.f;
    // entry j takes the input `hist - 1 - j` tokens before the last one; when that is itself a carried input, it sits
    // at a higher index than j, so ascending order is safe in place
    for (int j = 0; j < hist; ++j) state[((size_t)r.slot * hist + j) * C + ch] = input(r, t - hist + 1 + j, ch, bias);
  }
}

// ---------------------------------------------------------------------------
// TASK_RGLRU: channels [c0, c1) of one block of the block-diagonal gates, all requests.
//   r = sigmoid(Ra u + ra), i = sigmoid(Ri u + ri), log a = -c r softplus(lambda), S = a S + sqrt(1 - a^2) i u,
//   out = scale * S * gelu_tanh(y)
// Gate products in 32-bit: a warp takes two channels (four weight rows) and eight tokens at a time.
// ---------------------------------------------------------------------------
template <int HYB, bool PAIR>
__device__ __forceinline__ void rglru_gates(const TaskDesc &d, const float *us, float *rs, float *is, int nt) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int bs = d.a[GL_BS], c0 = d.a[GL_C0], C = d.a[GL_C1] - c0, blk = d.a[GL_BLOCK];
  for (int it = warp; it * 2 < C; it += 8) {
    const int ca = c0 + it * 2, cb = min(ca + 1, d.a[GL_C1] - 1);
    const size_t ra = ((size_t)blk * bs + ca) * bs, rb = ((size_t)blk * bs + cb) * bs;
    for (int t8 = 0; t8 < nt; t8 += 8) {
      float acc[4][8];
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int u = 0; u < 8; ++u) acc[m][u] = 0.f;
      if (PAIR) {
        for (int k = 2 * lane; k < bs; k += 64) {
          uint32_t w[4];
          w[0] = __ldg(reinterpret_cast<const uint32_t *>(d.p[3] + 2 * (ra + k)));
          w[1] = __ldg(reinterpret_cast<const uint32_t *>(d.p[5] + 2 * (ra + k)));
          w[2] = __ldg(reinterpret_cast<const uint32_t *>(d.p[3] + 2 * (rb + k)));
          w[3] = __ldg(reinterpret_cast<const uint32_t *>(d.p[5] + 2 * (rb + k)));
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const float2 x = *reinterpret_cast<const float2 *>(us + (size_t)min(t8 + u, nt - 1) * bs + k);
#pragma unroll
            for (int m = 0; m < 4; ++m) acc[m][u] = fmaf(bf16_hi(w[m]), x.y, fmaf(bf16_lo(w[m]), x.x, acc[m][u]));
          }
        }
      } else {
        for (int k = lane; k < bs; k += 32) {
          const float w[4] = {bf16_at(d.p[3], ra + k), bf16_at(d.p[5], ra + k), bf16_at(d.p[3], rb + k), bf16_at(d.p[5], rb + k)};
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const float x = us[(size_t)min(t8 + u, nt - 1) * bs + k];
#pragma unroll
            for (int m = 0; m < 4; ++m) acc[m][u] = fmaf(w[m], x, acc[m][u]);
          }
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const float v = warp_sum(acc[m][u]);
          if (lane == u && t8 + u < nt) ((m & 1) ? is : rs)[(size_t)(t8 + u) * C + ((m < 2 ? ca : cb) - c0)] = v;
        }
    }
  }
}

template <int HYB>
__device__ __forceinline__ void run_rglru(const Ctx &c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  if (B <= 0) return;
  const int tid = threadIdx.x;
  const int bs = d.a[GL_BS], c0 = d.a[GL_C0], C = d.a[GL_C1] - c0, TG = d.a[GL_TG], blk = d.a[GL_BLOCK], width = d.a[GL_WIDTH];
  float *state = *reinterpret_cast<float *const *>(&d.a[GL_STATE]);
  T *outp = *reinterpret_cast<T *const *>(&d.a[GL_OUT]);
  const float oscale = __int_as_float(d.a[GL_OSCALE]), gate_c = __int_as_float(d.a[GL_GATE_C]);
  TokenRec *rec = reinterpret_cast<TokenRec *>(c.s.xtile);
  float *us = reinterpret_cast<float *>(c.s.xtile + kTokenMapBytes);   // [TG][bs]
  float *rs = us + (size_t)TG * bs;                                     // [TG][C]  gate r, then a
  float *is = rs + (size_t)TG * C;                                      // [TG][C]  gate i, then b, then S
  token_map(P, B, rec, reinterpret_cast<int *>(us));
  const int gch = blk * bs + c0;   // first channel of this task
  float carry = 0.f;               // state of channel tid between token groups
  for (int tb = 0; tb < B; tb += TG) {
    const int nt = min(TG, B - tb);
    for (int i = tid; i < nt * bs; i += kConsumerThreads) {
      const int t = i / bs, k = i - t * bs;
      us[i] = __ldcg(reinterpret_cast<const float *>(d.p[0]) + (size_t)(tb + t) * d.a[GL_LDU] + (size_t)blk * bs + k);
    }
    consumer_sync();
    if ((bs & 1) == 0) rglru_gates<HYB, true>(d, us, rs, is, nt);
    else rglru_gates<HYB, false>(d, us, rs, is, nt);
    consumer_sync();
    for (int i = tid; i < nt * C; i += kConsumerThreads) {
      const int t = i / C, ch = i - t * C, g = gch + ch;
      const float r = sigmoid_f(rs[i] + bf16_at(d.p[4], g)), gi = sigmoid_f(is[i] + bf16_at(d.p[6], g));
      const float la = -gate_c * r * softplus_f(bf16_at(d.p[7], g));
      float a = decay_exp(la), b = sqrtf(-expm1f(2.0f * la)) * gi * us[(size_t)t * bs + c0 + ch];
      const TokenRec &tr = rec[tb + t];
      if (tr.flags & 1) {   // the request's carried state enters here; nothing flows in from the previous token
        if (!(tr.flags & 4)) b = fmaf(a, __ldcg(state + (size_t)tr.slot * width + g), b);
        a = 0.f;
      }
      rs[i] = a;
      is[i] = b;
    }
    consumer_sync();
    if (tid < C) {
      float S = carry;
      for (int t = 0; t < nt; ++t) {
        S = fmaf(rs[(size_t)t * C + tid], S, is[(size_t)t * C + tid]);
        is[(size_t)t * C + tid] = S;
      }
      carry = S;
    }
    consumer_sync();
    for (int i = tid; i < nt * C; i += kConsumerThreads) {
      const int t = i / C, ch = i - t * C, g = gch + ch;
      const float S = is[i];
      const TokenRec &tr = rec[tb + t];
      if (tr.flags & 2) state[(size_t)tr.slot * width + g] = S;
      const float y = gelu_tanh_f(__ldcg(reinterpret_cast<const float *>(d.p[1]) + (size_t)(tb + t) * d.a[GL_LDP] + d.a[GL_YOFF] + g) +
                                  bf16_at(d.p[2], g));
      store_elt(outp + (size_t)(tb + t) * d.a[GL_LDO] + d.a[GL_OCOL] + g, S * y * oscale);
    }
    consumer_sync();
  }
}

// ---------------------------------------------------------------------------
// TASK_MLSTM: (request, head, range of value columns).  Matrix memory S [dim, columns] in registers, 4 columns x RPT
// rows per thread; the columns of the task are walked in sub-blocks of 4 CQ.  Per token
//   m' = max(f + m, i), S = exp(f + m - m') S + exp(i - m') k v^T, n likewise, o = S^T q / (max(|n q|, exp(-m')) + 1e-6)
// Every task keeps its own copy of (n, m), so that tasks of one head share nothing while they run.  The normalised and
// gated output needs the whole head: the last task of the (request, head) to finish writes it.
// ---------------------------------------------------------------------------
template <int HYB, int RPT>
__device__ __forceinline__ void mlstm_body(const Ctx &c, const TaskDesc &d, const SeqView &sv, int CQ) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = d.a[ML_H], h = d.a[ML_HEAD], dim = d.a[ML_DIM], vdim = d.a[ML_VDIM], vdimp = d.a[ML_VDIMP], TC = d.a[ML_TC];
  const int vc = 4 * CQ, RG = kConsumerThreads / CQ, qd = tid % CQ, rg = tid / CQ;
  const float *proj = reinterpret_cast<const float *>(d.p[0]) + (size_t)sv.q0 * d.a[ML_LDP];
  const int ldp = d.a[ML_LDP];
  const bool fresh = sv.pos0 == 0;
  float *nm = reinterpret_cast<float *>(d.p[5]) + ((size_t)(sv.slot * H + h) * d.a[ML_NCHUNK] + d.a[ML_CHUNK]) * (dim + 1);
  float *Sg = reinterpret_cast<float *>(d.p[4]) + (size_t)(sv.slot * H + h) * dim * vdimp;
  float *raw = reinterpret_cast<float *>(d.p[6]) + (size_t)sv.q0 * d.a[ML_LDR] + (size_t)h * vdim;
  // shared memory
  float *dec = reinterpret_cast<float *>(c.s.xtile);   // [64] exp(f + m - m')
  float *inp = dec + kMaxLinearTokens;                 // [64] exp(i - m')
  float *den = inp + kMaxLinearTokens;                 // [64] exp(-m'), then the denominator
  float *nred = den + kMaxLinearTokens;                // [TC][8]
  float *ks = nred + TC * 8;                           // [TC][dim] input-scaled keys
  float *qs = ks + (size_t)TC * dim;                   // [TC][dim]
  float *vs = qs + (size_t)TC * dim;                   // [TC][vc]
  float *red = vs + (size_t)TC * vc;                   // [TC][8 warps][vc]
  const float cap = __int_as_float(d.a[ML_CAP]), qscale = __int_as_float(d.a[ML_QSCALE]);
  // gates of all tokens, then the running maximum (one thread: a handful of operations per token)
  for (int t = tid; t < sv.nq; t += kConsumerThreads) {
    const float ip = __ldcg(proj + (size_t)t * ldp + d.a[ML_IOFF] + h) + bf16_at(d.p[1], h);
    const float fp = __ldcg(proj + (size_t)t * ldp + d.a[ML_FOFF] + h) + bf16_at(d.p[2], h);
    inp[t] = cap * tanhf(ip / cap);
    dec[t] = -softplus_f(-cap * tanhf(fp / cap));
  }
  consumer_sync();
  if (tid == 0) {
    float m = fresh ? 0.f : __ldcg(nm + dim);
    for (int t = 0; t < sv.nq; ++t) {
      const float fm = dec[t] + m, i = inp[t];
      m = fmaxf(fm, i);
      dec[t] = fm - m;
      inp[t] = i - m;
      den[t] = -m;
    }
    nm[dim] = m;
  }
  consumer_sync();
  for (int t = tid; t < sv.nq; t += kConsumerThreads) {
    dec[t] = decay_exp(dec[t]);
    inp[t] = expf(inp[t]);
    den[t] = expf(den[t]);
  }
  constexpr int NR = 4;   // rows of n per thread: dim <= 1024
  float n[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    n[i] = (!fresh && row < dim) ? __ldcg(nm + row) : 0.f;
  }
  for (int v0 = d.a[ML_V0]; v0 < d.a[ML_V1]; v0 += vc) {
    const bool col_ok = v0 + 4 * qd < vdimp && v0 + 4 * qd < d.a[ML_V1];
    const bool first = v0 == d.a[ML_V0];
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int row = rg + i * RG;
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && col_ok && row < dim) S[i] = __ldcg(reinterpret_cast<const float4 *>(Sg + (size_t)row * vdimp + v0 + 4 * qd));
    }
    for (int tb = 0; tb < sv.nq; tb += TC) {
      const int nt = min(TC, sv.nq - tb);
      consumer_sync();   // gates are final / the previous trip's readers are done
      for (int i = tid; i < nt * dim; i += kConsumerThreads) {
        const int t = i / dim, r = i - t * dim;
        const float *pr = proj + (size_t)(tb + t) * ldp + h * dim + r;
        ks[i] = __ldcg(pr + d.a[ML_KOFF]) * inp[tb + t];
        qs[i] = __ldcg(pr + d.a[ML_QOFF]) * qscale;
      }
      for (int i = tid; i < nt * vc; i += kConsumerThreads) {
        const int t = i / vc, col = v0 + i - t * vc;
        vs[i] = col < vdim ? __ldcg(proj + (size_t)(tb + t) * ldp + d.a[ML_VOFF] + (size_t)h * vdim + col) : 0.f;
      }
      consumer_sync();
      for (int t = 0; t < nt; ++t) {
        const float a = dec[tb + t];
        const float4 v = *reinterpret_cast<const float4 *>(vs + t * vc + 4 * qd);
        const float *kt = ks + (size_t)t * dim, *qt = qs + (size_t)t * dim;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          const int row = rg + i * RG;
          if (row < dim) {
            const float k = kt[row], q = qt[row];
            S[i].x = fmaf(a, S[i].x, k * v.x); o.x = fmaf(q, S[i].x, o.x);
            S[i].y = fmaf(a, S[i].y, k * v.y); o.y = fmaf(q, S[i].y, o.y);
            S[i].z = fmaf(a, S[i].z, k * v.z); o.z = fmaf(q, S[i].z, o.z);
            S[i].w = fmaf(a, S[i].w, k * v.w); o.w = fmaf(q, S[i].w, o.w);
          }
        }
        for (int s = CQ; s < 32; s <<= 1) {
          o.x += __shfl_xor_sync(0xffffffffu, o.x, s);
          o.y += __shfl_xor_sync(0xffffffffu, o.y, s);
          o.z += __shfl_xor_sync(0xffffffffu, o.z, s);
          o.w += __shfl_xor_sync(0xffffffffu, o.w, s);
        }
        if (lane < CQ) *reinterpret_cast<float4 *>(red + (size_t)(t * 8 + warp) * vc + 4 * lane) = o;
        if (first) {
          float p = 0.f;
#pragma unroll
          for (int i = 0; i < NR; ++i) {
            const int row = tid + i * kConsumerThreads;
            if (row < dim) {
              n[i] = fmaf(a, n[i], kt[row]);
              p = fmaf(n[i], qt[row], p);
            }
          }
          p = warp_sum(p);
          if (lane == 0) nred[t * 8 + warp] = p;
        }
      }
      consumer_sync();
      if (first) {
        if (tid < nt) {
          float s = 0.f;
#pragma unroll
          for (int w = 0; w < 8; ++w) s += nred[tid * 8 + w];
          den[tb + tid] = fmaxf(fabsf(s), den[tb + tid]) + 1e-6f;
        }
        consumer_sync();
      }
      for (int i = tid; i < nt * vc; i += kConsumerThreads) {
        const int t = i / vc, j = i - t * vc;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += red[(size_t)(t * 8 + w) * vc + j];
        if (v0 + j < vdim && v0 + j < d.a[ML_V1]) __stcg(raw + (size_t)(tb + t) * d.a[ML_LDR] + v0 + j, s / den[tb + t]);
      }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int row = rg + i * RG;
      if (col_ok && row < dim) *reinterpret_cast<float4 *>(Sg + (size_t)row * vdimp + v0 + 4 * qd) = S[i];
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    if (row < dim) nm[row] = n[i];
  }
  // ---- output of the head
  consumer_sync();
  if (d.a[ML_NCHUNK] > 1) {
    if (tid == 0) {
      unsigned int *ticket = &P.attn_tickets[d.a[ML_TICKET]];
      unsigned int old;
      asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(old) : "l"(ticket) : "memory");
      const bool last = old + 1u == (unsigned)d.a[ML_NCHUNK];
      if (last) *reinterpret_cast<volatile unsigned int *>(ticket) = 0u;
      c.s.flags[1] = last ? 1 : 0;
    }
    consumer_sync();
    if (c.s.flags[1] == 0) return;
  }
  const float eps = __int_as_float(d.a[ML_EPS]);
  T *out = reinterpret_cast<T *>(d.p[7]) + (size_t)sv.q0 * d.a[ML_LDO] + (size_t)h * vdim;
  for (int t = warp; t < sv.nq; t += 8) {
    const float *rt = raw + (size_t)t * d.a[ML_LDR];
    float ss = 0.f;
    for (int j = lane; j < vdim; j += 32) { const float v = __ldcg(rt + j); ss += v * v; }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int j = lane; j < vdim; j += 32) {
      const float g = __ldcg(proj + (size_t)t * ldp + d.a[ML_GOFF] + (size_t)h * vdim + j);
      store_elt(out + (size_t)t * d.a[ML_LDO] + j, __ldcg(rt + j) * inv * bf16_at(d.p[3], (size_t)h * vdim + j) * sigmoid_f(g));
    }
  }
}

template <int HYB>
__device__ __forceinline__ void run_mlstm(const Ctx &c, const TaskDesc &d) {
  const SeqView sv = seq_view(c.P, d.a[ML_SLOT]);
  if (sv.nq <= 0) return;
  const int dim = d.a[ML_DIM];
  const int CQ = dim <= 256 ? 16 : (dim <= 512 ? 8 : 4);      // at most 16 rows per thread
  const int rpt = (dim * CQ + kConsumerThreads - 1) / kConsumerThreads;
  if (rpt <= 4) mlstm_body<HYB, 4>(c, d, sv, CQ);
  else if (rpt <= 8) mlstm_body<HYB, 8>(c, d, sv, CQ);
  else mlstm_body<HYB, 16>(c, d, sv, CQ);
}

// ---------------------------------------------------------------------------
// greedy choice over float32 logits
// ---------------------------------------------------------------------------
__device__ __forceinline__ void run_argmax_partial_f32(const Ctx &c, const TaskDesc &d) {
  const int B = active_tokens(c.P);
  const float *logits = reinterpret_cast<const float *>(d.p[0]);
  const int c0 = d.a[0], c1 = d.a[1], cid = d.a[2], ldl = d.a[3], ldp = d.a[4];
  for (int b = 0; b < B; ++b) {
    float v = -INFINITY;
    long long i = 0x7fffffffffffffffLL;
    for (int j = c0 + threadIdx.x; j < c1; j += kConsumerThreads) argmax_merge(v, i, __ldcg(&logits[(size_t)b * ldl + j]), (long long)j);
    block_argmax(c, v, i);
    if (threadIdx.x == 0) {
      reinterpret_cast<float *>(d.p[1])[(size_t)b * ldp + cid] = v;
      reinterpret_cast<long long *>(d.p[2])[(size_t)b * ldp + cid] = i;
    }
  }
}
__device__ __forceinline__ void run_argmax_reduce_f32(const Ctx &c, const TaskDesc &d) {
  const int B = active_tokens(c.P);
  const float *pv = reinterpret_cast<const float *>(d.p[0]);
  const long long *pi = reinterpret_cast<const long long *>(d.p[1]);
  const int n = d.a[0], ldp = d.a[1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int b = warp; b < B; b += 8) {
    float v = -INFINITY;
    long long i = 0x7fffffffffffffffLL;
    for (int j = lane; j < n; j += 32) argmax_merge(v, i, __ldcg(&pv[(size_t)b * ldp + j]), __ldcg(&pi[(size_t)b * ldp + j]));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
      const long long i2 = __shfl_xor_sync(0xffffffffu, i, o);
      argmax_merge(v, i, v2, i2);
    }
    if (lane == 0) reinterpret_cast<long long *>(d.p[2])[b] = i;
  }
}

template <int HYB>
__device__ __forceinline__ void run_hybrid_task(const Ctx &c, const TaskDesc &d) {
  switch (d.type) {
    case TASK_BATCH: {
      Ctx cc = c;
      cc.tmem_base = 0u;
      run_batch(cc);
      break;
    }
    case TASK_EMBED_F32: run_embed_f32(c, d); break;
    case TASK_RESIDUAL_NORM: run_residual_norm<HYB>(c, d); break;
    case TASK_LINEAR_F32: if (HYB == HYB_F32) run_linear_f32(c, d); break;
    case TASK_QKV_APPEND: run_qkv_append<HYB>(c, d); break;
    case TASK_EXT_ATTENTION: run_ext_attention<HYB>(c, d); break;
    case TASK_SHORT_CONV: run_short_conv(c, d); break;
    case TASK_RGLRU: run_rglru<HYB>(c, d); break;
    case TASK_MLSTM: run_mlstm<HYB>(c, d); break;
    case TASK_ARGMAX_PARTIAL: run_argmax_partial_f32(c, d); break;
    case TASK_ARGMAX_REDUCE: run_argmax_reduce_f32(c, d); break;
    case TASK_SAMPLING_PARTIAL: run_sampling_partial<float>(c, d); break;
    case TASK_SAMPLING_REDUCE: run_sampling_reduce(c, d); break;
    default: break;
  }
}

}  // namespace mpk
