// Task bodies of hybrid graphs: decoders whose layers mix softmax attention with recurrent state.
//
//   float32 residual stream      TASK_EMBED_F32, TASK_RESIDUAL_NORM
//   attention                    TASK_QKV_APPEND (norms, rotation, cache rows), TASK_LATENT_APPEND (latent rows that serve
//                                as keys and values), TASK_EXT_ATTENTION (any head size, score scale, soft cap, sinks, sliding
//                                window, distance bias), TASK_DIFF_COMBINE (differential attention)
//   activations                  TASK_POLY_NORM (beside those in the epilogues of linears)
//   recurrences                  TASK_SHORT_CONV, TASK_RGLRU (gated diagonal), TASK_SELECTIVE_SCAN (diagonal, input-dependent steps),
//                                TASK_MLSTM and TASK_GLA (matrix memories)
//   experts                      TASK_MOE_ROUTING, TASK_MOE_GEMM (megakernel.cuh); their sum is part of TASK_RESIDUAL_NORM
//   32-bit graphs                TASK_LINEAR_F32, TASK_MOE_GEMM_F32
//
// A recurrent layer keeps its state in float32 tensors indexed by the request's state slot, which the batching task
// hands out at admission; a request whose batch portion starts at position 0 starts from a zero state, so slots are
// reused without being cleared.  Every body walks the tokens of the batch by request (qo_indptr), whatever mixture of
// prompt portions and single decoded tokens it holds.
//
// HYB = HYB_BF16: matrix operands, the KV cache and the operands handed to projections are bf16, everything else is
// float32.  HYB = HYB_F32: those are float32 as well.
//
// The bodies are functions of their own (__noinline__): inlined side by side into the task switch they share one register
// allocation, and every variant added makes the linear loop and the others spill.  They take the context by value: a
// reference would keep it in local memory for the whole kernel.
#pragma once
#include <stddef.h>

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
// A 64-bit value (pointer) kept in two of a descriptor's integers.
__device__ __forceinline__ uint64_t wide_arg(const TaskDesc &d, int i) { return *reinterpret_cast<const uint64_t *>(&d.a[i]); }
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Phase stamp i (0..3) of a task's profiler record.
__device__ __forceinline__ void stamp(const KernelParams &P, int task, int i) {
  if (threadIdx.x == 0 && P.profiler != nullptr && (uint64_t)(task + 1) * 8 <= P.profiler_entries)
    P.profiler[(size_t)task * 8 + 4 + i] = globaltimer_ns();
}
__device__ __forceinline__ void stamp(const Ctx &c, int task, int i) { stamp(c.P, task, i); }
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

// Four bf16 values as floats (8-byte aligned).
__device__ __forceinline__ float4 bf16x4_at(uint64_t base, int i) {
  const uint2 v = __ldg(reinterpret_cast<const uint2 *>(base + 2ull * i));
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ void store_elt4(__nv_bfloat16 *p, float4 v) {
  *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ void store_elt4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }

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

// The request batch token t belongs to: as many requests end at or before the token.  Called by a whole warp.
__device__ __forceinline__ int request_of(const KernelParams &P, int t) {
  const int lane = threadIdx.x & 31, mbr = P.max_num_batched_requests;
  int k = 0;
  for (int b = 0; b < mbr; b += 32) {
    const bool before = b + lane < mbr && __ldcg(&P.meta.qo_indptr[b + lane + 1]) <= t;
    const int n = __popc(__ballot_sync(0xffffffffu, before));
    k += n;
    if (n < 32) break;
  }
  return k;
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
  const float factor = __int_as_float(d.a[E_LDI2]);
  for (int t = t0; t < t1; ++t) {
    const long long id = __ldcg(reinterpret_cast<const long long *>(&ids[t]));
    const bool in_table = id >= 0 && id < (long long)d.a[E_AUX];   // ids outside the table read as a zero row
    for (int j = threadIdx.x; j < width; j += kConsumerThreads)
      out[(size_t)t * d.a[E_LDO] + j] = in_table ? bf16_at(d.p[1], (size_t)id * d.a[E_LDI] + j) * factor : 0.f;
  }
}

// Rows with further terms: the bigram of the token and the one before it, and sines and cosines of the position.  Angles are turns in
// units of 2^-64, position times frequency, so that their reduction is exact.
static __device__ __noinline__ void run_embed_sum(const Ctx c, const TaskDesc &d) {
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  const int t1 = min(d.a[E_T1], B), width = d.a[E_WIDTH];
  const long long *ids = reinterpret_cast<const long long *>(d.p[0]);
  const long long *freq = reinterpret_cast<const long long *>(d.p[4]);
  const float factor = __int_as_float(d.a[E_LDI2]);
  const bool vec = ((width | d.a[E_LDI] | d.a[E_LDB] | d.a[E_LDO] | d.a[E_LDC]) & 3) == 0 && ((d.p[1] | d.p[3]) & 7) == 0 && ((d.p[2] | d.p[5]) & 15) == 0;
  for (int t = d.a[E_T0]; t < t1; ++t) {
    const long long id = __ldcg(ids + t);
    const bool in_table = id >= 0 && id < (long long)d.a[E_AUX];
    const int k = request_of(P, t);
    const SeqView s = seq_view(P, k);
    const int pos = s.pos0 + t - s.q0;
    unsigned long long pair = (unsigned)d.a[E_BUCKETS];
    if (d.p[3] && pos > 0) {
      const int row = P.meta_static ? k : __ldcg(&P.meta.request_ids[k]);
      const unsigned long long prev = t > s.q0 ? __ldcg(ids + t - 1) : __ldcg(reinterpret_cast<const long long *>(P.meta.tokens) + (size_t)row * P.max_seq_length + pos - 1);
      pair = (prev * wide_arg(d, E_PREV) + (unsigned long long)id * wide_arg(d, E_CUR)) % pair;
    }
    float *out = reinterpret_cast<float *>(d.p[2]) + (size_t)t * d.a[E_LDO], *copy = reinterpret_cast<float *>(d.p[5]) + (size_t)t * d.a[E_LDC];
    const uint64_t row1 = d.p[1] + 2ull * (size_t)id * d.a[E_LDI], row2 = d.p[3] + 2ull * (size_t)pair * d.a[E_LDB];
    auto angle = [&](int i) {   // of columns 2 i and 2 i + 1, in half turns
      return (float)(int)((unsigned long long)pos * (unsigned long long)__ldg(freq + i) >> 32) * (1.0f / 2147483648.0f);
    };
    if (vec) {
      constexpr int NV = 4;   // 4096 columns at a time
      for (int j0 = threadIdx.x * 4; j0 < width; j0 += NV * kConsumerThreads * 4) {
        float4 a[NV], b[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int j = j0 + i * kConsumerThreads * 4;
          a[i] = j < width && in_table ? bf16x4_at(row1, j) : make_float4(0.f, 0.f, 0.f, 0.f);
          b[i] = j < width && d.p[3] ? bf16x4_at(row2, j) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int j = j0 + i * kConsumerThreads * 4;
          if (j >= width) break;
          float4 v = make_float4(fmaf(a[i].x, factor, b[i].x), fmaf(a[i].y, factor, b[i].y), fmaf(a[i].z, factor, b[i].z), fmaf(a[i].w, factor, b[i].w));
          if (freq) {
            float s0, c0, s1, c1;
            sincospif(angle(j >> 1), &s0, &c0);
            sincospif(angle((j >> 1) + 1), &s1, &c1);
            v.x += s0; v.y += c0; v.z += s1; v.w += c1;
          }
          *reinterpret_cast<float4 *>(out + j) = v;
          if (d.p[5]) *reinterpret_cast<float4 *>(copy + j) = v;
        }
      }
      continue;
    }
    for (int j = threadIdx.x; j < width; j += kConsumerThreads) {
      float v = in_table ? bf16_at(row1, j) * factor : 0.f;
      if (d.p[3]) v += bf16_at(row2, j);
      if (freq) v += (j & 1) ? cospif(angle(j >> 1)) : sinpif(angle(j >> 1));
      out[j] = v;
      if (d.p[5]) copy[j] = v;
    }
  }
}

// What joins the stream beside the sublayer output y (pointers are null where a layer has no such term).
struct NormTerms {
  const float *add, *experts, *ew, *gate;   // added stream, expert outputs and their weights, logit whose sigmoid scales y
  uint64_t row, bias;                       // row added to every token, bias of the output norm
  int slots;
  float factor;                             // of y's norm
  float *results;                           // this token's row of the earlier results, or null: their weighted sum becomes the stream
};
__device__ __forceinline__ NormTerms norm_terms(const TaskDesc &d, int t) {
  NormTerms n;
  n.slots = d.a[RN_SLOTS];
  n.factor = __int_as_float(d.a[RN_POST]);
  n.add = reinterpret_cast<const float *>(wide_arg(d, RN_ADD));
  n.experts = reinterpret_cast<const float *>(wide_arg(d, RN_EXP));
  n.ew = reinterpret_cast<const float *>(wide_arg(d, RN_EW));
  n.gate = reinterpret_cast<const float *>(wide_arg(d, RN_GATE));
  if (n.add) n.add += (size_t)t * d.a[RN_LDADD];
  if (n.experts) n.experts += (size_t)t * n.slots * d.a[2];
  if (n.ew) n.ew += (size_t)t * d.a[RN_LDEW];
  if (n.gate) n.gate += (size_t)t * d.a[RN_LDGATE];
  n.row = wide_arg(d, RN_ROW);
  n.bias = wide_arg(d, RN_BIAS);
  n.results = reinterpret_cast<float *>(d.p[6]);
  if (n.results) n.results += (size_t)t * d.a[2];
  return n;
}

// x += the given terms, then out = norm(x): one token row at a time.  VEC consecutive elements per thread and step; the row
// stays in shared memory between the passes (every element is touched by one thread only).
template <int HYB, int VEC>
__device__ __forceinline__ void residual_norm_rows(const Ctx &c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const int B = active_tokens(c.P);
  const int t0 = d.a[0], t1 = min(d.a[1], B), W = d.a[2];
  const float eps = __int_as_float(d.a[6]);
  const float off = (d.a[7] & 2) ? 1.0f : 0.0f;
  const bool layer_norm = (d.a[7] & 4) != 0;
  const bool has_y = d.p[1] != 0, has_post = d.p[2] != 0, has_out = d.p[3] != 0, has_copy = !has_out && d.p[4] != 0;
  float *row = reinterpret_cast<float *>(c.s.xtile);
  for (int t = t0; t < t1; ++t) {
    float *x = reinterpret_cast<float *>(d.p[0]) + (size_t)t * d.a[3];
    float *xo = reinterpret_cast<float *>(d.p[5]) + (size_t)t * d.a[8];
    const float *y = reinterpret_cast<const float *>(d.p[1]) + (size_t)t * d.a[4];
    T *out = reinterpret_cast<T *>(d.p[4]) + (size_t)t * d.a[5];
    const NormTerms nt = norm_terms(d, t);
    const bool moved = has_y || nt.add || nt.experts || nt.row;
    float inv = nt.gate ? sigmoid_f(__ldcg(nt.gate)) : 1.f;
    if (has_post && nt.slots > 0) {   // the experts' sum is part of what is normed
      float ss = 0.f;
      for (int j = threadIdx.x; j < W; j += kConsumerThreads) {
        float v = has_y ? __ldcg(y + j) : 0.f;
        for (int k = 0; k < nt.slots; ++k) v = fmaf(__ldcg(nt.ew + k), __ldcg(nt.experts + (size_t)k * W + j), v);
        row[j] = v;
        ss += v * v;
      }
      inv = nt.factor / sqrtf(block_sum(ss, c.s.red) / (float)W + eps);   // (its barrier: the row is complete)
    } else if (has_y && has_post) {
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
      inv = nt.factor / sqrtf(block_sum(ss, c.s.red) / (float)W + eps);
    }
    float ss = 0.f, sum = 0.f;
    for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC) {
      float xv[VEC], yv[VEC];
      if (VEC == 4) {
        *reinterpret_cast<float4 *>(xv) = __ldcg(reinterpret_cast<const float4 *>(x + j));
        if (has_y || has_post) *reinterpret_cast<float4 *>(yv) = has_post ? *reinterpret_cast<const float4 *>(row + j)
                                                              : __ldcg(reinterpret_cast<const float4 *>(y + j));
      } else {
        xv[0] = __ldcg(x + j);
        if (has_y || has_post) yv[0] = has_post ? row[j] : __ldcg(y + j);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (has_y || has_post) xv[e] += has_post ? yv[e] * inv * (off + bf16_at(d.p[2], j + e)) : yv[e] * inv;
        for (int k = 0; k < (has_post ? 0 : nt.slots); ++k) xv[e] = fmaf(__ldcg(nt.ew + k), __ldcg(nt.experts + (size_t)k * W + j + e), xv[e]);
        if (nt.add) xv[e] += __ldcg(nt.add + j + e);
        if (nt.row) xv[e] += bf16_at(nt.row, j + e);
        if (nt.results) {
          const int last = d.a[RN_TERMS] - 1;
          nt.results[(size_t)last * d.a[RN_HSTRIDE] + j + e] = xv[e];
          xv[e] *= bf16_at(d.p[7], last);
          for (int k = 0; k < last; ++k) xv[e] = fmaf(bf16_at(d.p[7], k), __ldcg(nt.results + (size_t)k * d.a[RN_HSTRIDE] + j + e), xv[e]);
        }
        ss += xv[e] * xv[e];
        sum += xv[e];
        row[j + e] = xv[e];
        if (moved) xo[j + e] = xv[e];
        if (has_copy) store_elt(out + j + e, xv[e]);
      }
    }
    if (has_out) {
      float mean = 0.f;
      if (layer_norm) {   // the variance from deviations, not as a difference of two large sums
        mean = block_sum(sum, c.s.red + 16) / (float)W;
        ss = 0.f;
        for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC)
#pragma unroll
          for (int e = 0; e < VEC; ++e) { const float v = row[j + e] - mean; ss += v * v; }
      }
      const float inv2 = 1.0f / sqrtf(block_sum(ss, c.s.red + 8) / (float)W + eps);
      for (int j = threadIdx.x * VEC; j < W; j += kConsumerThreads * VEC) {
#pragma unroll
        for (int e = 0; e < VEC; ++e)
          store_elt(out + j + e, (row[j + e] - mean) * inv2 * (off + bf16_at(d.p[3], j + e)) + (nt.bias ? bf16_at(nt.bias, j + e) : 0.f));
      }
    }
    consumer_sync();   // the reduction slots are used again by the next row
  }
}
// The same for aligned rows of at most 4096 columns: row, sublayer output and both weights sit in registers, every load of
// a row is in flight before the first reduction.
template <int HYB>
__device__ __forceinline__ void residual_norm_wide(const Ctx &c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  constexpr int NV = 4;
  const int B = active_tokens(c.P);
  const int t0 = d.a[0], t1 = min(d.a[1], B), W = d.a[2], tid = threadIdx.x;
  const float eps = __int_as_float(d.a[6]);
  const float off = (d.a[7] & 2) ? 1.0f : 0.0f;
  const bool layer_norm = (d.a[7] & 4) != 0;
  const bool has_y = d.p[1] != 0, has_post = d.p[2] != 0, has_out = d.p[3] != 0;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  auto fma4 = [](float4 &a, float w, const float4 &v) {
    a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
  };
  for (int t = t0; t < t1; ++t) {
    float *x = reinterpret_cast<float *>(d.p[0]) + (size_t)t * d.a[3];
    float *xo = reinterpret_cast<float *>(d.p[5]) + (size_t)t * d.a[8];
    const float *y = reinterpret_cast<const float *>(d.p[1]) + (size_t)t * d.a[4];
    const NormTerms nt = norm_terms(d, t);
    float4 xv[NV], yv[NV], wp[NV], wn[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = (i * kConsumerThreads + tid) * 4;
      const bool in = j < W;
      yv[i] = in && has_y ? __ldcg(reinterpret_cast<const float4 *>(y + j)) : zero;
      xv[i] = in ? __ldcg(reinterpret_cast<const float4 *>(x + j)) : zero;
      wp[i] = in && has_post ? bf16x4_at(d.p[2], j) : zero;
      wn[i] = in && has_out ? bf16x4_at(d.p[3], j) : zero;
    }
    // the weighted sum over the experts: part of what is normed, or added to the stream
    auto add_experts = [&](float4 (&to)[NV]) {
      for (int k = 0; k < nt.slots; k += 2) {   // two experts' rows in flight
        float4 e[2][NV];
        float w[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          w[u] = k + u < nt.slots ? __ldcg(nt.ew + k + u) : 0.f;
#pragma unroll
          for (int i = 0; i < NV; ++i) {
            const int j = (i * kConsumerThreads + tid) * 4;
            e[u][i] = j < W && k + u < nt.slots ? __ldcg(reinterpret_cast<const float4 *>(nt.experts + (size_t)(k + u) * W + j)) : zero;
          }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < NV; ++i) fma4(to[i], w[u], e[u][i]);
      }
    };
    if (has_post) add_experts(yv);
    if (has_y || has_post) {
      float inv = nt.gate ? sigmoid_f(__ldcg(nt.gate)) : 1.f;
      if (has_post) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) ss += yv[i].x * yv[i].x + yv[i].y * yv[i].y + yv[i].z * yv[i].z + yv[i].w * yv[i].w;
        inv = nt.factor / sqrtf(block_sum(ss, c.s.red) / (float)W + eps);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const float ox = has_post ? off + wp[i].x : 1.f, oy = has_post ? off + wp[i].y : 1.f, oz = has_post ? off + wp[i].z : 1.f,
                    ow = has_post ? off + wp[i].w : 1.f;
        xv[i].x += yv[i].x * inv * ox; xv[i].y += yv[i].y * inv * oy;
        xv[i].z += yv[i].z * inv * oz; xv[i].w += yv[i].w * inv * ow;
      }
    }
    if (!has_post) add_experts(xv);
    if (nt.add || nt.row) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int j = (i * kConsumerThreads + tid) * 4;
        if (j >= W) break;
        if (nt.add) fma4(xv[i], 1.f, __ldcg(reinterpret_cast<const float4 *>(nt.add + j)));
        if (nt.row) fma4(xv[i], 1.f, bf16x4_at(nt.row, j));
      }
    }
    if (nt.results) {
      const int last = d.a[RN_TERMS] - 1;
      const float w = bf16_at(d.p[7], last);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int j = (i * kConsumerThreads + tid) * 4;
        if (j < W) *reinterpret_cast<float4 *>(nt.results + (size_t)last * d.a[RN_HSTRIDE] + j) = xv[i];
        xv[i].x *= w; xv[i].y *= w; xv[i].z *= w; xv[i].w *= w;
      }
      for (int k = 0; k < last; k += 2) {   // two earlier results in flight
        float4 e[2][NV];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < NV; ++i) {
            const int j = (i * kConsumerThreads + tid) * 4;
            e[u][i] = j < W && k + u < last ? __ldcg(reinterpret_cast<const float4 *>(nt.results + (size_t)(k + u) * d.a[RN_HSTRIDE] + j)) : zero;
          }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const float wk = k + u < last ? bf16_at(d.p[7], k + u) : 0.f;
#pragma unroll
          for (int i = 0; i < NV; ++i) fma4(xv[i], wk, e[u][i]);
        }
      }
    }
    if (has_y || nt.slots > 0 || nt.add || nt.row) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int j = (i * kConsumerThreads + tid) * 4;
        if (j < W) *reinterpret_cast<float4 *>(xo + j) = xv[i];
      }
    }
    if (!has_out && d.p[4] != 0) {   // the stream as it is
      T *out = reinterpret_cast<T *>(d.p[4]) + (size_t)t * d.a[5];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int j = (i * kConsumerThreads + tid) * 4;
        if (j < W) store_elt4(out + j, xv[i]);
      }
    }
    if (has_out) {
      if (layer_norm) {
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) sum += xv[i].x + xv[i].y + xv[i].z + xv[i].w;
        const float mean = block_sum(sum, c.s.red + 16) / (float)W;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if ((i * kConsumerThreads + tid) * 4 < W) { xv[i].x -= mean; xv[i].y -= mean; xv[i].z -= mean; xv[i].w -= mean; }
      }
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) ss += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
      const float inv = 1.0f / sqrtf(block_sum(ss, c.s.red + 8) / (float)W + eps);
      T *out = reinterpret_cast<T *>(d.p[4]) + (size_t)t * d.a[5];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int j = (i * kConsumerThreads + tid) * 4;
        if (j >= W) break;
        const float4 b = nt.bias ? bf16x4_at(nt.bias, j) : zero;
        store_elt4(out + j, make_float4(xv[i].x * inv * (off + wn[i].x) + b.x, xv[i].y * inv * (off + wn[i].y) + b.y,
                                        xv[i].z * inv * (off + wn[i].z) + b.z, xv[i].w * inv * (off + wn[i].w) + b.w));
      }
    }
    if (t + 1 < t1) consumer_sync();   // the reduction slots are used again by the next row
  }
}
template <int HYB>
__device__ __noinline__ void run_residual_norm(const Ctx c, const TaskDesc &d) {
  if (d.a[2] <= 4096 && ((d.a[2] | d.a[3] | d.a[4] | d.a[5] | d.a[8]) & 3) == 0 && ((d.p[0] | d.p[1] | d.p[4] | d.p[5]) & 15) == 0 &&
      ((d.p[2] | d.p[3] | wide_arg(d, RN_BIAS) | wide_arg(d, RN_ROW)) & 7) == 0 && (d.a[RN_LDADD] & 3) == 0 &&
      ((wide_arg(d, RN_ADD) | wide_arg(d, RN_EXP) | d.p[6]) & 15) == 0 && (d.a[RN_HSTRIDE] & 3) == 0) {
    residual_norm_wide<HYB>(c, d);
    return;
  }
  if (((d.a[2] | d.a[3] | d.a[4] | d.a[8]) & 3) == 0 && ((d.p[0] | d.p[1] | d.p[5]) & 15) == 0) residual_norm_rows<HYB, 4>(c, d);
  else residual_norm_rows<HYB, 1>(c, d);
}

// ---------------------------------------------------------------------------
// linear layers in 32-bit arithmetic: one warp per output column (one weight row, or a gate row and its up row), eight tokens
// at a time
// ---------------------------------------------------------------------------
// Products of weight row `wrow` with eight rows of xs [nt][K], starting at t8: acc[u] belongs to token min(t8 + u, nt - 1), its
// sum over the lanes is still to be taken.
__device__ __forceinline__ void dot8_f32(uint64_t w, size_t wrow, const float *xs, int K, int t8, int nt, float (&acc)[8]) {
  const float *xr[8];
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    acc[u] = 0.f;
    xr[u] = xs + (size_t)min(t8 + u, nt - 1) * K;
  }
  for (int k = threadIdx.x & 31; k < K; k += 32) {
    const float v = bf16_at(w, wrow + k);
#pragma unroll
    for (int u = 0; u < 8; ++u) acc[u] = fmaf(v, xr[u][k], acc[u]);
  }
}
// Output column n of `nt` tokens in xs; emit(t, value) is called by one lane.  W points to the weight's first row.
template <class F>
__device__ __forceinline__ void column_f32(uint64_t w, size_t ldw, const float *xs, int K, int n, int nt, int act, float cap, F emit) {
  const int lane = threadIdx.x & 31;
  const bool gated = act == ACT_GATED_SILU || act == ACT_GATED_GELU;
  const size_t row = gated ? (size_t)(n >> 1) * 4 + (n & 1) : n;
  for (int t8 = 0; t8 < nt; t8 += 8) {
    float acc[8], up[8];
    dot8_f32(w, row * ldw, xs, K, t8, nt, acc);
    if (gated) dot8_f32(w, (row + 2) * ldw, xs, K, t8, nt, up);
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      float v = warp_sum(acc[u]);
      if (gated) {
        const float g = warp_sum(up[u]);
        v = (act == ACT_GATED_SILU ? silu_exact_f(v) : gelu_tanh_f(v)) * g;
      } else if (act == ACT_RELU2) {
        v = fmaxf(v, 0.f);
        v *= v;
      } else if (act == ACT_SOFTCAP) {
        v = cap * tanhf(v / cap);
      } else if (act == ACT_SCALE) {
        v *= cap;
      }
      if (lane == u && t8 + u < nt) emit(t8 + u, v);
    }
  }
}
static __device__ __noinline__ void run_linear_f32(const Ctx c, const TaskDesc &d) {
  const int B = active_tokens(c.P);
  const int n0 = d.a[0], n1 = d.a[1], K = d.a[2], TT = d.a[7];
  const int tid = threadIdx.x, warp = tid >> 5;
  float *xs = reinterpret_cast<float *>(c.s.xtile);   // [TT][K]
  const float *x = reinterpret_cast<const float *>(d.p[1]);
  float *out = reinterpret_cast<float *>(d.p[2]);
  for (int tb = 0; tb < B; tb += TT) {
    const int nt = min(TT, B - tb);
    if (tb > 0) consumer_sync();
    for (int t = 0; t < nt; ++t)
      for (int k = tid; k < K; k += kConsumerThreads) xs[(size_t)t * K + k] = __ldcg(x + (size_t)(tb + t) * d.a[4] + k);
    consumer_sync();
    for (int n = n0 + warp; n < n1; n += 8)
      column_f32(d.p[0], d.a[3], xs, K, n, nt, d.a[6], __int_as_float(d.a[8]), [&](int t, float v) {
        if (d.p[4]) v *= sigmoid_f(__ldcg(reinterpret_cast<const float *>(d.p[4]) + (size_t)(tb + t) * d.a[9] + n));
        out[(size_t)(tb + t) * d.a[5] + n] = d.p[3] ? v + bf16_at(d.p[3], n) : v;
      });
  }
}
// Expert projections: the active experts one after the other, the tokens routed to each gathered in shared memory.
static __device__ __noinline__ void run_moe_gemm_f32(const Ctx c, const TaskDesc &d) {
  const int B = min(active_tokens(c.P), kMaxLinearTokens);
  const int n0 = d.a[0], n1 = d.a[1], K = d.a[2], TT = d.a[7], slots = d.a[9], ldr = d.a[10], E = d.a[11];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int *routing = reinterpret_cast<const int *>(d.p[4]), *active = reinterpret_cast<const int *>(d.p[5]);
  float *xs = reinterpret_cast<float *>(c.s.xtile);                      // [TT][K]
  int *list = reinterpret_cast<int *>(xs + (size_t)TT * K);              // [64] token * slots + slot
  const float *x = reinterpret_cast<const float *>(d.p[1]);
  float *out = reinterpret_cast<float *>(d.p[2]);
  const int n_act = min(__ldcg(&active[E]), E);
  for (int j = 0; j < n_act; ++j) {
    const int e = __ldcg(&active[j]);
    consumer_sync();   // the previous expert's readers are done
    if (warp == 0) {
      int cnt = 0;
      for (int b = 0; b < B; b += 32) {
        const int r = b + lane < B ? __ldcg(&routing[(size_t)e * ldr + b + lane]) : 0;
        const unsigned bal = __ballot_sync(0xffffffffu, r != 0);
        if (r != 0) list[cnt + __popc(bal & ((1u << lane) - 1u))] = (b + lane) * slots + r - 1;
        cnt += __popc(bal);
      }
      if (lane == 0) c.s.flags[8] = cnt;
    }
    consumer_sync();
    const int cnt = c.s.flags[8];
    for (int tb = 0; tb < cnt; tb += TT) {
      const int nt = min(TT, cnt - tb);
      if (tb > 0) consumer_sync();
      for (int t = 0; t < nt; ++t) {
        const int it = list[tb + t];
        const float *xr = x + (size_t)(d.a[8] ? it : it / slots) * d.a[4];
        for (int k = tid; k < K; k += kConsumerThreads) xs[(size_t)t * K + k] = __ldcg(xr + k);
      }
      consumer_sync();
      for (int n = n0 + warp; n < n1; n += 8)
        column_f32(d.p[0] + (uint64_t)e * d.a[12] * K * 2, K, xs, K, n, nt, d.a[6], 0.f,
                   [&](int t, float v) { out[(size_t)list[tb + t] * d.a[5] + n] = v; });
    }
  }
}

// ---------------------------------------------------------------------------
// TASK_QKV_APPEND: one warp per (token, head, map).  q: norm, rotate, store; k: norm, rotate, store in the cache page of its
// position together with the value row.  The norm is an RMS norm with a weight in front of the rotation, or a unit norm behind it.
// Two maps (differential attention): a cache row holds both maps' keys side by side; a query row, one per map, has zeros where
// the other map's key lies, so that attention over the whole row gives the map's own scores and a value row serves both.
// ---------------------------------------------------------------------------
template <int HYB>
__device__ __noinline__ void run_qkv_append(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hq = d.a[QA_HQ], hkv = d.a[QA_HKV], dim = d.a[QA_DIM], dimp = d.a[QA_DIMP], vdim = d.a[QA_VDIM], vdimp = d.a[QA_VDIMP];
  const int rot = d.a[QA_ROT], half = rot >> 1, page = d.a[QA_PAGE], maps = d.a[QA_MAPS];
  const bool pairs = d.a[QA_PAIRS] != 0;
  const float eps = __int_as_float(d.a[QA_EPS]);
  const int heads = (hq + (d.p[2] ? hkv : 0)) * maps, first = d.a[QA_T0], tasks = d.a[QA_T1];
  for (int item = first * 8 + warp; item < B * heads; item += tasks * 8) {
    const int t = item / heads, hm = item - t * heads, h = hm / maps, map = hm - h * maps;
    const SeqView s = seq_view(P, request_of(P, t));
    const int pos = s.pos0 + t - s.q0;
    const bool is_q = h < hq;
    const float *src = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[QA_LDP] +
                       (is_q ? d.a[QA_QOFF] + hm * dim : d.a[QA_KOFF] + (hm - hq * maps) * dim);
    const uint64_t norm = is_q ? d.p[6] : d.p[7];
    const size_t trow = (size_t)min(pos, d.a[QA_ROWS] - 1) * half;
    const float *cosT = reinterpret_cast<const float *>(d.p[4]) + trow, *sinT = reinterpret_cast<const float *>(d.p[5]) + trow;
    auto value = [&](int i) { return norm ? __ldcg(src + i) * bf16_at(norm, i) : __ldcg(src + i); };   // (the norm's factor comes last)
    auto rotated = [&](int i) {
      const float v = value(i);
      if (i >= rot) return v;
      const bool lower = pairs ? !(i & 1) : i < half;
      const int f = pairs ? i >> 1 : (lower ? i : i - half);
      const float w = value(pairs ? i ^ 1 : (lower ? i + half : i - half));
      return lower ? v * __ldg(cosT + f) - w * __ldg(sinT + f) : v * __ldg(cosT + f) + w * __ldg(sinT + f);
    };
    float inv = 1.f;
    if (norm || d.a[QA_NORM]) {
      float ss = 0.f;
      for (int i = lane; i < dim; i += 32) { const float v = norm ? __ldcg(src + i) : rotated(i); ss += v * v; }
      inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
    }
    T *dst;
    if (is_q) {
      dst = reinterpret_cast<T *>(d.p[1]) + (size_t)t * d.a[QA_LDQ] + (size_t)hm * dimp;
      if (maps > 1)
        for (int i = lane; i < dimp; i += 32)
          if (i / dim != map) store_elt(dst + i, 0.f);
    } else {
      const int pg = pos / page;
      const size_t cell = ((size_t)__ldcg(&P.meta.paged_kv_indices[s.kv0 + pg]) * page + (pos - pg * page)) * hkv + (h - hq);
      dst = reinterpret_cast<T *>(d.p[2]) + cell * dimp;
      T *vdst = reinterpret_cast<T *>(d.p[3]) + cell * vdimp;
      const float *vsrc = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[QA_LDP] + d.a[QA_VOFF] + (h - hq) * vdim;
      if (map == 0)
        for (int i = lane; i < vdim; i += 32) store_elt(vdst + i, __ldcg(vsrc + i));
    }
    dst += map * dim;
    for (int i = lane; i < dim; i += 32) store_elt(dst + i, rotated(i) * inv);
  }
}

// The norms span all heads and nothing is rotated: a block takes a token's queries, or its keys and values.
template <int HYB>
__device__ __noinline__ void run_qkv_append_whole(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  constexpr int NR = 16;   // a row's first 4096 columns, in registers
  const KernelParams &P = c.P;
  const int B = active_tokens(P), tid = threadIdx.x;
  const int hq = d.a[QA_HQ], hkv = d.a[QA_HKV], dim = d.a[QA_DIM], dimp = d.a[QA_DIMP], vdim = d.a[QA_VDIM], vdimp = d.a[QA_VDIMP], page = d.a[QA_PAGE];
  const int parts = d.p[2] ? 2 : 1;
  for (int item = d.a[QA_T0]; item < B * parts; item += d.a[QA_T1]) {
    const int t = item / parts;
    const bool is_q = item == t * parts;
    const SeqView s = seq_view(P, request_of(P, t));
    const int pos = s.pos0 + t - s.q0, n = (is_q ? hq : hkv) * dim;
    const float *row = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[QA_LDP];
    const float *src = row + (is_q ? d.a[QA_QOFF] : d.a[QA_KOFF]);
    const uint64_t norm = is_q ? d.p[6] : d.p[7];
    float x[NR], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int j = i * kConsumerThreads + tid;
      x[i] = j < n ? __ldcg(src + j) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) ss += x[i] * x[i];
    for (int j = NR * kConsumerThreads + tid; j < n; j += kConsumerThreads) { const float v = __ldcg(src + j); ss += v * v; }
    float inv = 1.0f / sqrtf(block_sum(ss, c.s.red) / (float)n + __int_as_float(d.a[QA_EPS]));
    if (is_q && d.a[QA_EVERY] > 0) inv *= 1.0f + __int_as_float(d.a[QA_TEMP]) * logf((float)((pos + 1) / d.a[QA_EVERY] + 1));
    T *dst = reinterpret_cast<T *>(d.p[1]) + (size_t)t * d.a[QA_LDQ], *vdst = nullptr;
    if (!is_q) {
      const int pg = pos / page;
      const size_t cell = ((size_t)__ldcg(&P.meta.paged_kv_indices[s.kv0 + pg]) * page + (pos - pg * page)) * hkv;
      dst = reinterpret_cast<T *>(d.p[2]) + cell * dimp;
      vdst = reinterpret_cast<T *>(d.p[3]) + cell * vdimp;
    }
    // the keys as projected are the values: they are in registers already
    const bool same = !is_q && d.a[QA_VOFF] == d.a[QA_KOFF] && vdim == dim;
    auto place = [&](int j, float v) {
      const int h = dim == dimp && (is_q || vdim == vdimp) ? 0 : j / dim;
      store_elt(dst + j + h * (dimp - dim), v * bf16_at(norm, j) * inv);
      if (same) store_elt(vdst + j + h * (vdimp - vdim), v);
    };
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int j = i * kConsumerThreads + tid;
      if (j < n) place(j, x[i]);
    }
    for (int j = NR * kConsumerThreads + tid; j < n; j += kConsumerThreads) place(j, __ldcg(src + j));
    if (!is_q && !same)
      for (int j = tid; j < hkv * vdim; j += kConsumerThreads) store_elt(vdst + j + j / vdim * (vdimp - vdim), __ldcg(row + d.a[QA_VOFF] + j));
    consumer_sync();   // the reduction slots are used again
  }
}

// ---------------------------------------------------------------------------
// TASK_LATENT_APPEND: one warp per (token, head) rotates the head's rotary query part into its columns of q (behind the
// `rank` latent columns, which a grouped linear writes); one more warp per token writes the token's cache row: the latent,
// RMS-normed, and the rotated key part all heads share.
// ---------------------------------------------------------------------------
template <int HYB>
__device__ __noinline__ void run_latent_append(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rank = d.a[LA_RANK], rot = d.a[LA_ROT], half = rot >> 1, dimp = d.a[LA_DIMP], page = d.a[LA_PAGE];
  const int H = rot > 0 ? d.a[LA_H] : 0;   // heads with something to rotate
  for (int item = d.a[LA_T0] * 8 + warp; item < B * (H + 1); item += d.a[LA_T1] * 8) {
    const int t = item / (H + 1), h = item - t * (H + 1);
    const SeqView s = seq_view(P, request_of(P, t));
    const int pos = s.pos0 + t - s.q0;
    const float *row = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[LA_LDP];
    const float *src;   // what is rotated
    T *dst;
    if (h < H) {
      src = row + d.a[LA_QOFF] + h * rot;
      dst = reinterpret_cast<T *>(d.p[2]) + (size_t)t * d.a[LA_LDQ] + (size_t)h * dimp + rank;
    } else {
      const float *lat = row + d.a[LA_KVOFF];
      const int pg = pos / page;
      T *cell = reinterpret_cast<T *>(d.p[3]) + ((size_t)__ldcg(&P.meta.paged_kv_indices[s.kv0 + pg]) * page + (pos - pg * page)) * dimp;
      float x[16], ss = 0.f;   // 512 columns in registers, all loads in flight
#pragma unroll
      for (int u = 0; u < 16; ++u) x[u] = u * 32 + lane < rank ? __ldcg(lat + u * 32 + lane) : 0.f;
#pragma unroll
      for (int u = 0; u < 16; ++u) ss += x[u] * x[u];
      for (int i = 512 + lane; i < rank; i += 32) { const float v = __ldcg(lat + i); ss += v * v; }
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)rank + __int_as_float(d.a[LA_EPS]));
#pragma unroll
      for (int u = 0; u < 16; ++u)
        if (u * 32 + lane < rank) store_elt(cell + u * 32 + lane, x[u] * inv * bf16_at(d.p[1], u * 32 + lane));
      for (int i = 512 + lane; i < rank; i += 32) store_elt(cell + i, __ldcg(lat + i) * inv * bf16_at(d.p[1], i));
      src = lat + rank;
      dst = cell + rank;
    }
    const size_t trow = (size_t)min(pos, d.a[LA_ROWS] - 1) * half;
    const float *cosT = reinterpret_cast<const float *>(d.p[4]) + trow, *sinT = reinterpret_cast<const float *>(d.p[5]) + trow;
    for (int i = lane; i < half; i += 32) {
      const float u = __ldcg(src + i), v = __ldcg(src + i + half), cs = __ldg(cosT + i), sn = __ldg(sinT + i);
      store_elt(dst + i, u * cs - v * sn);
      store_elt(dst + i + half, v * cs + u * sn);
    }
  }
}

// ---------------------------------------------------------------------------
// TASK_EXT_ATTENTION: (request, kv head, chunk of the keys).  The M rows of a task are the (token, query head of the
// group) pairs, row r = token r / G, head r % G.  Chunks are merged by the last task of the (request, kv head) to
// arrive, or by a layer of TASK_ATTN_MERGE.  Scores live in base 2 (bf16) or base e (float32): exp_dom undoes the same base everywhere.
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

// Logit of the sink that joins head h's denominator, in the domain's base.
template <int HYB>
__device__ __forceinline__ float sink_logit(const TaskDesc &d, int h) {
  return d.p[4] ? bf16_at(d.p[4], h) * (HYB == HYB_F32 ? 1.0f : 1.4426950408889634f) : 0.f;
}
// What a distance takes off a score, in the domain's base: r1 ln(1 + r2 distance).
template <int HYB>
__device__ __forceinline__ float distance_bias(float r1, float r2, int distance) {
  const float x = r2 * (float)max(distance, 0);
  return r1 * (HYB == HYB_F32 ? log1pf(x) : __log2f(1.0f + x));
}
// Keys of a request in the order the tasks walk them.  Without a window: positions 0, 1, ....  With one, positions that no token
// of the portion sees are left out: first `kept` positions (a multiple of eight that covers the ones kept for good), then
// everything from `shift` positions further on (a multiple of eight too, so that eight keys stay in one page).
struct AttnKeys {
  int kept, shift, len;   // len: keys in this order
  __device__ __forceinline__ int pos(int i) const { return i < kept ? i : i + shift; }
};
__device__ __forceinline__ AttnKeys attn_keys(const TaskDesc &d, const SeqView &sv) {
  AttnKeys k;
  const int window = d.a[XA_WINDOW];
  const int first = window > 0 ? max(0, sv.pos0 - window + 1) & ~7 : 0;
  k.kept = min((d.a[XA_KEEP] + 7) & ~7, first);
  k.shift = first - k.kept;
  k.len = sv.pos0 + sv.nq - k.shift;
  return k;
}
struct AttnOut {   // where a task's rows go, and the keys
  int hq, G, head, q0, ks, chunk, n_act, vdim, ldo, ocol, srec, rec0;
  float oscale;
  bool sink, f32;
  AttnKeys keys;
  int window, keep;   // keys a position sees at most (very large without a window), first positions it sees all the same
  // Does the row at position p not see the key at position `key` <= p?
  __device__ __forceinline__ bool outside(int key, int p) const { return p - key >= window && key >= keep; }
};
// Element i of an output row that is float32 or of the activation type.
template <class T>
__device__ __forceinline__ void store_out(const TaskDesc &d, bool f32, size_t i, float v) {
  if (f32) reinterpret_cast<float *>(d.p[3])[i] = v;
  else store_elt(reinterpret_cast<T *>(d.p[3]) + i, v);
}
// Partial record of a row (max, sum, then the unnormalised columns) of this task's chunk; the chunks of a row lie side by side.
__device__ __forceinline__ float *attn_record(const KernelParams &P, const AttnOut &o, int r) {
  return P.attn_scratch + ((size_t)o.rec0 + (size_t)r * o.ks + o.chunk) * o.srec;
}
// How the NC tasks of a (request, kv head) share its work: over the tiles of RT query rows first and over the keys with what is
// left: a prompt portion has rows enough and needs no merge, a decoded token has one tile and all its tasks share the keys.
struct AttnSplit {
  int rows, tiles, parts, ks, per, n_act;   // rows, row tiles, row parts, key chunks at most, keys of a chunk, chunks with keys
};
__device__ __forceinline__ AttnSplit attn_split(const SeqView &sv, int len, int G, int NC, int RT) {
  AttnSplit a;
  a.rows = sv.nq * G;
  a.tiles = (a.rows + RT - 1) / RT;
  a.parts = min(NC, a.tiles);
  a.ks = min(NC / a.parts, 32);
  a.per = max(64, ((len + a.ks - 1) / a.ks + 63) & ~63);
  a.n_act = (len + a.per - 1) / a.per;
  return a;
}
// Row r with (max m, sum l); val(col) gives the unnormalised output column.  Called by one warp.
template <int HYB, class F>
__device__ __forceinline__ void attn_emit_row(const Ctx &c, const TaskDesc &d, const AttnOut &o, int r, float m, float l, F val) {
  typedef typename HybElt<HYB>::T T;
  const int lane = threadIdx.x & 31;
  const int tok = o.q0 + r / o.G, hq_idx = o.head * o.G + r % o.G;
  if (o.n_act == 1) {
    const float sk = o.sink ? sink_logit<HYB>(d, hq_idx) : 0.f;
    const float M = o.sink ? fmaxf(m, sk) : m;
    const float w = m == -INFINITY ? 0.f : exp_dom<HYB>(m - M);
    const float L = l * w + (o.sink ? exp_dom<HYB>(sk - M) : 0.f);
    const float f = L > 0.f ? w / L * o.oscale : 0.f;
    const size_t out = (size_t)tok * o.ldo + o.ocol + (size_t)hq_idx * o.vdim;
    for (int j0 = 0; j0 < o.vdim; j0 += 32) {   // (val may shuffle: the whole warp calls it)
      const float v = val(j0 + lane);
      if (j0 + lane < o.vdim) store_out<T>(d, o.f32, out + j0 + lane, v * f);
    }
  } else {
    float *rec = attn_record(c.P, o, r);
    if (lane == 0) {
      __stcg(rec, m);
      __stcg(rec + 1, l);
    }
    for (int j0 = 0; j0 < o.vdim; j0 += 32) {
      const float v = val(j0 + lane);
      if (j0 + lane < o.vdim) __stcg(rec + kXaRecHead + j0 + lane, v);
    }
  }
}

// Merge of the chunks' records by the last arriver (at most 32 chunks).
template <int HYB>
__device__ __noinline__ void attn_merge(const Ctx c, const TaskDesc &d, const AttnOut &o, int part, int row0, int row1) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  consumer_sync();
  if (threadIdx.x == 0) {
    unsigned int *ticket = &P.attn_tickets[d.a[XA_TICKET] + part];
    unsigned int old;
    asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(old) : "l"(ticket) : "memory");
    const bool last = old + 1u == (unsigned)o.n_act;
    if (last) *reinterpret_cast<volatile unsigned int *>(ticket) = 0u;
    c.s.flags[1] = last ? 1 : 0;
  }
  consumer_sync();
  if (c.s.flags[1] == 0) return;
  // an item is 32 output columns of a row; its chunks' records are fetched sixteen at a time
  const int cols = (o.vdim + 31) >> 5;
  for (int item = warp + row0 * cols; item < row1 * cols; item += 8) {
    const int r = item / cols, j = (item - r * cols) * 32 + lane;
    const int tok = o.q0 + r / o.G, hq_idx = o.head * o.G + r % o.G;
    const float *rec = P.attn_scratch + ((size_t)o.rec0 + (size_t)r * o.ks) * o.srec;
    const bool v = lane < o.n_act;
    const float m = v ? __ldcg(rec + (size_t)lane * o.srec) : -INFINITY;
    const float l = v ? __ldcg(rec + (size_t)lane * o.srec + 1) : 0.f;
    float x[16], x2[16];
#pragma unroll
    for (int u = 0; u < 16; ++u) x[u] = (u < o.n_act && j < o.vdim) ? __ldcg(rec + (size_t)u * o.srec + kXaRecHead + j) : 0.f;
    if (o.n_act > 16) {
#pragma unroll
      for (int u = 0; u < 16; ++u) x2[u] = (16 + u < o.n_act && j < o.vdim) ? __ldcg(rec + (size_t)(16 + u) * o.srec + kXaRecHead + j) : 0.f;
    }
    float M = warp_max(m);
    const float sk = o.sink ? sink_logit<HYB>(d, hq_idx) : 0.f;
    if (o.sink) M = fmaxf(M, sk);
    const float w = m == -INFINITY ? 0.f : exp_dom<HYB>(m - M);
    const float L = warp_sum(l * w) + (o.sink ? exp_dom<HYB>(sk - M) : 0.f);
    const float f = L > 0.f ? o.oscale / L : 0.f;
    float acc = 0.f;
#pragma unroll
    for (int u = 0; u < 16; ++u) acc = fmaf(__shfl_sync(0xffffffffu, w, u), x[u], acc);
    if (o.n_act > 16) {
#pragma unroll
      for (int u = 0; u < 16; ++u) acc = fmaf(__shfl_sync(0xffffffffu, w, 16 + u), x2[u], acc);
    }
    if (j < o.vdim)
      store_out<T>(d, o.f32, (size_t)tok * o.ldo + o.ocol + (size_t)hq_idx * o.vdim + j, acc * f);
  }
}

// What a warp's 16-row tile needs to know of its queries.
struct AttnRows {
  float scale, cap, cap2;
  int kend;         // end of the task's keys
  int p_lo, p_hi;   // positions of this lane's two rows
  int p_all;        // keys up to here are not ahead of any row of the tile
  int p_far;        // keys from here on are in the window of every row
  bool two;         // rows 8 .. 15 of the tile hold queries
  float r1[2], r2[2];   // distance bias of this lane's two rows
};
template <bool BIAS>
__device__ __forceinline__ AttnRows attn_rows(const TaskDesc &d, const SeqView &sv, const AttnOut &ao, int first, int n, int kend) {
  AttnRows w;
  w.scale = __int_as_float(d.a[XA_SCALE]);
  w.cap = __int_as_float(d.a[XA_CAP]);
  w.cap2 = w.cap > 0.f ? 2.0f * 1.4426950408889634f / w.cap : 0.f;
  w.kend = kend;
  const int r = first + ((threadIdx.x & 31) >> 2), G = ao.G;
  w.p_lo = sv.pos0 + r / G;
  w.p_hi = sv.pos0 + (r + 8) / G;
  w.p_all = sv.pos0 + first / G;
  w.p_far = sv.pos0 + (first + n - 1) / G - ao.window + 1;
  w.two = n > 8;
  if (BIAS) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = ao.head * G + (r + 8 * i) % G;
      w.r1[i] = bf16_at(d.p[5], h);
      w.r2[i] = bf16_at(d.p[6], h);
    }
  }
  return w;
}
// Eight keys (rows at kaddr / vaddr, this lane's ldmatrix addresses) against a 16-row query tile: scores, online softmax,
// P V.  The first is number key0 (below w.kend) of the request's keys and lies at position `at`.
template <int D, int ON, bool TWO, bool BIAS>
__device__ __forceinline__ void attn_octet(const AttnRows &w, const AttnOut &ao, const uint32_t (&qf)[TWO ? 1 : D / 16][2], uint32_t qa, uint32_t kaddr,
                                           uint32_t vaddr, int key0, int at, float (&m_run)[2], float (&l_run)[2], float (&o)[ON / 8][4]) {
  float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int kk = 0; kk < D / 32; ++kk) {
    uint32_t b[4];
    ldmatrix_x4(b, kaddr + kk * 64u);
    if (!TWO) {
      const uint32_t a0[4] = {qf[TWO ? 0 : 2 * kk][0], 0u, qf[TWO ? 0 : 2 * kk][1], 0u};
      const uint32_t a1[4] = {qf[TWO ? 0 : 2 * kk + 1][0], 0u, qf[TWO ? 0 : 2 * kk + 1][1], 0u};
      mma_bf16_16816(s, a0, b[0], b[1]);
      mma_bf16_16816(s2, a1, b[2], b[3]);
    } else {
      uint32_t a0[4], a1[4];
      ldmatrix_x4(a0, qa + kk * 64u);
      ldmatrix_x4(a1, qa + kk * 64u + 32u);
      mma_bf16_16816(s, a0, b[0], b[1]);
      mma_bf16_16816(s2, a1, b[2], b[3]);
    }
  }
  float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    if (e >= 2 && !(TWO && w.two)) { s[e] = -INFINITY; continue; }
    s[e] = attn_score<HYB_BF16>(s[e] + s2[e], w.scale, w.cap, w.cap2);
    if (BIAS) s[e] -= distance_bias<HYB_BF16>(w.r1[e >> 1], w.r2[e >> 1], (e < 2 ? w.p_lo : w.p_hi) - at - 2 * ((int)threadIdx.x & 3) - (e & 1));
  }
  if (at + 7 > w.p_all || key0 + 8 > w.kend || at < w.p_far) {
    const int off = 2 * (threadIdx.x & 3);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int o = off + (e & 1), p = e < 2 ? w.p_lo : w.p_hi;
      if (key0 + o >= w.kend || at + o > p || ao.outside(at + o, p)) s[e] = -INFINITY;
    }
  }
  mx[0] = fmaxf(s[0], s[1]);
  mx[1] = fmaxf(s[2], s[3]);
  float ms[2], corr[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
    const float mn = fmaxf(m_run[i], mx[i]);
    ms[i] = mn == -INFINITY ? 0.f : mn;
    corr[i] = exp2f(m_run[i] - ms[i]);
    m_run[i] = mn;
  }
  if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
    l_run[0] *= corr[0];
    l_run[1] *= corr[1];
#pragma unroll
    for (int i = 0; i < ON / 8; ++i) {
      o[i][0] *= corr[0]; o[i][1] *= corr[0];
      o[i][2] *= corr[1]; o[i][3] *= corr[1];
    }
  }
  float p[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    p[e] = exp2f(s[e] - ms[e >> 1]);
    l_run[e >> 1] += p[e];
  }
  const uint32_t h0 = pack_bf16(p[0], p[1]), h1 = pack_bf16(p[2], p[3]);
  const uint32_t r0 = pack_bf16(p[0] - bf16_lo(h0), p[1] - bf16_hi(h0)), r1 = pack_bf16(p[2] - bf16_lo(h1), p[3] - bf16_hi(h1));
  // value and remainder side by side in one k = 16 product: the V octet serves both halves
  const uint32_t pa[4] = {h0, h1, r0, r1};
#pragma unroll
  for (int vq = 0; vq < ON / 32; ++vq) {
    uint32_t b[4];
    ldmatrix_x4_trans(b, vaddr + vq * 64u);
#pragma unroll
    for (int i = 0; i < 4; ++i) mma_bf16_16816(o[4 * vq + i], pa, b[i], b[i]);
  }
}

// Rows [first, first + nrow) from the records [split][row of `stride`] of (max, sum, D columns) in shared memory.
template <int D>
__device__ __forceinline__ void attn_emit_splits(const Ctx &c, const TaskDesc &d, const AttnOut &ao, const float *comb, int stride, int WK,
                                                 int first, int nrow) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int r = warp; r < nrow; r += 8) {
    const float *cr = comb + (size_t)r * (D + 2);
    const size_t step = (size_t)stride * (D + 2);
    // lane w holds split w's weight
    const float mw = lane < WK ? cr[lane * step] : -INFINITY;
    const float M = warp_max(mw);
    const float wgt = mw == -INFINITY ? 0.f : exp2f(mw - M);
    const float L = warp_sum(lane < WK ? cr[lane * step + 1] * wgt : 0.f);
    attn_emit_row<HYB_BF16>(c, d, ao, first + r, M, L, [&](int j) {
      float v = 0.f;
      for (int w = 0; w < WK; ++w) v = fmaf(__shfl_sync(0xffffffffu, wgt, w), cr[w * step + 2 + min(j, D - 1)], v);
      return v;
    });
  }
}

// One tile of query rows (decoding, or a task's share of a prompt portion): every warp streams its own octets of keys, w,
// w + 8, ..., through its own ring -- no block barrier in the loop -- and the eight partial results are combined at the end.
template <int D, bool TWO, bool BIAS>
__device__ __noinline__ void ext_attention_stream(const Ctx c, const TaskDesc &d, const SeqView sv, const AttnOut &ao, int k0, int k1,
                                                  int row0, int nrow, int task) {
  constexpr int PITCH = D * 2 + 16, STEP = 16 * PITCH, PIECES = D / 8, RSTEP = 32 / PIECES;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nstg = d.a[XA_STAGES], page = d.a[XA_PAGE];
  const AttnKeys keys = ao.keys;
  const int kend = min(k1, sv.pos0 + (row0 + nrow - 1) / ao.G + 1 - keys.shift);
  const int noct = kend > k0 ? (kend - k0 + 7) >> 3 : 0, mine = noct > warp ? (noct - warp + 7) >> 3 : 0;
  uint8_t *qs = c.s.xtile;                                                      // [16][PITCH]
  const uint32_t ring = smem_u32(qs) + (16 + warp * nstg * 16) * PITCH;         // this warp's stages: eight K rows, then eight V rows
  // (everything below is live through the key loop: 32-bit offsets in units of 16 bytes)
  const int piece = lane % PIECES, rl = lane / PIECES;
  const uint32_t krow = d.a[XA_HKV] * (d.a[XA_DIMP] >> 3), vrow = d.a[XA_HKV] * (d.a[XA_VDIMP] >> 3);   // between positions
  const bool kin = piece < (d.a[XA_DIMP] >> 3), vin = piece < (d.a[XA_VDIMP] >> 3);
  const uint4 *kg = reinterpret_cast<const uint4 *>(d.p[1]) + ao.head * (d.a[XA_DIMP] >> 3) + piece + rl * krow;
  const uint4 *vg = reinterpret_cast<const uint4 *>(d.p[2]) + ao.head * (d.a[XA_VDIMP] >> 3) + piece + rl * vrow;
  const int32_t *pages = c.P.meta.paged_kv_indices + sv.kv0;
  // page of the next octet to request, looked up one request ahead of its use
  int pos = k0 + warp * 8;
  int pid = pos < kend ? __ldcg(pages + keys.pos(pos) / page) : 0;
  auto issue = [&](int slot) {
    if (pos < kend) {
      const uint32_t row = (uint32_t)pid * page + keys.pos(pos) % page;
      const uint32_t dst = ring + slot * STEP + rl * PITCH + piece * 16;
      const int left = kend - pos - rl;   // rows of this lane's stride that exist
#pragma unroll
      for (int i = 0; i < 8 / RSTEP; ++i) {
        const uint32_t kd = dst + i * RSTEP * PITCH, vd = kd + 8 * PITCH;
        const bool in = i * RSTEP < left;
        if (in && kin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(kd), "l"(kg + (size_t)((row + i * RSTEP) * krow)) : "memory");
        else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(kd), "r"(0) : "memory");
        if (in && vin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(vd), "l"(vg + (size_t)((row + i * RSTEP) * vrow)) : "memory");
        else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(vd), "r"(0) : "memory");
      }
      pos += 64;
      pid = pos < kend ? __ldcg(pages + keys.pos(pos) / page) : 0;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (int i = 0; i < nstg - 1; ++i) issue(i);
  {
    const uint8_t *qg = reinterpret_cast<const uint8_t *>(d.p[0]);
    const int G = ao.G, kp = d.a[XA_DIMP] >> 3;
    for (int i = tid; i < 16 * PIECES; i += kConsumerThreads) {
      const int r = i / PIECES, p = i % PIECES, row = row0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nrow && p < kp)
        v = __ldcg(reinterpret_cast<const uint4 *>(qg + ((size_t)(sv.q0 + row / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + row % G) * kp * 8) * 2) + p);
      *reinterpret_cast<uint4 *>(qs + r * PITCH + p * 16) = v;
    }
  }
  consumer_sync();
  stamp(c, task, 0);
  const AttnRows w = attn_rows<BIAS>(d, sv, ao, row0, nrow, kend);
  const uint32_t qa = smem_u32(qs) + (uint32_t)((lane & 15) * PITCH + (lane >> 4) * 16);
  uint32_t qf[TWO ? 1 : D / 16][2];   // rows 0 .. 7 only: two of a fragment's four registers
  if (!TWO) {
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk)
      ldmatrix_x2(qf[TWO ? 0 : kk], smem_u32(qs) + (uint32_t)((lane & 7) * PITCH + ((lane >> 3) & 1) * 16 + kk * 32));
  }
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const uint32_t lane_off = (uint32_t)((lane & 7) * PITCH + (lane >> 3) * 16);
  int slot = 0;
#pragma unroll 1
  for (int i = 0; i < mine; ++i) {
    if (nstg >= 4) asm volatile("cp.async.wait_group 2;" ::: "memory");
    else if (nstg == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();   // the octet has landed for every lane, and every lane is done with the slot refilled next
    issue(slot == 0 ? nstg - 1 : slot - 1);
    const uint32_t ka = ring + slot * STEP + lane_off;
    const int key0 = k0 + (warp + 8 * i) * 8;
    attn_octet<D, D, TWO, BIAS>(w, ao, qf, qa, ka, ka + 8 * PITCH, key0, keys.pos(key0), m_run, l_run, o);
    if (++slot == nstg) slot = 0;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  consumer_sync();   // the rings become the combine area
  stamp(c, task, 2);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
  }
  float *comb = reinterpret_cast<float *>(qs + 16 * PITCH);   // [8 warps][16 rows][D + 2]
  float *c0 = comb + (size_t)(warp * 16 + (lane >> 2)) * (D + 2), *c1 = c0 + 8 * (D + 2);
  if ((lane & 3) == 0) {
    c0[0] = m_run[0]; c0[1] = l_run[0];
    c1[0] = m_run[1]; c1[1] = l_run[1];
  }
#pragma unroll
  for (int i = 0; i < D / 8; ++i) {
    const int col = 2 + i * 8 + 2 * (lane & 3);
    *reinterpret_cast<float2 *>(c0 + col) = make_float2(o[i][0], o[i][1]);
    if (w.two) *reinterpret_cast<float2 *>(c1 + col) = make_float2(o[i][2], o[i][3]);
  }
  consumer_sync();
  attn_emit_splits<D>(c, d, ao, comb, 16, 8, row0, nrow);
}

// At most eight query rows (decoding): the transposed products, so that no half of an accumulator is idle.  Sixteen keys
// are the M rows of S^T = K Q^T and the reduction of O^T = V^T P^T; an 8 x 8 block of P turns from accumulator to operand
// layout with movmatrix.  Every warp streams its own sixteen-key steps, as two octets, through its ring of four octets.
__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}
template <int D, bool BIAS>
__device__ __noinline__ void ext_attention_decode(const Ctx c, const TaskDesc &d, const SeqView sv, const AttnOut &ao, int k0, int k1,
                                                  int row0, int nrow, int task) {
  constexpr int PITCH = D * 2 + 16, OCT = 8 * PITCH, PIECES = D / 8, RSTEP = 32 / PIECES, STEPS = 2;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int page = d.a[XA_PAGE];
  const AttnKeys keys = ao.keys;
  const int kend = min(k1, sv.pos0 + (row0 + nrow - 1) / ao.G + 1 - keys.shift);
  const int nstep = kend > k0 ? (kend - k0 + 15) >> 4 : 0, mine = nstep > warp ? (nstep - warp + 7) >> 3 : 0;
  uint8_t *qs = c.s.xtile;                                                   // [16][PITCH]
  // this warp's steps: sixteen K rows, then sixteen V rows
  const uint32_t ring = smem_u32(qs) + 16 * PITCH + warp * STEPS * 4 * OCT;
  const int piece = lane % PIECES, rl = lane / PIECES;
  const uint32_t krow = d.a[XA_HKV] * (d.a[XA_DIMP] >> 3), vrow = d.a[XA_HKV] * (d.a[XA_VDIMP] >> 3);
  const bool kin = piece < (d.a[XA_DIMP] >> 3), vin = piece < (d.a[XA_VDIMP] >> 3);
  const uint4 *kg = reinterpret_cast<const uint4 *>(d.p[1]) + ao.head * (d.a[XA_DIMP] >> 3) + piece + rl * krow;
  const uint4 *vg = reinterpret_cast<const uint4 *>(d.p[2]) + ao.head * (d.a[XA_VDIMP] >> 3) + piece + rl * vrow;
  const int32_t *pages = c.P.meta.paged_kv_indices + sv.kv0;
  int pos = k0 + warp * 16;
  auto page_of = [&](int key) { return key < kend ? __ldcg(pages + keys.pos(key) / page) : 0; };
  int pid0 = page_of(pos), pid1 = page_of(pos + 8);   // of the next step to request
  auto issue = [&](int slot) {
    if (pos < kend) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int p0 = pos + h * 8, left = kend - p0 - rl;
        const uint32_t row = (uint32_t)(h ? pid1 : pid0) * page + keys.pos(p0) % page;
        const uint32_t dst = ring + slot * 4 * OCT + h * OCT + rl * PITCH + piece * 16;
#pragma unroll
        for (int i = 0; i < 8 / RSTEP; ++i) {
          const uint32_t kd = dst + i * RSTEP * PITCH, vd = kd + 2 * OCT;
          const bool in = i * RSTEP < left;
          if (in && kin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(kd), "l"(kg + (size_t)((row + i * RSTEP) * krow)) : "memory");
          else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(kd), "r"(0) : "memory");
          if (in && vin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(vd), "l"(vg + (size_t)((row + i * RSTEP) * vrow)) : "memory");
          else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(vd), "r"(0) : "memory");
        }
      }
      pos += 128;
      pid0 = page_of(pos);
      pid1 = page_of(pos + 8);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0);
  issue(1);
  {
    const uint8_t *qg = reinterpret_cast<const uint8_t *>(d.p[0]);
    const int G = ao.G, kp = d.a[XA_DIMP] >> 3;
    for (int i = tid; i < 8 * PIECES; i += kConsumerThreads) {
      const int r = i / PIECES, p = i % PIECES, row = row0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nrow && p < kp)
        v = __ldcg(reinterpret_cast<const uint4 *>(qg + ((size_t)(sv.q0 + row / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + row % G) * kp * 8) * 2) + p);
      *reinterpret_cast<uint4 *>(qs + r * PITCH + p * 16) = v;
    }
  }
  consumer_sync();
  stamp(c, task, 0);
  const float scale = __int_as_float(d.a[XA_SCALE]), cap = __int_as_float(d.a[XA_CAP]);
  const float cap2 = cap > 0.f ? 2.0f * 1.4426950408889634f / cap : 0.f;
  uint32_t qf[D / 16][2];
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk)
    ldmatrix_x2(qf[kk], smem_u32(qs) + (uint32_t)((lane & 7) * PITCH + ((lane >> 3) & 1) * 16 + kk * 32));
  // this lane's two queries (columns of S^T), their positions, and the range of keys that needs no mask
  const int q0 = row0 + 2 * (lane & 3);
  const int p_a = sv.pos0 + q0 / ao.G, p_b = sv.pos0 + (q0 + 1) / ao.G, p_all = sv.pos0 + row0 / ao.G;
  const int p_far = sv.pos0 + (row0 + nrow - 1) / ao.G - ao.window + 1;
  float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};   // distance bias of the two
  if (BIAS) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = ao.head * ao.G + (q0 + i) % ao.G;
      r1[i] = bf16_at(d.p[5], h);
      r2[i] = bf16_at(d.p[6], h);
    }
  }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  float o[D / 16][4];
#pragma unroll
  for (int i = 0; i < D / 16; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const uint32_t k_off = (uint32_t)((lane & 15) * PITCH + (lane >> 4) * 16);
  const uint32_t v_off = (uint32_t)(2 * OCT + ((lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 16);
#pragma unroll 1
  for (int i = 0; i < mine; ++i) {
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncwarp();
    const uint32_t st = ring + (i & 1) * 4 * OCT;
    const int key0 = k0 + (warp + 8 * i) * 16;
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t a[4];
      ldmatrix_x4(a, st + k_off + kk * 32u);
      if (kk & 1) mma_bf16_16816(s2, a, qf[kk][0], qf[kk][1]);
      else mma_bf16_16816(s, a, qf[kk][0], qf[kk][1]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = attn_score<HYB_BF16>(s[e] + s2[e], scale, cap, cap2);
    const int at0 = keys.pos(key0), at1 = keys.pos(key0 + 8);
    if (BIAS) {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] -= distance_bias<HYB_BF16>(r1[e & 1], r2[e & 1], ((e & 1) ? p_b : p_a) - (e >> 1 ? at1 : at0) - (lane >> 2));
    }
    if (at1 + 7 > p_all || key0 + 16 > kend || at0 < p_far) {   // e: key g + 8 (e / 2), query 2 q + (e & 1)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int at = (e >> 1 ? at1 : at0) + (lane >> 2), p = (e & 1) ? p_b : p_a;
        if (key0 + (lane >> 2) + (e >> 1) * 8 >= kend || at > p || ao.outside(at, p)) s[e] = -INFINITY;
      }
    }
    float x0 = fmaxf(s[0], s[2]), x1 = fmaxf(s[1], s[3]);
#pragma unroll
    for (int sh = 4; sh < 32; sh <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, sh));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, sh));
    }
    const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);
    const float b0 = n0 == -INFINITY ? 0.f : n0, b1 = n1 == -INFINITY ? 0.f : n1;
    const float c0 = exp2f(m0 - b0), c1 = exp2f(m1 - b1);
    m0 = n0;
    m1 = n1;
    const float p0 = exp2f(s[0] - b0), p1 = exp2f(s[1] - b1), p2 = exp2f(s[2] - b0), p3 = exp2f(s[3] - b1);
    if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {   // (columns of O^T are queries as well: 2 q, 2 q + 1)
      l0 *= c0;
      l1 *= c1;
#pragma unroll
      for (int t = 0; t < D / 16; ++t) {
        o[t][0] *= c0; o[t][1] *= c1;
        o[t][2] *= c0; o[t][3] *= c1;
      }
    }
    l0 += p0 + p2;
    l1 += p1 + p3;
    // weights as a bf16 value and a bf16 remainder
    const uint32_t h0 = pack_bf16(p0, p1), h1 = pack_bf16(p2, p3);
    const uint32_t r0 = pack_bf16(p0 - bf16_lo(h0), p1 - bf16_hi(h0)), r1 = pack_bf16(p2 - bf16_lo(h1), p3 - bf16_hi(h1));
    const uint32_t hb0 = movmatrix_trans(h0), hb1 = movmatrix_trans(h1), rb0 = movmatrix_trans(r0), rb1 = movmatrix_trans(r1);
#pragma unroll
    for (int t = 0; t < D / 16; ++t) {
      uint32_t a[4];
      ldmatrix_x4_trans(a, st + v_off + t * 32u);
      mma_bf16_16816(o[t], a, hb0, hb1);
      mma_bf16_16816(o[t], a, rb0, rb1);
    }
    __syncwarp();   // every lane is done with the step that is refilled now
    issue(i & 1);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  consumer_sync();   // the rings become the combine area
  stamp(c, task, 2);
#pragma unroll
  for (int sh = 4; sh < 32; sh <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, sh);
    l1 += __shfl_xor_sync(0xffffffffu, l1, sh);
  }
  float *comb = reinterpret_cast<float *>(qs + 16 * PITCH);   // [8 warps][8 queries][D + 2]
  float *ca = comb + (size_t)(warp * 8 + 2 * (lane & 3)) * (D + 2), *cb = ca + (D + 2);
  if (lane < 4) {
    ca[0] = m0; ca[1] = l0;
    cb[0] = m1; cb[1] = l1;
  }
#pragma unroll
  for (int t = 0; t < D / 16; ++t) {
    const int col = 2 + t * 16 + (lane >> 2);
    ca[col] = o[t][0]; cb[col] = o[t][1];
    ca[col + 8] = o[t][2]; cb[col + 8] = o[t][3];
  }
  consumer_sync();
  attn_emit_splits<D>(c, d, ao, comb, 8, 8, row0, nrow);
}

// bf16: QK^T and PV on mma.sync.  Head sizes are padded to D columns in shared memory.  The eight warps are split over
// row tiles (16 rows), key octets and, for D = 256, halves of the output columns; the key split is combined in shared
// memory.  The probabilities enter PV as a bf16 value and a bf16 remainder, so that the weights keep 16 bits.
template <int D, bool BIAS>
__device__ __noinline__ void ext_attention_mma(const Ctx c, const TaskDesc &d, const SeqView sv, const AttnOut &ao, int k0, int k1,
                                                  int row0, int rows, int task) {
  constexpr int ON = D < 128 ? D : 128, WN = D / ON, KEYS = D > 128 ? 32 : 64, NSUB = KEYS / 8, PITCH = D * 2 + 16;
  constexpr int WMAX = 8 / WN, MROWS = WMAX * 16, TILE = KEYS * PITCH;
  const KernelParams &P = c.P;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int G = ao.G, hkv = d.a[XA_HKV], dimp = d.a[XA_DIMP], vdimp = d.a[XA_VDIMP], page = d.a[XA_PAGE];
  const int RB = min(MROWS, ext_attention_rows(P.max_num_batched_tokens * G));   // rows of a block (all of them in small graphs)
  uint8_t *qs = c.s.xtile;                // [RB][PITCH]
  uint8_t *st = qs + RB * PITCH;          // ring of stages, each KEYS K rows, then KEYS V rows
  const int nstg = d.a[XA_STAGES];
  int *cells = reinterpret_cast<int *>(st + nstg * 2 * TILE);   // [kXaCells] cache row (page * page size + offset) of every eighth key
  const uint8_t *qg = reinterpret_cast<const uint8_t *>(d.p[0]);
  const uint8_t *kg = reinterpret_cast<const uint8_t *>(d.p[1]), *vg = reinterpret_cast<const uint8_t *>(d.p[2]);
  const int kp = dimp >> 3, vp = vdimp >> 3;   // 16-byte pieces of a row
  // eight consecutive keys lie in one page when pages hold a multiple of eight positions
  const int ncell = (page & 7) == 0 && k1 - k0 <= 8 * kXaCells ? (k1 - k0 + 7) >> 3 : 0;
  const AttnKeys keys = ao.keys;
  auto cell_row = [&](int i) {
    const int key = keys.pos(i), pg = key / page;
    return __ldcg(&P.meta.paged_kv_indices[sv.kv0 + pg]) * page + (key - pg * page);
  };
  for (int i = tid; i < ncell; i += kConsumerThreads) cells[i] = cell_row(k0 + 8 * i);

  for (int rb = row0; rb < rows; rb += RB) {
    const int nrow = min(RB, rows - rb), mt = (nrow + 15) >> 4;
    const int WM = mt <= 1 ? 1 : (mt <= 2 ? 2 : (mt <= 4 ? 4 : WMAX));
    const int WK = WMAX / WM;                                      // <= NSUB
    const int wn = warp % WN, w2 = warp / WN, wm = w2 % WM, wk = w2 / WM;
    const int kend = min(k1, sv.pos0 + (rb + nrow - 1) / G + 1 - keys.shift);   // keys past the last row's position are not needed
    if (rb > row0) consumer_sync();
    for (int i = tid; i < WM * 16 * (D / 8); i += kConsumerThreads) {
      const int r = i / (D / 8), p = i - r * (D / 8);
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nrow && p < kp) {
        const int row = rb + r;
        v = __ldcg(reinterpret_cast<const uint4 *>(qg + ((size_t)(sv.q0 + row / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + row % G) * dimp) * 2) + p);
      }
      *reinterpret_cast<uint4 *>(qs + r * PITCH + p * 16) = v;
    }
    auto issue = [&](int it, int stg) {
      const int base = k0 + it * KEYS;
      const int p = tid % (D / 8);
      uint8_t *dst = st + stg * 2 * TILE + (tid / (D / 8)) * PITCH + p * 16;
      constexpr int STEP = kConsumerThreads / (D / 8);   // rows of a pass
#pragma unroll
      for (int pass = 0; pass < KEYS / STEP; ++pass) {
        const int key = base + pass * STEP + tid / (D / 8);
        uint8_t *kd = dst + pass * STEP * PITCH, *vd = kd + TILE;
        const bool in = key < kend;
        size_t cell = 0;
        if (in) cell = (size_t)(ncell > 0 ? cells[(key - k0) >> 3] + ((key - k0) & 7) : cell_row(key)) * hkv + ao.head;
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
    const AttnRows w = attn_rows<BIAS>(d, sv, ao, rb + wm * 16, min(nrow - wm * 16, 16), kend);
    const int ntiles = kend > k0 ? (kend - k0 + KEYS - 1) / KEYS : 0;
    consumer_sync();   // queries and cells
    stamp(c, task, 0);
    // nstg - 1 tiles in flight; one commit per trip, empty past the last tile, so that the wait counts trips
    for (int i = 0; i < nstg - 1; ++i) {
      if (i < ntiles) issue(i, i);
      else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    const uint32_t qa = smem_u32(qs) + (uint32_t)((wm * 16 + (lane & 15)) * PITCH + (lane >> 4) * 16);
    const uint32_t qf[1][2] = {{0u, 0u}};   // (the fragments come from shared memory)
    const uint32_t lane_off = (uint32_t)((lane & 7) * PITCH + (lane >> 3) * 16);
    int stg = 0;
    for (int it = 0; it < ntiles; ++it) {
      if (nstg >= 4) asm volatile("cp.async.wait_group 2;" ::: "memory");
      else if (nstg == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
      else asm volatile("cp.async.wait_group 0;" ::: "memory");
      consumer_sync();   // tile `it` has landed for everyone, and everyone is done with the stage refilled next
      if (it == 0) stamp(c, task, 1);
      if (it + nstg - 1 < ntiles) issue(it + nstg - 1, stg == 0 ? nstg - 1 : stg - 1);
      else asm volatile("cp.async.commit_group;" ::: "memory");
      const int base = k0 + it * KEYS;
      const uint32_t kt = smem_u32(st + stg * 2 * TILE) + lane_off, vt = kt + TILE + wn * ON * 2;
      if (++stg == nstg) stg = 0;
      if (wm >= mt) continue;
      // this warp's octets of keys, one at a time
#pragma unroll 1
      for (int j = wk; j < NSUB; j += WK) {
        const int key0 = base + j * 8;
        if (key0 >= kend) break;
        attn_octet<D, ON, true, BIAS>(w, ao, qf, qa, kt + (uint32_t)(j * 8 * PITCH), vt + (uint32_t)(j * 8 * PITCH), key0, keys.pos(key0), m_run, l_run, o);
      }
    }
    consumer_sync();   // the stages become the combine area
    stamp(c, task, 2);
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
        if (w.two) *reinterpret_cast<float2 *>(c1 + col) = make_float2(o[i][2], o[i][3]);
      }
    }
    consumer_sync();
    attn_emit_splits<D>(c, d, ao, comb, WM * 16, WK, rb, nrow);
  }
}

// Shared key / value rows (latent attention: one kv head, the leading vdim columns of a key are its value), bf16 on mma.sync.  A
// tile of 16 query rows meets KEYS keys at a time, and every key row is brought to shared memory once for both products:
//   scores   the warps split the keys in groups of 16 and the row width KS ways; partial sums meet in shared memory
//   softmax  a warp takes RT / 8 rows, online in base 2; weights go back as a bf16 value and a bf16 remainder, so that they
//            keep 16 bits
//   output   every warp owns eight-column tiles w, w + 8, ... of all rows; a tile's output is formed beside the next one's scores
//
// (with a few KB of L1 beside the shared memory a spilled variable of the key loop costs an L2 round trip: areas of fixed size
// come first, so that their addresses are one base plus constants, and everything is addressed in 32 bits)
__device__ __forceinline__ float lds_f32(uint32_t a) {
  float v;
  asm volatile("ld.shared.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ float4 lds_f32x4(uint32_t a) {
  float4 v;
  asm volatile("ld.shared.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ float2 lds_f32x2(uint32_t a) {
  float2 v;
  asm volatile("ld.shared.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ int lds_s32(uint32_t a) {
  int v;
  asm volatile("ld.shared.s32 %0, [%1];" : "=r"(v) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ void sts_f32(uint32_t a, float v) { asm volatile("st.shared.f32 [%0], %1;" ::"r"(a), "f"(v) : "memory"); }
__device__ __forceinline__ void sts_f32x2(uint32_t a, float v, float w) { asm volatile("st.shared.v2.f32 [%0], {%1, %2};" ::"r"(a), "f"(v), "f"(w) : "memory"); }
__device__ __forceinline__ void sts_bf16(uint32_t a, __nv_bfloat16 v) {
  asm volatile("st.shared.b16 [%0], %1;" ::"r"(a), "h"(__bfloat16_as_ushort(v)) : "memory");
}
__device__ __forceinline__ void sts_zero16(uint32_t a) { asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(a), "r"(0) : "memory"); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
// (the arguments and the loop's constants too: they stay in shared memory and are read where they are used)
struct alignas(16) LatentArgs {
  AttnOut ao;
  alignas(16) int keys;           // keys of the chunk the rows see
  int pieces, table, ntiles;      // 16-byte pieces of a cache row, the table of cache rows is used, key tiles
  const uint4 *rows;              // this layer's cache
  const int32_t *pages;           // the request's pages
  float scale, cap;
  int page, k0;
  int q0, pos0, row0, nrow, task, stages;
};
constexpr uint32_t kLatentHot = offsetof(LatentArgs, keys);
static_assert(offsetof(LatentArgs, rows) == kLatentHot + 16, "read as one vector and one pointer");
static_assert(sizeof(LatentArgs) <= 256, "the reduction slots hold 64 words");
__device__ __forceinline__ int4 lds_v4(uint32_t a) {
  int4 v;
  asm volatile("ld.shared.v4.s32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ uint64_t lds_u64(uint32_t a) {
  uint64_t v;
  asm volatile("ld.shared.u64 %0, [%1];" : "=l"(v) : "r"(a) : "memory");
  return v;
}
// Cache row of a key, where the table does not hold it (page sizes that are no multiple of eight, very long chunks).
static __device__ __noinline__ int latent_cell(const int32_t *pages, int page, int key) { return __ldcg(pages + key / page) * page + key % page; }

template <int KEYS>
__device__ __noinline__ void latent_attention_mma(const KernelParams &P, uint32_t sm, const TaskDesc &d, const LatentArgs &la) {
  constexpr int RT = 16, KW = KEYS / 16, KS = 8 / KW, SP = KEYS + 4, PP = KEYS * 2 + 16, NV = 8;
  constexpr int RPW = RT * KEYS / 256;             // row sets a warp's lanes hold in the softmax (32 / KEYS rows at a time)
  // shared memory: partial scores [KS][RT][SP], weights [value, remainder][RT][PP], rescale factors [RT] (at the end m and l [2][RT]),
  // cache row of every eighth key [kXaCells], queries [RT][pitch], ring of key tiles [stages][KEYS][pitch]
  constexpr uint32_t oP = KS * RT * SP * 4, oC = oP + 2 * RT * PP, oCell = oC + 8 * RT, oQ = (oCell + kXaCells * 4 + 15) & ~15u;
  const uint32_t args = smem_u32(&la);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t pitch = ((la.pieces + 7) & ~7) * 16 + 16;   // rows padded to whole 64-column blocks
  const uint32_t ring = sm + oQ + RT * pitch;
  {
    const int row0 = la.row0, nrow = la.nrow, pieces = la.pieces, padded = (pieces + 7) & ~7;
    if (la.table)
      for (int i = tid; i < (la.keys + 7) >> 3; i += kConsumerThreads)
        asm volatile("st.shared.s32 [%0], %1;" ::"r"(sm + oCell + i * 4), "r"(latent_cell(la.pages, la.page, la.k0 + 8 * i)) : "memory");
    // queries, and zeros where no copy reaches
    const uint4 *qg = reinterpret_cast<const uint4 *>(d.p[0]);
    const int G = la.ao.G, ldq = d.a[XA_LDQ] >> 3;
    for (int r = warp; r < RT; r += 8) {
      const uint32_t dst = sm + oQ + r * pitch;
      const uint4 *src = qg + (size_t)(la.q0 + (row0 + r) / G) * ldq + (size_t)((row0 + r) % G) * pieces;
      for (int p = lane; p < padded; p += 32) {
        if (r < nrow && p < pieces) cp_async16(dst + p * 16, src + p);
        else sts_zero16(dst + p * 16);
      }
    }
    if (pieces < padded)
      for (int r = warp; r < la.stages * KEYS; r += 8)
        for (int p = pieces + lane; p < padded; p += 32) sts_zero16(ring + r * pitch + p * 16);
  }
  consumer_sync();   // (the table of cache rows)
  stamp(P, la.task, 0);
  auto issue = [&](int it, uint32_t dst) {
    const int4 h = lds_v4(args + kLatentHot);   // keys, pieces, table, tiles
    if (it < h.w) {
      const uint4 *rows = reinterpret_cast<const uint4 *>(lds_u64(args + kLatentHot + 16)) + lane;
      dst += warp * pitch + lane * 16;
#pragma unroll
      for (int r = 0; r < KEYS / 8; ++r, dst += 8 * pitch) {
        const int key = it * KEYS + warp + 8 * r;   // of the chunk
        if (key < h.x) {
          int cell;
          if (h.z) cell = lds_s32(sm + oCell + (key >> 3) * 4) + (key & 7);
          else cell = latent_cell(la.pages, la.page, la.k0 + key);
          const uint4 *src = rows + (size_t)cell * h.y;
          for (int p = lane; p < h.y; p += 32) cp_async16(dst + (p - lane) * 16, src + (p - lane));
        } else {   // a masked key has weight 0, and 0 x NaN would be NaN
          for (int p = lane; p < h.y; p += 32) sts_zero16(dst + (p - lane) * 16);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (int i = 0; i < la.stages - 2; ++i) issue(i, ring + i * KEYS * pitch);   // (the queries join the first group)
  const int nv = (la.ao.vdim >> 3) > warp ? ((la.ao.vdim >> 3) - warp + 7) >> 3 : 0;   // this warp's column tiles
  // softmax: this lane's key of the tile, its first row and how far behind that row set the key lies
  const int skey = lane % KEYS, srow = warp * (RT / 8) + lane / KEYS;
  int seen[RPW];
  float m_run[RPW], l_run[RPW];
#pragma unroll
  for (int i = 0; i < RPW; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
    seen[i] = la.pos0 + (la.row0 + srow + i * (32 / KEYS)) / la.ao.G - la.k0 - skey;   // distance from this lane's key of the first tile
  }
  float o[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  // Trip `it`: scores of tile `it` and, in between, output of tile `it - 1`, whose weights the softmax left behind
  uint32_t slot = 0, before = ring;   // ring slot of tile `it`, address of tile `it - 1`
#pragma unroll 1
  for (int it = 0;; ++it) {
    const uint32_t nstg = lds_s32(args + offsetof(LatentArgs, stages)), ntiles = lds_s32(args + offsetof(LatentArgs, ntiles));
    if (nstg >= 4) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    consumer_sync();   // the tile has landed for everyone, the weights of the one before are final, the one before that is free
    if (it == 0) stamp(P, la.task, 1);
    const uint32_t kt = ring + slot * (KEYS * pitch);
    issue(it + nstg - 2, ring + (slot >= 2 ? slot - 2 : slot + nstg - 2) * (KEYS * pitch));
    if (++slot == nstg) slot = 0;
    {
      const int kw = warp % KW, ks = warp / KW, ksteps = it < (int)ntiles ? (int)(pitch >> 5) : 0;   // 16-column steps of a row
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const uint32_t ka = kt + (uint32_t)((kw * 16 + (lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 16);
      const uint32_t qa = sm + oQ + (uint32_t)((lane & 15) * pitch + (lane >> 4) * 16);
      int kk = ks;
      if (it > 0) {
        const float c0 = lds_f32(sm + oC + (lane >> 2) * 4), c1 = lds_f32(sm + oC + (8 + (lane >> 2)) * 4);
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
          for (int i = 0; i < NV; ++i) {
            o[i][0] *= c0; o[i][1] *= c0;
            o[i][2] *= c1; o[i][3] *= c1;
          }
        }
        // 16 keys and two column tiles at a time (one past the last is read, not used), a step of the scores beside each
        const uint32_t pa = sm + oP + (uint32_t)((lane & 15) * PP + (lane >> 4) * 16);
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          uint32_t p[2][4];
#pragma unroll
          for (int h = 0; h < 2; ++h) ldmatrix_x4(p[h], pa + (uint32_t)(h * RT * PP + k * 32));
          const uint32_t va = before + (uint32_t)(k * 16 + (lane & 15)) * pitch + warp * 16 + (lane >> 4) * 128u;
#pragma unroll
          for (int i = 0; i < NV; i += 2) {
            if (i >= nv) break;
            uint32_t v[4], a[4], b[4];
            ldmatrix_x4_trans(v, va + i * 128u);
            if (kk < ksteps) {
              ldmatrix_x4(b, ka + kk * 32u);
              ldmatrix_x4(a, qa + kk * 32u);
              mma_bf16_16816(s[0], a, b[0], b[1]);
              mma_bf16_16816(s[1], a, b[2], b[3]);
              kk += KS;
            }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              mma_bf16_16816(o[i], p[h], v[0], v[1]);
              if (i + 1 < nv) mma_bf16_16816(o[i + 1], p[h], v[2], v[3]);
            }
          }
        }
      }
#pragma unroll 2
      for (; kk < ksteps; kk += KS) {
        uint32_t a[4], b[4];
        ldmatrix_x4(b, ka + kk * 32u);
        ldmatrix_x4(a, qa + kk * 32u);
        mma_bf16_16816(s[0], a, b[0], b[1]);
        mma_bf16_16816(s[1], a, b[2], b[3]);
      }
      before = kt;
      if (it == (int)ntiles) break;
      const uint32_t sr = sm + (uint32_t)(((ks * RT + (lane >> 2)) * SP + kw * 16 + 2 * (lane & 3)) * 4);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        sts_f32x2(sr + n * 32, s[n][0], s[n][1]);
        sts_f32x2(sr + (8 * SP + n * 8) * 4, s[n][2], s[n][3]);
      }
    }
    consumer_sync();
    {   // ---- softmax
      const uint32_t sa = sm + (uint32_t)((srow * SP + skey) * 4), pa = sm + oP + (uint32_t)(srow * PP + skey * 2);
      const float scale = lds_f32(args + offsetof(LatentArgs, scale)), cap = lds_f32(args + offsetof(LatentArgs, cap));
      const float cap2 = cap > 0.f ? 2.0f * 1.4426950408889634f / cap : 0.f;
      // keys past the chunk's end are in nobody's window
      const int window = it * KEYS + skey < lds_s32(args + kLatentHot) ? lds_s32(args + offsetof(LatentArgs, ao) + offsetof(AttnOut, window)) : 0;
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int r = i * (32 / KEYS);
        float v = 0.f;
#pragma unroll
        for (int p = 0; p < KS; ++p) v += lds_f32(sa + (p * RT + r) * SP * 4);
        v = attn_score<HYB_BF16>(v, scale, cap, cap2);
        if ((unsigned)(seen[i] - it * KEYS) >= (unsigned)window) v = -INFINITY;
        float mx = v;
#pragma unroll
        for (int sh = KEYS / 2; sh > 0; sh >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, sh));
        const float mn = fmaxf(m_run[i], mx), ms = mn == -INFINITY ? 0.f : mn;
        const float corr = exp2f(m_run[i] - ms), p = exp2f(v - ms);
        m_run[i] = mn;
        l_run[i] = l_run[i] * corr + p;
        const __nv_bfloat16 hi = __float2bfloat16_rn(p);
        sts_bf16(pa + r * PP, hi);
        sts_bf16(pa + (RT + r) * PP, __float2bfloat16_rn(p - bf16_to_f(hi)));
        if (skey == 0) sts_f32(sm + oC + (srow + r) * 4, corr);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  stamp(P, la.task, 2);
  // running maximum and sum of every row
  consumer_sync();
#pragma unroll
  for (int i = 0; i < RPW; ++i) {
    float l = l_run[i];
#pragma unroll
    for (int sh = KEYS / 2; sh > 0; sh >>= 1) l += __shfl_xor_sync(0xffffffffu, l, sh);
    if (skey == 0) {
      sts_f32(sm + oC + (srow + i * (32 / KEYS)) * 4, m_run[i]);
      sts_f32(sm + oC + (RT + srow + i * (32 / KEYS)) * 4, l);
    }
  }
  consumer_sync();
  const AttnOut &ao = la.ao;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = h * 8 + (lane >> 2), row = la.row0 + r;
    if (r >= la.nrow) continue;
    const float mx = lds_f32(sm + oC + r * 4), l = lds_f32(sm + oC + (RT + r) * 4);
    const int col0 = warp * 8 + 2 * (lane & 3);
    if (ao.n_act == 1) {
      const int hq_idx = row % ao.G;
      const float sk = ao.sink ? sink_logit<HYB_BF16>(d, hq_idx) : 0.f;
      const float M = ao.sink ? fmaxf(mx, sk) : mx;
      const float w = mx == -INFINITY ? 0.f : exp2f(mx - M);
      const float L = l * w + (ao.sink ? exp2f(sk - M) : 0.f);
      const float f = L > 0.f ? w / L * ao.oscale : 0.f;
      __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(d.p[3]) + (size_t)(la.q0 + row / ao.G) * ao.ldo + ao.ocol + (size_t)hq_idx * ao.vdim + col0;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i < nv) *reinterpret_cast<uint32_t *>(out + i * 64) = pack_bf16(o[i][2 * h] * f, o[i][2 * h + 1] * f);
    } else {
      float *rec = attn_record(P, ao, row);
      if (warp == 0 && (lane & 3) == 0) {
        __stcg(rec, mx);
        __stcg(rec + 1, l);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i < nv) __stcg(reinterpret_cast<float2 *>(rec + kXaRecHead + col0 + i * 64), make_float2(o[i][2 * h], o[i][2 * h + 1]));
    }
  }
}

// 32-bit: one warp per row, 32 keys at a time (a lane per key for the scores, a lane per output column for PV)
static __device__ __noinline__ void ext_attention_f32(const Ctx c, const TaskDesc &d, const SeqView sv, const AttnOut &ao, int k0, int k1,
                                                  int row0, int rows) {
  constexpr int NO = 16;   // output columns per lane: value sizes up to 512
  const KernelParams &P = c.P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = ao.G, hkv = d.a[XA_HKV], dimp = d.a[XA_DIMP], vdimp = d.a[XA_VDIMP], page = d.a[XA_PAGE];
  const float scale = __int_as_float(d.a[XA_SCALE]), cap = __int_as_float(d.a[XA_CAP]);
  float *q = reinterpret_cast<float *>(c.s.xtile) + warp * dimp;
  const float *qg = reinterpret_cast<const float *>(d.p[0]);
  const float *kg = reinterpret_cast<const float *>(d.p[1]), *vg = reinterpret_cast<const float *>(d.p[2]);
  const AttnKeys keys = ao.keys;
  const bool bias = d.p[5] != 0;
  auto cell_of = [&](int key) {
    const int pg = key / page;
    return ((size_t)__ldcg(&P.meta.paged_kv_indices[sv.kv0 + pg]) * page + (key - pg * page)) * hkv + ao.head;
  };
  for (int r = row0 + warp; r < rows; r += 8) {
    const int pos = sv.pos0 + r / G, kend = min(k1, pos + 1 - keys.shift);
    __syncwarp();
    for (int i = lane; i < dimp; i += 32) q[i] = __ldcg(qg + (size_t)(sv.q0 + r / G) * d.a[XA_LDQ] + (size_t)(ao.head * G + r % G) * dimp + i);
    __syncwarp();
    const int hb = ao.head * G + r % G;
    const float r1 = bias ? bf16_at(d.p[5], hb) : 0.f, r2 = bias ? bf16_at(d.p[6], hb) : 0.f;
    float m = -INFINITY, l = 0.f, o[NO];
#pragma unroll
    for (int i = 0; i < NO; ++i) o[i] = 0.f;
    for (int kb = k0; kb < kend; kb += 32) {
      const int at = keys.pos(kb + lane);
      const bool seen = kb + lane < kend && !ao.outside(at, pos);
      float s = -INFINITY;
      size_t cell = 0;
      if (seen) {
        cell = cell_of(at);
        const float4 *kr = reinterpret_cast<const float4 *>(kg + cell * dimp);
        float dot = 0.f;
        for (int i = 0; i < dimp >> 2; ++i) {
          const float4 kv = __ldcg(kr + i), qv = *reinterpret_cast<const float4 *>(q + 4 * i);
          dot += kv.x * qv.x + kv.y * qv.y + kv.z * qv.z + kv.w * qv.w;
        }
        s = attn_score<HYB_F32>(dot, scale, cap, 0.f);
        if (bias) s -= distance_bias<HYB_F32>(r1, r2, pos - at);
      }
      const float mn = fmaxf(m, warp_max(s));
      if (mn == -INFINITY) continue;   // none of these keys is seen
      const float corr = expf(m - mn), p = seen ? expf(s - mn) : 0.f;
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

// Head sizes padded to D columns, bf16: the body for the task's rows.
template <int D, bool BIAS>
__device__ __forceinline__ void ext_attention_sized(const Ctx &c, const TaskDesc &d, const SeqView &sv, const AttnOut &ao, int k0, int k1, int row0,
                                                    int row1, int task) {
  if constexpr (D <= 128) {
    const int n = row1 - row0;
    if (n <= 16 && (d.a[XA_PAGE] & 7) == 0) {
      if (n <= 8 && d.a[XA_STAGES] >= 3) ext_attention_decode<D, BIAS>(c, d, sv, ao, k0, k1, row0, n, task);
      else if (n <= 8) ext_attention_stream<D, false, BIAS>(c, d, sv, ao, k0, k1, row0, n, task);
      else ext_attention_stream<D, true, BIAS>(c, d, sv, ao, k0, k1, row0, n, task);
      return;
    }
  }
  ext_attention_mma<D, BIAS>(c, d, sv, ao, k0, k1, row0, row1, task);
}

template <int HYB>
__device__ __forceinline__ void run_ext_attention(const Ctx &c, const TaskDesc &d, int task) {
  const SeqView sv = seq_view(c.P, d.a[XA_SLOT]);
  if (sv.nq <= 0) return;
  // shared by the block, in shared memory: in registers it would be live through the key loops (every thread writes the
  // same values, and the previous task is done with it)
  AttnOut &ao = *reinterpret_cast<AttnOut *>(c.s.red);
  constexpr int RT = 16;
  const int NC = d.a[XA_NCHUNK];
  ao.hq = d.a[XA_HQ];
  ao.G = ao.hq / d.a[XA_HKV];
  ao.head = d.a[XA_HEAD];
  ao.q0 = sv.q0;
  ao.vdim = d.a[XA_VDIM];
  ao.ldo = d.a[XA_LDO];
  ao.ocol = d.a[XA_OCOL];
  ao.srec = d.a[XA_SREC];
  ao.oscale = __int_as_float(d.a[XA_OSCALE]);
  ao.sink = d.a[XA_SINK] != 0;
  ao.f32 = d.a[XA_OUTF32] != 0;
  ao.window = d.a[XA_WINDOW] > 0 ? d.a[XA_WINDOW] : 1 << 30;
  ao.keep = d.a[XA_KEEP];
  ao.keys = attn_keys(d, sv);
  const AttnSplit sp = attn_split(sv, ao.keys.len, ao.G, NC, RT);
  const int part = d.a[XA_CHUNK] % sp.parts;
  ao.chunk = d.a[XA_CHUNK] / sp.parts;
  ao.ks = sp.ks;
  ao.n_act = sp.n_act;
  ao.rec0 = (d.a[XA_SLOT] * d.a[XA_HKV] + ao.head) * RT * NC;
  if (ao.chunk >= ao.n_act) return;   // (n_act <= ks: this also ends the tasks beyond parts * ks)
  const int k0 = ao.chunk * sp.per, k1 = min(ao.keys.len, k0 + sp.per);
  const int row0 = sp.tiles * part / sp.parts * RT, row1 = min(sp.rows, sp.tiles * (part + 1) / sp.parts * RT);
  if (HYB == HYB_F32) {
    ext_attention_f32(c, d, sv, ao, k0, k1, row0, row1);
  } else if (d.a[XA_SHARED]) {
    LatentArgs &la = *reinterpret_cast<LatentArgs *>(c.s.red);   // (begins with `ao`)
    const int keys = d.a[XA_KEYS];
    for (int r = row0; r < row1; r += 16) {
      if (r > row0) consumer_sync();
      // keys in front of the first row's window and past the last row's position are not needed
      const int n = min(16, row1 - r), shift = ao.keys.shift, kend = min(k1 + shift, sv.pos0 + (r + n - 1) / ao.G + 1);
      const int first = max(k0 + shift, (sv.pos0 + r / ao.G - ao.window + 1) & ~7);
      la.keys = max(kend - first, 0);
      la.pieces = d.a[XA_DIMP] >> 3;
      la.table = (d.a[XA_PAGE] & 7) == 0 && la.keys <= 8 * kXaCells;   // eight consecutive keys lie in one page
      la.ntiles = (la.keys + keys - 1) / keys;
      la.rows = reinterpret_cast<const uint4 *>(d.p[1]);
      la.pages = c.P.meta.paged_kv_indices + sv.kv0;
      la.scale = __int_as_float(d.a[XA_SCALE]);
      la.cap = __int_as_float(d.a[XA_CAP]);
      la.page = d.a[XA_PAGE]; la.k0 = first; la.q0 = sv.q0; la.pos0 = sv.pos0; la.row0 = r; la.nrow = n; la.task = task; la.stages = d.a[XA_STAGES];
      if (keys == 32) latent_attention_mma<32>(c.P, smem_u32(c.s.xtile), d, la);
      else latent_attention_mma<16>(c.P, smem_u32(c.s.xtile), d, la);
    }
  } else {
    const int w = max(d.a[XA_DIMP], d.a[XA_VDIMP]);
    if (d.p[5]) {
      if (w <= 64) ext_attention_sized<64, true>(c, d, sv, ao, k0, k1, row0, row1, task);
      else if (w <= 128) ext_attention_sized<128, true>(c, d, sv, ao, k0, k1, row0, row1, task);
      else ext_attention_sized<256, true>(c, d, sv, ao, k0, k1, row0, row1, task);
    } else {
      if (w <= 64) ext_attention_sized<64, false>(c, d, sv, ao, k0, k1, row0, row1, task);
      else if (w <= 128) ext_attention_sized<128, false>(c, d, sv, ao, k0, k1, row0, row1, task);
      else ext_attention_sized<256, false>(c, d, sv, ao, k0, k1, row0, row1, task);
    }
  }
  stamp(c, task, 3);
  if (ao.n_act > 1 && !d.a[XA_MERGE]) attn_merge<HYB>(c, d, ao, part, row0, row1);
}

// TASK_ATTN_MERGE: the chunks' records of an attention layer with wide values, spread over all workers.  A warp takes 128 columns
// of a (token, query head).
template <int HYB>
__device__ __noinline__ void run_attn_merge(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hq = d.a[XA_HQ], hkv = d.a[XA_HKV], G = hq / hkv, vdim = d.a[XA_VDIM], srec = d.a[XA_SREC], NC = d.a[XA_NCHUNK];
  const int RT = 16, cols = (vdim + 127) >> 7;
  for (int item = d.a[XA_SLOT] * 8 + warp; item < B * hq * cols; item += d.a[XA_CHUNK] * 8) {
    const int row = item / cols, j = (item - row * cols) * 128 + lane * 4, t = row / hq, h = row - t * hq;
    const int k = request_of(P, t);
    const SeqView sv = seq_view(P, k);
    const AttnSplit a = attn_split(sv, attn_keys(d, sv).len, G, NC, RT);
    if (a.n_act == 1) continue;   // the attention task wrote the output
    const int r = (t - sv.q0) * G + h % G;
    const float *rec = P.attn_scratch + ((size_t)(k * hkv + h / G) * RT * NC + (size_t)r * a.ks) * srec;
    const bool v = lane < a.n_act;
    const float m = v ? __ldcg(rec + (size_t)lane * srec) : -INFINITY, l = v ? __ldcg(rec + (size_t)lane * srec + 1) : 0.f;
    const float sk = d.a[XA_SINK] ? sink_logit<HYB>(d, h) : 0.f;
    float M = warp_max(m);
    if (d.a[XA_SINK]) M = fmaxf(M, sk);
    const float w = m == -INFINITY ? 0.f : exp_dom<HYB>(m - M);
    const float L = warp_sum(l * w) + (d.a[XA_SINK] ? exp_dom<HYB>(sk - M) : 0.f);
    const float f = L > 0.f ? __int_as_float(d.a[XA_OSCALE]) / L : 0.f;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int u = 0; u < a.n_act; ++u) {
      const float wu = __shfl_sync(0xffffffffu, w, u);
      const float4 x = j < vdim ? __ldcg(reinterpret_cast<const float4 *>(rec + (size_t)u * srec + kXaRecHead + j)) : make_float4(0.f, 0.f, 0.f, 0.f);
      acc.x = fmaf(wu, x.x, acc.x); acc.y = fmaf(wu, x.y, acc.y); acc.z = fmaf(wu, x.z, acc.z); acc.w = fmaf(wu, x.w, acc.w);
    }
    const size_t out = (size_t)t * d.a[XA_LDO] + d.a[XA_OCOL] + (size_t)h * vdim + j;
    const float o[4] = {acc.x * f, acc.y * f, acc.z * f, acc.w * f};
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (j + e < vdim) store_out<T>(d, d.a[XA_OUTF32] != 0, out + e, o[e]);
  }
}

// ---------------------------------------------------------------------------
// TASK_DIFF_COMBINE (Ye et al., "Differential Transformer"): per token and head, the difference of the two maps' outputs, divided
// by its root mean square over the head's values, times a factor.  One warp per (token, head).
// ---------------------------------------------------------------------------
template <int HYB>
__device__ __noinline__ void run_diff_combine(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const int B = active_tokens(c.P), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = d.a[2], vdim = d.a[3];
  const float lambda = __int_as_float(d.a[6]), factor = __int_as_float(d.a[7]), eps = __int_as_float(d.a[8]);
  for (int item = d.a[0] * 8 + warp; item < B * H; item += d.a[1] * 8) {
    const int t = item / H, h = item - t * H;
    const float *a = reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[4] + (size_t)2 * h * vdim;
    T *out = reinterpret_cast<T *>(d.p[1]) + (size_t)t * d.a[5] + (size_t)h * vdim;
    float ss = 0.f;
    if (vdim <= 256) {   // the row in registers, all loads in flight
      float x[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int j = i * 32 + lane;
        x[i] = j < vdim ? __ldcg(a + j) - lambda * __ldcg(a + vdim + j) : 0.f;
        ss += x[i] * x[i];
      }
      const float f = factor / sqrtf(warp_sum(ss) / (float)vdim + eps);
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i * 32 + lane < vdim) store_elt(out + i * 32 + lane, x[i] * f);
      continue;
    }
    for (int j = lane; j < vdim; j += 32) { const float x = __ldcg(a + j) - lambda * __ldcg(a + vdim + j); ss += x * x; }
    const float f = factor / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int j = lane; j < vdim; j += 32) store_elt(out + j, (__ldcg(a + j) - lambda * __ldcg(a + vdim + j)) * f);
  }
}

// ---------------------------------------------------------------------------
// TASK_POLY_NORM: a N(z) + b N(z^2) + c N(z^3) + e, N dividing a token's values by their root mean square.  One block per token; with the
// three factors known the sum is a cubic in z.
// ---------------------------------------------------------------------------
// One token: emit4(column, values) or emit(column, value) receives the activations of the row's N columns.  Ends with a barrier.
template <class F4, class F>
__device__ __forceinline__ void poly_norm_row(const Ctx &c, const float *z, int N, bool vec, uint64_t coefficients, float eps, F4 emit4, F emit) {
  constexpr int NV = 16;   // 16384 columns in registers, all loads in flight
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float4 x[NV];
  float s[3] = {0.f, 0.f, 0.f};
  auto powers = [&](float v) {
    const float q = v * v;
    s[0] += q;
    s[1] = fmaf(q, q, s[1]);
    s[2] = fmaf(q * q, q, s[2]);
  };
  vec = vec && N <= NV * kConsumerThreads * 4;
  if (vec) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = (i * kConsumerThreads + tid) * 4;
      x[i] = j < N ? __ldcg(reinterpret_cast<const float4 *>(z + j)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (i * kConsumerThreads * 4 >= N) break;
      powers(x[i].x); powers(x[i].y); powers(x[i].z); powers(x[i].w);
    }
  } else {
#pragma unroll 4
    for (int j = tid; j < N; j += kConsumerThreads) powers(__ldcg(z + j));
  }
#pragma unroll
  for (int k = 0; k < 3; ++k) {
    s[k] = warp_sum(s[k]);
    if (lane == 0) c.s.red[8 * k + warp] = s[k];
  }
  consumer_sync();
  float f[3];
#pragma unroll
  for (int k = 0; k < 3; ++k) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) v += c.s.red[8 * k + w];
    f[k] = bf16_at(coefficients, k) / sqrtf(v / (float)N + eps);
  }
  const float k0 = bf16_at(coefficients, 3);
  auto cubic = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, f[2], f[1]), f[0]), k0); };
  if (vec) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int j = (i * kConsumerThreads + tid) * 4;
      if (i * kConsumerThreads * 4 >= N) break;
      if (j < N) emit4(j, make_float4(cubic(x[i].x), cubic(x[i].y), cubic(x[i].z), cubic(x[i].w)));
    }
  } else {
#pragma unroll 4
    for (int j = tid; j < N; j += kConsumerThreads) emit(j, cubic(__ldcg(z + j)));
  }
  consumer_sync();   // the reduction slots are used again
}
template <int HYB>
__device__ __noinline__ void run_poly_norm(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const int t1 = min(d.a[1], active_tokens(c.P)), N = d.a[2];
  const bool vec = ((N | d.a[3] | d.a[4]) & 3) == 0 && ((d.p[0] | d.p[2]) & 15) == 0;
  for (int t = d.a[0]; t < t1; ++t) {
    T *out = reinterpret_cast<T *>(d.p[2]) + (size_t)t * d.a[4];
    poly_norm_row(c, reinterpret_cast<const float *>(d.p[0]) + (size_t)t * d.a[3], N, vec, d.p[1], __int_as_float(d.a[5]),
                  [&](int j, float4 v) { store_elt4(out + j, v); }, [&](int j, float v) { store_elt(out + j, v); });
  }
}
// PRO_POLY (graphs of one or two tokens): the same rows as the activation tile of the linear behind them, zeros in the padding columns.
static __device__ __noinline__ void stage_poly(const Ctx c, const TaskDesc &d, int B) {
  const int N = d.a[L_GROUPS], K = d.a[L_K];
  const bool vec = ((N | d.a[L_LDX]) & 3) == 0 && (d.p[1] & 15) == 0;
  for (int b = 0; b < B; ++b) {
    __nv_bfloat16 *row = reinterpret_cast<__nv_bfloat16 *>(c.s.xtile + (size_t)b * (K * 2 + kRowPadBytes));
    for (int j = N + threadIdx.x; j < K; j += kConsumerThreads) store_elt(row + j, 0.f);
    poly_norm_row(c, reinterpret_cast<const float *>(d.p[1]) + (size_t)b * d.a[L_LDX], N, vec, d.p[4], __int_as_float(d.a[L_EPS]),
                  [&](int j, float4 v) { store_elt4(row + j, v); }, [&](int j, float v) { store_elt(row + j, v); });
  }
}

// ---------------------------------------------------------------------------
// TASK_SHORT_CONV: out[t][ch] = bias[ch] + sum_j taps[ch][j] in[t - (taps - 1) + j][ch], inputs before the portion come
// from the carried state (zeros before the sequence).  A task owns a channel range of every request.
// ---------------------------------------------------------------------------
// Up to kConvWindow + 1 taps: a warp takes 32 channels and a run of up to eight consecutive tokens, with every input it
// needs (the tokens of its run, the ones before them, carried ones where a request starts) in registers before anything
// is stored.
constexpr int kConvWindow = 4;
template <int HYB>
__device__ __forceinline__ void short_conv_window(const Ctx &c, const TaskDesc &d, const TokenRec *rec, int B) {
  typedef typename HybElt<HYB>::T T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int C = d.a[2], taps = d.a[3], hist = taps - 1;
  const float *in = reinterpret_cast<const float *>(d.p[0]) + d.a[5];
  float *state = reinterpret_cast<float *>(d.p[4]);
  float *out = reinterpret_cast<float *>(d.p[5]);
  const int per = (B + 7) >> 3, t0 = warp * per, n = max(0, min(per, B - t0));
  for (int cb = d.a[0]; cb < d.a[1]; cb += 32) {
    const int ch = cb + lane;
    const bool ok = ch < d.a[1];
    float x[8 + kConvWindow], w[kConvWindow + 1];
    float prev[8][kConvWindow];   // prev[u][j]: the input j + 1 tokens before token t0 + u
    const float ib = (ok && d.p[1]) ? bf16_at(d.p[1], ch) : 0.f, ob = (ok && d.p[3]) ? bf16_at(d.p[3], ch) : 0.f;
#pragma unroll
    for (int j = 0; j <= kConvWindow; ++j) w[j] = (ok && j <= hist) ? bf16_at(d.p[2], (size_t)ch * taps + hist - j) : 0.f;
#pragma unroll
    for (int i = 0; i < 8 + kConvWindow; ++i) {   // x[i]: batch token t0 - kConvWindow + i
      const int t = t0 - kConvWindow + i;
      x[i] = (ok && n > 0 && t >= 0 && i < n + kConvWindow) ? __ldcg(in + (size_t)t * d.a[4] + ch) + ib : 0.f;
    }
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const int t = t0 + u;
      const TokenRec r = rec[u < n ? t : 0];
#pragma unroll
      for (int j = 0; j < kConvWindow; ++j) {
        const int src = t - 1 - j;
        prev[u][j] = src >= r.q0 ? x[kConvWindow + u - 1 - j] : 0.f;
        if (ok && u < n && j < hist && src < r.q0 && !(r.flags & 4))
          prev[u][j] = __ldcg(state + ((size_t)r.slot * hist + (hist + src - r.q0)) * C + ch);
      }
    }
    consumer_sync();   // all carried inputs have been read
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (!ok || u >= n) continue;
      const TokenRec r = rec[t0 + u];
      const float cur = x[kConvWindow + u];
      float v = fmaf(w[0], cur, ob);
#pragma unroll
      for (int j = 0; j < kConvWindow; ++j) v = fmaf(w[j + 1], prev[u][j], v);
      if (d.a[7] == 1) v = v * sigmoid_f(v);
      out[(size_t)(t0 + u) * d.a[6] + ch] = v;
      if (d.p[6]) store_elt(reinterpret_cast<T *>(d.p[6]) + (size_t)(t0 + u) * d.a[8] + ch, v);
      if (r.flags & 2) {   // the last `hist` inputs, oldest first
#pragma unroll
        for (int j = 0; j < kConvWindow; ++j)
          if (j < hist) state[((size_t)r.slot * hist + hist - 1 - j) * C + ch] = j == 0 ? cur : prev[u][j - 1];
      }
    }
  }
}

template <int HYB>
__device__ __noinline__ void run_short_conv(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  if (B <= 0) return;
  TokenRec *rec = reinterpret_cast<TokenRec *>(c.s.xtile);
  token_map(P, B, rec, reinterpret_cast<int *>(c.s.xtile + kTokenMapBytes));
  if (d.a[3] <= kConvWindow + 1) {
    short_conv_window<HYB>(c, d, rec, B);
    return;
  }
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
    if (d.p[6]) store_elt(reinterpret_cast<T *>(d.p[6]) + (size_t)t * d.a[8] + ch, v);
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
// Gate products, plain form: a warp takes two channels (four weight rows) and eight tokens at a time.
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

// The gate products on the tensor cores without losing 32-bit precision: the weights are bf16 as they are, u is the exact
// sum of three bf16 numbers, so three products with float32 accumulation give u's full mantissa.  A unit is (16 rows of one
// gate matrix, half of the columns); `af` holds the first unit's first kGateSteps weight fragments, loaded before the tokens
// were known.
constexpr int kGateSteps = 8;
struct GateUnit {
  uint64_t w;        // gate matrix
  int ch, k0, k1;    // first channel of the 16 (relative to the task), column range
  int mat;
};
__device__ __forceinline__ GateUnit gate_unit(const TaskDesc &d, int u) {
  const int bs = d.a[GL_BS], half = ((bs + 31) >> 5) << 4;
  GateUnit g;
  g.mat = (u >> 1) & 1;
  g.w = d.p[g.mat ? 5 : 3];
  g.ch = (u >> 2) * 16;
  g.k0 = (u & 1) ? half : 0;
  g.k1 = (u & 1) ? bs : min(half, bs);
  return g;
}
__device__ __forceinline__ void gate_fragment(const TaskDesc &d, const GateUnit &g, int k, uint32_t (&a)[4]) {
  const int lane = threadIdx.x & 31, bs = d.a[GL_BS], c0 = d.a[GL_C0], C = d.a[GL_C1] - c0;
#pragma unroll
  for (int i = 0; i < 4; ++i) {   // rows g, g + 8; columns 2 q, 2 q + 8
    const int ch = g.ch + (lane >> 2) + (i & 1) * 8, col = k + 2 * (lane & 3) + (i >> 1) * 8;
    a[i] = (ch < C && col < g.k1) ? __ldg(reinterpret_cast<const uint32_t *>(g.w + 2 * (((size_t)d.a[GL_BLOCK] * bs + c0 + ch) * bs + col))) : 0u;
  }
}
// us: [3][TG][pitch] bf16 (columns past bs are zeros); part: [half][matrix][TG][C] sums.
__device__ __forceinline__ void rglru_gates_mma(const TaskDesc &d, const __nv_bfloat16 *us, int pitch, float *part, int nt,
                                                uint32_t (&af)[kGateSteps][4], bool have) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int C = d.a[GL_C1] - d.a[GL_C0], TG = d.a[GL_TG], units = ((C + 15) >> 4) * 4;
  for (int u = warp; u < units; u += 8) {
    const GateUnit g = gate_unit(d, u);
    for (int n0 = 0; n0 < nt; n0 += 32) {
      float acc[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
      for (int kb = g.k0; kb < g.k1; kb += 16 * kGateSteps) {
        if (!have) {
#pragma unroll
          for (int st = 0; st < kGateSteps; ++st) gate_fragment(d, g, kb + 16 * st, af[st]);
        }
        have = false;
#pragma unroll
        for (int st = 0; st < kGateSteps; ++st) {
          const int k = kb + 16 * st;
          if (k >= g.k1) break;
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            if (n0 + n * 8 >= nt) break;
            const __nv_bfloat16 *x = us + (size_t)(n0 + n * 8 + (lane >> 2)) * pitch + k + 2 * (lane & 3);
#pragma unroll
            for (int h = 0; h < 3; ++h) {
              const uint32_t *xp = reinterpret_cast<const uint32_t *>(x + (size_t)h * TG * pitch);
              mma_bf16_16816(acc[n], af[st], xp[0], xp[4]);
            }
          }
        }
      }
      float *out = part + (size_t)((u & 1) * 2 + g.mat) * TG * C;
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = n0 + n * 8 + 2 * (lane & 3) + (e & 1), ch = g.ch + (lane >> 2) + (e >> 1) * 8;
          if (t < nt && ch < C) out[(size_t)t * C + ch] = acc[n][e];
        }
    }
  }
}

template <int HYB>
__device__ __noinline__ void run_rglru(const Ctx c, const TaskDesc &d) {
  typedef typename HybElt<HYB>::T T;
  const KernelParams &P = c.P;
  const int B = active_tokens(P);
  if (B <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int bs = d.a[GL_BS], c0 = d.a[GL_C0], C = d.a[GL_C1] - c0, TG = d.a[GL_TG], blk = d.a[GL_BLOCK], width = d.a[GL_WIDTH];
  const bool mma = HYB == HYB_BF16 && (bs & 1) == 0;
  const int gch = blk * bs + c0;   // first channel of this task
  uint32_t af[kGateSteps][4];
  if (mma && warp < ((C + 15) >> 4) * 4) {
    const GateUnit g = gate_unit(d, warp);
#pragma unroll
    for (int st = 0; st < kGateSteps; ++st) gate_fragment(d, g, g.k0 + 16 * st, af[st]);
  }
  float *state = *reinterpret_cast<float *const *>(&d.a[GL_STATE]);
  T *outp = *reinterpret_cast<T *const *>(&d.a[GL_OUT]);
  const float oscale = __int_as_float(d.a[GL_OSCALE]), gate_c = __int_as_float(d.a[GL_GATE_C]);
  TokenRec *rec = reinterpret_cast<TokenRec *>(c.s.xtile);
  float *chp = reinterpret_cast<float *>(c.s.xtile + kTokenMapBytes);   // [4][64] per channel: gate biases, decay * softplus(lambda), y bias
  float *part = chp + 256;                                              // [half][matrix][TG][C]; [0][0] then holds a, [0][1] b and then S
  float *us = part + 4 * (size_t)TG * C;                                // [TG][bs], or three bf16 parts [3][TG][pitch]
  const int pitch = ((bs + 15) & ~15) + 8;
  __nv_bfloat16 *uh = reinterpret_cast<__nv_bfloat16 *>(us);
  if (tid < C) {
    chp[tid] = bf16_at(d.p[4], gch + tid);
    chp[64 + tid] = bf16_at(d.p[6], gch + tid);
    chp[128 + tid] = gate_c * softplus_f(bf16_at(d.p[7], gch + tid));
    chp[192 + tid] = bf16_at(d.p[2], gch + tid);
  }
  token_map(P, B, rec, reinterpret_cast<int *>(us));
  float *rs = part, *is = part + (size_t)TG * C;
  float carry = 0.f;               // state of channel tid between token groups
  for (int tb = 0; tb < B; tb += TG) {
    const int nt = min(TG, B - tb);
    const float *ug = reinterpret_cast<const float *>(d.p[0]) + (size_t)tb * d.a[GL_LDU] + (size_t)blk * bs;
    const float *yg = reinterpret_cast<const float *>(d.p[1]) + (size_t)tb * d.a[GL_LDP] + d.a[GL_YOFF] + gch;
    for (int t = warp; t < nt; t += 8) {
#pragma unroll 8
      for (int k = lane; k < (mma ? pitch - 8 : bs); k += 32) {
        const float v = k < bs ? __ldcg(ug + (size_t)t * d.a[GL_LDU] + k) : 0.f;
        if (mma) {
          const __nv_bfloat16 h = __float2bfloat16_rn(v);
          const float r1 = v - bf16_to_f(h);
          const __nv_bfloat16 m = __float2bfloat16_rn(r1);
          uh[(size_t)t * pitch + k] = h;
          uh[(size_t)(TG + t) * pitch + k] = m;
          uh[(size_t)(2 * TG + t) * pitch + k] = __float2bfloat16_rn(r1 - bf16_to_f(m));
        } else {
          us[(size_t)t * bs + k] = v;
        }
      }
    }
    // the elementwise inputs of this thread's first items travel while the gates are formed
    float y0[4], u0[4];
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int i = tid + q * kConsumerThreads, t = i / C, ch = i - t * C;
      y0[q] = i < nt * C ? __ldcg(yg + (size_t)t * d.a[GL_LDP] + ch) : 0.f;
      u0[q] = i < nt * C ? __ldcg(ug + (size_t)t * d.a[GL_LDU] + c0 + ch) : 0.f;
    }
    consumer_sync();
    if (mma) rglru_gates_mma(d, uh, pitch, part, nt, af, tb == 0 && warp < ((C + 15) >> 4) * 4);
    else if ((bs & 1) == 0) rglru_gates<HYB, true>(d, us, rs, is, nt);
    else rglru_gates<HYB, false>(d, us, rs, is, nt);
    consumer_sync();
#pragma unroll 1
    for (int q = 0; q * kConsumerThreads < nt * C; ++q) {
      const int i = tid + q * kConsumerThreads;
      if (i >= nt * C) break;
      const int t = i / C, ch = i - t * C;
      float rp = rs[i], ip = is[i];
      if (mma) { rp += part[2 * (size_t)TG * C + i]; ip += part[3 * (size_t)TG * C + i]; }
      const float u = q == 0 ? u0[0] : q == 1 ? u0[1] : q == 2 ? u0[2] : q == 3 ? u0[3] : __ldcg(ug + (size_t)t * d.a[GL_LDU] + c0 + ch);
      const float r = sigmoid_f(rp + chp[ch]), gi = sigmoid_f(ip + chp[64 + ch]);
      const float la = -r * chp[128 + ch];
      float a = decay_exp(la), b = sqrtf(-expm1f(2.0f * la)) * gi * u;
      const TokenRec &tr = rec[tb + t];
      if (tr.flags & 1) {   // the request's carried state enters here; nothing flows in from the previous token
        if (!(tr.flags & 4)) b = fmaf(a, __ldcg(state + (size_t)tr.slot * width + gch + ch), b);
        a = 0.f;
      }
      rs[i] = a;
      is[i] = b;
    }
    consumer_sync();
    if (tid < C) {
      float S = carry;
#pragma unroll 4
      for (int t = 0; t < nt; ++t) {
        S = fmaf(rs[(size_t)t * C + tid], S, is[(size_t)t * C + tid]);
        is[(size_t)t * C + tid] = S;
      }
      carry = S;
    }
    consumer_sync();
#pragma unroll 1
    for (int q = 0; q * kConsumerThreads < nt * C; ++q) {
      const int i = tid + q * kConsumerThreads;
      if (i >= nt * C) break;
      const int t = i / C, ch = i - t * C;
      const float S = is[i];
      const TokenRec &tr = rec[tb + t];
      if (tr.flags & 2) state[(size_t)tr.slot * width + gch + ch] = S;
      const float yp = q == 0 ? y0[0] : q == 1 ? y0[1] : q == 2 ? y0[2] : q == 3 ? y0[3] : __ldcg(yg + (size_t)t * d.a[GL_LDP] + ch);
      store_elt(outp + (size_t)(tb + t) * d.a[GL_LDO] + d.a[GL_OCOL] + gch + ch, S * gelu_tanh_f(yp + chp[192 + ch]) * oscale);
    }
    consumer_sync();
  }
}

// ---------------------------------------------------------------------------
// TASK_SELECTIVE_SCAN (Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces"): a channel range of every
// request.  Per channel c and state n
//   dt = softplus(W_dt low + b),  S = exp(-dt exp(A_log)) S + dt u B,  y = (sum_n S C + D u) * silu(z)
// SS_LANES neighbouring lanes share a channel, four states each, so that a block walks 256 / SS_LANES channels at a time through the
// tokens of the batch; the step sizes' low-rank product is part of the task.  A request's state enters at its first token of the
// batch and is written back at its last; every thread copies its own piece of the states to come into its own cells of a ring.
// The phases are functions of their own, called one after the other: what one keeps in registers is not spilled in another's loop (a
// further level of calls would cost every task body registers).
// ---------------------------------------------------------------------------
// Shared memory of a task.
struct ScanMem {
  TokenRec *rec;        // [64]
  int *seqs;            // [64] state slot of the batch's requests in order, -1: starts from zeros
  int *tok;             // [64] state slot << 2 | first token of its request in the batch << 1 | last one
  int *qo;              // [requests + 1]
  float *bc;            // [B][2 NP] B, C
  float *us;            // [B][CP] inputs
  float *dts;           // [B][CP] step sizes, then read-outs
  float *low;           // [B][scan_pitch] columns of the low-rank part
  __nv_bfloat16 *w;     // [CP][scan_pitch] weights of the step sizes
  float *gate;          // [B][CP] (in the place of low and w, once the step sizes are there)
  float4 *ring;         // [kScanRing][256] states to come (likewise)
};
__device__ __forceinline__ ScanMem scan_mem(const Ctx &c, const TaskDesc &d, int B) {
  const int NP = d.a[SS_NP], CP = kConsumerThreads / d.a[SS_LANES];
  ScanMem m;
  m.rec = reinterpret_cast<TokenRec *>(c.s.xtile);
  m.seqs = reinterpret_cast<int *>(c.s.xtile + kTokenMapBytes);
  m.tok = m.seqs + kMaxLinearTokens;
  m.qo = m.tok + kMaxLinearTokens;
  m.bc = reinterpret_cast<float *>(m.qo + ((c.P.max_num_batched_requests + 4) & ~3));
  m.us = m.bc + B * 2 * NP;
  m.dts = m.us + B * CP;
  m.low = m.gate = m.dts + B * CP;
  m.w = reinterpret_cast<__nv_bfloat16 *>(m.low + B * scan_pitch(d.a[SS_RANK]));
  m.ring = reinterpret_cast<float4 *>(m.gate + B * CP);
  return m;
}
// `rows` rows of `bytes` bytes, 16-byte asynchronous copies: one warp per row, or WIDE (a power of two) neighbouring threads per row.
template <int WIDE = 32>
__device__ __forceinline__ void scan_copy(uint32_t dst, int pitch, const void *src, int ld, int rows, int bytes) {
#pragma unroll 1
  for (int t = threadIdx.x / WIDE; t < rows; t += kConsumerThreads / WIDE)
    for (int j = threadIdx.x % WIDE * 16; j < bytes; j += WIDE * 16)
      cp_async16(dst + t * pitch + j, reinterpret_cast<const uint8_t *>(src) + (size_t)t * ld + j);
}
// The same for floats at any alignment.
__device__ __forceinline__ void scan_copy_plain(float *dst, int pitch, const float *src, int ld, int rows, int cols) {
  for (int i = threadIdx.x; i < rows * cols; i += kConsumerThreads) dst[i / cols * pitch + i % cols] = __ldcg(src + (size_t)(i / cols) * ld + i % cols);
}
__device__ __forceinline__ bool scan_aligned(const TaskDesc &d) {
  return ((d.a[SS_C0] | d.a[SS_C] | d.a[SS_N] | d.a[SS_LDU] | d.a[SS_LDL] | d.a[SS_LDG] | d.a[SS_GOFF]) & 3) == 0 && (d.a[SS_RANK] & 7) == 0 &&
         ((d.p[0] | d.p[1] | d.p[2] | d.p[3]) & 15) == 0;
}
// Requests what the task needs for channels [cb, cb + nc): inputs, B and C, columns [r0, ..) of the low-rank part and of its weights;
// then the places of the batch's tokens.
template <int HYB>
__device__ __noinline__ void scan_load(const Ctx c, const TaskDesc &d, int B, int cb, int nc, int r0) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rank = d.a[SS_RANK], NP = d.a[SS_NP], N = d.a[SS_N], CP = kConsumerThreads / d.a[SS_LANES], pitch = scan_pitch(rank);
  const int rn = min(pitch - 8, rank - r0), rpad = (rn + 15) & ~15;
  const bool vec = scan_aligned(d);
  const ScanMem m = scan_mem(c, d, B);
  const float *low = reinterpret_cast<const float *>(d.p[1]);
  const float *u = reinterpret_cast<const float *>(d.p[0]) + cb;
  const __nv_bfloat16 *w = reinterpret_cast<const __nv_bfloat16 *>(d.p[3]) + (size_t)cb * rank + r0;
  const bool first = r0 == 0 && cb == d.a[SS_C0];
  if (vec) {
    if (HYB == HYB_BF16) scan_copy(smem_u32(m.w), pitch * 2, w, rank * 2, nc, rn * 2);
    scan_copy(smem_u32(m.low), pitch * 4, low + r0, d.a[SS_LDL] * 4, B, rn * 4);
    if (r0 == 0) scan_copy<16>(smem_u32(m.us), CP * 4, u, d.a[SS_LDU] * 4, B, nc * 4);
    if (first) scan_copy<8>(smem_u32(m.bc), NP * 8, low + rank, d.a[SS_LDL] * 4, B, NP * 8);
  } else {
    if (HYB == HYB_BF16)
      for (int i = tid; i < nc * rn; i += kConsumerThreads) m.w[i / rn * pitch + i % rn] = __ldg(w + (size_t)(i / rn) * rank + i % rn);
    scan_copy_plain(m.low, pitch, low + r0, d.a[SS_LDL], B, rn);
    if (r0 == 0) scan_copy_plain(m.us, CP, u, d.a[SS_LDU], B, nc);
    if (first)
      for (int i = tid; i < B * 2 * NP; i += kConsumerThreads) {
        const int t = i / (2 * NP), j = i - t * 2 * NP, n = j % NP;
        m.bc[i] = n < N ? __ldcg(low + (size_t)t * d.a[SS_LDL] + rank + (j < NP ? n : N + n)) : 0.f;
      }
  }
  if (rpad > rn) {   // columns up to a whole 16: zeros on both sides
    const int z = rpad - rn;
    for (int i = tid; i < B * z; i += kConsumerThreads) m.low[i / z * pitch + rn + i % z] = 0.f;
    if (HYB == HYB_BF16)
      for (int i = tid; i < nc * z; i += kConsumerThreads) m.w[i / z * pitch + rn + i % z] = __float2bfloat16_rn(0.f);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (first) {
    token_map(c.P, B, m.rec, m.qo);
    if (warp == 0) {
      const int f0 = lane < B ? m.rec[lane].flags : 0, f1 = 32 + lane < B ? m.rec[32 + lane].flags : 0;
      const unsigned b0 = __ballot_sync(0xffffffffu, f0 & 1), b1 = __ballot_sync(0xffffffffu, f1 & 1), before = (1u << lane) - 1u;
      m.seqs[lane] = m.seqs[32 + lane] = -1;
      __syncwarp();
      if (f0 & 1) m.seqs[__popc(b0 & before)] = f0 & 4 ? -1 : m.rec[lane].slot;
      if (f1 & 1) m.seqs[__popc(b0) + __popc(b1 & before)] = f1 & 4 ? -1 : m.rec[32 + lane].slot;
      if (lane < B) m.tok[lane] = m.rec[lane].slot << 2 | (f0 & 1) << 1 | (f0 & 2) >> 1;
      if (32 + lane < B) m.tok[32 + lane] = m.rec[32 + lane].slot << 2 | (f1 & 1) << 1 | (f1 & 2) >> 1;
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  consumer_sync();
}
// Three bf16 parts of two neighbouring values; their sum is the float32 value.
__device__ __forceinline__ void split3(const float2 v, uint32_t (&p)[3]) {
  p[0] = pack_bf16(v.x, v.y);
  const float a = v.x - bf16_lo(p[0]), b = v.y - bf16_hi(p[0]);
  p[1] = pack_bf16(a, b);
  p[2] = pack_bf16(a - bf16_lo(p[1]), b - bf16_hi(p[1]));
}
// Step sizes from the columns at hand (added to what earlier columns gave).  Tensor cores, without losing 32-bit precision: the
// weights are bf16 as they are, the low-rank part is split into three bf16 numbers.  A unit of a warp is 16 MT channels x 8 tokens.
template <int MT>
__device__ __forceinline__ void scan_products(const ScanMem &m, int B, int nc, int CP, int pitch, int rn, bool add) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = (B + 7) >> 3, units = (nc + 16 * MT - 1) / (16 * MT) * groups;
#pragma unroll 1
  for (int u = warp; u < units; u += 8) {
    const int t0 = u % groups * 8, c0 = u / groups * 16 * MT;
    // (rows past the channels or the batch repeat the last one; what they give is not stored)
    uint32_t wa[MT];
#pragma unroll
    for (int i = 0; i < MT; ++i) wa[i] = smem_u32(m.w + min(c0 + 16 * i + (lane & 15), nc - 1) * pitch) + (uint32_t)(lane >> 4) * 16u;
    const uint32_t xa = smem_u32(m.low + min(t0 + (lane >> 2), B - 1) * pitch + 2 * (lane & 3));
    float acc[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll 1
    for (int k = 0; k < rn; k += 16) {
      uint32_t a[MT][4], p0[3], p1[3];
      split3(lds_f32x2(xa + 4 * k), p0);
      split3(lds_f32x2(xa + 4 * k + 32), p1);
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmatrix_x4(a[i], wa[i] + 2 * k);
#pragma unroll
      for (int h = 0; h < 3; ++h)
#pragma unroll
        for (int i = 0; i < MT; ++i) mma_bf16_16816(acc[i], a[i], p0[h], p1[h]);
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = t0 + 2 * (lane & 3) + (e & 1), ch = c0 + 16 * i + (lane >> 2) + (e >> 1) * 8;
        if (t < B && ch < nc) m.dts[t * CP + ch] = add ? m.dts[t * CP + ch] + acc[i][e] : acc[i][e];
      }
  }
}
template <int HYB>
__device__ __noinline__ void scan_steps(const Ctx c, const TaskDesc &d, int B, int cb, int nc, int r0) {
  const int tid = threadIdx.x;
  const int rank = d.a[SS_RANK], CP = kConsumerThreads / d.a[SS_LANES], pitch = scan_pitch(rank), rn = min(pitch - 8, rank - r0);
  const ScanMem m = scan_mem(c, d, B);
  const bool last = r0 + rn >= rank;
  // a thread keeps its channel in what follows
  const int ch = tid % CP, tstep = kConsumerThreads / CP;
  const float bias = last && ch < nc ? bf16_at(d.p[4], cb + ch) : 0.f;
  if (HYB == HYB_BF16) {
    // (as many units as warps, if there are channels enough)
    if (B <= 16) scan_products<1>(m, B, nc, CP, pitch, rn, r0 > 0);
    else if (B <= 32) scan_products<2>(m, B, nc, CP, pitch, rn, r0 > 0);
    else scan_products<4>(m, B, nc, CP, pitch, rn, r0 > 0);
  } else {
#pragma unroll 1
    for (int i = tid; i < nc * ((B + 7) >> 3); i += kConsumerThreads) {   // a channel, eight tokens
      const int ch = i % nc, t0 = i / nc * 8;
      const size_t row = (size_t)(cb + ch) * rank + r0;
      float acc[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) acc[u] = 0.f;
#pragma unroll 8
      for (int k = 0; k < rn; ++k) {
        const float w = bf16_at(d.p[3], row + k);
#pragma unroll
        for (int u = 0; u < 8; ++u) acc[u] = fmaf(w, m.low[min(t0 + u, B - 1) * pitch + k], acc[u]);
      }
#pragma unroll
      for (int u = 0; u < 8; ++u)
        if (t0 + u < B) m.dts[(t0 + u) * CP + ch] = r0 > 0 ? m.dts[(t0 + u) * CP + ch] + acc[u] : acc[u];
    }
  }
  consumer_sync();
  if (!last) return;
  // the gate travels while the recurrence is walked
  if (scan_aligned(d)) scan_copy<16>(smem_u32(m.gate), CP * 4, reinterpret_cast<const float *>(d.p[2]) + d.a[SS_GOFF] + cb, d.a[SS_LDG] * 4, B, nc * 4);
#pragma unroll 2
  for (int t = ch < nc ? tid / CP : B; t < B; t += tstep) m.dts[t * CP + ch] = softplus_f(m.dts[t * CP + ch] + bias);
  consumer_sync();
}

// Two float32 values in one 64-bit register, and the arithmetic that takes both at once.
__device__ __forceinline__ uint64_t f2(float x, float y) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float2 f2_parts(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
// exp(x) for x <= 0, to the last bit near 1 (a decay that is applied once per token must not be off to one side): exp(x) = 2^n exp(r)
// with n = round(x / ln 2) and the Taylor series of exp(r) - 1, without branches and conversions.
__device__ __forceinline__ uint64_t scan_decay2(uint64_t v) {
  constexpr float kRound = 12582912.0f;   // 1.5 x 2^23: added, it leaves the nearest integer in the low bits
  auto both = [](float x) { return f2(x, x); };
  const float2 u = f2_parts(v);
  const uint64_t x = f2(fmaxf(u.x, -87.0f), fmaxf(u.y, -87.0f));
  const uint64_t t = fma2(x, both(1.44269504f), both(kRound));
  const uint64_t r = fma2(add2(t, both(-kRound)), both(-0.69314718f), x);   // |r| <= 0.35
  uint64_t p = fma2(r, both(1.0f / 720.0f), both(1.0f / 120.0f));
  p = fma2(p, r, both(1.0f / 24.0f));
  p = fma2(p, r, both(1.0f / 6.0f));
  p = fma2(p, r, both(0.5f));
  p = fma2(p, mul2(r, r), r);                                               // exp(r) - 1
  const float2 n = f2_parts(t);
  const uint64_t s = f2(__int_as_float((__float_as_int(n.x) << 23) + 0x3f800000), __int_as_float((__float_as_int(n.y) << 23) + 0x3f800000));
  return fma2(s, p, s);
}
struct ScanState { uint64_t a, b; };   // four states of a thread
__device__ __forceinline__ ScanState scan_state(const float4 v) { return ScanState{f2(v.x, v.y), f2(v.z, v.w)}; }
__device__ __forceinline__ ScanState lds_state(uint32_t a) {
  ScanState v;
  asm volatile("ld.shared.v2.b64 {%0, %1}, [%2];" : "=l"(v.a), "=l"(v.b) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ void scan_update(ScanState &S, const ScanState &e, const ScanState &x) {
  S.a = fma2(e.a, S.a, x.a);
  S.b = fma2(e.b, S.b, x.b);
}
__device__ __forceinline__ float scan_read(const ScanState &S, const ScanState &k) {
  const float2 y = f2_parts(fma2(S.a, k.a, mul2(S.b, k.b)));
  return y.x + y.y;
}

// The recurrence over channels [cb, cb + nc).  Four tokens at a time where none of them begins or ends a request, or where all of them
// are single tokens of requests of their own; else one by one.
static __device__ __noinline__ void scan_walk(const Ctx c, const TaskDesc &d, int B, int cb, int nc) {
  const int tid = threadIdx.x, N = d.a[SS_N], NP = d.a[SS_NP], LPC = d.a[SS_LANES], CP = kConsumerThreads / LPC, stride = d.a[SS_C] * NP;
  const int ch = tid / LPC, n0 = tid % LPC * 4, q = tid & 3;
  const bool on = ch < nc && n0 < NP;          // this thread holds states (the others walk along and write nothing)
  float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 4; ++e)
    if (on && n0 + e < N) a[e] = bf16_at(d.p[5], (size_t)(cb + ch) * N + n0 + e);
  const ScanMem m = scan_mem(c, d, B);
  float *mine = reinterpret_cast<float *>(wide_arg(d, SS_STATE)) + (on ? (size_t)(cb + ch) * NP + n0 : 0);
  const uint32_t ring = smem_u32(m.ring + tid), rows = (uint32_t)(B * CP) * 4u, step = (uint32_t)CP * 4u, bstep = (uint32_t)NP * 8u;
  constexpr uint32_t kSlot = kConsumerThreads * 16;
  uint32_t tok = smem_u32(m.tok), bc = smem_u32(m.bc + min(n0, NP - 4)), cell = smem_u32(m.us + ch);   // (dts lies `rows` bytes behind us)
  uint32_t put = ring, get = ring, next = smem_u32(m.seqs), seq = next;   // ring cells and requests to fetch and to use next
  const uint32_t end = next + 4 * kMaxLinearTokens;
  auto turn = [&](uint32_t at) { return at + kSlot == ring + kScanRing * kSlot ? ring : at + kSlot; };
  auto slot_of = [&](uint32_t at) { return on && at < end ? lds_s32(min(at, end - 4)) : -1; };   // of a request, -1: nothing to fetch
  auto fetch = [&](int slot) {
    asm volatile("{\n.reg .pred p;\nsetp.ge.s32 p, %2, 0;\n@p cp.async.cg.shared.global [%0], [%1], 16;\n}" ::"r"(put), "l"(mine + (size_t)max(slot, 0) * stride), "r"(slot)
                 : "memory");
    asm volatile("cp.async.commit_group;" ::: "memory");
    next += 4;
    put = turn(put);
  };
  auto entering = [&](int slot) {   // the state a request brings
    const ScanState s = lds_state(get);
    get = turn(get);
    return ScanState{slot >= 0 ? s.a : 0ull, slot >= 0 ? s.b : 0ull};
  };
  auto leaving = [&](const ScanState &S, int slot) {
    const float2 lo = f2_parts(S.a), hi = f2_parts(S.b);
    *reinterpret_cast<float4 *>(mine + (size_t)slot * stride) = make_float4(lo.x, lo.y, hi.x, hi.y);
  };
#pragma unroll 1
  for (int j = 0; j < kScanRing - 1; ++j) fetch(slot_of(next));   // (the gate's copies join the first group)
  const ScanState A = scan_state(make_float4(-expf(a[0]), -expf(a[1]), -expf(a[2]), -expf(a[3])));
  ScanState S{0ull, 0ull};
#pragma unroll 1
  for (int t = 0; t < B;) {
    const int4 info = lds_v4(tok & ~15u);
    const bool four = (t & 3) == 0 && t + 4 <= B, plain = four && ((info.x | info.y | info.z | info.w) & 3) == 0;
    if (plain || (four && (info.x & info.y & info.z & info.w & 3) == 3)) {
      ScanState e[4], x[4], k[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float dt = lds_f32(cell + rows + i * step), du = dt * lds_f32(cell + i * step);
        const ScanState b = lds_state(bc + i * bstep);
        k[i] = lds_state(bc + i * bstep + NP * 4u);
        e[i].a = scan_decay2(mul2(f2(dt, dt), A.a));
        e[i].b = scan_decay2(mul2(f2(dt, dt), A.b));
        x[i].a = mul2(f2(du, du), b.a);
        x[i].b = mul2(f2(du, du), b.b);
      }
      float y[4];
      if (plain) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          scan_update(S, e[i], x[i]);
          y[i] = scan_read(S, k[i]);
        }
      } else {
        const int slot[4] = {info.x >> 2, info.y >> 2, info.z >> 2, info.w >> 2};
        int from[4], then[4];
        ScanState s[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          from[i] = slot_of(seq + 4 * i);
          then[i] = slot_of(next + 4 * i);
        }
        seq += 16;
        asm volatile("cp.async.wait_group %0;" ::"n"(kScanRing - 5) : "memory");   // the four oldest of kScanRing - 1
#pragma unroll
        for (int i = 0; i < 4; ++i) s[i] = entering(from[i]);
#pragma unroll
        for (int i = 0; i < 4; ++i) scan_update(s[i], e[i], x[i]);
        if (on)
#pragma unroll
          for (int i = 0; i < 4; ++i) leaving(s[i], slot[i]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          y[i] = scan_read(s[i], k[i]);
          fetch(then[i]);
        }
      }
      // sums over the lanes of a channel; lane q of the last four ends up with token q's
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] = on ? y[i] : 0.f;
      for (int s = LPC >> 1; s > 2; s >>= 1)
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] += __shfl_xor_sync(0xffffffffu, y[i], s);
      float y0 = q & 2 ? y[2] : y[0], y1 = q & 2 ? y[3] : y[1];
      y0 += __shfl_xor_sync(0xffffffffu, q & 2 ? y[0] : y[2], 2);
      y1 += __shfl_xor_sync(0xffffffffu, q & 2 ? y[1] : y[3], 2);
      const float sum = (q & 1 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, q & 1 ? y0 : y1, 1);
      if (ch < nc && n0 < 16) sts_f32(cell + rows + q * step, sum);   // (the step sizes there have been read before the shuffles)
      t += 4; cell += 4 * step; bc += 4 * bstep; tok += 16;
      continue;
    }
    const int here = lds_s32(tok);
    const float dt = lds_f32(cell + rows), du = dt * lds_f32(cell);
    const ScanState b = lds_state(bc), k = lds_state(bc + NP * 4u);
    if (here & 2) {
      fetch(slot_of(next));
      asm volatile("cp.async.wait_group %0;" ::"n"(kScanRing - 1) : "memory");
      S = entering(slot_of(seq));
      seq += 4;
    }
    scan_update(S, ScanState{scan_decay2(mul2(f2(dt, dt), A.a)), scan_decay2(mul2(f2(dt, dt), A.b))}, ScanState{mul2(f2(du, du), b.a), mul2(f2(du, du), b.b)});
    if ((here & 1) && on) leaving(S, here >> 2);
    float y = on ? scan_read(S, k) : 0.f;
    for (int s = LPC >> 1; s > 0; s >>= 1) y += __shfl_xor_sync(0xffffffffu, y, s);
    if (ch < nc && n0 == 0) sts_f32(cell + rows, y);
    ++t; cell += step; bc += bstep; tok += 4;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  consumer_sync();
}

// (y + D u) * silu(z)
template <int HYB>
__device__ __noinline__ void scan_emit(const Ctx c, const TaskDesc &d, int B, int cb, int nc) {
  typedef typename HybElt<HYB>::T T;
  const int tid = threadIdx.x, CP = kConsumerThreads / d.a[SS_LANES];
  const ScanMem m = scan_mem(c, d, B);
  T *out = reinterpret_cast<T *>(d.p[7]) + cb;
  if (scan_aligned(d) && (d.a[SS_LDO] & 3) == 0 && ((d.p[6] | d.p[7]) & 15) == 0) {
    const int j = tid % (CP >> 2) * 4;   // a thread keeps its channels
    const float4 D = j < nc ? bf16x4_at(d.p[6], cb + j) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
    for (int t = j < nc ? tid / (CP >> 2) : B; t < B; t += kConsumerThreads * 4 / CP) {
      const float4 y = *reinterpret_cast<const float4 *>(m.dts + t * CP + j), u = *reinterpret_cast<const float4 *>(m.us + t * CP + j);
      const float4 z = *reinterpret_cast<const float4 *>(m.gate + t * CP + j);
      store_elt4(out + (size_t)t * d.a[SS_LDO] + j, make_float4(fmaf(D.x, u.x, y.x) * silu_exact_f(z.x), fmaf(D.y, u.y, y.y) * silu_exact_f(z.y),
                                                                fmaf(D.z, u.z, y.z) * silu_exact_f(z.z), fmaf(D.w, u.w, y.w) * silu_exact_f(z.w)));
    }
  } else {
#pragma unroll 1
    for (int i = tid; i < B * nc; i += kConsumerThreads) {
      const int t = i / nc, j = i - t * nc;
      const float z = __ldcg(reinterpret_cast<const float *>(d.p[2]) + (size_t)t * d.a[SS_LDG] + d.a[SS_GOFF] + cb + j);
      store_elt(out + (size_t)t * d.a[SS_LDO] + j, fmaf(bf16_at(d.p[6], cb + j), m.us[t * CP + j], m.dts[t * CP + j]) * silu_exact_f(z));
    }
  }
  consumer_sync();   // the next channels reuse the arrays and the ring
}

template <int HYB>
__device__ __forceinline__ void run_selective_scan(const Ctx &c, const TaskDesc &d, int task) {
  const int B = min(active_tokens(c.P), kMaxLinearTokens);
  if (B <= 0) return;
#pragma unroll 1
  for (int cb = d.a[SS_C0]; cb < d.a[SS_C1]; cb += kConsumerThreads / d.a[SS_LANES]) {
    const int nc = min(kConsumerThreads / d.a[SS_LANES], d.a[SS_C1] - cb);
#pragma unroll 1
    for (int r0 = 0; r0 < d.a[SS_RANK]; r0 += kScanRank) {
      scan_load<HYB>(c, d, B, cb, nc, r0);
      stamp(c, task, 0);
      scan_steps<HYB>(c, d, B, cb, nc, r0);
    }
    stamp(c, task, 1);
    scan_walk(c, d, B, cb, nc);
    stamp(c, task, 2);
    scan_emit<HYB>(c, d, B, cb, nc);
  }
}

// ---------------------------------------------------------------------------
// TASK_MLSTM: (request, head, range of value columns).  Matrix memory S [dim, columns] in registers: a thread holds RPT
// consecutive rows of 4 columns, the block 4 CQ columns of all rows (256 RPT / CQ of them; keys and queries are padded with
// zeros up to that, so padding rows stay zero); the columns of the task are walked in sub-blocks.  Per token
//   m' = max(f + m, i), S = exp(f + m - m') S + exp(i - m') k v^T, n likewise, o = S^T q / (max(|n q|, exp(-m')) + 1e-6)
// Every task keeps its own copy of (n, m), so that tasks of one head share nothing while they run.  The normalised and
// gated output needs the whole head: the last task of the (request, head) to finish writes it.
// ---------------------------------------------------------------------------
struct MlstmView {
  const float *proj;   // projections of the request's first token
  float *nm, *S, *raw;
  int ldp, H, h, dim, vdim, vdimp, V0, V1, chunks;
  bool fresh;
};
__device__ __forceinline__ MlstmView mlstm_view(const TaskDesc &d, const SeqView &sv) {
  MlstmView m;
  m.ldp = d.a[ML_LDP]; m.H = d.a[ML_H]; m.h = d.a[ML_HEAD]; m.dim = d.a[ML_DIM]; m.vdim = d.a[ML_VDIM]; m.vdimp = d.a[ML_VDIMP];
  m.V0 = d.a[ML_V0]; m.V1 = d.a[ML_V1]; m.chunks = d.a[ML_NCHUNK];
  m.fresh = sv.pos0 == 0;
  m.proj = reinterpret_cast<const float *>(d.p[0]) + (size_t)sv.q0 * m.ldp;
  m.nm = reinterpret_cast<float *>(d.p[5]) + ((size_t)(sv.slot * m.H + m.h) * m.chunks + d.a[ML_CHUNK]) * (m.dim + 1);
  m.S = reinterpret_cast<float *>(d.p[4]) + (size_t)(sv.slot * m.H + m.h) * m.dim * m.vdimp;
  m.raw = reinterpret_cast<float *>(d.p[6]) + (size_t)sv.q0 * d.a[ML_LDR] + (size_t)m.h * m.vdim;
  return m;
}
// log gates from the pre-activations
__device__ __forceinline__ float mlstm_log_i(float pre, float cap) { return cap * tanhf(pre / cap); }
__device__ __forceinline__ float mlstm_log_f(float pre, float cap) { return -softplus_f(-cap * tanhf(pre / cap)); }

// True for the task that finishes a (request, head).  Ends with a barrier.
__device__ __forceinline__ bool last_of_head(const Ctx &c, int ticket_id, int chunks) {
  consumer_sync();
  if (chunks == 1) return true;
  if (threadIdx.x == 0) {
    unsigned int *ticket = &c.P.attn_tickets[ticket_id];
    unsigned int old;
    asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(old) : "l"(ticket) : "memory");
    const bool last = old + 1u == (unsigned)chunks;
    if (last) *reinterpret_cast<volatile unsigned int *>(ticket) = 0u;
    c.s.flags[1] = last ? 1 : 0;
  }
  consumer_sync();
  return c.s.flags[1] != 0;
}

// One step of S and the read-out for this thread's rows (k scaled by the input gate).
template <int RPT>
__device__ __forceinline__ float4 mlstm_step(float4 (&S)[RPT], float a, const float4 v, const float *kt, const float *qt) {
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RPT; i += 4) {
    const float4 k4 = *reinterpret_cast<const float4 *>(kt + i), q4 = *reinterpret_cast<const float4 *>(qt + i);
    const float k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float4 &s = S[i + e];
      s.x = fmaf(a, s.x, k[e] * v.x); o.x = fmaf(q[e], s.x, o.x);
      s.y = fmaf(a, s.y, k[e] * v.y); o.y = fmaf(q[e], s.y, o.y);
      s.z = fmaf(a, s.z, k[e] * v.z); o.z = fmaf(q[e], s.z, o.z);
      s.w = fmaf(a, s.w, k[e] * v.w); o.w = fmaf(q[e], s.w, o.w);
    }
  }
  return o;
}
// Sum over the row groups of a warp (lanes that differ above bit log2(CQ)); valid in lanes < CQ.
template <int CQ>
__device__ __forceinline__ float4 mlstm_warp_rows(float4 o) {
#pragma unroll
  for (int s = CQ; s < 32; s <<= 1) {
    o.x += __shfl_xor_sync(0xffffffffu, o.x, s);
    o.y += __shfl_xor_sync(0xffffffffu, o.y, s);
    o.z += __shfl_xor_sync(0xffffffffu, o.z, s);
    o.w += __shfl_xor_sync(0xffffffffu, o.w, s);
  }
  return o;
}

// A portion of several tokens.
template <int HYB, int CQ, int RPT>
__device__ __noinline__ void mlstm_portion(const Ctx c, const TaskDesc &d, const SeqView sv, int task) {
  typedef typename HybElt<HYB>::T T;
  constexpr int VC = 4 * CQ, RG = kConsumerThreads / CQ, ROWS = RG * RPT;
  constexpr int NR = (ROWS + kConsumerThreads - 1) / kConsumerThreads;   // rows of n per thread
  const MlstmView m = mlstm_view(d, sv);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qd = tid % CQ, r0 = tid / CQ * RPT, TC = d.a[ML_TC];
  // shared memory
  float *dec = reinterpret_cast<float *>(c.s.xtile);   // [64] exp(f + m - m')
  float *inp = dec + kMaxLinearTokens;                 // [64] exp(i - m')
  float *den = inp + kMaxLinearTokens;                 // [64] exp(-m'), then the denominator
  float *nred = den + kMaxLinearTokens;                // [TC][8]
  float *ks = nred + TC * 8;                           // [TC][ROWS] input-scaled keys
  float *qs = ks + (size_t)TC * ROWS;                  // [TC][ROWS]
  float *vs = qs + (size_t)TC * ROWS;                  // [TC][VC]
  float *red = vs + (size_t)TC * VC;                   // [TC][8 warps][VC]
  const float cap = __int_as_float(d.a[ML_CAP]), qscale = __int_as_float(d.a[ML_QSCALE]);
  // gates of all tokens, then the running maximum (one thread: a handful of operations per token)
  for (int t = tid; t < sv.nq; t += kConsumerThreads) {
    inp[t] = mlstm_log_i(__ldcg(m.proj + (size_t)t * m.ldp + d.a[ML_IOFF] + m.h) + bf16_at(d.p[1], m.h), cap);
    dec[t] = mlstm_log_f(__ldcg(m.proj + (size_t)t * m.ldp + d.a[ML_FOFF] + m.h) + bf16_at(d.p[2], m.h), cap);
  }
  consumer_sync();
  if (tid == 0) {
    float run = m.fresh ? 0.f : __ldcg(m.nm + m.dim);
    for (int t = 0; t < sv.nq; ++t) {
      const float fm = dec[t] + run, i = inp[t];
      run = fmaxf(fm, i);
      dec[t] = fm - run;
      inp[t] = i - run;
      den[t] = -run;
    }
    m.nm[m.dim] = run;
  }
  consumer_sync();
  for (int t = tid; t < sv.nq; t += kConsumerThreads) {
    dec[t] = decay_exp(dec[t]);
    inp[t] = expf(inp[t]);
    den[t] = expf(den[t]);
  }
  stamp(c, task, 0);
  float n[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    n[i] = (!m.fresh && row < m.dim) ? __ldcg(m.nm + row) : 0.f;
  }
  for (int v0 = m.V0; v0 < m.V1; v0 += VC) {
    const bool col_ok = v0 + 4 * qd < m.V1;
    const bool first = v0 == m.V0;
    float4 S[RPT];
    float *Sp = m.S + (size_t)r0 * m.vdimp + v0 + 4 * qd;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!m.fresh && col_ok && r0 + i < m.dim) S[i] = __ldcg(reinterpret_cast<const float4 *>(Sp + (size_t)i * m.vdimp));
    }
    for (int tb = 0; tb < sv.nq; tb += TC) {
      const int nt = min(TC, sv.nq - tb);
      consumer_sync();   // gates are final / the previous trip's readers are done
      // warp w takes tokens w, w + 8; a lane's loads of a token are independent and in flight together
      const float *pk = m.proj + (size_t)tb * m.ldp + d.a[ML_KOFF] + m.h * m.dim, *pq = m.proj + (size_t)tb * m.ldp + d.a[ML_QOFF] + m.h * m.dim;
      const float *pv = m.proj + (size_t)tb * m.ldp + d.a[ML_VOFF] + (size_t)m.h * m.vdim + v0;
      for (int t = warp; t < nt; t += 8) {
        const float in = inp[tb + t];
#pragma unroll 8
        for (int r = lane; r < ROWS; r += 32) {
          const bool ok = r < m.dim;
          ks[(size_t)t * ROWS + r] = ok ? __ldcg(pk + (size_t)t * m.ldp + r) * in : 0.f;
          qs[(size_t)t * ROWS + r] = ok ? __ldcg(pq + (size_t)t * m.ldp + r) * qscale : 0.f;
        }
#pragma unroll
        for (int r = lane; r < VC; r += 32) vs[t * VC + r] = v0 + r < m.vdim ? __ldcg(pv + (size_t)t * m.ldp + r) : 0.f;
      }
      consumer_sync();
      for (int t = 0; t < nt; ++t) {
        const float a = dec[tb + t];
        const float *kt = ks + (size_t)t * ROWS, *qt = qs + (size_t)t * ROWS;
        const float4 v = *reinterpret_cast<const float4 *>(vs + t * VC + 4 * qd);
        const float4 o = mlstm_warp_rows<CQ>(mlstm_step<RPT>(S, a, v, kt + r0, qt + r0));
        if (lane < CQ) *reinterpret_cast<float4 *>(red + (size_t)(t * 8 + warp) * VC + 4 * lane) = o;
        if (first) {
          float p = 0.f;
#pragma unroll
          for (int i = 0; i < NR; ++i) {
            const int row = tid + i * kConsumerThreads;
            if (row < ROWS) {
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
      for (int i = tid; i < nt * VC; i += kConsumerThreads) {
        const int t = i / VC, j = i % VC;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += red[(size_t)(t * 8 + w) * VC + j];
        if (v0 + j < m.vdim && v0 + j < m.V1) __stcg(m.raw + (size_t)(tb + t) * d.a[ML_LDR] + v0 + j, s / den[tb + t]);
      }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      if (col_ok && r0 + i < m.dim) *reinterpret_cast<float4 *>(Sp + (size_t)i * m.vdimp) = S[i];
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    if (row < m.dim) m.nm[row] = n[i];
  }
  stamp(c, task, 1);
  // ---- output of the head
  if (!last_of_head(c, d.a[ML_TICKET], m.chunks)) return;
  stamp(c, task, 2);
  const float eps = __int_as_float(d.a[ML_EPS]);
  T *out = reinterpret_cast<T *>(d.p[7]) + (size_t)sv.q0 * d.a[ML_LDO] + (size_t)m.h * m.vdim;
  for (int t = warp; t < sv.nq; t += 8) {
    const float *rt = m.raw + (size_t)t * d.a[ML_LDR];
    const float *gt = m.proj + (size_t)t * m.ldp + d.a[ML_GOFF] + (size_t)m.h * m.vdim;
    float ss = 0.f;
    if (m.vdim <= 512) {   // the row and its gates in registers, all loads in flight
      float x[16], g[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const bool in = i * 32 + lane < m.vdim;
        x[i] = in ? __ldcg(rt + i * 32 + lane) : 0.f;
        g[i] = in ? __ldcg(gt + i * 32 + lane) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) ss += x[i] * x[i];
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)m.vdim + eps);
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (i * 32 + lane < m.vdim)
          store_elt(out + (size_t)t * d.a[ML_LDO] + i * 32 + lane, x[i] * inv * bf16_at(d.p[3], (size_t)m.h * m.vdim + i * 32 + lane) * sigmoid_f(g[i]));
      continue;
    }
    for (int j = lane; j < m.vdim; j += 32) { const float v = __ldcg(rt + j); ss += v * v; }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)m.vdim + eps);
    for (int j = lane; j < m.vdim; j += 32)
      store_elt(out + (size_t)t * d.a[ML_LDO] + j, __ldcg(rt + j) * inv * bf16_at(d.p[3], (size_t)m.h * m.vdim + j) * sigmoid_f(__ldcg(gt + j)));
  }
}

// One token (decoding): the state is what has to move.  Every thread copies its own piece of the next sub-block into its
// own shared-memory cells while it works on the current one, starting before anything else is known of the token.
template <int HYB, int CQ, int RPT>
__device__ __noinline__ void mlstm_single(const Ctx c, const TaskDesc &d, const SeqView sv, int task) {
  typedef typename HybElt<HYB>::T T;
  constexpr int VC = 4 * CQ, RG = kConsumerThreads / CQ, ROWS = RG * RPT;
  constexpr int NR = (ROWS + kConsumerThreads - 1) / kConsumerThreads;
  const MlstmView m = mlstm_view(d, sv);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qd = tid % CQ, r0 = tid / CQ * RPT;
  float4 *ring = reinterpret_cast<float4 *>(c.s.xtile) + tid;                  // [2][RPT][256], this thread's cells
  float *ks = reinterpret_cast<float *>(c.s.xtile) + 8 * RPT * kConsumerThreads;   // [ROWS] input-scaled keys
  float *qs = ks + ROWS;                                                       // [ROWS]
  float *red = qs + ROWS;                                                      // [2][8 warps][VC]
  float *misc = red + 16 * VC;                                                 // [16]
  const int nrow = min(RPT, m.dim - r0);                                       // real rows of this thread (may be <= 0)
  float *Sp = m.S + (size_t)r0 * m.vdimp + m.V0 + 4 * qd;                      // its piece of the current sub-block
  auto fetch = [&](int v0, int slot, const float *src) {
    if (!m.fresh && v0 + 4 * qd < m.V1) {
      const uint32_t dst = smem_u32(ring + slot * RPT * kConsumerThreads);
#pragma unroll
      for (int i = 0; i < RPT; ++i, src += m.vdimp)
        if (i < nrow)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + (uint32_t)(i * kConsumerThreads * 16)), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(m.V0, 0, Sp);
  fetch(m.V0 + VC, 1, Sp + VC);
  const float cap = __int_as_float(d.a[ML_CAP]), qscale = __int_as_float(d.a[ML_QSCALE]);
  float kq[NR][2], n[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    const bool ok = row < m.dim;
    kq[i][0] = ok ? __ldcg(m.proj + d.a[ML_KOFF] + m.h * m.dim + row) : 0.f;
    kq[i][1] = ok ? __ldcg(m.proj + d.a[ML_QOFF] + m.h * m.dim + row) : 0.f;
    n[i] = ok && !m.fresh ? __ldcg(m.nm + row) : 0.f;
  }
  const float li = mlstm_log_i(__ldcg(m.proj + d.a[ML_IOFF] + m.h) + bf16_at(d.p[1], m.h), cap);
  const float fm = mlstm_log_f(__ldcg(m.proj + d.a[ML_FOFF] + m.h) + bf16_at(d.p[2], m.h), cap) + (m.fresh ? 0.f : __ldcg(m.nm + m.dim));
  const float run = fmaxf(fm, li), a = decay_exp(fm - run), b = expf(li - run);
  float p = 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = tid + i * kConsumerThreads;
    if (row < ROWS) {
      const float k = kq[i][0] * b, q = kq[i][1] * qscale;
      ks[row] = k;
      qs[row] = q;
      n[i] = fmaf(a, n[i], k);
      p = fmaf(n[i], q, p);
      if (row < m.dim) m.nm[row] = n[i];
    }
  }
  const float den = fmaxf(fabsf(block_sum(p, misc)), expf(-run)) + 1e-6f;   // (its barrier also orders reads of nm[dim] before the write)
  if (tid == 0) m.nm[m.dim] = run;
  stamp(c, task, 0);
  int par = 0;
  for (int v0 = m.V0; v0 < m.V1; v0 += VC, par ^= 1, Sp += VC) {
    const bool col_ok = v0 + 4 * qd < m.V1;
    float4 S[RPT];
    asm volatile("cp.async.wait_group 1;" ::: "memory");
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      S[i] = !m.fresh && col_ok && i < nrow ? ring[(par * RPT + i) * kConsumerThreads] : make_float4(0.f, 0.f, 0.f, 0.f);
    const float *pv = m.proj + d.a[ML_VOFF] + (size_t)m.h * m.vdim + v0 + 4 * qd;
    float4 v;
    v.x = v0 + 4 * qd < m.vdim ? __ldcg(pv) : 0.f;
    v.y = v0 + 4 * qd + 1 < m.vdim ? __ldcg(pv + 1) : 0.f;
    v.z = v0 + 4 * qd + 2 < m.vdim ? __ldcg(pv + 2) : 0.f;
    v.w = v0 + 4 * qd + 3 < m.vdim ? __ldcg(pv + 3) : 0.f;
    const float4 o = mlstm_warp_rows<CQ>(mlstm_step<RPT>(S, a, v, ks + r0, qs + r0));
    fetch(v0 + 2 * VC, par, Sp + 2 * VC);
    if (lane < CQ) *reinterpret_cast<float4 *>(red + (size_t)(par * 8 + warp) * VC + 4 * lane) = o;
    float *dst = Sp;
#pragma unroll
    for (int i = 0; i < RPT; ++i, dst += m.vdimp)
      if (col_ok && i < nrow) *reinterpret_cast<float4 *>(dst) = S[i];
    consumer_sync();
    if (tid < VC && v0 + tid < m.vdim && v0 + tid < m.V1) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += red[(size_t)(par * 8 + w) * VC + tid];
      __stcg(m.raw + v0 + tid, s / den);
    }
  }
  stamp(c, task, 1);
  if (!last_of_head(c, d.a[ML_TICKET], m.chunks)) return;
  stamp(c, task, 2);
  const float *gt = m.proj + d.a[ML_GOFF] + (size_t)m.h * m.vdim;
  T *out = reinterpret_cast<T *>(d.p[7]) + (size_t)sv.q0 * d.a[ML_LDO] + (size_t)m.h * m.vdim;
  float ss = 0.f;
  for (int j = tid; j < m.vdim; j += kConsumerThreads) { const float x = __ldcg(m.raw + j); ss += x * x; }
  const float inv = 1.0f / sqrtf(block_sum(ss, misc + 8) / (float)m.vdim + __int_as_float(d.a[ML_EPS]));
  for (int j = tid; j < m.vdim; j += kConsumerThreads)
    store_elt(out + j, __ldcg(m.raw + j) * inv * bf16_at(d.p[3], (size_t)m.h * m.vdim + j) * sigmoid_f(__ldcg(gt + j)));
}

template <int HYB, int CQ, int RPT>
__device__ __forceinline__ void mlstm_body(const Ctx &c, const TaskDesc &d, const SeqView &sv, int task) {
  if (sv.nq == 1) mlstm_single<HYB, CQ, RPT>(c, d, sv, task);
  else mlstm_portion<HYB, CQ, RPT>(c, d, sv, task);
}
template <int HYB>
__device__ __forceinline__ void run_mlstm(const Ctx &c, const TaskDesc &d, int task) {
  const SeqView sv = seq_view(c.P, d.a[ML_SLOT]);
  if (sv.nq <= 0) return;
  const int dim = d.a[ML_DIM];
  switch (mlstm_quads(dim)) {
    case 16:
      if (mlstm_rows_per_thread(dim) == 4) mlstm_body<HYB, 16, 4>(c, d, sv, task);
      else mlstm_body<HYB, 16, 8>(c, d, sv, task);
      break;
    case 8: mlstm_body<HYB, 8, 8>(c, d, sv, task); break;
    case 4: mlstm_body<HYB, 4, 8>(c, d, sv, task); break;
    default: mlstm_body<HYB, 2, 8>(c, d, sv, task); break;
  }
}

// ---------------------------------------------------------------------------
// TASK_GLA: (request, head, range of value columns).  Gated linear attention: the matrix memory S [dim, columns] decays by a
// factor per key channel,
//   S = diag(alpha) S + k v^T, o = S^T q,  alpha = sigmoid(a2 (a1 h) + b)^(1 / tau)
// Thread layout and column walk are those of TASK_MLSTM.  The low-rank decay product is part of the task: a1 h is read from
// the projections, a2's rows of the head from the weight.  The last task of the (request, head) to finish writes the head's
// normed and gated output.
// ---------------------------------------------------------------------------
struct GlaView {
  const float *proj;   // projections of the request's first token
  float *S, *raw;
  int ldp, H, h, dim, vdim, vdimp, V0, V1, chunks, rank;
  bool fresh;
};
__device__ __forceinline__ GlaView gla_view(const TaskDesc &d, const SeqView &sv) {
  GlaView m;
  m.ldp = d.a[GA_LDP]; m.H = d.a[GA_H]; m.h = d.a[GA_HEAD]; m.dim = d.a[GA_DIM]; m.vdim = d.a[GA_VDIM]; m.vdimp = d.a[GA_VDIMP];
  m.V0 = d.a[GA_V0]; m.V1 = d.a[GA_V1]; m.chunks = d.a[GA_NCHUNK]; m.rank = d.a[GA_RANK];
  m.fresh = sv.pos0 == 0;
  m.proj = reinterpret_cast<const float *>(d.p[0]) + (size_t)sv.q0 * m.ldp;
  m.S = reinterpret_cast<float *>(d.p[4]) + (size_t)(sv.slot * m.H + m.h) * m.dim * m.vdimp;
  m.raw = reinterpret_cast<float *>(d.p[6]) + (size_t)sv.q0 * d.a[GA_LDR] + (size_t)m.h * m.vdim;
  return m;
}
__device__ __forceinline__ float gla_decay(float z, float inv_tau) { return decay_exp(-softplus_f(-z) * inv_tau); }

// One step of S and the read-out for this thread's rows.
template <int RPT>
__device__ __forceinline__ float4 gla_step(float4 (&S)[RPT], const float *at, const float4 v, const float *kt, const float *qt) {
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RPT; i += 4) {
    const float4 a4 = *reinterpret_cast<const float4 *>(at + i), k4 = *reinterpret_cast<const float4 *>(kt + i),
                 q4 = *reinterpret_cast<const float4 *>(qt + i);
    const float a[4] = {a4.x, a4.y, a4.z, a4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float4 &s = S[i + e];
      s.x = fmaf(a[e], s.x, k[e] * v.x); o.x = fmaf(q[e], s.x, o.x);
      s.y = fmaf(a[e], s.y, k[e] * v.y); o.y = fmaf(q[e], s.y, o.y);
      s.z = fmaf(a[e], s.z, k[e] * v.z); o.z = fmaf(q[e], s.z, o.z);
      s.w = fmaf(a[e], s.w, k[e] * v.w); o.w = fmaf(q[e], s.w, o.w);
    }
  }
  return o;
}

// Output of a head for token rows t0, t0 + step, ...: unit norm over the head, weight, silu of the gate.  One warp per token.
template <int HYB>
__device__ __forceinline__ void gla_emit(const TaskDesc &d, const GlaView &m, const SeqView &sv, int t0, int step) {
  typedef typename HybElt<HYB>::T T;
  const int lane = threadIdx.x & 31;
  const float eps = __int_as_float(d.a[GA_EPS]);
  T *out = reinterpret_cast<T *>(d.p[7]) + (size_t)sv.q0 * d.a[GA_LDO] + (size_t)m.h * m.vdim;
  for (int t = t0; t < sv.nq; t += step) {
    const float *rt = m.raw + (size_t)t * d.a[GA_LDR];
    const float *gt = m.proj + (size_t)t * m.ldp + d.a[GA_GOFF] + (size_t)m.h * m.vdim;
    float ss = 0.f;
    if (m.vdim <= 512) {   // the row and its gates in registers, all loads in flight
      float x[16], g[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const bool in = i * 32 + lane < m.vdim;
        x[i] = in ? __ldcg(rt + i * 32 + lane) : 0.f;
        g[i] = in ? __ldcg(gt + i * 32 + lane) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) ss += x[i] * x[i];
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)m.vdim + eps);
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (i * 32 + lane < m.vdim)
          store_elt(out + (size_t)t * d.a[GA_LDO] + i * 32 + lane, x[i] * inv * bf16_at(d.p[3], i * 32 + lane) * silu_exact_f(g[i]));
      continue;
    }
    for (int j = lane; j < m.vdim; j += 32) { const float v = __ldcg(rt + j); ss += v * v; }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)m.vdim + eps);
    for (int j = lane; j < m.vdim; j += 32)
      store_elt(out + (size_t)t * d.a[GA_LDO] + j, __ldcg(rt + j) * inv * bf16_at(d.p[3], j) * silu_exact_f(__ldcg(gt + j)));
  }
}

// A portion of several tokens.
template <int HYB, int CQ, int RPT>
__device__ __noinline__ void gla_portion(const Ctx c, const TaskDesc &d, const SeqView sv, int task) {
  constexpr int VC = 4 * CQ, RG = kConsumerThreads / CQ, ROWS = RG * RPT;
  constexpr int GT = 8;   // tokens whose decays a thread forms together
  const GlaView m = gla_view(d, sv);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qd = tid % CQ, r0 = tid / CQ * RPT, TC = d.a[GA_TC];
  // shared memory
  float *as = reinterpret_cast<float *>(c.s.xtile);    // [TC][ROWS] decays
  float *ks = as + (size_t)TC * ROWS;                  // [TC][ROWS]
  float *qs = ks + (size_t)TC * ROWS;                  // [TC][ROWS]
  float *vs = qs + (size_t)TC * ROWS;                  // [TC][VC]
  float *red = vs + (size_t)TC * VC;                   // [TC][8 warps][VC]
  float *low = red + (size_t)TC * 8 * VC;              // [TC][rank]
  const float inv_tau = __int_as_float(d.a[GA_INVTAU]), qscale = __int_as_float(d.a[GA_QSCALE]);
  stamp(c, task, 0);
  for (int v0 = m.V0; v0 < m.V1; v0 += VC) {
    const bool col_ok = v0 + 4 * qd < m.V1;
    float4 S[RPT];
    float *Sp = m.S + (size_t)r0 * m.vdimp + v0 + 4 * qd;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!m.fresh && col_ok && r0 + i < m.dim) S[i] = __ldcg(reinterpret_cast<const float4 *>(Sp + (size_t)i * m.vdimp));
    }
    for (int tb = 0; tb < sv.nq; tb += TC) {
      const int nt = min(TC, sv.nq - tb);
      consumer_sync();   // the previous trip's readers are done
      // warp w takes tokens w, w + 8; a lane's loads of a token are independent and in flight together
      const float *pk = m.proj + (size_t)tb * m.ldp + d.a[GA_KOFF] + m.h * m.dim, *pq = m.proj + (size_t)tb * m.ldp + d.a[GA_QOFF] + m.h * m.dim;
      const float *pv = m.proj + (size_t)tb * m.ldp + d.a[GA_VOFF] + (size_t)m.h * m.vdim + v0;
      const float *pa = m.proj + (size_t)tb * m.ldp + d.a[GA_AOFF];
      for (int t = warp; t < nt; t += 8) {
#pragma unroll 8
        for (int r = lane; r < ROWS; r += 32) {
          const bool ok = r < m.dim;
          ks[(size_t)t * ROWS + r] = ok ? __ldcg(pk + (size_t)t * m.ldp + r) : 0.f;
          qs[(size_t)t * ROWS + r] = ok ? __ldcg(pq + (size_t)t * m.ldp + r) * qscale : 0.f;
        }
#pragma unroll
        for (int r = lane; r < VC; r += 32) vs[t * VC + r] = v0 + r < m.vdim ? __ldcg(pv + (size_t)t * m.ldp + r) : 0.f;
        for (int j = lane; j < m.rank; j += 32) low[t * m.rank + j] = __ldcg(pa + (size_t)t * m.ldp + j);
      }
      consumer_sync();
      // decays: an item is (row, GT tokens)
      for (int it = tid; it < ROWS * ((nt + GT - 1) / GT); it += kConsumerThreads) {
        const int r = it % ROWS, tg = it / ROWS * GT;
        float z[GT];
        const bool ok = r < m.dim;
        const float bias = ok ? bf16_at(d.p[2], m.h * m.dim + r) : 0.f;
#pragma unroll
        for (int u = 0; u < GT; ++u) z[u] = bias;
        if (ok) {
          const size_t wr = (size_t)(m.h * m.dim + r) * m.rank;
          for (int j = 0; j < m.rank; ++j) {
            const float w = bf16_at(d.p[1], wr + j);
#pragma unroll
            for (int u = 0; u < GT; ++u) z[u] = fmaf(w, low[min(tg + u, nt - 1) * m.rank + j], z[u]);
          }
        }
#pragma unroll
        for (int u = 0; u < GT; ++u)
          if (tg + u < nt) as[(size_t)(tg + u) * ROWS + r] = ok ? gla_decay(z[u], inv_tau) : 0.f;
      }
      consumer_sync();
      for (int t = 0; t < nt; ++t) {
        const float *at = as + (size_t)t * ROWS, *kt = ks + (size_t)t * ROWS, *qt = qs + (size_t)t * ROWS;
        const float4 v = *reinterpret_cast<const float4 *>(vs + t * VC + 4 * qd);
        const float4 o = mlstm_warp_rows<CQ>(gla_step<RPT>(S, at + r0, v, kt + r0, qt + r0));
        if (lane < CQ) *reinterpret_cast<float4 *>(red + (size_t)(t * 8 + warp) * VC + 4 * lane) = o;
      }
      consumer_sync();
      for (int i = tid; i < nt * VC; i += kConsumerThreads) {
        const int t = i / VC, j = i % VC;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += red[(size_t)(t * 8 + w) * VC + j];
        if (v0 + j < m.vdim && v0 + j < m.V1) __stcg(m.raw + (size_t)(tb + t) * d.a[GA_LDR] + v0 + j, s);
      }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      if (col_ok && r0 + i < m.dim) *reinterpret_cast<float4 *>(Sp + (size_t)i * m.vdimp) = S[i];
  }
  stamp(c, task, 1);
  if (!last_of_head(c, d.a[GA_TICKET], m.chunks)) return;
  stamp(c, task, 2);
  gla_emit<HYB>(d, m, sv, warp, 8);
}

// One token (decoding): the state is what has to move, streamed as in mlstm_single.
template <int HYB, int CQ, int RPT>
__device__ __noinline__ void gla_single(const Ctx c, const TaskDesc &d, const SeqView sv, int task) {
  constexpr int VC = 4 * CQ, RG = kConsumerThreads / CQ, ROWS = RG * RPT;
  const GlaView m = gla_view(d, sv);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qd = tid % CQ, r0 = tid / CQ * RPT;
  float4 *ring = reinterpret_cast<float4 *>(c.s.xtile) + tid;                  // [2][RPT][256], this thread's cells
  float *as = reinterpret_cast<float *>(c.s.xtile) + 8 * RPT * kConsumerThreads;   // [ROWS]
  float *ks = as + ROWS;                                                       // [ROWS]
  float *qs = ks + ROWS;                                                       // [ROWS]
  float *red = qs + ROWS;                                                      // [2][8 warps][VC]
  float *low = red + 16 * VC;                                                  // [rank]
  const int nrow = min(RPT, m.dim - r0);                                       // real rows of this thread (may be <= 0)
  float *Sp = m.S + (size_t)r0 * m.vdimp + m.V0 + 4 * qd;                      // its piece of the current sub-block
  auto fetch = [&](int v0, int slot, const float *src) {
    if (!m.fresh && v0 + 4 * qd < m.V1) {
      const uint32_t dst = smem_u32(ring + slot * RPT * kConsumerThreads);
#pragma unroll
      for (int i = 0; i < RPT; ++i, src += m.vdimp)
        if (i < nrow)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + (uint32_t)(i * kConsumerThreads * 16)), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(m.V0, 0, Sp);
  fetch(m.V0 + VC, 1, Sp + VC);
  const float inv_tau = __int_as_float(d.a[GA_INVTAU]), qscale = __int_as_float(d.a[GA_QSCALE]);
  for (int j = tid; j < m.rank; j += kConsumerThreads) low[j] = __ldcg(m.proj + d.a[GA_AOFF] + j);
  for (int r = tid; r < ROWS; r += kConsumerThreads) {
    const bool ok = r < m.dim;
    ks[r] = ok ? __ldcg(m.proj + d.a[GA_KOFF] + m.h * m.dim + r) : 0.f;
    qs[r] = ok ? __ldcg(m.proj + d.a[GA_QOFF] + m.h * m.dim + r) * qscale : 0.f;
  }
  consumer_sync();
  for (int r = tid; r < ROWS; r += kConsumerThreads) {
    float z = 0.f;
    if (r < m.dim) {
      z = bf16_at(d.p[2], m.h * m.dim + r);
      const size_t wr = (size_t)(m.h * m.dim + r) * m.rank;
#pragma unroll 16
      for (int j = 0; j < m.rank; ++j) z = fmaf(bf16_at(d.p[1], wr + j), low[j], z);
    }
    as[r] = r < m.dim ? gla_decay(z, inv_tau) : 0.f;
  }
  consumer_sync();
  stamp(c, task, 0);
  int par = 0;
  for (int v0 = m.V0; v0 < m.V1; v0 += VC, par ^= 1, Sp += VC) {
    const bool col_ok = v0 + 4 * qd < m.V1;
    float4 S[RPT];
    asm volatile("cp.async.wait_group 1;" ::: "memory");
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      S[i] = !m.fresh && col_ok && i < nrow ? ring[(par * RPT + i) * kConsumerThreads] : make_float4(0.f, 0.f, 0.f, 0.f);
    const float *pv = m.proj + d.a[GA_VOFF] + (size_t)m.h * m.vdim + v0 + 4 * qd;
    float4 v;
    v.x = v0 + 4 * qd < m.vdim ? __ldcg(pv) : 0.f;
    v.y = v0 + 4 * qd + 1 < m.vdim ? __ldcg(pv + 1) : 0.f;
    v.z = v0 + 4 * qd + 2 < m.vdim ? __ldcg(pv + 2) : 0.f;
    v.w = v0 + 4 * qd + 3 < m.vdim ? __ldcg(pv + 3) : 0.f;
    const float4 o = mlstm_warp_rows<CQ>(gla_step<RPT>(S, as + r0, v, ks + r0, qs + r0));
    fetch(v0 + 2 * VC, par, Sp + 2 * VC);
    if (lane < CQ) *reinterpret_cast<float4 *>(red + (size_t)(par * 8 + warp) * VC + 4 * lane) = o;
    float *dst = Sp;
#pragma unroll
    for (int i = 0; i < RPT; ++i, dst += m.vdimp)
      if (col_ok && i < nrow) *reinterpret_cast<float4 *>(dst) = S[i];
    consumer_sync();
    if (tid < VC && v0 + tid < m.vdim && v0 + tid < m.V1) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += red[(size_t)(par * 8 + w) * VC + tid];
      __stcg(m.raw + v0 + tid, s);
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  stamp(c, task, 1);
  if (!last_of_head(c, d.a[GA_TICKET], m.chunks)) return;
  stamp(c, task, 2);
  if (warp == 0) gla_emit<HYB>(d, m, sv, 0, 1);
}

template <int HYB, int CQ, int RPT>
__device__ __forceinline__ void gla_body(const Ctx &c, const TaskDesc &d, const SeqView &sv, int task) {
  if (sv.nq == 1) gla_single<HYB, CQ, RPT>(c, d, sv, task);
  else gla_portion<HYB, CQ, RPT>(c, d, sv, task);
}
template <int HYB>
__device__ __forceinline__ void run_gla(const Ctx &c, const TaskDesc &d, int task) {
  const SeqView sv = seq_view(c.P, d.a[GA_SLOT]);
  if (sv.nq <= 0) return;
  const int dim = d.a[GA_DIM];
  switch (mlstm_quads(dim)) {
    case 16:
      if (mlstm_rows_per_thread(dim) == 4) gla_body<HYB, 16, 4>(c, d, sv, task);
      else gla_body<HYB, 16, 8>(c, d, sv, task);
      break;
    case 8: gla_body<HYB, 8, 8>(c, d, sv, task); break;
    case 4: gla_body<HYB, 4, 8>(c, d, sv, task); break;
    default: gla_body<HYB, 2, 8>(c, d, sv, task); break;
  }
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

static __device__ __noinline__ void run_moe_routing_hybrid(const Ctx c, const TaskDesc &d) { run_moe_routing(c, d); }

template <int HYB>
__device__ __forceinline__ void run_hybrid_task(const Ctx &c, const TaskDesc &d, int task) {
  switch (d.type) {
    case TASK_BATCH: {
      Ctx cc = c;
      cc.tmem_base = 0u;
      run_batch(cc);
      break;
    }
    case TASK_EMBED_F32:
      if (d.p[3] | d.p[4] | d.p[5]) run_embed_sum(c, d);
      else run_embed_f32(c, d);
      break;
    case TASK_POLY_NORM: run_poly_norm<HYB>(c, d); break;
    case TASK_RESIDUAL_NORM: run_residual_norm<HYB>(c, d); break;
    case TASK_LINEAR_F32: if (HYB == HYB_F32) run_linear_f32(c, d); break;
    case TASK_MOE_ROUTING: run_moe_routing_hybrid(c, d); break;
    case TASK_MOE_GEMM_F32: if (HYB == HYB_F32) run_moe_gemm_f32(c, d); break;
    case TASK_LATENT_APPEND: run_latent_append<HYB>(c, d); break;
    case TASK_GLA: run_gla<HYB>(c, d, task); break;
    case TASK_ATTN_MERGE: run_attn_merge<HYB>(c, d); break;
    case TASK_QKV_APPEND:
      if (d.a[QA_WHOLE]) run_qkv_append_whole<HYB>(c, d);
      else run_qkv_append<HYB>(c, d);
      break;
    case TASK_EXT_ATTENTION: run_ext_attention<HYB>(c, d, task); break;
    case TASK_SHORT_CONV: run_short_conv<HYB>(c, d); break;
    case TASK_SELECTIVE_SCAN: run_selective_scan<HYB>(c, d, task); break;
    case TASK_DIFF_COMBINE: run_diff_combine<HYB>(c, d); break;
    case TASK_RGLRU: run_rglru<HYB>(c, d); break;
    case TASK_MLSTM: run_mlstm<HYB>(c, d, task); break;
    case TASK_ARGMAX_PARTIAL: run_argmax_partial_f32(c, d); break;
    case TASK_ARGMAX_REDUCE: run_argmax_reduce_f32(c, d); break;
    case TASK_SAMPLING_PARTIAL: run_sampling_partial<float>(c, d); break;
    case TASK_SAMPLING_REDUCE: run_sampling_reduce(c, d); break;
    default: break;
  }
}

}  // namespace mpk
