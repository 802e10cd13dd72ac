// Device-resident records shared by the host task-graph compiler and the megakernel.
//
// Counterpart of TaskDesc / EventDesc / RuntimeConfig in the reference
// (include/mirage/persistent_kernel/runtime_header.h:219-364), re-thought for a
// statically scheduled runtime: every worker CTA owns a fixed, ordered slice of the
// task array, events are plain 64-bit counters in HBM that grow monotonically
// across launches, and there are no scheduler CTAs or queues to pop.
#pragma once
#include <stdint.h>

namespace mpk {

constexpr int kMaxDeps = 3;
constexpr int kConsumerThreads = 256;          // 8 compute warps
constexpr int kBlockThreads = kConsumerThreads + 32;  // + 1 weight-streaming warp
constexpr int kChunkRows = 16;                 // weight rows per streamed chunk, at most (one mma m-tile)
constexpr int kChunkColsMax = 2048;            // k extent of a chunk, at most (the graph compiler may settle for 1024)
constexpr int kRowPadBytes = 16;               // shared-memory row padding: conflict-free ldmatrix
constexpr int stage_bytes_for(int chunk_cols) { return kChunkRows * (chunk_cols * 2 + kRowPadBytes); }
constexpr int kPartialBytes = 8 * 1024;        // per-task partial-sum slots
constexpr int kMiscBytes = 1536;               // barriers, descriptors, flags (1 KB) + the attention stash ring
constexpr int kMaxLinearTokens = 64;           // eight mma n-tiles of 8 tokens, one per compute warp
constexpr int kFp8TaskRows = 64;               // weight rows of one FP8 linear task (their scales are staged in shared memory)
constexpr int kTcSlotBytes = 16 * 1024;        // weight ring slot of graphs whose linears run on tcgen05 (1 KB multiples: swizzle atoms)
constexpr int kTmemCols = 512;                 // tensor-memory columns a worker CTA allocates (all of them: one CTA per SM)
constexpr int kTcKBlock = 64;                  // bf16 columns of one 128-byte swizzle row (an e4m3 row holds 128)
constexpr int kTcSfCols = 64;                  // tensor-memory columns kept for scale factors: 8 warps x (4 for A + 4 for B)
constexpr int kTcAccCols = kTmemCols - kTcSfCols;   // columns available to the accumulators of a task
constexpr int kTcFp8MaxTiles = 4;              // row tiles of one FP8 tcgen05 task (their scale words are staged in shared memory)

enum TaskType : uint32_t {
  TASK_NOP = 0,
  TASK_BATCH = 1,          // device-side continuous batching (prepare_next_batch)
  TASK_EMBED = 2,
  TASK_RMSNORM = 3,
  TASK_LINEAR = 4,         // weight-streaming GEMV with fused prologue/epilogue
  TASK_ATTENTION = 5,      // paged split-KV GQA decode attention
  TASK_SILU_MUL = 6,
  TASK_ARGMAX_PARTIAL = 7,
  TASK_ARGMAX_REDUCE = 8,
  TASK_ALLREDUCE = 9,      // sum the per-rank inbox slots (+ residual)
  TASK_ELEMENTWISE_ADD = 10,
  TASK_TENSOR_INIT = 11,
  TASK_QUANTIZE_FP8 = 12,  // per-token, per-128-group e4m3 quantisation (UE8M0 or float32 scales)
  TASK_MOE_ROUTING = 13,   // group-aware sigmoid top-k routing
  TASK_MOE_GEMM = 14,      // expert projections over the active experts (bf16, or e4m3 with float32 scales)
  TASK_MOE_SILU_MUL = 15,  // silu(gate) * up on [token, slot, gate | up]
  TASK_MOE_MUL_SUM_ADD = 16,  // weighted sum over expert slots + residual
  TASK_MLA_APPEND = 17,    // new [c_latent | k_pe] rows -> paged latent cache
  TASK_MLA_DECODE = 18,    // absorbed MLA decode of one (token, kv split, 16-head group): partial O + LSE
  TASK_MLA_REDUCE = 19,    // merge the splits
  TASK_SAMPLING_PARTIAL = 20,   // Gumbel-max sampling over one column range of the vocabulary
  TASK_SAMPLING_REDUCE = 21,    // merge of the column ranges (equal keys: highest index)
  TASK_ARGMAX_EXCHANGE = 22,    // argmax merge over a vocabulary sharded across ranks (pairs exchanged through the inboxes)
  TASK_AR_PUSH = 23,            // copy a column slice of a local bf16 tensor into every rank's inbox as fp32 (allreduce whose
                                // input is not produced by a bf16 linear); fields as TASK_ALLREDUCE with p[0] = the tensor
  // ---- hybrid graphs (recurrent and extended-attention layers; hybrid_tasks.cuh) ----
  TASK_EMBED_F32 = 24,          // token ids -> float32 rows of a bf16 table
  TASK_RESIDUAL_NORM = 25,      // x += norm(y) on a float32 residual stream, and the next layer's normed input
  TASK_LINEAR_F32 = 26,         // float32 activations x bf16 weights in 32-bit arithmetic
  TASK_QKV_APPEND = 27,         // rotation and unit norms of q and k, new k / v rows into the paged cache
  TASK_EXT_ATTENTION = 28,      // paged attention with free head sizes, score soft cap and sink
  TASK_SHORT_CONV = 29,         // causal per-channel convolution with carried inputs
  TASK_RGLRU = 30,              // gated diagonal linear recurrence
  TASK_MLSTM = 31,              // matrix-memory recurrence with exponential gates
  TASK_GLA = 32,                // gated linear attention (matrix state, a decay per key channel)
  TASK_LATENT_APPEND = 33,      // latent attention: cache rows and rotated query parts
  TASK_MOE_GEMM_F32 = 34,       // expert projections in 32-bit arithmetic
  TASK_ATTN_MERGE = 35,         // merge of an attention layer's key chunks
  TASK_SELECTIVE_SCAN = 36,     // selective state space recurrence
  TASK_DIFF_COMBINE = 37,       // differential attention: difference of the two maps' outputs, unit norm per head
  TASK_POLY_NORM = 38,          // activation: weighted sum of the normed powers of a token's values
};

// Which family of megakernel instantiations runs a graph (template parameter HYB of the kernel).
// Thread layout of a matrix-memory task: value-column quads and key rows per thread (256 threads).
#ifdef __CUDACC__
#define MPK_HD __host__ __device__
#else
#define MPK_HD
#endif
MPK_HD constexpr int mlstm_quads(int dim) { return dim <= 128 ? 16 : (dim <= 256 ? 8 : (dim <= 512 ? 4 : 2)); }
MPK_HD constexpr int mlstm_rows_per_thread(int dim) { return dim > 64 ? 8 : 4; }
MPK_HD constexpr int mlstm_rows(int dim) { return kConsumerThreads / mlstm_quads(dim) * mlstm_rows_per_thread(dim); }

// Query rows a bf16 extended-attention task keeps in shared memory: whole 16-row tiles, a power of two of them (the
// warps are split over the tiles), at most as many as the graph can batch.
MPK_HD constexpr int ext_attention_rows(int rows) {
  int r = 16;
  while (r < rows) r *= 2;
  return r;
}

// Selective scan: lanes that share a channel's state (four values each; at least four, so that the channels of a pass fit), slots of the ring of states to come, columns of the
// low-rank step sizes staged at a time.
MPK_HD constexpr int scan_lanes(int n) {
  int l = 4;
  while (4 * l < n) l *= 2;
  return l;
}
constexpr int kScanRing = 12, kScanRank = 256;
MPK_HD constexpr int scan_pitch(int rank) { return (rank < kScanRank ? (rank + 15) / 16 * 16 : kScanRank) + 8; }   // of staged rows, elements
// The low-rank part and its weights are staged where the gate and the ring will be.
MPK_HD constexpr int scan_staged_bytes(int tokens, int rank, int channels) {
  const int a = tokens * scan_pitch(rank) * 4 + channels * scan_pitch(rank) * 2, b = tokens * channels * 4, ring = kScanRing * kConsumerThreads * 16;
  return a > b + ring ? a : b + ring;
}

enum : int { HYB_NONE = 0, HYB_BF16 = 1, HYB_F32 = 2 };
// Activations of hybrid linears (mpk_activation of include/mpk_b200.h).
enum : int { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SOFTCAP = 2, ACT_GATED_SILU = 3, ACT_GATED_GELU = 4, ACT_SCALE = 5 };

// Online mode: control word of a token-table row (KernelParams.meta.request_ctl[row], written by the host between
// launches; request_ctl[rows + row] is the device's "live" flag).
enum : int {
  REQ_FREE = 0,    // row unused (the device sets it when a request retires)
  REQ_RUN = 1,     // runs its prompt, then decodes until EOS or the table's end
  REQ_HOLD = 2,    // runs the tokens supplied so far (prompt_lengths[row]) and then keeps its pages and state
  REQ_CLOSE = 3,   // retires once the supplied tokens have run
};

// prologue applied while staging the activation tile of a linear task
enum Prologue : int32_t { PRO_PLAIN = 0, PRO_RMSNORM = 1, PRO_SILU_MUL = 2,
                          PRO_RESNORM = 3,   // hybrid graphs: x_out = x + norm(y) on the float32 stream, activation = norm(x_out)
                          PRO_POLY = 4 };      // hybrid graphs: activation = sum of normed powers of float32 values (TASK_POLY_NORM)
// epilogue of a linear task
enum Epilogue : int32_t {
  EPI_STORE = 0,        // out = bf16(acc)
  EPI_RESIDUAL = 1,     // out = bf16(acc + residual)
  EPI_PUSH_F32 = 2,     // fp32 partial rows pushed into every rank's inbox slot [my_rank] (+ counter increments)
  EPI_PUSH_LL = 3,      // {bf16 partial, 16-bit sequence} words pushed into every rank's inbox: self-validating
  EPI_STORE_F32 = 5,    // out = acc, float32 (hybrid graphs)
  EPI_RELU2 = 6,        // out = bf16(max(acc, 0)^2) (hybrid graphs)
  EPI_SOFTCAP = 7,      // out = cap * tanh(acc / cap), float32 (hybrid graphs)
  EPI_GATED_SILU = 8,   // rows [gate, gate, up, up]: out[2k + i] = bf16(silu(gate_i) * up_i) (hybrid graphs)
  EPI_GATED_GELU = 9,   // the same with the tanh form of gelu
  EPI_BIAS_F32 = 10,    // out = acc + bias, float32 (hybrid graphs)
  EPI_SCALE_F32 = 11,   // out = factor * acc, float32 (hybrid graphs)
  EPI_GATE_SIGMOID = 12,  // out = bf16(acc * sigmoid(gate)), the gate float32 (hybrid graphs)
  EPI_SILU_PAIR = 4,    // rows interleaved [gate, gate, up, up]: out[2k + i] = bf16(silu(gate_i)) * up_i
};

// flags
constexpr uint32_t TF_SAME_X_AS_PREV = 1u << 0;    // activation tile already staged by the previous task
constexpr uint32_t TF_STREAM_AFTER_DEP = 1u << 1;  // weight operand is produced inside the graph: do not prefetch
constexpr uint32_t TF_REMOTE_TRIGGER = 1u << 2;    // trigger event lives on every rank (peer atomics)
constexpr uint32_t TF_FP8 = 1u << 3;               // linear task: e4m3 weights and activations with UE8M0 block scales
constexpr uint32_t TF_TC = 1u << 4;                // linear task on the tcgen05 path: weight tiles arrive by tensor-map TMA in the
                                                   // 128-byte-swizzled K-major layout, accumulators live in tensor memory
constexpr uint32_t TF_DEP0_REMOTE = 1u << 8;       // dependency i (bit 8 + i) is incremented by peers: system-scope acquire

struct alignas(16) TaskDesc {
  uint32_t type;
  uint32_t flags;
  int32_t dep_event[kMaxDeps];   // -1: none
  uint32_t dep_need[kMaxDeps];   // arrivals per iteration that complete the dependency
  int32_t trig_event;            // -1: none
  int32_t layer;                 // index of the layer this task was cut from (profiling / dumps)
  uint64_t p[8];                 // pointers, meaning per type
  int32_t a[28];                 // integers, meaning per type
};
constexpr int kDescVecs = 14;
static_assert(sizeof(TaskDesc) == 16 * kDescVecs, "TaskDesc must stay 224 bytes (14 x 16-byte vectors)");

// ---- TASK_LINEAR -----------------------------------------------------------
//  p[0] W [N,K] bf16 (row stride a[3])   p[1] x source   p[2] out   p[3] residual
//  p[4] gamma (PRO_RMSNORM)              p[5] inbox base (EPI_PUSH_F32, local address of slot 0)
//  a[0] n0  a[1] n1  a[2] K  a[3] ldw  a[4] ld_x  a[5] ld_out  a[6] ld_res
//  a[7] prologue  a[8] epilogue  a[9] eps bits  a[10] silu groups
//  a[11] KT (k tile of the activation)  a[12] KC (k extent of a streamed chunk)  a[13] inbox slot stride (floats)  a[14] N
//  a[18] weight rows per streamed chunk (8 or 16)
//  FP8 (TF_FP8): p[6] weight scales, p[7] activation scales, packed UE8M0 (4 exponents per uint32);
//        a[23], a[24] strides (uint32 units) of the weight scales over (row, packed k); a[25], a[26] of the
//        activation scales over (token, packed k).  K, KT, KC, ld* are in elements (= bytes).
//  a[19] 1 + index of the allreduce whose pushed partials the prologue gathers (0: none); then p[6] residual,
//        p[7] tensor that receives the reduced activations, a[20] ld residual, a[21] ld of that tensor,
//        a[22] inbox slot stride of that allreduce (words)
//  PRO_RESNORM: p[1] x f32  p[3] weight of y's norm or null  p[4] weight of the output norm  p[6] y f32 or null  p[7] x_out f32 (or
//        null), a[20] ld y, a[21] ld x_out, a[22] flags (2: weights stored around zero, 4: layer norm), a[10] width (K minus the
//        zero padding), p[5] norm bias or null, 64-bit values a[LR_ADD] added stream or null (ld a[LR_LDADD]), a[LR_ROW] added row or null
//        a[LR_POST] factor of y's norm (bits); p[4] null: the activation is the stream as it is
//        flag 8: the stream is the weighted sum of a[L_LDR] results: a[LR_ADD] results f32 (a[LR_LDADD] floats apart, rows of a[10]; the last is
//        written), a[LR_ROW] their weights bf16
//  PRO_POLY: p[1] z f32  p[4] coefficients bf16 [4], a[10] columns of z (K minus the zero padding), a[9] eps bits
//  EPI_SOFTCAP, EPI_SCALE_F32: a[23] cap / factor bits;  EPI_BIAS_F32: 64-bit value a[LR_BIAS];  EPI_GATE_SIGMOID: p[3] gate f32, a[6] its ld
//  a[15] allreduce index within the iteration  a[16] allreduces per iteration  a[17] stride between the two inbox buffers (floats)
//  tcgen05 path (TF_TC): a[18] rows of one weight tile (the TMA box height, a multiple of 8, at most 128; the task's rows are
//        cut into ceil(rows / a[18]) tiles, each one 128-lane accumulator), a[12] = 64 x (k blocks of 64 columns per ring slot),
//        a[27] index of the task's tensor map (dims {64, rows of the task, K / 64}, box {64, a[18], a[12] / 64}, 128-byte swizzle)
enum { L_N0 = 0, L_N1, L_K, L_LDW, L_LDX, L_LDO, L_LDR, L_PRO, L_EPI, L_EPS, L_GROUPS, L_KT, L_KC, L_SLOT, L_N, L_ARIDX, L_NAR, L_PARSTRIDE, L_ROWS,
       L_GATHER, L_G_LDRES, L_G_LDOUT, L_G_SLOT, L_WS_S0, L_WS_S1, L_XS_S0, L_XS_S1, L_TMAP };
static_assert(L_TMAP == 27, "TaskDesc::a has 28 entries");
enum { LR_POST = 13, LR_ADD = 14, LR_ROW = 16, L_CAP = 23, LR_BIAS = 24, LR_LDADD = 26 };   // hybrid graphs (the fields of allreduces and FP8 tasks are free there)
// ---- TASK_ATTENTION ----------------------------------------------------------
//  p[0] qkv  p[1] k_cache  p[2] v_cache  p[3] q_norm  p[4] k_norm  p[5] cos  p[6] sin  p[7] out
//  a[0] slot  a[1] kv head  a[2] chunk  a[3] num chunks  a[4] local q heads  a[5] local kv heads
//  a[6] head_dim  a[7] page_size  a[8] flags(1 qk_norm, 2 rope, 4 contiguous cache)  a[9] ld_qkv
//  a[10] ld_out  a[11] eps bits  a[12] rope table rows  a[13] cache seq (contiguous mode)
//  a[14] ticket bank offset  a[15] event of the batching task (-1: none)  a[16] its arrivals per iteration
enum { A_SLOT = 0, A_HEAD, A_CHUNK, A_NCHUNK, A_HQ, A_HKV, A_HD, A_PAGE, A_FLAGS, A_LDQKV, A_LDO, A_EPS, A_ROPE_ROWS, A_CSEQ,
       A_TICKET, A_EARLY_EV, A_EARLY_NEED };
// ---- TASK_EMBED / RMSNORM / SILU / ADD / INIT ---------------------------------
//  rows [a[0],a[1]) of the token dimension, width a[2]; p[0] in  p[1] weight/second input  p[2] out
//  a[3] ld_in  a[4] ld_out  a[5] eps bits | silu groups | vocab  a[6] ld_in2
enum { E_T0 = 0, E_T1, E_WIDTH, E_LDI, E_LDO, E_AUX, E_LDI2 };
// ---- TASK_MOE_ROUTING: p[0] logits [B, E] (zeroed after reading)  p[1] bias f32 [E]  p[2] weights f32 [B, topk]
//      p[3] routing i32 [E, ld]  p[4] active i32 [E + 1];  a[0] E  a[1] topk  a[2] groups  a[3] groups kept
//      a[4] scaling bits  a[5] ld logits  a[6] ld weights  a[7] ld routing  a[8] logits are f32  a[12] logits stay as they are
//      a[13] weights are the scores, not renormalised over the chosen experts
// ---- TASK_MOE_GEMM: linear-task fields (L_*) describe one expert's panel; p[0] weights [E, N, K]  p[1] x  p[2] out
//      p[4] routing  p[5] active list  p[6] weight scales f32 [E, N, K/128]  p[7] x scales f32 [rows, K/128];
//      a[L_EPI] EPI_STORE, EPI_STORE_F32, EPI_RELU2, EPI_GATED_*
//      a[M_NEXP] experts  a[M_NTOPK]  a[M_PER_SLOT] 1: x has one row per (token, slot)  a[M_LDR] ld routing
//      a[M_ESTRIDE] elements between experts
enum { M_NEXP = 19, M_NTOPK, M_PER_SLOT, M_LDR, M_ESTRIDE };
// ---- TASK_MOE_SILU_MUL: p[0] in [rows, 2I]  p[2] out [rows, I]; a[0] r0 a[1] r1 a[2] I a[3] ld in a[4] ld out a[5] rows per token
// ---- TASK_MOE_MUL_SUM_ADD: p[0] in [B, topk, H]  p[1] weights f32 [B, topk]  p[2] out  p[3] residual;
//      a[0] c0 a[1] c1 (columns) a[2] H a[3] topk a[4] ld out a[5] ld residual a[6] ld weights a[7] tokens
// ---- TASK_MLA_APPEND: p[0] c_latent_new  p[1] k_pe_new  p[2] cache [pages, page, d_k];  a[0] slot  a[1] ld c_latent
//      a[2] ld k_pe  a[3] page  a[4] d_k  a[5] d_v
// ---- TASK_MLA_DECODE: p[0] q [tokens, H * 576]  p[1] cache (paged, or contiguous [requests * kv_len, 576])
//      p[2] partial O bf16 [(token * H + head) * S + split][512]  p[3] partial LSE f32 [(token * H + head) * S + split]
//      a[0] token  a[1] split  a[2] first head  a[3] H  a[4] S  a[5] page (0: contiguous)  a[6] ld q  a[7] scale bits
//      a[8] q_len (contiguous mode)  a[9] kv_len (contiguous mode)
// ---- TASK_MLA_REDUCE: p[0] partial O  p[1] partial LSE  p[2] out [tokens, H * 512];  a[0] r0  a[1] r1 (rows = token * H + head)
//      a[2] H  a[3] S  a[4] ld out
// ---- TASK_QUANTIZE_FP8: rows [a[0],a[1]) of p[0] (bf16, width a[2], ld a[3]) -> p[1] e4m3 (ld a[4] bytes), p[2] scales;
//      a[5] 1: packed UE8M0 uint32, 0: float32; a[7], a[8] strides of the scale tensor over (token, packed k | group)
// ---- TASK_ARGMAX_PARTIAL:  p[0] logits p[1] value p[2] index  a[0] c0 a[1] c1 a[2] chunk id a[3] ld_logits a[4] ld_part
// ---- TASK_SAMPLING_PARTIAL: as TASK_ARGMAX_PARTIAL (the value is the bf16 key), plus a[6] / a[7] philox seed (low /
//                            high word), a[8] rows per reference task (the noise of row b is that of row b % a[8]),
//                            a[9] vocabulary size
// ---- TASK_ARGMAX_REDUCE:   p[0] value p[1] index p[2] out ids  a[0] num partials a[1] ld_part
// ---- TASK_SAMPLING_REDUCE:  as TASK_ARGMAX_REDUCE, but equal values go to the highest index
// ---- TASK_ARGMAX_EXCHANGE:  as TASK_ARGMAX_REDUCE, plus a[2] first column of this rank, p[5] word offset of the
//      exchange area inside an inbox buffer ([world][tokens] x {value | seq, index | seq} 64-bit words), a[L_ARIDX],
//      a[L_NAR], a[L_PARSTRIDE] as for the allreduce
// ---- hybrid tasks --------------------------------------------------------------
// ---- TASK_EMBED_F32: p[0] ids  p[1] table bf16  p[2] out f32;  a[E_*] as TASK_EMBED (a[E_AUX] = vocabulary, a[E_LDI2] factor bits)
//      p[3] bigram table bf16 [buckets + 1, a[E_LDB]] or null  p[4] position frequencies int64 [(width + 1) / 2] or null  p[5] second copy of the output
//      or null, a[E_LDC] its ld;  bigram row (previous id * mul_prev + id * mul_cur) mod buckets, 64-bit values a[E_PREV], a[E_CUR]
enum { E_LDB = 7, E_BUCKETS, E_LDC, E_PREV = 10, E_CUR = 12 };
// ---- TASK_RESIDUAL_NORM: rows [a[0], a[1]), width a[2]; p[0] x f32 (in place)  p[1] y f32 or null  p[2] weight of y's norm or
//      null (plain sum)  p[3] weight of the output norm or null (out is the new x)  p[4] out (bf16, f32 with flag 1) or null  p[5] new x (= p[0]: in place);
//      a[3] ld x  a[4] ld y  a[5] ld out  a[6] eps bits  a[7] flags (1: out f32, 2: weights stored around zero, 4: layer norm)  a[8] ld
//      of the new x;  64-bit values, 0 if absent: a[RN_BIAS] norm bias, a[RN_ADD] added stream, a[RN_ROW] added row, a[RN_EXP] expert
//      outputs f32 [tokens, slots, width], a[RN_EW] their weights f32, a[RN_GATE] f32 column, y is multiplied by its sigmoid
//      a[RN_POST] factor of y's norm (bits); with that norm the experts' sum is part of what is normed
//      p[6] earlier results f32 or null (then a[RN_TERMS] >= 2 of them, a[RN_HSTRIDE] floats apart, rows of `width`), p[7] their weights bf16: the sum
//      x + y goes to the last of the a[RN_TERMS] results, and the new stream is the weighted sum of all of them
enum { RN_LDADD = 9, RN_BIAS = 10, RN_ADD = 12, RN_ROW = 14, RN_EXP = 16, RN_EW = 18, RN_GATE = 20, RN_SLOTS = 22, RN_LDEW, RN_LDGATE, RN_POST, RN_TERMS, RN_HSTRIDE };
// ---- TASK_LINEAR_F32: p[0] W bf16 [N, K]  p[1] x f32  p[2] out f32;  a[0] n0  a[1] n1  a[2] K  a[3] ldw  a[4] ld x  a[5] ld out
//      a[6] activation (mpk_activation)  a[7] tokens per shared-memory tile  a[8] soft cap / factor bits  p[3] bias bf16 or null  p[4] gate f32 or null (the output
//      is multiplied by its sigmoid)  a[9] ld gate
// ---- TASK_MOE_GEMM_F32: p[0] W bf16 [E, N, K]  p[1] x f32  p[2] out f32  p[4] routing  p[5] active list;  a[0] n0  a[1] n1  a[2] K  a[4] ld x
//      a[5] ld out (of a slot)  a[6] activation  a[7] tokens per shared-memory tile  a[8] x rows per (token, slot)  a[9] slots  a[10] ld routing
//      a[11] experts  a[12] rows N of an expert
// ---- TASK_QKV_APPEND: tokens [a[0], a[1]); p[0] projections f32  p[1] q out  p[2] k cache  p[3] v cache  p[4] cos f32  p[5] sin f32
//      p[6] q norm  p[7] k norm (bf16 [dim], null: none);  p[2] null: queries only;  a[QA_*] below
//      QA_WHOLE: the norms span all heads (weights [heads * dim]), nothing is rotated;  queries are multiplied by
//      1 + QA_TEMP (bits) * ln(floor((position + 1) / QA_EVERY) + 1) where QA_EVERY > 0
enum { QA_T0 = 0, QA_T1, QA_LDP, QA_QOFF, QA_KOFF, QA_VOFF, QA_HQ, QA_HKV, QA_DIM, QA_DIMP, QA_VDIM, QA_VDIMP, QA_ROT, QA_NORM,
       QA_EPS, QA_PAGE, QA_LDQ, QA_ROWS, QA_PAIRS, QA_MAPS, QA_WHOLE, QA_TEMP, QA_EVERY };
// ---- TASK_EXT_ATTENTION: p[0] q [tokens, hq * dimp]  p[1] k cache  p[2] v cache  p[3] out;  a[XA_*] below
enum { XA_SLOT = 0, XA_HEAD, XA_CHUNK, XA_NCHUNK, XA_HQ, XA_HKV, XA_DIMP, XA_VDIM, XA_VDIMP, XA_PAGE, XA_LDQ, XA_LDO, XA_OCOL,
       XA_SCALE, XA_CAP, XA_SINK, XA_OSCALE, XA_TICKET, XA_SREC, XA_STAGES, XA_SHARED, XA_KEYS, XA_MERGE, XA_WINDOW, XA_KEEP, XA_OUTF32 };
//      p[4] sinks bf16 [hq] or null; XA_SHARED: values are key columns; XA_KEYS: keys of a tile of
//      theirs; XA_MERGE: a layer of TASK_ATTN_MERGE follows (its tasks: the same fields, task a[XA_SLOT] of a[XA_CHUNK]);
//      XA_WINDOW: keys a position sees at most, itself included (0: all)  XA_KEEP: first keys it sees all the same
//      p[5], p[6] distance bias bf16 [hq] or null: r1 * ln(1 + r2 * distance) comes off the score
constexpr int kXaRecHead = 4;   // floats in front of a record's columns
constexpr int kXaCells = 320;   // cache rows of a chunk's key octets kept in shared memory
// ---- TASK_SHORT_CONV: channels [a[0], a[1]); p[0] in f32  p[1] in bias bf16 or null  p[2] taps bf16 [channels, taps]
//      p[3] bias bf16 or null  p[4] carried inputs f32 [slots, taps - 1, channels]  p[5] out f32  p[6] copy of out in the activation type or null
//      a[2] channels  a[3] taps  a[4] ld in  a[5] in column offset  a[6] ld out  a[7] activation (0 none, 1 silu)  a[8] ld copy
// ---- TASK_RGLRU: p[0] u f32 [tokens, width]  p[1] projections f32 (output branch)  p[2] y bias bf16  p[3] ra  p[4] ra bias  p[5] ri
//      p[6] ri bias  p[7] lambda (bf16, all);  a[GL_*]; state and output pointers are 64-bit values in a[GL_STATE], a[GL_OUT]
enum { GL_BLOCK = 0, GL_C0, GL_C1, GL_BS, GL_WIDTH, GL_LDU, GL_LDP, GL_YOFF, GL_LDO, GL_OCOL, GL_OSCALE, GL_OUTF32, GL_GATE_C, GL_TG,
       GL_STATE = 20, GL_OUT = 22 };
// ---- TASK_MLSTM: p[0] projections f32  p[1] input-gate bias  p[2] forget-gate bias  p[3] output norm weight (bf16)
//      p[4] matrix state f32 [slots, heads, dim, vdimp]  p[5] normaliser state f32 [slots, heads, chunks, dim + 1] (n, then m)
//      p[6] readout scratch f32 [tokens, heads * vdim]  p[7] out;  a[ML_*]
enum { ML_SLOT = 0, ML_HEAD, ML_CHUNK, ML_NCHUNK, ML_H, ML_DIM, ML_VDIM, ML_VDIMP, ML_V0, ML_V1, ML_CAP, ML_EPS, ML_LDP, ML_QOFF,
       ML_KOFF, ML_VOFF, ML_GOFF, ML_IOFF, ML_FOFF, ML_LDO, ML_OUTF32, ML_QSCALE, ML_TICKET, ML_TC, ML_LDR };
// ---- TASK_GLA: p[0] projections f32  p[1] a2 bf16 [heads * dim, rank]  p[2] a2 bias bf16  p[3] output norm weight bf16 [vdim]
//      p[4] matrix state f32 [slots, heads, dim, vdimp]  p[6] readout scratch f32 [tokens, heads * vdim]  p[7] out;  a[GA_*]
enum { GA_SLOT = 0, GA_HEAD, GA_CHUNK, GA_NCHUNK, GA_H, GA_DIM, GA_VDIM, GA_VDIMP, GA_V0, GA_V1, GA_EPS, GA_LDP, GA_QOFF, GA_KOFF, GA_VOFF,
       GA_GOFF, GA_AOFF, GA_RANK, GA_LDO, GA_QSCALE, GA_TICKET, GA_TC, GA_LDR, GA_INVTAU };
// ---- TASK_LATENT_APPEND: items [a[0] of a[1] tasks]; p[0] projections f32  p[1] latent norm weight bf16  p[2] q out  p[3] cache [pages, page, 1, dimp]
//      p[4] cos f32  p[5] sin f32;  a[LA_*]
enum { LA_T0 = 0, LA_T1, LA_LDP, LA_QOFF, LA_KVOFF, LA_H, LA_RANK, LA_ROT, LA_DIMP, LA_EPS, LA_PAGE, LA_LDQ, LA_ROWS };
// ---- TASK_SELECTIVE_SCAN: channels [a[SS_C0], a[SS_C1]) of all requests; p[0] u f32  p[1] low f32 [tokens, rank | B | C]  p[2] gate f32
//      p[3] dt weight bf16 [channels, rank]  p[4] dt bias  p[5] A_log [channels, n]  p[6] D  p[7] out;  64-bit value a[SS_STATE] f32 [slots, channels, np]
enum { SS_C0 = 0, SS_C1, SS_C, SS_RANK, SS_N, SS_NP, SS_LANES, SS_LDU, SS_LDL, SS_LDG, SS_GOFF, SS_LDO, SS_STATE };
// ---- TASK_DIFF_COMBINE: task a[0] of a[1]; p[0] maps f32 [tokens, heads * 2 * vdim]  p[1] out;  a[2] heads  a[3] vdim  a[4] ld in  a[5] ld out
//      a[6] lambda  a[7] factor  a[8] eps (bits)
// ---- TASK_POLY_NORM: rows [a[0], a[1]), width a[2]; p[0] z f32  p[1] coefficients bf16 [4]  p[2] out (activation type);  a[3] ld z  a[4] ld out  a[5] eps bits
// ---- TASK_ALLREDUCE:       p[0] inbox base p[1] residual (or null) p[2] out
//  a[0] c0 a[1] c1 (columns) a[2] world a[3] slot stride (floats) a[4] ld_out a[5] ld_res a[6] N
//  a[7] allreduce index  a[8] allreduces per iteration  a[9] stride between the two inbox buffers (floats)
struct BatchMeta {
  int32_t *step;
  int64_t *tokens;
  int64_t *input_tokens;
  int64_t *output_tokens;
  int32_t *prompt_lengths;
  int32_t *qo_indptr;
  int32_t *paged_kv_indptr;
  int32_t *paged_kv_indices;
  int32_t *paged_kv_last_page_len;
  int32_t *paged_kv_indices_snapshot;
  // private scheduler state owned by the handle
  int32_t *request_ids;      // [max_num_batched_requests]
  int32_t *page_queue;       // [max_num_pages]
  int32_t *sched_scalars;    // [0] page_queue_head [1] page_queue_tail [2] next_request_id
  int32_t *state_slots;      // [max_num_batched_requests] recurrent-state slot of each batch slot
  int32_t *request_ctl;      // [2][total_num_requests] online mode only, else null
};

struct DeviceStatus {
  int32_t error;
  int32_t where;
  int32_t worker;
  int32_t task;
  int32_t all_done;
  int32_t active_tokens;
  unsigned long long iteration;   // completed launches; the running launch uses iteration + 1
  unsigned int exit_ticket;
  unsigned int pad;
  unsigned long long t_start[8];  // globaltimer at entry of CTA 0, ring indexed by iteration & 7
  unsigned long long t_end[8];    // globaltimer when the last CTA left
};

constexpr int kMaxWorld = 8;

struct KernelParams {
  const TaskDesc *tasks;
  const int32_t *worker_begin;          // [num_workers + 1]
  unsigned long long *counters;         // [num_events] local event counters
  unsigned long long *peer_counters[kMaxWorld];  // the same array on every rank (index = rank)
  float *peer_inbox[kMaxWorld];         // exchange region of every rank
  DeviceStatus *status;
  BatchMeta meta;
  float *attn_scratch;                  // split-KV partials
  unsigned int *attn_tickets;           // [max_requests * kv_heads] per attention layer slot
  uint64_t *profiler;
  uint64_t profiler_entries;
  long long eos_token_id;
  int32_t num_workers;
  int32_t test_mode;
  int32_t world_size, rank;
  int32_t max_seq_length, max_num_batched_requests, max_num_batched_tokens, max_num_pages, page_size;
  int32_t total_num_requests;
  int32_t num_stages;                   // weight pipeline depth
  int32_t stage_bytes;                  // bytes of one stage: 16 rows x (chunk columns x 2 + 16)
  uint32_t poll_sleep_ns;               // back-off between two polls of an event counter (0: none)
  int32_t quiet_streaming;              // hold the weight stream back while attention tasks run
  int32_t kv_l2_prefetch;               // streaming warp prefetches attention K/V rows into L2
  int32_t max_inflight;                 // chunks the streamer keeps in flight (<= num_stages)
  int32_t ll_row_words;                 // words of one token row in a rank's inbox slot when all fused allreduces have the same
                                        // width (0: they differ): the batching task clears rows that go idle (see ll_seq)
  int32_t ll_buffer_words;              // words between the two inbox buffers
  int32_t tp_extensions;                // batch-1 graphs of several ranks: run the instantiation with the argmax exchange and the
                                        // all-ranks-in-flight allreduce prologue (set when the graph holds an exchange task)
  int32_t hybrid;                       // host side: HYB_* family of the graph
  int32_t general_kernel;               // host side: launch the instantiation with FP8 and > 8-token linear tasks
  int32_t x_tile_bytes;                 // bytes reserved for the activation tile
  uint32_t spin_limit;                  // polls before a wait gives up
  const void *tmaps;                    // array of 128-byte tensor maps (one per tcgen05 linear task), 64-byte aligned
  int32_t use_tmem;                     // the graph has tcgen05 tasks: every worker CTA allocates tensor memory
  int32_t tc_tokens;                    // token rows of the activation operand tile (batched tokens rounded up to 16)
  int32_t meta_static;                  // the batch description is the caller's and final at launch (test mode, online_notoken):
                                        // the graph has no batching task
};

}  // namespace mpk
