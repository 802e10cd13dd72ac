// Task-graph compiler (host).  See task_graph.h.
#include "task_graph.h"

#include <algorithm>
#include <cstring>
#include <map>
#include <set>
#include <sstream>

namespace mpk {
namespace {

constexpr int kSmemBudget = 232448;   // 227 KB opt-in dynamic shared memory per CTA on sm_100
constexpr int ST_META = 0;            // batch description written by the batching task
constexpr int ST_META_OUT = 1;        // output_tokens (written by argmax, read by the batching task)

int elt_size(int dtype) {
  switch (dtype) {
    case MPK_BF16: case MPK_F16: case MPK_I16: return 2;
    case MPK_F32: case MPK_I32: case MPK_U32: return 4;
    case MPK_I64: case MPK_U64: return 8;
    default: return 1;
  }
}

int float_bits(float f) {
  int i;
  std::memcpy(&i, &f, 4);
  return i;
}


struct Builder {
  GraphInputs in;
  CompiledGraph *g;
  int64_t exchange_base_words = 0;   // start of the argmax-exchange area inside an inbox buffer
  std::string *err;
  const mpk_config &cfg;
  const std::vector<TensorInfo> &T;
  std::vector<LayerInfo> &L;
  int W;
  int nb_max;
  std::vector<std::vector<TaskDesc>> per_worker;
  std::vector<std::vector<int>> per_worker_exec;
  int rot = 0;
  static constexpr int kMaxFoldedTerms = 16;   // results a linear's prologue averages at most: every task of the linear reads them all
  TaskDesc xattn_task;      // the last extended-attention task (its merge layer shares the fields)
  int hybrid_tickets = 0;   // arrival tickets handed to the tasks of hybrid graphs
  std::map<int, std::map<int, int>> slices;   // storage -> (first column -> id) of outputs that layers write by column range

  Builder(GraphInputs i, CompiledGraph *out, std::string *e)
      : in(i), g(out), err(e), cfg(*i.cfg), T(*i.tensors), L(*i.layers), W(i.num_workers) {
    nb_max = std::min(std::max(cfg.max_num_batched_tokens, 1), (int)kMaxLinearTokens);
  }

  // largest activation tile: 64 KB up to 8 tokens (three 64 KB weight stages remain), 129 KB beyond (two 32 KB stages)
  int64_t x_tile_cap() const { return nb_max <= 8 ? 64 * 1024 + 256 : 64 * (1024 * 2 + kRowPadBytes); }

  // Does the graph run on the general instantiation of the megakernel (more than 8 batched tokens, or any FP8 /
  // expert / latent-attention / sampling layer)?
  bool general_graph() const {
    if (nb_max > 8 || cfg.max_num_batched_tokens > 8) return true;
    if (g->hybrid) return false;
    for (const auto &l : L)
      if (l.op >= MPK_OP_QUANTIZE_FP8) return true;
    return false;
  }

  // More than 8 batched tokens: bf16 linears whose K is a multiple of 64 run on tcgen05 (swap-AB, weights = M = 128,
  // tokens = N = tc_np() <= 64).  The activation operand tile is [K / 64][tc_np()][128 bytes], swizzled.
  // Graphs without a batching task: test mode, and online_notoken (one forward per call on a batch description the
  // caller manages; include/mirage/persistent_kernel/persistent_kernel.cuh:370-411 is the reference's counterpart).
  bool no_batch_task() const { return cfg.test_mode || cfg.mode == MPK_MODE_ONLINE_NOTOKEN; }
  int tc_np() const { return (nb_max + 15) / 16 * 16; }
  bool tc_linear(int64_t K) const { return nb_max > 8 && K % kTcKBlock == 0; }
  // FP8 linears on tcgen05 (block-scaled MMA): K a multiple of 512 (one packed scale word spans 512 columns).  The
  // operand tile is [KT / 128][tc_np()][128 bytes]; behind it sit the scale words of the k tile: 512 bytes per 512
  // columns for the activations and for each of up to kTcFp8MaxTiles row tiles.
  bool tc_linear_fp8(int64_t K) const { return nb_max > 8 && K % 512 == 0; }
  int64_t fp8_tc_tile_bytes(int64_t KT) const { return (int64_t)tc_np() * KT + (int64_t)(kTcFp8MaxTiles + 1) * KT; }
  // The e4m3 activation tile with its scale words may run on into the partial-sum area that follows the tile buffer
  // (these tasks keep no partial sums there), and the buffer may grow until five 16 KB ring slots remain (what the
  // 129 KB bf16 tile leaves as well): at 64 tokens that admits k tiles of 2048 instead of 1024, i.e. half as many
  // stage / drain pauses per task.
  static int64_t fp8_tc_tile_cap() { return (kSmemBudget - kMiscBytes - kPartialBytes - 5 * kTcSlotBytes) / 256 * 256; }
  int64_t linear_tile_bytes(int64_t K) const {
    return tc_linear(K) ? (int64_t)tc_np() * K * 2 : (int64_t)nb_max * (K * 2 + kRowPadBytes);
  }

  // activation tile of an FP8 linear: [tokens, KT] e4m3 rows padded by 16 bytes, then one scale exponent per
  // (token, 128-group) and per (weight row of the task, 128-group)
  static int64_t fp8_tile_bytes(int ntok, int64_t KT) {
    return (int64_t)ntok * (KT + kRowPadBytes) + 16 + (int64_t)ntok * (KT / 128) + 16 + (int64_t)kFp8TaskRows * (KT / 128) + 16;
  }

  // activation tile of an FP8 expert projection: as above, with the float32 scales kept raw (4 bytes each)
  static int64_t moe_fp8_tile_bytes(int ntok, int64_t KT) {
    return (int64_t)ntok * (KT + kRowPadBytes) + 16 + 4 * ((int64_t)ntok * (KT / 128) + 4) + 4 * (int64_t)kFp8TaskRows * (KT / 128) + 16;
  }

  int fail(int code, const std::string &msg) {
    *err = msg;
    return code;
  }

  // inputs / outputs (tensor ids) of a layer, after folding
  void layer_io(const LayerInfo &l, std::vector<int> *ins, std::vector<int> *outs) const {
    auto add = [](std::vector<int> *v, int t) { if (t >= 0) v->push_back(t); };
    switch (l.op) {
      case MPK_OP_EMBED: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); add(ins, norm_tensor(l, 3)); add(ins, norm_tensor(l, 4)); add(outs, norm_tensor(l, 5)); break;
      case MPK_OP_RMSNORM: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_RMSNORM_LINEAR:
        add(ins, l.t[0]); add(ins, l.t[1]); add(ins, l.t[2]); add(outs, l.t[3]); break;
      case MPK_OP_LINEAR: case MPK_OP_SPLITK_LINEAR: case MPK_OP_LINEAR_RESIDUAL: {
        if (l.gather_ar >= 0) {   // the activations arrive through the inbox; the layer materialises them
          add(ins, l.gather_res);
          add(outs, l.gather_out);
        } else {
          add(ins, l.prologue == PRO_PLAIN ? l.t[0] : l.pro_src);
        }
        if (l.prologue == PRO_RMSNORM || l.prologue == PRO_RESNORM || l.prologue == PRO_POLY) add(ins, l.pro_gamma);
        if (l.prologue == PRO_RESNORM) {
          for (int t : {l.pro_y, l.pro_post, l.pro_bias, l.pro_add, l.pro_row}) add(ins, t);
          add(outs, l.pro_xout);
          if (l.pro_terms > 0) add(outs, l.pro_add);   // the results it averages: one of them is its own
        }
        add(ins, l.t[1]);
        const int y = l.op == MPK_OP_LINEAR_RESIDUAL ? l.t[3] : l.t[2];
        if (l.op == MPK_OP_LINEAR_RESIDUAL) add(ins, l.t[2]);
        if (l.op == MPK_OP_LINEAR) add(ins, norm_tensor(l, 3));
        if (l.op == MPK_OP_SPLITK_LINEAR) add(ins, y);
        if (!l.push) add(outs, l.silu_out >= 0 ? l.silu_out : y);
        break;
      }
      case MPK_OP_ATTENTION: case MPK_OP_PAGED_ATTENTION:
        for (int i = 0; i < 7; ++i) add(ins, l.t[i]);
        add(outs, l.t[1]); add(outs, l.t[2]); add(outs, l.t[7]);
        break;
      case MPK_OP_SILU_MUL: add(ins, l.t[0]); add(outs, l.t[1]); break;
      case MPK_OP_AR_PUSH: add(ins, l.t[0]); break;
      case MPK_OP_ALLREDUCE: {
        if (l.ar_producer < 0) {   // before plan_allreduce(): plain reader of its input
          add(ins, l.t[0]);
        } else {                   // fused: reads the producer's residual, the partials arrive by push
          const LayerInfo &p = L[l.ar_producer];
          if (p.op == MPK_OP_LINEAR_RESIDUAL) add(ins, p.t[2]);
          if (p.op == MPK_OP_SPLITK_LINEAR) add(ins, p.t[2]);
        }
        add(outs, l.t[2]);
        break;
      }
      case MPK_OP_ARGMAX_PARTIAL: case MPK_OP_SAMPLING_PARTIAL:
        add(ins, l.t[0]); add(outs, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_ARGMAX_REDUCE: case MPK_OP_SAMPLING_REDUCE: case MPK_OP_ARGMAX_EXCHANGE:
        add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_ELEMENTWISE_ADD: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_TENSOR_INIT: add(outs, l.t[0]); break;
      case MPK_OP_QUANTIZE_FP8: add(ins, l.t[0]); add(outs, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_LINEAR_FP8: for (int i = 0; i < 4; ++i) add(ins, l.t[i]); add(outs, l.t[4]); break;
      case MPK_OP_MOE_TOPK_SIGMOID:
        add(ins, l.t[0]); add(ins, l.t[1]);
        if (!keeps_logits(l)) add(outs, l.t[0]);
        add(outs, l.t[2]); add(outs, l.t[3]); add(outs, l.t[4]); break;
      case MPK_OP_MOE_TOPK_SOFTMAX:
        add(ins, l.t[0]); add(outs, l.t[1]); add(outs, l.t[2]); add(outs, l.t[3]); break;
      case MPK_OP_MOE_W13_LINEAR: case MPK_OP_MOE_W2_LINEAR:
        for (int i = 0; i < 4; ++i) add(ins, l.t[i]); add(outs, l.t[4]); break;
      case MPK_OP_MOE_W13_FP8: case MPK_OP_MOE_W2_FP8:
        for (int i = 0; i < 6; ++i) add(ins, l.t[i]); add(outs, l.t[6]); break;
      case MPK_OP_MOE_SILU_MUL: add(ins, l.t[0]); add(outs, l.t[1]); break;
      case MPK_OP_MOE_MUL_SUM_ADD: add(ins, l.t[0]); add(ins, l.t[1]); add(ins, l.t[2]); add(outs, l.t[3]); break;
      case MPK_OP_MLA_KV_GATHER: add(ins, l.t[0]); add(ins, l.t[1]); add(ins, l.t[2]); add(outs, l.t[2]); break;
      case MPK_OP_MLA_DECODE: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); add(outs, l.t[3]); break;
      case MPK_OP_MLA_REDUCE: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_RESIDUAL_NORM:
        for (int i = 0; i < 14; ++i) if (i != 4 && i != 5) add(ins, norm_tensor(l, i));
        if (resnorm_moves(l)) add(outs, resnorm_out(l));
        add(outs, norm_tensor(l, 12));
        add(outs, l.t[4]);
        break;
      case MPK_OP_QKV_APPEND: add(ins, l.t[0]); for (int i = 4; i < 8; ++i) add(ins, norm_tensor(l, i)); for (int i = 1; i < 4; ++i) add(outs, l.t[i]); break;
      case MPK_OP_ATTN_MERGE: add(ins, l.t[3]); add(outs, l.t[3]); break;
      case MPK_OP_EXT_ATTENTION:
        for (int i = 0; i < 3; ++i) add(ins, l.t[i]);
        for (int i = 4; i < 7; ++i) add(ins, norm_tensor(l, i));
        add(outs, l.t[3]);
        break;
      case MPK_OP_SHORT_CONV: for (int i = 0; i < 5; ++i) add(ins, l.t[i]); add(outs, l.t[4]); add(outs, l.t[5]); add(outs, norm_tensor(l, 6)); break;
      case MPK_OP_SELECTIVE_SCAN: for (int i = 0; i < 8; ++i) add(ins, l.t[i]); add(outs, l.t[7]); add(outs, l.t[8]); break;
      case MPK_OP_DIFF_COMBINE: add(ins, l.t[0]); add(outs, l.t[1]); break;
      case MPK_OP_POLY_NORM: add(ins, l.t[0]); add(ins, l.t[1]); add(outs, l.t[2]); break;
      case MPK_OP_RGLRU: for (int i = 0; i < 9; ++i) add(ins, l.t[i]); add(outs, l.t[8]); add(outs, l.t[9]); break;
      case MPK_OP_MLSTM: for (int i = 0; i < 6; ++i) add(ins, l.t[i]); for (int i = 4; i < 8; ++i) add(outs, l.t[i]); break;
      case MPK_OP_GLA: for (int i = 0; i < 5; ++i) add(ins, l.t[i]); for (int i = 4; i < 7; ++i) add(outs, l.t[i]); break;
      case MPK_OP_LATENT_APPEND:
        add(ins, l.t[0]); add(ins, l.t[1]); add(ins, l.t[4]); add(ins, l.t[5]); add(outs, l.t[2]); add(outs, l.t[3]); break;
      case MPK_OP_GROUPED_LINEAR: add(ins, l.t[0]); add(ins, l.t[1]); add(ins, norm_tensor(l, 3)); add(outs, l.t[2]); break;
      case MPK_OP_LINEAR_FP8_RESIDUAL: for (int i = 0; i < 5; ++i) add(ins, l.t[i]); add(outs, l.t[5]); break;
      default: break;
    }
  }

  bool raw_reads(const LayerInfo &l, int storage) const {
    // does the un-folded layer read this storage?
    std::vector<int> ins, outs;
    layer_io(l, &ins, &outs);
    for (int t : ins) if (T[t].storage == storage) return true;
    return false;
  }
  bool raw_writes(const LayerInfo &l, int storage) const {
    std::vector<int> ins, outs;
    layer_io(l, &ins, &outs);
    for (int t : outs) if (T[t].storage == storage) return true;
    return false;
  }

  int check_arity() {
    for (size_t i = 0; i < L.size(); ++i) {
      static const std::map<int, int> need = {
          {MPK_OP_EMBED, 3}, {MPK_OP_RMSNORM, 3}, {MPK_OP_RMSNORM_LINEAR, 4}, {MPK_OP_LINEAR, 3},
          {MPK_OP_LINEAR_RESIDUAL, 4}, {MPK_OP_SPLITK_LINEAR, 3}, {MPK_OP_ATTENTION, 8},
          {MPK_OP_PAGED_ATTENTION, 8}, {MPK_OP_SILU_MUL, 2}, {MPK_OP_ALLREDUCE, 3},
          {MPK_OP_ARGMAX_PARTIAL, 3}, {MPK_OP_ARGMAX_REDUCE, 3}, {MPK_OP_ELEMENTWISE_ADD, 3},
          {MPK_OP_TENSOR_INIT, 1}, {MPK_OP_QUANTIZE_FP8, 3}, {MPK_OP_LINEAR_FP8, 5}, {MPK_OP_LINEAR_FP8_RESIDUAL, 6},
          {MPK_OP_MOE_TOPK_SIGMOID, 5}, {MPK_OP_MOE_W13_LINEAR, 5}, {MPK_OP_MOE_W2_LINEAR, 5}, {MPK_OP_MOE_W13_FP8, 7},
          {MPK_OP_MOE_W2_FP8, 7}, {MPK_OP_MOE_SILU_MUL, 2}, {MPK_OP_MOE_MUL_SUM_ADD, 4},
          {MPK_OP_MLA_KV_GATHER, 3}, {MPK_OP_MLA_DECODE, 4}, {MPK_OP_MLA_REDUCE, 3},
          {MPK_OP_SAMPLING_PARTIAL, 3}, {MPK_OP_SAMPLING_REDUCE, 3}, {MPK_OP_ARGMAX_EXCHANGE, 3},
          {MPK_OP_MOE_TOPK_SOFTMAX, 4}, {MPK_OP_RESIDUAL_NORM, 5}, {MPK_OP_QKV_APPEND, 6}, {MPK_OP_EXT_ATTENTION, 4},
          {MPK_OP_SHORT_CONV, 6}, {MPK_OP_RGLRU, 10}, {MPK_OP_MLSTM, 8}, {MPK_OP_GLA, 7}, {MPK_OP_LATENT_APPEND, 6},
          {MPK_OP_GROUPED_LINEAR, 3}, {MPK_OP_ATTN_MERGE, 4}, {MPK_OP_SELECTIVE_SCAN, 9}, {MPK_OP_DIFF_COMBINE, 2},
          {MPK_OP_POLY_NORM, 3}};
      auto it = need.find(L[i].op);
      if (it == need.end()) return fail(MPK_ERR_UNSUPPORTED, "layer " + std::to_string(i) + ": unknown op");
      if ((int)L[i].t.size() < it->second)
        return fail(MPK_ERR_INVALID, "layer " + std::to_string(i) + ": expected " + std::to_string(it->second) +
                                         " tensors");
      for (int t : L[i].t)
        if (t >= (int)T.size()) return fail(MPK_ERR_INVALID, "layer " + std::to_string(i) + ": bad tensor id");
    }
    return MPK_OK;
  }

  // ---- folding ----------------------------------------------------------------
  void fold_layers() {
    // RMSNORM_LINEAR is a linear with a norm prologue from the start.
    for (auto &l : L)
      if (l.op == MPK_OP_RMSNORM_LINEAR) {
        LayerInfo n = l;
        n.op = MPK_OP_LINEAR;
        n.t = {l.t[0], l.t[2], l.t[3]};
        n.prologue = PRO_RMSNORM;
        n.pro_src = l.t[0];
        n.pro_gamma = l.t[1];
        l = n;
      }
    for (size_t i = 0; i < L.size(); ++i) {
      LayerInfo &p = L[i];
      if (p.folded || (p.op != MPK_OP_RMSNORM && p.op != MPK_OP_SILU_MUL)) continue;
      const int y = p.op == MPK_OP_RMSNORM ? p.t[2] : p.t[1];
      const int src = p.t[0];
      if (T[y].owner == 0) continue;   // caller-visible buffer: keep it materialised
      std::vector<size_t> consumers;
      bool ok = true;
      for (size_t j = i + 1; j < L.size() && ok; ++j) {
        const LayerInfo &c = L[j];
        const bool reads = raw_reads(c, T[y].storage);
        if (reads) {
          const bool lin = (c.op == MPK_OP_LINEAR || c.op == MPK_OP_LINEAR_RESIDUAL ||
                            c.op == MPK_OP_SPLITK_LINEAR) && c.prologue == PRO_PLAIN && c.t[0] == y;
          // y must not also be this consumer's residual / accumulate operand
          const bool other_use = (c.op == MPK_OP_LINEAR_RESIDUAL && T[c.t[2]].storage == T[y].storage);
          if (!lin || other_use) ok = false;
          else consumers.push_back(j);
          // the norm prologue needs the whole row in the activation tile
          if (ok && p.op == MPK_OP_RMSNORM && linear_tile_bytes(T[c.t[1]].dim(1)) > x_tile_cap()) ok = false;
        }
        if (raw_writes(c, T[y].storage)) break;           // y redefined: later readers see the new value
      }
      if (!ok || consumers.empty()) continue;
      // no layer between the producer and its last consumer may overwrite the source
      for (size_t j = i + 1; j < consumers.back() && ok; ++j)
        if (raw_writes(L[j], T[src].storage)) ok = false;
      if (!ok) continue;
      for (size_t j : consumers) {
        LayerInfo &c = L[j];
        if (p.op == MPK_OP_RMSNORM) {
          c.prologue = PRO_RMSNORM;
          c.pro_src = src;
          c.pro_gamma = p.t[1];
        } else {
          c.prologue = PRO_SILU_MUL;
          c.pro_src = src;
          c.pro_groups = std::max(p.grid[0], 1);
        }
      }
      p.folded = true;
      g->num_folded++;
    }
  }

  // Stream tensor a residual_norm layer writes: its own output (t[5]) or the input in place.
  static int norm_tensor(const LayerInfo &l, size_t i) { return i < l.t.size() ? l.t[i] : -1; }
  static int resnorm_out(const LayerInfo &l) { return norm_tensor(l, 5) >= 0 ? l.t[5] : l.t[0]; }
  // Does the layer add anything to the stream?
  static bool resnorm_moves(const LayerInfo &l) {
    return l.t[1] >= 0 || norm_tensor(l, 7) >= 0 || norm_tensor(l, 8) >= 0 || norm_tensor(l, 9) >= 0;
  }
  static int norm_flags(const LayerInfo &l) { return (l.params[1] ? 2 : 0) | (l.params.size() > 2 && l.params[2] == 1 ? 4 : 0); }
  // columns of x a residual_norm layer works on
  int64_t norm_columns(const LayerInfo &l) const { return l.params.size() > 5 && l.params[5] > 0 ? l.params[5] : T[l.t[0]].dim(1); }
  static int norm_factor(const LayerInfo &l) { return l.params.size() > 4 ? bits_of(l.params[4]) : 0x3f800000; }   // (1.0f)
  static bool keeps_logits(const LayerInfo &l) { return l.params.size() > 5 && l.params[5] != 0; }

  // Hybrid graphs of one or two tokens: a residual_norm layer whose result feeds linears becomes their prologue, which
  // spares the chain a task group.  (With more tokens the rows are spread over the workers instead of being formed by all.)
  void fold_residual_norms() {
    if (g->hybrid != HYB_BF16 || nb_max > 2 || cfg.max_num_batched_tokens > 2) return;
    for (size_t i = 0; i < L.size(); ++i) {
      LayerInfo &p = L[i];
      if (p.op != MPK_OP_RESIDUAL_NORM || p.t[4] < 0) continue;
      const int x = p.t[0], y = p.t[1], out = p.t[4], xo = resnorm_out(p), add = norm_tensor(p, 7), row = norm_tensor(p, 8), bias = norm_tensor(p, 6);
      if (norm_tensor(p, 9) >= 0 || norm_tensor(p, 11) >= 0) continue;   // the sum over experts is formed once, not by every task
      const int results = norm_tensor(p, 12), terms = results >= 0 ? (int)T[p.t[13]].dim(0) : 0;
      if (results >= 0 && (add >= 0 || row >= 0 || terms > kMaxFoldedTerms || ((uint64_t)T[results].ptr & 15) || T[results].strides[0] % 4)) continue;
      const bool moves = resnorm_moves(p);
      auto aligned = [&](int t) { return T[t].ld() % 4 == 0 && ((uint64_t)T[t].ptr & 15) == 0; };
      const int64_t D = norm_columns(p);
      if (T[out].owner == 0 || D > 4096 || D % 4 || !aligned(x) || (p.t[3] >= 0 && ((uint64_t)T[p.t[3]].ptr & 7)) || p.params.size() < 2) continue;
      if (moves && (T[xo].storage == T[x].storage || !aligned(xo) || T[xo].dtype != MPK_F32 || T[xo].dim(1) != D)) continue;
      if ((y >= 0 && !aligned(y)) || (add >= 0 && (!aligned(add) || T[add].dtype != MPK_F32 || T[add].dim(1) != D))) continue;
      if ((bias >= 0 && ((uint64_t)T[bias].ptr & 7)) || (row >= 0 && ((uint64_t)T[row].ptr & 7))) continue;
      if (p.t[2] >= 0 && ((uint64_t)T[p.t[2]].ptr & 7)) continue;
      std::vector<size_t> consumers;
      bool ok = true;
      for (size_t j = i + 1; j < L.size() && ok; ++j) {
        const LayerInfo &c = L[j];
        if (raw_reads(c, T[out].storage)) {
          if (c.op != MPK_OP_LINEAR || c.prologue != PRO_PLAIN || c.t[0] != out || T[c.t[1]].dim(1) > 4096 ||
              linear_tile_bytes(T[c.t[1]].dim(1)) > x_tile_cap()) ok = false;
          else consumers.push_back(j);
        }
        if (raw_writes(c, T[out].storage)) break;
      }
      if (!ok || consumers.size() != 1) continue;
      for (size_t j = i + 1; j < consumers[0] && ok; ++j)   // nothing in between may touch what the prologue reads or writes
        for (int t : {x, y, xo, add, results})
          if (t >= 0 && (raw_writes(L[j], T[t].storage) || (t == xo && moves && raw_reads(L[j], T[t].storage)))) ok = false;
      if (!ok) continue;
      LayerInfo &c = L[consumers[0]];
      c.prologue = PRO_RESNORM;
      c.pro_src = x; c.pro_y = y; c.pro_post = p.t[2]; c.pro_gamma = p.t[3];
      c.pro_bias = bias; c.pro_add = add; c.pro_row = row;
      c.pro_xout = moves ? xo : -1;
      c.pro_cols = (int)D;
      c.pro_terms = terms;
      if (terms > 0) { c.pro_add = results; c.pro_row = p.t[13]; }
      c.pro_eps = bits_of(p.params[0]); c.pro_flags = norm_flags(p) | (terms > 0 ? 8 : 0); c.pro_factor = norm_factor(p);
      p.folded = true;
      g->num_folded++;
    }
  }

  // The same for the sum of normed powers in front of a linear.
  void fold_poly_norms() {
    if (g->hybrid != HYB_BF16 || nb_max > 2 || cfg.max_num_batched_tokens > 2) return;
    for (size_t i = 0; i < L.size(); ++i) {
      LayerInfo &p = L[i];
      if (p.op != MPK_OP_POLY_NORM || p.params.empty() || T[p.t[2]].owner == 0) continue;
      const int z = p.t[0], out = p.t[2];
      std::vector<size_t> consumers;
      bool ok = true;
      for (size_t j = i + 1; j < L.size() && ok; ++j) {
        const LayerInfo &c = L[j];
        if (raw_reads(c, T[out].storage)) {
          if (c.op != MPK_OP_LINEAR || c.prologue != PRO_PLAIN || c.t[0] != out || linear_tile_bytes(T[c.t[1]].dim(1)) > x_tile_cap()) ok = false;
          else consumers.push_back(j);
        }
        if (raw_writes(c, T[out].storage)) break;
      }
      if (!ok || consumers.size() != 1) continue;
      for (size_t j = i + 1; j < consumers[0] && ok; ++j)
        if (raw_writes(L[j], T[z].storage)) ok = false;
      if (!ok || T[z].dtype != MPK_F32 || T[p.t[1]].dtype != MPK_BF16 || T[p.t[1]].dim(0) != 4 || T[z].dim(1) > T[L[consumers[0]].t[1]].dim(1)) continue;
      LayerInfo &c = L[consumers[0]];
      c.prologue = PRO_POLY;
      c.pro_src = z; c.pro_gamma = p.t[1]; c.pro_cols = (int)T[z].dim(1); c.pro_eps = bits_of(p.params[0]);
      p.folded = true;
      g->num_folded++;
    }
  }

  // ---- allreduce fusion: linear -> allreduce becomes push epilogue + reduce tasks -----
  int plan_allreduce() {
    auto pushing_linear = [&](int j) {
      return j >= 0 && (L[j].op == MPK_OP_LINEAR || L[j].op == MPK_OP_LINEAR_RESIDUAL || L[j].op == MPK_OP_SPLITK_LINEAR);
    };
    auto producer_of = [&](size_t i) {
      for (int j = (int)i - 1; j >= 0; --j)
        if (!L[j].folded && raw_writes(L[j], T[L[i].t[0]].storage)) return j;
      return -1;
    };
    // An allreduce whose input comes from anything but a bf16 linear (an FP8 linear, the weighted sum of a
    // mixture-of-experts block, ...) gets a push stage of its own in front of it: the input is materialised by its
    // producer as usual and copied into the ranks' inboxes by TASK_AR_PUSH tasks.
    for (size_t i = 0; i < L.size(); ++i) {
      if (L[i].op != MPK_OP_ALLREDUCE) continue;
      if (cfg.world_size <= 1) return fail(MPK_ERR_INVALID, "allreduce_layer with world_size 1");
      const int prod = producer_of(i);
      if (prod < 0) return fail(MPK_ERR_UNSUPPORTED, "allreduce input is not produced inside the graph");
      if (pushing_linear(prod)) continue;
      if (T[L[i].t[0]].dtype != MPK_BF16 || T[L[i].t[0]].dims.size() != 2)
        return fail(MPK_ERR_UNSUPPORTED, "allreduce input must be a 2-D bf16 tensor");
      LayerInfo p;
      p.op = MPK_OP_AR_PUSH;
      p.t = {L[i].t[0]};
      L.insert(L.begin() + i, p);
      ++i;
    }
    int idx = 0;
    for (size_t i = 0; i < L.size(); ++i) {
      LayerInfo &a = L[i];
      if (a.op != MPK_OP_ALLREDUCE) continue;
      const int x = a.t[0];
      int prod = (i > 0 && L[i - 1].op == MPK_OP_AR_PUSH && L[i - 1].t[0] == x) ? (int)i - 1 : producer_of(i);
      if (prod < 0 || !(pushing_linear(prod) || L[prod].op == MPK_OP_AR_PUSH))
        return fail(MPK_ERR_UNSUPPORTED, "allreduce input must be produced by a linear layer");
      for (size_t j = prod + 1; j < L.size(); ++j) {
        if (j != i && !L[j].folded && raw_reads(L[j], T[x].storage) && j < i)
          return fail(MPK_ERR_UNSUPPORTED, "allreduce input has another reader before the allreduce");
      }
      L[prod].push = true;
      L[prod].ar_index = idx;
      a.ar_producer = prod;
      a.ar_index = idx++;
    }
    // an argmax exchange is one more instance in the same sequence (its words live in their own area of the inbox)
    for (auto &a : L)
      if (a.op == MPK_OP_ARGMAX_EXCHANGE) {
        if (cfg.world_size <= 1) return fail(MPK_ERR_INVALID, "argmax exchange with world_size 1");
        a.ar_index = idx++;
      }
    g->num_allreduce = idx;
    fold_allreduce();
    return MPK_OK;
  }

  // Fold an allreduce into the linears that consume its result: the producer pushes self-validating words,
  // the consumers' prologue gathers, reduces, adds the residual and materialises the tensor.  No task and
  // no event remain for the allreduce itself.
  void fold_allreduce() {
    // Only for graphs of at most 8 batched tokens.  The fused form makes EVERY consumer CTA poll and read the whole
    // [world][tokens][K] inbox: 8 KB per rank at one token, but 128 KB per rank at 16 -- at 8 ranks 148 CTAs pulling
    // 2 MB each per allreduce, measured at 12.2 ms per 16-token step on 8 GPUs against 6.0 ms on one.  With more
    // tokens the allreduce stays a task group of its own: fp32 partials pushed by the producer's epilogue, summed once
    // by reduce tasks spread over the workers, read as an ordinary activation by the consumers.
    if (cfg.max_num_batched_tokens > 8) return;
    auto is_lin = [](int op) { return op == MPK_OP_LINEAR || op == MPK_OP_LINEAR_RESIDUAL || op == MPK_OP_SPLITK_LINEAR; };
    for (size_t i = 0; i < L.size(); ++i) {
      LayerInfo &a = L[i];
      if (a.op != MPK_OP_ALLREDUCE || a.ar_producer < 0) continue;
      if (L[a.ar_producer].op == MPK_OP_AR_PUSH) continue;   // (fp32 slots + remote event: summed by TASK_ALLREDUCE)
      LayerInfo &prod = L[a.ar_producer];
      const int y = a.t[2];
      const int res = (prod.op == MPK_OP_LINEAR_RESIDUAL || prod.op == MPK_OP_SPLITK_LINEAR) ? prod.t[2] : -1;
      if (T[y].dims.size() != 2 || T[y].dtype != MPK_BF16) continue;
      std::vector<size_t> consumers;
      bool ok = true;
      for (size_t j = i + 1; j < L.size() && ok; ++j) {
        const LayerInfo &c = L[j];
        if (c.folded) continue;
        if (raw_reads(c, T[y].storage)) {
          const bool as_input = is_lin(c.op) && c.gather_ar < 0 &&
                                ((c.prologue == PRO_RMSNORM && c.pro_src == y) || (c.prologue == PRO_PLAIN && c.t[0] == y)) &&
                                T[c.t[1]].dim(1) == T[y].dim(1);
          const bool as_pushed_residual = is_lin(c.op) && c.push && c.t[2] == y && !as_input &&
                                          !(c.prologue == PRO_PLAIN && c.t[0] == y) && c.pro_src != y;
          const bool as_ar_residual = c.op == MPK_OP_ALLREDUCE;
          if (as_input) consumers.push_back(j);
          else if (!as_pushed_residual && !as_ar_residual) ok = false;
        }
        if (j != i && raw_writes(c, T[y].storage)) break;
      }
      if (!ok || consumers.empty()) continue;
      for (size_t j : consumers) {
        L[j].gather_ar = a.ar_index;
        L[j].gather_res = res;
        L[j].gather_out = y;
      }
      prod.push_ll = true;
      a.folded = true;
      g->num_folded++;
    }
  }

  // ---- shared-memory plan ---------------------------------------------------------
  int plan_smem() {
    const int ntok = std::min(std::max(cfg.max_num_batched_tokens, 1), (int)kMaxLinearTokens);
    int64_t need = 24 * 1024;
    for (const auto &l : L) {
      if (l.folded) continue;
      if (hybrid_op(l.op)) {
        need = std::max<int64_t>(need, hybrid_smem(l) - kPartialBytes);
        if (l.op == MPK_OP_GROUPED_LINEAR && g->hybrid == HYB_BF16 && tc_linear(T[l.t[1]].dim(2))) g->use_tmem = true;
      } else if (g->hybrid == HYB_F32 && l.op == MPK_OP_LINEAR) {
        const int64_t K = T[l.t[1]].dim(1);
        need = std::max<int64_t>(need, (int64_t)linear_f32_tokens(K) * K * 4 - kPartialBytes);
      } else if (l.op == MPK_OP_LINEAR || l.op == MPK_OP_LINEAR_RESIDUAL || l.op == MPK_OP_SPLITK_LINEAR) {
        const int64_t K = T[l.t[1]].dim(1);
        need = std::max(need, std::min<int64_t>(linear_tile_bytes(K), x_tile_cap()));
        if (tc_linear(K) && T[l.t[1]].dtype == MPK_BF16) g->use_tmem = true;
      } else if (l.op == MPK_OP_LINEAR_FP8 || l.op == MPK_OP_LINEAR_FP8_RESIDUAL) {
        const int64_t K = T[l.t[2]].dim(1);
        if (tc_linear_fp8(K)) {
          g->use_tmem = true;
          int64_t KT = K;
          while (KT > 512 && (fp8_tc_tile_bytes(KT) - kPartialBytes > fp8_tc_tile_cap() || K % KT != 0 || KT % 512 != 0)) KT -= 512;
          need = std::max<int64_t>(need, fp8_tc_tile_bytes(KT) - kPartialBytes);
        } else {
          need = std::max(need, std::min<int64_t>(fp8_tile_bytes(ntok, K), x_tile_cap()));
        }
      } else if (l.op == MPK_OP_MOE_W13_FP8 || l.op == MPK_OP_MOE_W2_FP8) {
        need = std::max(need, std::min<int64_t>(moe_fp8_tile_bytes(ntok, T[l.t[2]].dim(2)), x_tile_cap()));
      } else if (g->hybrid == HYB_F32 && (l.op == MPK_OP_MOE_W13_LINEAR || l.op == MPK_OP_MOE_W2_LINEAR)) {
        const int64_t K = T[l.t[1]].dim(2);
        need = std::max<int64_t>(need, (int64_t)linear_f32_tokens(K) * K * 4 + 256 - kPartialBytes);
      } else if (l.op == MPK_OP_MOE_W13_LINEAR || l.op == MPK_OP_MOE_W2_LINEAR) {
        const int64_t K = T[l.t[1]].dim(2);
        need = std::max(need, std::min<int64_t>((int64_t)ntok * (K * 2 + kRowPadBytes), x_tile_cap()));
        if (g->hybrid && tc_linear(K)) {
          g->use_tmem = true;
          need = std::max<int64_t>(need, (int64_t)tc_np() * kTcKBlock * 2 * 4);   // four k blocks of all tokens' rows at least
        }
      } else if (l.op == MPK_OP_MLA_DECODE) {
        need = std::max<int64_t>(need, 16 * (576 * 2 + 16) + 64 * (576 * 2 + 16) + 16 * (64 * 2 + 16) + 2 * 8 * 16 * 4);
      } else if (l.op == MPK_OP_MOE_TOPK_SIGMOID || l.op == MPK_OP_MOE_TOPK_SOFTMAX) {
        const int64_t E = T[l.t[l.op == MPK_OP_MOE_TOPK_SIGMOID ? 3 : 2]].dim(0);
        need = std::max(need, 8 * (2 * E + 64) * 4 + E * 4 + 64);
      } else if (l.op == MPK_OP_ATTENTION || l.op == MPK_OP_PAGED_ATTENTION) {
        const int G = (int)(l.params[0] / l.params[1]);
        int64_t attn = (int64_t)G * (128 + 16 + 8 * 128) * 4 + (int64_t)cfg.max_num_batched_tokens * 512;
        // the general instantiation streams cached K/V rows through 32 KB stages (two at least) beside the query
        // heads, the per-warp maxima / sums, 256 page ids and the rows of the new tokens
        if (general_graph()) {
          const int64_t new_rows = (std::min(cfg.max_num_batched_tokens, 64) + 7) / 8 * 8;
          attn = 8 * 272 + (int64_t)G * 64 + 1024 + 2 * new_rows * 272 + 2 * (8 * 2 * 8 * 272);   // two stages per warp
        }
        need = std::max(need, attn - kPartialBytes);
      }
    }
    if (!no_batch_task()) need = std::max<int64_t>(need, (int64_t)(16 * cfg.max_num_batched_requests + 20 + (cfg.mode == MPK_MODE_ONLINE ? cfg.total_num_requests : 0)) * 4 - kPartialBytes);
    need = (need + 255) / 256 * 256;
    // 64 KB stages (4 KB row segments) when at least three of them fit, else 32 KB stages
    const int64_t room = kSmemBudget - kMiscBytes - kPartialBytes - need;
    g->x_tile_bytes = (int)need;
    g->tc_tokens = tc_np();
    if (g->use_tmem) {
      // tcgen05 graphs: a ring of 16 KB slots (whole swizzle atoms), each filled by one tensor-map TMA; tasks that
      // still stream padded rows (FP8, expert projections) take the widest chunk such a slot holds
      const int stages = (int)(room / kTcSlotBytes);
      if (stages < 2) return fail(MPK_ERR_UNSUPPORTED, "activation tile leaves fewer than 2 weight stages");
      g->stage_bytes = kTcSlotBytes;
      g->chunk_cols = 448;                 // 16 rows x (448 x 2 + 16) bytes <= 16 KB
      g->num_stages = std::min(stages, 8);
      return MPK_OK;
    }
    int cols = kChunkColsMax;
    if (room / stage_bytes_for(cols) < (nb_max <= 8 ? 3 : 2)) cols = kChunkColsMax / 2;
    const int stages = (int)(room / stage_bytes_for(cols));
    if (stages < 2) return fail(MPK_ERR_UNSUPPORTED, "activation tile leaves fewer than 2 weight stages");
    g->chunk_cols = cols;
    g->stage_bytes = stage_bytes_for(cols);
    g->num_stages = std::min(stages, 8);   // (the kernel uses the upper half of its 16-entry barrier arrays as scratch)
    return MPK_OK;
  }

  // ---- task emission ----------------------------------------------------------------
  TaskDesc blank(uint32_t type, int layer) {
    TaskDesc d;
    std::memset(&d, 0, sizeof(d));
    d.type = type;
    d.layer = layer;
    for (int i = 0; i < kMaxDeps; ++i) d.dep_event[i] = -1;
    d.trig_event = -1;
    return d;
  }
  void put(int worker, const TaskDesc &d, int exec) {
    per_worker[worker].push_back(d);
    per_worker_exec[worker].push_back(exec);
    g->exec[exec].num_tasks++;
  }

  int emit_linear(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &w = T[l.t[1]];
    const int yid = l.op == MPK_OP_LINEAR_RESIDUAL ? l.t[3] : l.t[2];
    const TensorInfo &y = T[yid];
    if (w.dims.size() != 2 || w.dtype != MPK_BF16)
      return fail(MPK_ERR_UNSUPPORTED, "linear weight must be a 2-D bf16 tensor: " + w.name);
    if (w.strides[1] != 1) return fail(MPK_ERR_UNSUPPORTED, "linear weight must be row-major: " + w.name);
    const int N = (int)w.dim(0), K = (int)w.dim(1), ldw = (int)w.strides[0];
    if (cfg.max_num_batched_tokens > kMaxLinearTokens)
      return fail(MPK_ERR_UNSUPPORTED, "linear layers support at most 64 batched tokens in this build");
    if (K % 16 != 0 || ldw % 8 != 0) return fail(MPK_ERR_UNSUPPORTED, "linear K must be a multiple of 16: " + w.name);
    // k tiling of the activation tile: the fewest tiles whose [tokens, KT] slab fits the tile buffer
    const int ntok = std::min(std::max(cfg.max_num_batched_tokens, 1), (int)kMaxLinearTokens);
    const bool tc = g->use_tmem && tc_linear(K);
    const int kq = tc ? kTcKBlock : 16;   // granularity of a k tile
    int nkt = 1;
    while (nkt <= K / kq &&
           !(K % nkt == 0 && (K / nkt) % kq == 0 && linear_tile_bytes(K / nkt) <= g->x_tile_bytes))
      ++nkt;
    if (nkt > K / kq) return fail(MPK_ERR_UNSUPPORTED, "cannot tile K for " + w.name);
    const int KT = K / nkt;
    const bool f32_source = l.prologue == PRO_RESNORM || l.prologue == PRO_POLY;   // formed from float32 values by the prologue
    if ((l.prologue == PRO_RMSNORM || f32_source) && nkt != 1)
      return fail(MPK_ERR_UNSUPPORTED, "rmsnorm prologue needs the whole row in shared memory: " + w.name);
    // k extent of a streamed chunk: the largest multiple of 16 that divides KT and fits a stage
    // Chunk geometry: 16 rows (one mma m-tile) x KC columns.  The copy engine handles a fixed number of bulk
    // copies per unit time, so row segments should be long: KC is as wide as the stage allows.
    const int R = kChunkRows;
    int KC = std::min(KT, g->chunk_cols) / 16 * 16;
    while (KC > 16 && KT % KC != 0) KC -= 16;
    // with several k tiles the partial sums of a task wait in shared memory: two row groups at most
    const int cap = nkt > 1 ? 2 * R : (1 << 20);
    // source of the activation
    const int xsrc = l.prologue == PRO_PLAIN ? l.t[0] : l.pro_src;
    const TensorInfo &x = T[xsrc];
    if (l.prologue == PRO_SILU_MUL) {
      if (x.dim(1) != 2 * (int64_t)K || (K / l.pro_groups) % 8 != 0 || K % l.pro_groups != 0)
        return fail(MPK_ERR_INVALID, "silu_mul feeding " + w.name + ": bad gate|up width or group count");
    } else if (!f32_source && x.dim(x.dims.size() - 1) != K) {
      return fail(MPK_ERR_INVALID, "linear input width != K for " + w.name);
    }
    int epi = EPI_STORE;
    bool gated = false;
    const int bias = l.op == MPK_OP_LINEAR ? norm_tensor(l, 3) : -1;
    if (bias >= 0 && (y.dtype != MPK_F32 || T[bias].dtype != MPK_BF16 || T[bias].dim(0) < N || (!l.params.empty() && l.params[0])))
      return fail(MPK_ERR_INVALID, "linear bias: bf16 [rows], float32 output, no activation: " + w.name);
    uint64_t res_ptr = 0;
    int ldr = 0;
    if (l.op == MPK_OP_LINEAR_RESIDUAL) {
      const bool enable = l.params.empty() ? true : l.params[0] != 0;
      // With tensor parallelism the reference adds the residual on rank 0 only
      // (python/mirage/mpk/persistent_kernel.py:1783-1787); here the residual of a pushed
      // linear is added once by the reduce tasks instead, on every rank identically.
      if (enable && !l.push) { epi = EPI_RESIDUAL; res_ptr = (uint64_t)T[l.t[2]].ptr; ldr = (int)T[l.t[2]].ld(); }
    } else if (l.op == MPK_OP_SPLITK_LINEAR && !l.push) {
      epi = EPI_RESIDUAL; res_ptr = (uint64_t)y.ptr; ldr = (int)y.ld();
    }
    if (l.push) epi = l.push_ll ? EPI_PUSH_LL : EPI_PUSH_F32;
    if (x.dtype != MPK_BF16 && !f32_source) return fail(MPK_ERR_UNSUPPORTED, "linear input must be bf16: " + w.name);
    if (l.op == MPK_OP_LINEAR && !l.params.empty() && l.params[0] != 0) {
      epi = activation_epilogue(l.params[0]);
      if (g->hybrid != HYB_BF16 || epi == EPI_STORE || y.dtype != (capped(epi) ? MPK_F32 : MPK_BF16) || (capped(epi) && l.params.size() < 2))
        return fail(MPK_ERR_UNSUPPORTED, "linear activation: in hybrid graphs, bf16 output (soft cap, scale: float32): " + w.name);
      gated = epi == EPI_GATED_SILU || epi == EPI_GATED_GELU;
      if (gated && N % 4) return fail(MPK_ERR_INVALID, "gated linear: rows come as two gate rows, two up rows: " + w.name);
    } else if (y.dtype == MPK_F32) {
      if (g->hybrid != HYB_BF16 || epi != EPI_STORE) return fail(MPK_ERR_UNSUPPORTED, "float32 linear output needs a hybrid graph: " + w.name);
      epi = bias >= 0 ? EPI_BIAS_F32 : EPI_STORE_F32;
    } else if (y.dtype != MPK_BF16) {
      return fail(MPK_ERR_UNSUPPORTED, "linear output must be bf16 or float32: " + w.name);
    }
    uint64_t out_ptr = (uint64_t)y.ptr;
    int ldo = (int)y.ld();
    // (hybrid graphs: the output buffer may be padded to the k granularity of the next linear)
    const int out_cols = gated ? N / 2 : N;
    if (g->hybrid ? y.dim(y.dims.size() - 1) < out_cols : y.dim(y.dims.size() - 1) != N)
      return fail(MPK_ERR_INVALID, "linear output width != N for " + w.name);
    const int unit = l.silu_out >= 0 || gated ? 4 : 1;      // paired rows stay in one task
    if (l.silu_out >= 0) {
      if (epi != EPI_STORE || N % 4 != 0) return fail(MPK_ERR_INVALID, "activation epilogue on an unsupported linear: " + w.name);
      epi = EPI_SILU_PAIR;
      out_ptr = (uint64_t)T[l.silu_out].ptr;
      ldo = (int)T[l.silu_out].ld();
    }
    bool w_dynamic = false;
    for (const auto &o : L) if (!o.folded && raw_writes(o, w.storage)) w_dynamic = true;
    const int base = (N / unit) / W, rem = (N / unit) % W;
    // tcgen05 path: cut the widest worker panel into row tiles of RB <= 128 rows (one accumulator each) and give a
    // ring slot as many 64-column k blocks of such a tile as it holds; among the tilings near the minimum, take
    // the one that fills the slots best (the bytes in flight per worker are what hides the HBM latency)
    int tc_rb = 0, tc_nkb = 1, tc_task_rows = 0;
    if (tc) {
      const int cnt_max = (base + (rem ? 1 : 0)) * unit;
      const int kbt = KT / kTcKBlock;
      const int t_min = (cnt_max + 127) / 128;
      // Measured: an M = 128 bf16 tcgen05.mma with N <= 64 occupies the tensor pipe for about 43 cycles whatever N is
      // and however few of its 128 rows are real, and a worker must consume ~23 weight bytes per cycle to keep up
      // with its share of HBM.  A K = 16 step of a tile with r real rows consumes 32 r bytes: r must exceed ~31
      // for the MMAs to stay ahead of the stream, so tiles keep at least 40 real rows where the panel allows.
      const int need_rows = 40;
      double best = -1.0;
      for (int tiles = t_min; tiles <= t_min + 6; ++tiles) {
        const int rb = ((cnt_max + tiles - 1) / tiles + 7) / 8 * 8;
        if (rb > 128 || rb <= 0) continue;
        if (tiles > t_min && cnt_max / tiles < need_rows) break;
        int nkb = std::min(kbt, g->stage_bytes / (rb * 128));
        while (nkb > 1 && kbt % nkb != 0) --nkb;
        if (nkb < 1) continue;
        const double fill = (double)cnt_max / tiles * 128.0 * nkb / g->stage_bytes;
        if (fill > best * 1.05) { best = fill; tc_rb = rb; tc_nkb = nkb; }
      }
      if (tc_rb == 0) return fail(MPK_ERR_UNSUPPORTED, "cannot tile the rows of " + w.name);
      tc_task_rows = std::max(1, kTcAccCols / tc_np()) * tc_rb;   // accumulators of one task: tiles x tc_np() columns
      g->exec[ex].tc_rows = tc_rb;
      g->exec[ex].tc_kblocks = tc_nkb;
    }
    const int task_cap = tc ? tc_task_rows : cap;
    int row = 0;
    for (int i = 0; i < W; ++i) {
      const int worker = (i + rot) % W;
      const int cnt = (base + (i < rem ? 1 : 0)) * unit;
      bool first = true;
      for (int r = row; r < row + cnt; r += task_cap) {
        TaskDesc d = blank(TASK_LINEAR, li);
        if (!first && nkt == 1) d.flags |= TF_SAME_X_AS_PREV;
        if (w_dynamic) d.flags |= TF_STREAM_AFTER_DEP;
        d.p[0] = (uint64_t)w.ptr;
        d.p[1] = (uint64_t)x.ptr;
        d.p[2] = out_ptr;
        d.p[3] = res_ptr;
        d.p[4] = l.prologue == PRO_RMSNORM || l.prologue == PRO_POLY ? (uint64_t)T[l.pro_gamma].ptr : 0;
        d.p[5] = in.inbox_base_floats;
        if (l.gather_ar >= 0) {
          d.p[6] = l.gather_res >= 0 ? (uint64_t)T[l.gather_res].ptr : 0;
          d.p[7] = (uint64_t)T[l.gather_out].ptr;
          d.a[L_GATHER] = l.gather_ar + 1;
          d.a[L_G_LDRES] = l.gather_res >= 0 ? (int)T[l.gather_res].ld() : 0;
          d.a[L_G_LDOUT] = (int)T[l.gather_out].ld();
          d.a[L_G_SLOT] = cfg.max_num_batched_tokens * K;
        }
        if (l.prologue == PRO_RESNORM) {
          d.p[3] = l.pro_post >= 0 ? (uint64_t)T[l.pro_post].ptr : 0;
          d.p[4] = l.pro_gamma >= 0 ? (uint64_t)T[l.pro_gamma].ptr : 0;
          d.p[6] = l.pro_y >= 0 ? (uint64_t)T[l.pro_y].ptr : 0;
          d.p[7] = l.pro_xout >= 0 ? (uint64_t)T[l.pro_xout].ptr : 0;
          d.a[L_G_LDRES] = l.pro_y >= 0 ? (int)T[l.pro_y].ld() : 0;
          d.a[L_G_LDOUT] = l.pro_xout >= 0 ? (int)T[l.pro_xout].ld() : 0;
          d.a[L_G_SLOT] = l.pro_flags;
          d.p[5] = l.pro_bias >= 0 ? (uint64_t)T[l.pro_bias].ptr : 0;
          d.a[LR_LDADD] = l.pro_terms > 0 ? (int)T[l.pro_add].strides[0] : l.pro_add >= 0 ? (int)T[l.pro_add].ld() : 0;
        }
        d.a[L_N0] = r;
        d.a[L_N1] = std::min(r + task_cap, row + cnt);
        d.a[L_K] = K;
        d.a[L_LDW] = ldw;
        d.a[L_LDX] = (int)x.ld();
        d.a[L_LDO] = ldo;
        d.a[L_LDR] = l.prologue == PRO_RESNORM ? l.pro_terms : ldr;
        d.a[L_PRO] = l.prologue;
        d.a[L_EPI] = epi;
        d.a[L_EPS] = f32_source ? l.pro_eps : float_bits(1e-6f);
        d.a[L_GROUPS] = f32_source ? l.pro_cols : l.pro_groups;
        d.a[L_KT] = KT;
        d.a[L_KC] = KC;
        d.a[L_ROWS] = R;
        d.a[L_SLOT] = cfg.max_num_batched_tokens * N;
        d.a[L_N] = N;
        d.a[L_ARIDX] = std::max(l.ar_index, 0);
        d.a[L_NAR] = g->num_allreduce;
        d.a[L_PARSTRIDE] = (int)g->inbox_floats_per_buffer;
        if (capped(epi)) d.a[L_CAP] = bits_of(l.params[1]);
        if (epi == EPI_BIAS_F32) put_wide(&d, LR_BIAS, bias);
        if (l.prologue == PRO_RESNORM) {
          d.a[LR_POST] = l.pro_factor;
          put_wide(&d, LR_ADD, l.pro_add);
          put_wide(&d, LR_ROW, l.pro_row);
        }
        if (tc) {
          d.flags |= TF_TC;
          d.a[L_KC] = tc_nkb * kTcKBlock;
          d.a[L_ROWS] = tc_rb;
          d.a[L_TMAP] = (int)g->tmaps.size();
          TmapSpec m;
          m.base = (uint64_t)w.ptr + (uint64_t)r * (uint64_t)ldw * 2;
          m.rows = d.a[L_N1] - d.a[L_N0];
          m.ld_bytes = (int64_t)ldw * 2;
          m.kblocks = K / kTcKBlock;
          m.box_rows = tc_rb;
          m.box_kblocks = tc_nkb;
          m.elt_bytes = 2;
          g->tmaps.push_back(m);
        }
        put(worker, d, ex);
        g->weight_bytes += (int64_t)(d.a[L_N1] - d.a[L_N0]) * K * 2;
        first = false;
      }
      row += cnt;
    }
    return MPK_OK;
  }

  // Strides (in uint32 words) of a packed UE8M0 scale tensor over (outer index, packed k).  Accepted layouts:
  // logical [outer, packed_k] with any strides, or the physical column-major form [packed_k, aligned_outer]
  // that the reference's builders allocate (python/mirage/mpk/models/deepseek_v3/builder.py:166-174).
  int ue8m0_strides(const TensorInfo &s, int64_t outer, int64_t pk, bool activation, int *s_outer, int *s_pk) {
    if (s.dims.size() != 2 || (s.dtype != MPK_U32 && s.dtype != MPK_I32))
      return fail(MPK_ERR_INVALID, "packed UE8M0 scales must be a 2-D uint32 tensor: " + s.name);
    const bool logical = s.dim(0) >= outer && s.dim(1) == pk;
    const bool physical = s.dim(0) == pk && s.dim(1) >= outer;
    if (!logical && !physical)
      return fail(MPK_ERR_INVALID, "scale tensor " + s.name + " matches neither [outer, K/512] nor [K/512, outer]");
    // a square tensor fits both readings: activation scales are then taken in the physical form the
    // reference's quantiser writes, weight scales in the logical form its checkpoints converters attach
    if (physical && (!logical || activation)) {
      *s_outer = (int)s.strides[1]; *s_pk = (int)s.strides[0];
    } else {
      *s_outer = (int)s.strides[0]; *s_pk = (int)s.strides[1];
    }
    return MPK_OK;
  }

  // FP8 linear: e4m3 weights [N, K] and activations [tokens, K], UE8M0 scales per 128 columns of each row
  // (python/mirage/mpk/persistent_kernel.py:1584-1632).  Same streaming geometry as the bf16 linear with one
  // byte per element; a task covers at most kFp8TaskRows weight rows so that their scales fit in the tile.
  int emit_linear_fp8(int li, int ex) {
    const LayerInfo &l = L[li];
    const bool has_res = l.op == MPK_OP_LINEAR_FP8_RESIDUAL;
    const TensorInfo &x = T[l.t[0]], &xs = T[l.t[1]], &w = T[l.t[2]], &ws = T[l.t[3]];
    const TensorInfo &y = T[l.t[has_res ? 5 : 4]];
    if (w.dims.size() != 2 || w.dtype != MPK_F8E4M3 || x.dtype != MPK_F8E4M3 || w.strides[1] != 1)
      return fail(MPK_ERR_UNSUPPORTED, "linear_fp8 needs row-major 2-D e4m3 weight and activations: " + w.name);
    const int N = (int)w.dim(0), K = (int)w.dim(1), ldw = (int)w.strides[0];
    if (K % 128 != 0 || ldw % 16 != 0) return fail(MPK_ERR_UNSUPPORTED, "linear_fp8 K must be a multiple of 128: " + w.name);
    if (x.dim(x.dims.size() - 1) != K || x.ld() % 16 != 0) return fail(MPK_ERR_INVALID, "linear_fp8 input width != K for " + w.name);
    if (y.dim(y.dims.size() - 1) != N || y.dtype != MPK_BF16) return fail(MPK_ERR_INVALID, "linear_fp8 output must be bf16 [tokens, N]: " + w.name);
    if (cfg.max_num_batched_tokens > kMaxLinearTokens)
      return fail(MPK_ERR_UNSUPPORTED, "linear layers support at most 64 batched tokens in this build");
    const int64_t pk = (K / 128 + 3) / 4;
    int ws0, ws1, xs0, xs1;
    int rc = ue8m0_strides(ws, N, pk, false, &ws0, &ws1);
    if (rc) return rc;
    rc = ue8m0_strides(xs, cfg.max_num_batched_tokens, pk, true, &xs0, &xs1);
    if (rc) return rc;
    const int ntok = std::min(std::max(cfg.max_num_batched_tokens, 1), (int)kMaxLinearTokens);
    const bool tc = g->use_tmem && tc_linear_fp8(K);
    int nkt = 1;
    if (tc) {
      while (nkt <= K / 512 && !(K % nkt == 0 && (K / nkt) % 512 == 0 && fp8_tc_tile_bytes(K / nkt) <= g->x_tile_bytes + kPartialBytes)) ++nkt;
      if (nkt > K / 512) return fail(MPK_ERR_UNSUPPORTED, "cannot tile K for " + w.name);
    } else {
      while (nkt <= K / 128 && !(K % nkt == 0 && (K / nkt) % 128 == 0 && fp8_tile_bytes(ntok, K / nkt) <= g->x_tile_bytes)) ++nkt;
      if (nkt > K / 128) return fail(MPK_ERR_UNSUPPORTED, "cannot tile K for " + w.name);
    }
    const int KT = K / nkt;
    const int R = kChunkRows;
    int KC = std::min(KT, g->chunk_cols * 2) / 128 * 128;   // a stage holds twice as many one-byte columns
    while (KC > 128 && KT % KC != 0) KC -= 128;
    int cap = nkt > 1 ? 2 * R : kFp8TaskRows;
    bool w_dynamic = false;
    for (const auto &o : L) if (!o.folded && raw_writes(o, w.storage)) w_dynamic = true;
    const bool enable_res = has_res && (l.params.empty() || l.params[0] != 0);
    const int base = N / W, rem = N % W;
    // tcgen05 path: row tiles and k blocks per ring slot chosen as for the bf16 linears (a k block is 128 one-byte
    // columns); a task holds at most kTcFp8MaxTiles tiles
    int tc_rb = 0, tc_nkb = 1;
    if (tc) {
      const int cnt_max = base + (rem ? 1 : 0);
      const int kbt = KT / 128;
      const int t_min = (cnt_max + 127) / 128;
      double best = -1.0;
      for (int tiles = t_min; tiles <= t_min + 6; ++tiles) {
        const int rb = ((cnt_max + tiles - 1) / tiles + 7) / 8 * 8;
        if (rb > 128 || rb <= 0) continue;
        if (tiles > t_min && cnt_max / tiles < 40) break;
        int nkb = std::min(kbt, g->stage_bytes / (rb * 128));
        while (nkb > 1 && kbt % nkb != 0) --nkb;
        if (nkb < 1) continue;
        const double fill = (double)cnt_max / tiles * 128.0 * nkb / g->stage_bytes;
        if (fill > best * 1.05) { best = fill; tc_rb = rb; tc_nkb = nkb; }
      }
      if (tc_rb == 0) return fail(MPK_ERR_UNSUPPORTED, "cannot tile the rows of " + w.name);
      cap = std::min<int>(kTcFp8MaxTiles, std::max(1, kTcAccCols / tc_np())) * tc_rb;
      KC = tc_nkb * 128;
      g->exec[ex].tc_rows = tc_rb;
      g->exec[ex].tc_kblocks = tc_nkb;
    }
    int row = 0;
    for (int i = 0; i < W; ++i) {
      const int worker = (i + rot) % W;
      const int cnt = base + (i < rem ? 1 : 0);
      bool first = true;
      for (int r = row; r < row + cnt; r += cap) {
        TaskDesc d = blank(TASK_LINEAR, li);
        d.flags |= TF_FP8;
        if (!first && nkt == 1) d.flags |= TF_SAME_X_AS_PREV;
        if (w_dynamic) d.flags |= TF_STREAM_AFTER_DEP;
        d.p[0] = (uint64_t)w.ptr;
        d.p[1] = (uint64_t)x.ptr;
        d.p[2] = (uint64_t)y.ptr;
        d.p[3] = enable_res ? (uint64_t)T[l.t[4]].ptr : 0;
        d.p[6] = (uint64_t)ws.ptr;
        d.p[7] = (uint64_t)xs.ptr;
        d.a[L_N0] = r;
        d.a[L_N1] = std::min(r + cap, row + cnt);
        d.a[L_K] = K;
        d.a[L_LDW] = ldw;
        d.a[L_LDX] = (int)x.ld();
        d.a[L_LDO] = (int)y.ld();
        d.a[L_LDR] = enable_res ? (int)T[l.t[4]].ld() : 0;
        d.a[L_PRO] = PRO_PLAIN;
        d.a[L_EPI] = enable_res ? EPI_RESIDUAL : EPI_STORE;
        d.a[L_KT] = KT;
        d.a[L_KC] = KC;
        d.a[L_ROWS] = R;
        d.a[L_N] = N;
        d.a[L_WS_S0] = ws0; d.a[L_WS_S1] = ws1; d.a[L_XS_S0] = xs0; d.a[L_XS_S1] = xs1;
        if (tc) {
          d.flags |= TF_TC;
          d.a[L_ROWS] = tc_rb;
          d.a[L_TMAP] = (int)g->tmaps.size();
          TmapSpec m;
          m.base = (uint64_t)w.ptr + (uint64_t)r * (uint64_t)ldw;
          m.rows = d.a[L_N1] - d.a[L_N0];
          m.ld_bytes = ldw;
          m.kblocks = K / 128;
          m.box_rows = tc_rb;
          m.box_kblocks = tc_nkb;
          m.elt_bytes = 1;
          g->tmaps.push_back(m);
        }
        put(worker, d, ex);
        g->weight_bytes += (int64_t)(d.a[L_N1] - d.a[L_N0]) * K;
        first = false;
      }
      row += cnt;
    }
    return MPK_OK;
  }

  // Per-token, per-128-column quantisation to e4m3 (python/mirage/mpk/persistent_kernel.py:1561-1582):
  // a task takes a range of tokens and a range of 512-column packs.
  int emit_quantize_fp8(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]], &q = T[l.t[1]], &s = T[l.t[2]];
    const bool ue8m0 = l.params.empty() || l.params[0] != 0;
    if (x.dtype != MPK_BF16 || q.dtype != MPK_F8E4M3) return fail(MPK_ERR_INVALID, "quantize_fp8: bf16 in, e4m3 out");
    const int nd = (int)x.dims.size();
    const int64_t K = x.dim(nd - 1);
    int64_t rows = 1;
    for (int i = 0; i < nd - 1; ++i) rows *= x.dim(i);
    if (K % 128 != 0) return fail(MPK_ERR_UNSUPPORTED, "quantize_fp8 width must be a multiple of 128");
    if (x.strides[nd - 1] != 1 || q.strides[nd - 1] != 1 || (nd > 2 && (x.strides[nd - 2] != K || q.strides[nd - 2] != K)))
      return fail(MPK_ERR_UNSUPPORTED, "quantize_fp8 tensors must be dense in their leading dimensions");
    const int64_t ng = K / 128, pk = (ng + 3) / 4;
    int s0, s1;
    if (ue8m0) {
      if (nd != 2) return fail(MPK_ERR_UNSUPPORTED, "quantize_fp8 with packed scales takes 2-D tensors");
      const int rc = ue8m0_strides(s, rows, pk, true, &s0, &s1);
      if (rc) return rc;
    } else {
      if (s.dtype != MPK_F32 || (int64_t)(s.bytes / 4) < rows * ng) return fail(MPK_ERR_INVALID, "quantize_fp8 float32 scales must be [rows, K/128]");
      s0 = (int)ng; s1 = 1;
    }
    // tokens: with a 2-D input only the active tokens are quantised; higher-rank inputs (token x expert) are
    // treated as rows of the flattened tensor
    const int per_tok = (int)(rows / std::max<int64_t>(x.dim(0), 1));
    const int nt = (int)std::max<int64_t>(1, std::min<int64_t>(W, rows * pk));
    const int64_t units = rows * pk;
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_QUANTIZE_FP8, li);
      d.p[0] = (uint64_t)x.ptr; d.p[1] = (uint64_t)q.ptr; d.p[2] = (uint64_t)s.ptr;
      d.a[0] = (int)(units * i / nt); d.a[1] = (int)(units * (i + 1) / nt);   // (row, pack) units
      d.a[2] = (int)K; d.a[3] = (int)(nd == 2 ? x.strides[0] : K); d.a[4] = (int)(nd == 2 ? q.strides[0] : K);
      d.a[5] = ue8m0 ? 1 : 0; d.a[6] = per_tok; d.a[7] = s0; d.a[8] = s1; d.a[9] = (int)pk;
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  // Expert projections (python/mirage/mpk/persistent_kernel.py:1444-1559, 1652-1681): every worker owns a row
  // range of EVERY expert and walks the list of active experts at run time, so the work is balanced whatever the
  // routing; a worker with more rows than a task may hold gets several tasks.
  int emit_moe_gemm(int li, int ex) {
    const LayerInfo &l = L[li];
    const bool fp8 = l.op == MPK_OP_MOE_W13_FP8 || l.op == MPK_OP_MOE_W2_FP8;
    const bool w2 = l.op == MPK_OP_MOE_W2_LINEAR || l.op == MPK_OP_MOE_W2_FP8;
    const TensorInfo &x = T[l.t[0]], &w = T[l.t[fp8 ? 2 : 1]], &idx = T[l.t[fp8 ? 4 : 2]], &mask = T[l.t[fp8 ? 5 : 3]];
    const TensorInfo &y = T[l.t[fp8 ? 6 : 4]];
    if (w.dims.size() != 3 || y.dims.size() != 3 || (int)x.dims.size() != (w2 ? 3 : 2))
      return fail(MPK_ERR_INVALID, "expert projection: weight [E, N, K], output [B, topk, N]: " + w.name);
    // E counts the experts of the routing tensors; the weight tensor may hold a contiguous range of them starting at
    // params[0] (expert parallelism): experts outside never reach the active list, so addressing a virtual expert 0
    // params[0] panels below the tensor is enough
    const int E = (int)idx.dim(0), EW = (int)w.dim(0), ebase = l.params.empty() ? 0 : (int)l.params[0];
    const int N = (int)w.dim(1), K = (int)w.dim(2), topk = (int)y.dim(1);
    if (ebase < 0 || ebase + EW > E) return fail(MPK_ERR_INVALID, "expert projection: weight experts outside the routing range: " + w.name);
    const int want = fp8 ? MPK_F8E4M3 : MPK_BF16;
    if (g->hybrid == HYB_F32) return emit_moe_gemm_f32(li, ex);
    int epi = EPI_STORE, cols = N;
    if (g->hybrid && !w2 && l.params.size() > 1 && l.params[1]) {
      epi = activation_epilogue(l.params[1]);
      const bool gated = epi == EPI_GATED_SILU || epi == EPI_GATED_GELU;
      if ((!gated && epi != EPI_RELU2) || (gated && N % 4)) return fail(MPK_ERR_INVALID, "expert projection: gated activations or squared relu: " + w.name);
      if (gated) cols = N / 2;
    } else if (g->hybrid && y.dtype == MPK_F32) {
      epi = EPI_STORE_F32;
    }
    const int unit = cols < N ? 4 : 1;
    if (g->hybrid && fp8) return fail(MPK_ERR_UNSUPPORTED, "expert projection: bf16 in hybrid graphs: " + w.name);
    if (w.dtype != want || x.dtype != want || y.dtype != (epi == EPI_STORE_F32 ? MPK_F32 : MPK_BF16) || w.strides[2] != 1 || w.strides[1] != K ||
        w.strides[0] != (int64_t)N * K)
      return fail(MPK_ERR_UNSUPPORTED, "expert projection: dense " + std::string(fp8 ? "e4m3" : "bf16") + " weights, bf16 output: " + w.name);
    if (x.dim(x.dims.size() - 1) != K || (g->hybrid ? y.dim(2) < cols : y.dim(2) != N) || mask.dim(0) != E + 1 || idx.dtype != MPK_I32 ||
        mask.dtype != MPK_I32 || (w2 && x.dim(1) != topk) || topk > 255 || idx.dim(1) > 255)
      return fail(MPK_ERR_INVALID, "expert projection: shapes of " + w.name + " and its routing tensors disagree");
    const int kstep = g->hybrid ? 64 : 128;
    if (K % kstep != 0 || (int64_t)N * K >= (1ll << 31))
      return fail(MPK_ERR_UNSUPPORTED, "expert projection: K must be a multiple of 128 (hybrid graphs: 64): " + w.name);
    if ((((uint64_t)x.ptr | (uint64_t)w.ptr) & 15u) != 0)     // rows are gathered / streamed with 16-byte copies
      return fail(MPK_ERR_UNSUPPORTED, "expert projection: input and weight must start on a 16-byte boundary: " + w.name);
    if (cfg.max_num_batched_tokens > kMaxLinearTokens)
      return fail(MPK_ERR_UNSUPPORTED, "linear layers support at most 64 batched tokens in this build");
    if (fp8) {
      const TensorInfo &xs = T[l.t[1]], &ws = T[l.t[3]];
      if (xs.dtype != MPK_F32 || ws.dtype != MPK_F32 || (int64_t)(ws.bytes / 4) < (int64_t)EW * N * (K / 128) ||
          xs.dim(xs.dims.size() - 1) != K / 128)
        return fail(MPK_ERR_INVALID, "expert projection: float32 scales [.., K/128] expected: " + w.name);
      // the task copies scales four at a time (16-byte asynchronous copies) when a row holds a multiple of four
      if ((K / 128) % 4 == 0 && (((uint64_t)xs.ptr | (uint64_t)ws.ptr) & 15u) != 0)
        return fail(MPK_ERR_UNSUPPORTED, "expert projection: scale tensors must start on a 16-byte boundary: " + w.name);
    }
    if (g->hybrid && g->use_tmem && tc_linear(K)) {
      // tensor path: row tiles of the active experts, dealt out to one task per worker.  Tall tiles share one gather of the token
      // rows; short ones spread better when few experts are active.
      const int rb = N % 128 == 0 && (int64_t)std::min<int64_t>(E, (int64_t)cfg.max_num_batched_tokens * topk) * (N / 128) >= 4 * W ? 128 : N > 32 ? 64 : 32;
      int nkb = std::max(1, std::min(K / kTcKBlock, g->stage_bytes / (rb * 128)));
      while (K / kTcKBlock % nkb) --nkb;
      if (E * (int64_t)N >= (1ll << 31)) return fail(MPK_ERR_UNSUPPORTED, "expert projection: more rows than a tensor map holds: " + w.name);
      TmapSpec m;
      m.base = (uint64_t)w.ptr; m.rows = (int64_t)EW * N; m.ld_bytes = (int64_t)K * 2; m.kblocks = K / kTcKBlock; m.box_rows = rb; m.box_kblocks = nkb;
      if (ebase) return fail(MPK_ERR_UNSUPPORTED, "expert projection: hybrid graphs hold all experts: " + w.name);
      const int map = (int)g->tmaps.size();
      g->tmaps.push_back(m);
      g->exec[ex].tc_rows = rb;
      g->exec[ex].tc_kblocks = nkb;
      for (int i = 0; i < W; ++i) {
        TaskDesc d = blank(TASK_MOE_GEMM, li);
        d.flags |= TF_STREAM_AFTER_DEP | TF_TC;
        d.p[0] = (uint64_t)w.ptr; d.p[1] = (uint64_t)x.ptr; d.p[2] = (uint64_t)y.ptr; d.p[4] = (uint64_t)idx.ptr; d.p[5] = (uint64_t)mask.ptr;
        d.a[L_N0] = i; d.a[L_N1] = W; d.a[L_K] = K; d.a[L_LDX] = (int)x.ld(); d.a[L_LDO] = (int)y.ld(); d.a[L_EPI] = epi; d.a[L_KT] = K;
        d.a[L_KC] = nkb * kTcKBlock; d.a[L_ROWS] = rb; d.a[L_N] = N; d.a[L_TMAP] = map;
        d.a[M_NEXP] = E; d.a[M_NTOPK] = topk; d.a[M_PER_SLOT] = w2 ? 1 : 0; d.a[M_LDR] = (int)idx.dim(1);
        put((i + rot) % W, d, ex);
      }
      return MPK_OK;
    }
    const int ntok = std::min(std::max(cfg.max_num_batched_tokens, 1), (int)kMaxLinearTokens);
    auto tile_bytes = [&](int KT) { return fp8 ? moe_fp8_tile_bytes(ntok, KT) : (int64_t)ntok * (KT * 2 + kRowPadBytes); };
    int nkt = 1;
    while (nkt <= K / kstep && !(K % nkt == 0 && (K / nkt) % kstep == 0 && tile_bytes(K / nkt) <= g->x_tile_bytes)) ++nkt;
    if (nkt > K / kstep) return fail(MPK_ERR_UNSUPPORTED, "cannot tile K for " + w.name);
    const int KT = K / nkt;
    const int R = kChunkRows;
    const int step = fp8 ? 128 : 64;
    int KC = std::min(KT, g->chunk_cols * (fp8 ? 2 : 1)) / step * step;
    while (KC > step && KT % KC != 0) KC -= step;
    const int cap = nkt > 1 ? 2 * R : kFp8TaskRows;
    const int base = N / unit / W, rem = N / unit % W;
    int row = 0;
    for (int i = 0; i < W; ++i) {
      const int worker = (i + rot) % W;
      const int cnt = (base + (i < rem ? 1 : 0)) * unit;
      for (int r = row; r < row + cnt; r += cap) {
        TaskDesc d = blank(TASK_MOE_GEMM, li);
        d.flags |= TF_STREAM_AFTER_DEP | (fp8 ? TF_FP8 : 0u);
        d.p[0] = (uint64_t)w.ptr - (uint64_t)ebase * (uint64_t)N * K * (fp8 ? 1 : 2);
        d.p[1] = (uint64_t)x.ptr; d.p[2] = (uint64_t)y.ptr;
        d.p[4] = (uint64_t)idx.ptr; d.p[5] = (uint64_t)mask.ptr;
        if (fp8) {
          d.p[6] = (uint64_t)T[l.t[3]].ptr - (uint64_t)ebase * (uint64_t)N * (K / 128) * 4;
          d.p[7] = (uint64_t)T[l.t[1]].ptr;
        }
        d.a[L_N0] = r; d.a[L_N1] = std::min(r + cap, row + cnt); d.a[L_K] = K; d.a[L_LDW] = K;
        d.a[L_LDX] = (int)x.ld(); d.a[L_LDO] = (int)y.ld(); d.a[L_EPI] = epi; d.a[L_KT] = KT; d.a[L_KC] = KC; d.a[L_ROWS] = R; d.a[L_N] = N;
        d.a[M_NEXP] = E; d.a[M_NTOPK] = topk; d.a[M_PER_SLOT] = w2 ? 1 : 0; d.a[M_LDR] = (int)idx.dim(1);
        d.a[M_ESTRIDE] = N * K;
        put(worker, d, ex);
      }
      row += cnt;
    }
    return MPK_OK;
  }

  int emit_attention(int li, int ex, int attn_ordinal) {
    const LayerInfo &l = L[li];
    const bool paged = l.op == MPK_OP_PAGED_ATTENTION;
    if (l.params.size() < 4) return fail(MPK_ERR_INVALID, "attention needs [hq, hkv, qk_norm, rope] params");
    const int hq = (int)l.params[0], hkv = (int)l.params[1];
    const int qk_norm = (int)l.params[2], rope = (int)l.params[3];
    const TensorInfo &kc = T[l.t[1]];
    if (kc.dims.size() != 4 || kc.dim(3) != 128)
      return fail(MPK_ERR_UNSUPPORTED, "attention supports head_dim 128 caches [pages|batch, page|seq, kv_heads, 128]");
    if (hkv <= 0 || hq % hkv != 0) return fail(MPK_ERR_INVALID, "q heads must be a multiple of kv heads");
    const int G = hq / hkv;
    if (G != 1 && G != 2 && G != 4 && G != 8) return fail(MPK_ERR_UNSUPPORTED, "GQA group size must be 1, 2, 4 or 8");
    if (kc.dim(2) != hkv) return fail(MPK_ERR_INVALID, "kv cache head count != num_kv_heads");
    if (!cfg.qo_indptr && paged && !cfg.dry_run) return fail(MPK_ERR_INVALID, "paged attention needs the batch meta tensors");
    const int slots = paged ? cfg.max_num_batched_requests : std::max(l.grid[0], 1);
    const int page = paged ? (int)kc.dim(1) : (int)kc.dim(1);
    if (paged && page != cfg.page_size) return fail(MPK_ERR_INVALID, "kv cache page size != page_size");
    if (paged && general_graph() && page % 8 != 0)
      return fail(MPK_ERR_UNSUPPORTED, "with more than 8 batched tokens (or FP8 / expert layers) the page size must be a multiple of 8");
    const int max_seq = paged ? cfg.max_seq_length : (int)kc.dim(1);
    // chunks per (request, kv head): enough to give every worker a task, and with many requests enough that a
    // task stays near 128 rows at full length (the rows a task prefetches before its dependency wait are its
    // cheapest ones; long serial chunks are latency-bound)
    int NC = std::max(1, W / std::max(slots * hkv, 1));
    if (general_graph()) {
      // streamed K/V: long chunks are cheap (a task's fixed part is paid once), so a (request, kv head) pair is cut
      // only as far as it takes to occupy the workers, and into chunks of at most ~2048 positions so that requests
      // of very different lengths still spread evenly
      NC = std::max(NC, (max_seq + 2047) / 2048);
    } else {
      NC = std::max(NC, std::min((max_seq + 127) / 128, 16));
    }
    NC = std::min(NC, std::max(1, max_seq / 32));
    NC = std::min(NC, 32);
    const int rope_rows = rope ? (int)T[l.t[5]].dim(0) : 1;
    for (int s = 0; s < slots; ++s)
      for (int h = 0; h < hkv; ++h)
        for (int c = 0; c < NC; ++c) {
          TaskDesc d = blank(TASK_ATTENTION, li);
          for (int i = 0; i < 8; ++i) d.p[i] = l.t[i] >= 0 ? (uint64_t)T[l.t[i]].ptr : 0;
          d.a[A_SLOT] = s;
          d.a[A_HEAD] = h;
          d.a[A_CHUNK] = c;
          d.a[A_NCHUNK] = NC;
          d.a[A_HQ] = hq;
          d.a[A_HKV] = hkv;
          d.a[A_HD] = 128;
          d.a[A_PAGE] = page;
          d.a[A_FLAGS] = (qk_norm ? 1 : 0) | (rope ? 2 : 0) | (paged ? 0 : 4);
          d.a[A_LDQKV] = (int)T[l.t[0]].ld();
          d.a[A_LDO] = (int)T[l.t[7]].ld();
          d.a[A_EPS] = float_bits(1e-6f);
          d.a[A_ROPE_ROWS] = rope_rows;
          d.a[A_CSEQ] = (int)kc.dim(1);
          d.a[A_TICKET] = attn_ordinal;   // ticket bank
          d.a[A_EARLY_EV] = no_batch_task() ? -1 : 0;   // exec layer 0 is the batching task
          d.a[A_EARLY_NEED] = 1;
          put(((s * hkv + h) * NC + c + rot) % W, d, ex);
        }
    g->attn_scratch_floats =
        std::max<int64_t>(g->attn_scratch_floats, (int64_t)cfg.max_num_batched_tokens * hq * NC * 130);
    g->attn_tickets = std::max<int64_t>(g->attn_tickets, (int64_t)slots * hkv);
    return MPK_OK;
  }

  // ---- hybrid graphs: recurrent layers, extended attention, float32 residual stream --------------------------
  static bool hybrid_op(int op) { return op >= MPK_OP_RESIDUAL_NORM && op <= MPK_OP_POLY_NORM; }
  static bool expert_op(int op) { return op == MPK_OP_MOE_TOPK_SIGMOID || op == MPK_OP_MOE_TOPK_SOFTMAX || op == MPK_OP_MOE_W13_LINEAR || op == MPK_OP_MOE_W2_LINEAR; }
  static int activation_epilogue(int64_t act) {
    switch (act) {
      case MPK_ACT_RELU2: return EPI_RELU2;
      case MPK_ACT_SOFTCAP: return EPI_SOFTCAP;
      case MPK_ACT_SCALE: return EPI_SCALE_F32;
      case MPK_ACT_GATED_SILU: return EPI_GATED_SILU;
      case MPK_ACT_GATED_GELU_TANH: return EPI_GATED_GELU;
      default: return EPI_STORE;
    }
  }
  // Epilogues with a number of their own and a float32 output.
  static bool capped(int epi) { return epi == EPI_SOFTCAP || epi == EPI_SCALE_F32; }
  // A tensor's address (0: absent) into two of a descriptor's integers.
  void put_wide(TaskDesc *d, int i, int tensor) const {
    const uint64_t p = tensor >= 0 ? (uint64_t)T[tensor].ptr : 0;
    std::memcpy(&d->a[i], &p, 8);
  }
  static int round_up(int64_t v, int m) { return (int)((v + m - 1) / m * m); }
  static int bits_of(int64_t p) { return (int)(uint32_t)p; }

  int classify_hybrid() {
    bool any = false, f32 = false;
    for (const auto &l : L) any = any || hybrid_op(l.op);
    if (!any) return MPK_OK;
    if (cfg.world_size > 1) return fail(MPK_ERR_UNSUPPORTED, "hybrid graphs run on one rank");
    if (cfg.max_num_batched_tokens > kMaxLinearTokens)
      return fail(MPK_ERR_UNSUPPORTED, "hybrid graphs batch at most 64 tokens");
    for (size_t i = 0; i < L.size(); ++i) {
      const LayerInfo &l = L[i];
      const int act_out = l.op == MPK_OP_RESIDUAL_NORM || l.op == MPK_OP_EXT_ATTENTION || l.op == MPK_OP_RGLRU || l.op == MPK_OP_MLSTM ||
                                  l.op == MPK_OP_GLA || l.op == MPK_OP_SELECTIVE_SCAN || l.op == MPK_OP_DIFF_COMBINE || l.op == MPK_OP_POLY_NORM
                              ? (l.op == MPK_OP_RESIDUAL_NORM ? l.t[4] : l.op == MPK_OP_EXT_ATTENTION ? l.t[0] : l.t.back()) : -1;   // tensor of the graph's activation type
      if (act_out >= 0 && T[act_out].dtype == MPK_F32) f32 = true;
      if (hybrid_op(l.op) || l.op == MPK_OP_EMBED || l.op == MPK_OP_ARGMAX_PARTIAL || l.op == MPK_OP_ARGMAX_REDUCE ||
          l.op == MPK_OP_SAMPLING_PARTIAL || l.op == MPK_OP_SAMPLING_REDUCE || expert_op(l.op)) continue;
      if (l.op != MPK_OP_LINEAR) return fail(MPK_ERR_UNSUPPORTED, "layer " + std::to_string(i) + ": not available in a hybrid graph");
      if (T[l.t[0]].dtype == MPK_F32) f32 = true;
    }
    g->hybrid = f32 ? HYB_F32 : HYB_BF16;
    return MPK_OK;
  }
  int act_dtype() const { return g->hybrid == HYB_F32 ? MPK_F32 : MPK_BF16; }
  bool batch_meta_given() const {
    return cfg.dry_run || (cfg.qo_indptr && cfg.paged_kv_indptr && cfg.paged_kv_indices && cfg.paged_kv_last_page_len);
  }
  int linear_f32_tokens(int64_t K) const { return (int)std::max<int64_t>(1, std::min<int64_t>(nb_max, 98304 / (4 * std::max<int64_t>(K, 1)))); }
  int xattn_width(const LayerInfo &l) const {   // padded head size of the tensor-core body
    const int w = (int)std::max(T[l.t[1]].dim(3), T[l.t[2]].dim(3));
    return w <= 64 ? 64 : (w <= 128 ? 128 : 256);
  }
  // key / value tiles in flight: graphs of many tokens reserve a large activation tile anyway
  int xattn_stages() const { return nb_max > 8 ? 3 : 2; }
  // Tiles of attention over shared key / value rows: the largest that leave the weight ring its size (graphs of many tokens
  // reserve a large activation tile anyway; of few tokens what a ring of 32 KB stages leaves over).
  struct LatentPlan { int keys, stages; int64_t bytes; };
  LatentPlan latent_plan(const LayerInfo &l) const {
    const int64_t pitch = round_up(T[l.t[1]].dim(3), 64) * 2 + 16;
    const int64_t budget = nb_max > 8 ? kSmemBudget - kMiscBytes - 5 * kTcSlotBytes : kPartialBytes + 90 * 1024;
    LatentPlan p{0, 0, 0};
    for (int keys : {32, 16}) {
      const int64_t fixed = 32 + 16 * pitch + (int64_t)(8 / (keys / 16)) * 16 * (keys + 4) * 4 + 2 * 16 * (keys * 2 + 16) + 8 * 16 + kXaCells * 4;
      p.keys = keys;
      p.stages = (int)std::min<int64_t>(4, (budget - fixed) / (keys * pitch));
      if (p.stages < 3 && keys == 16) p.stages = 3;   // the smallest tiles: whatever they need
      p.bytes = fixed + p.stages * keys * pitch;
      if (p.stages >= 3) return p;
    }
    return p;
  }
  // shared memory of a token: gate sums and u, as float32 or as three bf16 parts
  static int64_t rglru_token_bytes(int bs, int C) { return 16 * C + 6 * (round_up(bs, 16) + 8); }
  void rglru_plan(const LayerInfo &l, int *C, int *TG) const {
    const int nb = (int)T[l.t[3]].dim(0), bs = (int)T[l.t[3]].dim(1);
    const int chunks = std::max(1, W / std::max(nb, 1));
    // 16 channels are one tile of the bf16 graphs' gate products
    *C = std::min(std::min(bs, 64), std::max(8, round_up((bs + chunks - 1) / chunks, g->hybrid == HYB_BF16 ? 16 : 2)));
    int tg = std::min(nb_max, (int)std::max<int64_t>(8, (int64_t)65536 / rglru_token_bytes(bs, *C)));
    *TG = std::max(1, tg > 8 ? tg / 8 * 8 : tg);
  }
  static int mlstm_tokens(int64_t dim) { return dim <= 512 ? 16 : 8; }
  int64_t hybrid_smem(const LayerInfo &l) const {
    const int64_t mbr = cfg.max_num_batched_requests;
    switch (l.op) {
      case MPK_OP_RESIDUAL_NORM: return norm_columns(l) * 4 + 16;
      case MPK_OP_EXT_ATTENTION: {
        if (g->hybrid == HYB_F32) return 8 * T[l.t[1]].dim(3) * 4;
        if (T[l.t[1]].storage == T[l.t[2]].storage) return latent_plan(l).bytes;
        const int D = xattn_width(l), pitch = D * 2 + 16, keys = D > 128 ? 32 : 64, wmax = D > 128 ? 4 : 8;
        const int G = (int)(l.params[0] / std::max<int64_t>(l.params[1], 1));
        const int64_t tile = (int64_t)std::min(wmax * 16, ext_attention_rows(cfg.max_num_batched_tokens * G)) * pitch +
                             xattn_stages() * 2 * keys * pitch + kXaCells * 4;
        // decoded tokens of graphs with room for it: sixteen query rows, two steps of 16 keys and values for each warp
        return std::max(tile, xattn_stages() >= 3 && D <= 128 ? (int64_t)(16 + 8 * 64) * pitch : 0);
      }
      case MPK_OP_SHORT_CONV: return kMaxLinearTokens * 16 + (mbr + 1) * 4;
      case MPK_OP_SELECTIVE_SCAN: {
        const int64_t np = round_up(l.params[1], 4), cp = kConsumerThreads / scan_lanes((int)l.params[1]);
        return kMaxLinearTokens * (16 + 8) + round_up(mbr + 1, 4) * 4 + 4 * nb_max * (2 * np + 2 * cp) +
               scan_staged_bytes(nb_max, (int)l.params[0], (int)cp);
      }
      case MPK_OP_GROUPED_LINEAR: {
        const int64_t K = T[l.t[1]].dim(2);
        if (g->hybrid == HYB_F32) return (int64_t)linear_f32_tokens(K) * K * 4;
        return std::min<int64_t>(linear_tile_bytes(K), x_tile_cap()) + kPartialBytes;   // (a linear task's partial sums stay behind the tile)
      }
      case MPK_OP_GLA: {
        const int64_t dim = l.params[1], rank = T[l.t[1]].dim(1), vc = MPK_MLSTM_COLUMNS(dim), TC = mlstm_tokens(dim), rows = mlstm_rows((int)dim);
        const int64_t portion = 4 * (TC * (3 * rows + vc) + TC * 8 * vc + TC * rank);
        const int64_t single = (int64_t)mlstm_rows_per_thread((int)dim) * kConsumerThreads * 32 + 4 * (3 * rows + 16 * vc + rank);
        return std::max(portion, single);
      }
      case MPK_OP_RGLRU: {
        int C, TG;
        rglru_plan(l, &C, &TG);
        const int bs = (int)T[l.t[3]].dim(1);
        return kMaxLinearTokens * 16 + 1024 + (int64_t)TG * 16 * C + std::max<int64_t>((int64_t)round_up(TG, 8) * 6 * (round_up(bs, 16) + 8), (mbr + 1) * 4);
      }
      case MPK_OP_MLSTM: {
        const int64_t dim = l.params[1], vc = MPK_MLSTM_COLUMNS(dim), TC = mlstm_tokens(dim), rows = mlstm_rows((int)dim);
        const int64_t portion = 4 * (3 * kMaxLinearTokens + TC * 8 + TC * (2 * rows + vc) + TC * 8 * vc);
        const int64_t single = (int64_t)mlstm_rows_per_thread((int)dim) * kConsumerThreads * 32 + 4 * (2 * rows + 16 * vc + 16);
        return std::max(portion, single);
      }
      default: return 0;
    }
  }

  int emit_linear_f32(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]], &w = T[l.t[1]], &y = T[l.t[2]];
    if (w.dims.size() != 2 || w.dtype != MPK_BF16 || w.strides[1] != 1 || x.dtype != MPK_F32 || y.dtype != MPK_F32)
      return fail(MPK_ERR_UNSUPPORTED, "32-bit linear: float32 input and output, row-major bf16 weight: " + w.name);
    const int N = (int)w.dim(0), K = (int)w.dim(1);
    const int act = l.params.empty() ? 0 : (int)l.params[0];
    const bool gated = act == MPK_ACT_GATED_SILU || act == MPK_ACT_GATED_GELU_TANH;
    const int cols = gated ? N / 2 : N;
    if (x.dim(1) != K || y.dim(1) < cols || (gated && N % 4) || act < 0 || act > MPK_ACT_SCALE || ((act == MPK_ACT_SOFTCAP || act == MPK_ACT_SCALE) && l.params.size() < 2))
      return fail(MPK_ERR_INVALID, "32-bit linear: shapes or activation of " + w.name);
    const int bias = norm_tensor(l, 3);
    if (bias >= 0 && (act || T[bias].dtype != MPK_BF16 || T[bias].dim(0) < N)) return fail(MPK_ERR_INVALID, "linear bias: bf16 [rows], no activation: " + w.name);
    const int nt = std::min(W, cols);
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_LINEAR_F32, li);
      d.p[0] = (uint64_t)w.ptr; d.p[1] = (uint64_t)x.ptr; d.p[2] = (uint64_t)y.ptr; d.p[3] = bias >= 0 ? (uint64_t)T[bias].ptr : 0;
      d.a[0] = (int)((int64_t)cols * i / nt); d.a[1] = (int)((int64_t)cols * (i + 1) / nt);
      d.a[2] = K; d.a[3] = (int)w.ld(); d.a[4] = (int)x.ld(); d.a[5] = (int)y.ld();
      d.a[6] = act;
      d.a[7] = linear_f32_tokens(K);
      d.a[8] = l.params.size() > 1 ? bits_of(l.params[1]) : 0;
      put((i + rot) % W, d, ex);
    }
    g->weight_bytes += (int64_t)N * K * 2;
    return MPK_OK;
  }

  int emit_moe_gemm_f32(int li, int ex) {
    const LayerInfo &l = L[li];
    const bool w2 = l.op == MPK_OP_MOE_W2_LINEAR;
    const TensorInfo &x = T[l.t[0]], &w = T[l.t[1]], &idx = T[l.t[2]], &mask = T[l.t[3]], &y = T[l.t[4]];
    const int E = (int)idx.dim(0), N = (int)w.dim(1), K = (int)w.dim(2), slots = (int)y.dim(1);
    const int act = !w2 && l.params.size() > 1 ? (int)l.params[1] : 0;
    const bool gated = act == MPK_ACT_GATED_SILU || act == MPK_ACT_GATED_GELU_TANH;
    const int cols = gated ? N / 2 : N;
    if (w.dtype != MPK_BF16 || x.dtype != MPK_F32 || y.dtype != MPK_F32 || w.strides[2] != 1 || w.strides[1] != K || w.strides[0] != (int64_t)N * K)
      return fail(MPK_ERR_UNSUPPORTED, "32-bit expert projection: float32 input and output, dense bf16 weights: " + w.name);
    if (w.dim(0) != E || mask.dim(0) != E + 1 || idx.dtype != MPK_I32 || mask.dtype != MPK_I32 || x.dim(x.dims.size() - 1) < K || y.dim(2) < cols ||
        (w2 && x.dim(1) != slots) || (act && !gated && act != MPK_ACT_RELU2) || (gated && N % 4))
      return fail(MPK_ERR_INVALID, "32-bit expert projection: shapes of " + w.name + " and its routing tensors disagree");
    const int nt = std::min(W, cols);
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_MOE_GEMM_F32, li);
      d.p[0] = (uint64_t)w.ptr; d.p[1] = (uint64_t)x.ptr; d.p[2] = (uint64_t)y.ptr; d.p[4] = (uint64_t)idx.ptr; d.p[5] = (uint64_t)mask.ptr;
      d.a[0] = (int)((int64_t)cols * i / nt); d.a[1] = (int)((int64_t)cols * (i + 1) / nt); d.a[2] = K;
      d.a[4] = (int)x.ld(); d.a[5] = (int)y.ld(); d.a[6] = act; d.a[7] = linear_f32_tokens(K); d.a[8] = w2 ? 1 : 0; d.a[9] = slots;
      d.a[10] = (int)idx.dim(1); d.a[11] = E; d.a[12] = N;
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  // One linear per group of columns: the same tasks as a linear layer's, cut at the group borders.
  int emit_grouped_linear(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]], &w = T[l.t[1]], &y = T[l.t[2]];
    if (l.params.size() < 3 || w.dims.size() != 3) return fail(MPK_ERR_INVALID, "grouped linear: weight [groups, N, K], params [x stride, y column, y stride]");
    const int G = (int)w.dim(0), N = (int)w.dim(1), K = (int)w.dim(2);
    const int64_t xs = l.params[0], yc = l.params[1], ys = l.params[2];
    if (w.dtype != MPK_BF16 || w.strides[2] != 1 || w.strides[1] != K || w.strides[0] != (int64_t)N * K || x.dtype != act_dtype() ||
        (y.dtype != act_dtype() && y.dtype != MPK_F32))
      return fail(MPK_ERR_UNSUPPORTED, "grouped linear: dense bf16 weight, input and output of the graph's activation type: " + w.name);
    if (xs < K || yc < 0 || ys < N || (G - 1) * xs + K > x.dim(1) || yc + (G - 1) * ys + N > y.dim(1))
      return fail(MPK_ERR_INVALID, "grouped linear: columns outside the input or output: " + w.name);
    const int gate = norm_tensor(l, 3);
    const int64_t gc = l.params.size() > 3 ? l.params[3] : 0, gs = l.params.size() > 4 ? l.params[4] : N;
    if (gate >= 0 && (T[gate].dtype != MPK_F32 || y.dtype != act_dtype() || gc < 0 || gs < N || gc + (G - 1) * gs + N > T[gate].dim(1)))
      return fail(MPK_ERR_INVALID, "grouped linear: float32 gate columns inside their tensor, output of the graph's activation type: " + w.name);
    const bool f32 = g->hybrid == HYB_F32;
    if (!f32 && (K % 16 || xs % 8 || ((uint64_t)x.ptr & 15) || ((uint64_t)w.ptr & 15) || x.ld() % 8))
      return fail(MPK_ERR_UNSUPPORTED, "grouped linear: K a multiple of 16, input columns on 16-byte boundaries: " + w.name);
    const int64_t rows = (int64_t)G * N;
    const bool tc = !f32 && g->use_tmem && tc_linear(K);
    if (!f32 && linear_tile_bytes(K) > g->x_tile_bytes) return fail(MPK_ERR_UNSUPPORTED, "grouped linear: K too large: " + w.name);
    const int esz_x = f32 ? 4 : 2, esz_y = y.dtype == MPK_F32 ? 4 : 2;
    int KC = std::min(K, g->chunk_cols) / 16 * 16;
    while (!f32 && KC > 16 && K % KC != 0) KC -= 16;
    // tcgen05: row tiles of at most 128 rows; a task holds as many accumulators as fit
    const int64_t widest = std::min<int64_t>((rows + W - 1) / W, N);
    int rb = 0, nkb = 1;
    if (tc) {
      const int tiles = (int)((widest + 127) / 128);
      rb = (int)std::min<int64_t>(128, ((widest + tiles - 1) / tiles + 7) / 8 * 8);
      nkb = std::max(1, std::min(K / kTcKBlock, g->stage_bytes / (rb * 128)));
      while (K / kTcKBlock % nkb) --nkb;
      g->exec[ex].tc_rows = rb;
      g->exec[ex].tc_kblocks = nkb;
    }
    const int cap = tc ? std::max(1, kTcAccCols / tc_np()) * rb : 1 << 20;
    for (int i = 0; i < W; ++i) {
      const int64_t end = rows * (i + 1) / W;
      int last = -1;
      for (int64_t r = rows * i / W; r < end;) {
        const int grp = (int)(r / N), n0 = (int)(r - (int64_t)grp * N);
        const int n1 = (int)std::min<int64_t>(std::min<int64_t>(N, end - (int64_t)grp * N), n0 + cap);
        TaskDesc d = blank(f32 ? TASK_LINEAR_F32 : TASK_LINEAR, li);
        d.p[0] = (uint64_t)w.ptr + (uint64_t)grp * N * K * 2;
        d.p[1] = (uint64_t)x.ptr + (uint64_t)grp * xs * esz_x;
        d.p[2] = (uint64_t)y.ptr + (uint64_t)(yc + grp * ys) * esz_y;
        const uint64_t gp = gate >= 0 ? (uint64_t)T[gate].ptr + (uint64_t)(gc + grp * gs) * 4 : 0;
        if (f32) {
          d.p[4] = gp; d.a[9] = gate >= 0 ? (int)T[gate].ld() : 0;
          d.a[0] = n0; d.a[1] = n1; d.a[2] = K; d.a[3] = K; d.a[4] = (int)x.ld(); d.a[5] = (int)y.ld(); d.a[7] = linear_f32_tokens(K);
        } else {
          if (grp == last) d.flags |= TF_SAME_X_AS_PREV;
          d.a[L_N0] = n0; d.a[L_N1] = n1; d.a[L_K] = K; d.a[L_LDW] = K; d.a[L_LDX] = (int)x.ld(); d.a[L_LDO] = (int)y.ld();
          d.a[L_PRO] = PRO_PLAIN; d.a[L_EPI] = gate >= 0 ? EPI_GATE_SIGMOID : y.dtype == MPK_F32 ? EPI_STORE_F32 : EPI_STORE; d.a[L_GROUPS] = 1;
          d.p[3] = gp; d.a[L_LDR] = gate >= 0 ? (int)T[gate].ld() : 0;
          d.a[L_KT] = K; d.a[L_KC] = KC; d.a[L_ROWS] = kChunkRows; d.a[L_N] = N;
          if (tc) {
            d.flags |= TF_TC;
            d.a[L_KC] = nkb * kTcKBlock; d.a[L_ROWS] = rb; d.a[L_TMAP] = (int)g->tmaps.size();
            TmapSpec m;
            m.base = d.p[0] + (uint64_t)n0 * K * 2;
            m.rows = n1 - n0; m.ld_bytes = (int64_t)K * 2; m.kblocks = K / kTcKBlock; m.box_rows = rb; m.box_kblocks = nkb; m.elt_bytes = 2;
            g->tmaps.push_back(m);
          }
        }
        put((i + rot) % W, d, ex);
        last = grp;
        r += n1 - n0;
      }
    }
    g->weight_bytes += rows * K * 2;
    return MPK_OK;
  }

  int emit_latent_append(int li, int ex) {
    const LayerInfo &l = L[li];
    if (l.params.size() < 6) return fail(MPK_ERR_INVALID, "latent_append needs 6 parameters");
    const int H = (int)l.params[0], rank = (int)l.params[1], rdim = (int)l.params[2];
    for (int i : {2, 4, 5})   // (nothing to rotate: they stand for themselves)
      if (l.t[i] < 0 && rdim) return fail(MPK_ERR_INVALID, "latent_append: q and tables are absent, but there is a rotated part");
    const TensorInfo &pr = T[l.t[0]], &nw = T[l.t[1]], &kc = T[l.t[3]], &q = T[l.t[l.t[2] >= 0 ? 2 : 3]], &cs = T[l.t[l.t[4] >= 0 ? 4 : 0]], &sn = T[l.t[l.t[5] >= 0 ? 5 : 0]];
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "latent_append needs the batch meta tensors");
    if (pr.dtype != MPK_F32 || nw.dtype != MPK_BF16 || q.dtype != act_dtype() || kc.dtype != act_dtype() || cs.dtype != MPK_F32 || sn.dtype != MPK_F32)
      return fail(MPK_ERR_INVALID, "latent_append: float32 projections and tables, bf16 norm weight, q and cache of the graph's activation type");
    if (H < 1 || rank < 1 || rdim < 0 || rdim % 2 || nw.dim(0) < rank || kc.dims.size() != 4 || kc.dim(1) != cfg.page_size || kc.dim(2) != 1 ||
        kc.dim(3) < rank + rdim || kc.dim(3) % 8 || (rdim > 0 && q.dim(1) != H * kc.dim(3)))
      return fail(MPK_ERR_INVALID, "latent_append: cache [pages, page, 1, latent + rotated size rounded up to 8], q [tokens, heads x that]");
    if (l.params[3] < 0 || l.params[4] < 0 || l.params[3] + (int64_t)H * rdim > pr.dim(1) || l.params[4] + rank + rdim > pr.dim(1))
      return fail(MPK_ERR_INVALID, "latent_append: columns outside the projections");
    if (rdim > 0 && (cs.dims.size() != 2 || cs.dim(1) != rdim / 2 || sn.dim(1) != rdim / 2 || cs.dim(0) != sn.dim(0)))
      return fail(MPK_ERR_INVALID, "latent_append: cos / sin tables [positions, rotated dims / 2]");
    const int nt = std::max(1, std::min(W, (nb_max * (rdim > 0 ? H + 1 : 1) + 7) / 8));
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_LATENT_APPEND, li);
      d.p[0] = (uint64_t)pr.ptr; d.p[1] = (uint64_t)nw.ptr; d.p[2] = (uint64_t)q.ptr; d.p[3] = (uint64_t)kc.ptr;
      d.p[4] = (uint64_t)cs.ptr; d.p[5] = (uint64_t)sn.ptr;
      d.a[LA_T0] = i; d.a[LA_T1] = nt; d.a[LA_LDP] = (int)pr.ld(); d.a[LA_QOFF] = (int)l.params[3]; d.a[LA_KVOFF] = (int)l.params[4];
      d.a[LA_H] = H; d.a[LA_RANK] = rank; d.a[LA_ROT] = rdim; d.a[LA_DIMP] = (int)kc.dim(3); d.a[LA_EPS] = bits_of(l.params[5]);
      d.a[LA_PAGE] = cfg.page_size; d.a[LA_LDQ] = (int)q.ld(); d.a[LA_ROWS] = rdim > 0 ? (int)cs.dim(0) : 1;
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_gla(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &pr = T[l.t[0]], &a2 = T[l.t[1]], &S = T[l.t[4]], &raw = T[l.t[5]], &o = T[l.t[6]];
    if (l.params.size() < 12 || a2.dims.size() != 2) return fail(MPK_ERR_INVALID, "gla: a2 [heads x dim, rank], 12 parameters");
    const int H = (int)l.params[0], dim = (int)l.params[1], vdim = (int)l.params[2], chunks = (int)l.params[11], rank = (int)a2.dim(1);
    const int slots = cfg.max_num_batched_requests;
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "gla needs the batch meta tensors");
    if (H < 1 || dim < 1 || vdim < 1 || rank < 1) return fail(MPK_ERR_INVALID, "gla: head count or sizes");
    if (dim > 1024 || rank > 512) return fail(MPK_ERR_UNSUPPORTED, "gla: key sizes up to 1024, decay rank up to 512");
    if (pr.dtype != MPK_F32 || S.dtype != MPK_F32 || raw.dtype != MPK_F32 || o.dtype != act_dtype() || S.dims.size() != 4 || S.dim(0) < slots ||
        S.dim(1) != H || S.dim(2) != dim || S.dim(3) < vdim || S.dim(3) % 4 || raw.dim(1) < (int64_t)H * vdim || o.dim(1) < (int64_t)H * vdim)
      return fail(MPK_ERR_INVALID, "gla: state [slots, heads, dim, vdim rounded up to 4], scratch and output [tokens, heads x vdim]");
    for (int i = 3; i < 8; ++i) {
      const int64_t w = i < 5 ? (int64_t)H * dim : (i < 7 ? (int64_t)H * vdim : rank);
      if (l.params[i] < 0 || l.params[i] + w > pr.dim(1)) return fail(MPK_ERR_INVALID, "gla: columns outside the projections");
    }
    if (a2.dtype != MPK_BF16 || a2.dim(0) != (int64_t)H * dim || a2.strides[0] != rank || a2.strides[1] != 1 || T[l.t[2]].dtype != MPK_BF16 ||
        T[l.t[2]].dim(0) < (int64_t)H * dim || T[l.t[3]].dtype != MPK_BF16 || T[l.t[3]].dim(0) < vdim)
      return fail(MPK_ERR_INVALID, "gla: bf16 a2 [heads x dim, rank], bias [heads x dim], norm [vdim]");
    const int vc = MPK_MLSTM_COLUMNS(dim), nsub = (vdim + vc - 1) / vc;
    if (chunks < 1 || chunks > nsub) return fail(MPK_ERR_INVALID, "gla: chunk count");
    for (int s = 0; s < slots; ++s)
      for (int h = 0; h < H; ++h)
        for (int ch = 0; ch < chunks; ++ch) {
          TaskDesc d = blank(TASK_GLA, li);
          for (int k = 0; k < 5; ++k) d.p[k] = (uint64_t)T[l.t[k]].ptr;
          d.p[6] = (uint64_t)raw.ptr; d.p[7] = (uint64_t)o.ptr;
          d.a[GA_SLOT] = s; d.a[GA_HEAD] = h; d.a[GA_CHUNK] = ch; d.a[GA_NCHUNK] = chunks; d.a[GA_H] = H; d.a[GA_DIM] = dim;
          d.a[GA_VDIM] = vdim; d.a[GA_VDIMP] = (int)S.dim(3); d.a[GA_V0] = nsub * ch / chunks * vc;
          d.a[GA_V1] = std::min(nsub * (ch + 1) / chunks * vc, (int)S.dim(3));
          d.a[GA_EPS] = bits_of(l.params[9]); d.a[GA_LDP] = (int)pr.ld(); d.a[GA_QOFF] = (int)l.params[3]; d.a[GA_KOFF] = (int)l.params[4];
          d.a[GA_VOFF] = (int)l.params[5]; d.a[GA_GOFF] = (int)l.params[6]; d.a[GA_AOFF] = (int)l.params[7]; d.a[GA_RANK] = rank;
          d.a[GA_LDO] = (int)o.ld(); d.a[GA_QSCALE] = bits_of(l.params[10]); d.a[GA_TICKET] = hybrid_tickets + s * H + h;
          d.a[GA_TC] = mlstm_tokens(dim); d.a[GA_LDR] = (int)raw.ld(); d.a[GA_INVTAU] = bits_of(l.params[8]);
          put(((s * H + h) * chunks + ch + rot) % W, d, ex);
        }
    hybrid_tickets += slots * H;
    return MPK_OK;
  }

  int emit_residual_norm(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]];
    auto opt = [&](int i) { return l.t[i] >= 0 ? (uint64_t)T[l.t[i]].ptr : 0; };
    const int D = (int)norm_columns(l);
    if (l.params.size() < 2 || x.dtype != MPK_F32 || x.dims.size() != 2) return fail(MPK_ERR_INVALID, "residual_norm: x must be float32 [tokens, width]");
    if (l.t[1] >= 0 && (T[l.t[1]].dtype != MPK_F32 || T[l.t[1]].dim(1) != D)) return fail(MPK_ERR_INVALID, "residual_norm: y must be float32 of x's width");
    for (int i = 2; i < 4; ++i)
      if (l.t[i] >= 0 && (T[l.t[i]].dtype != MPK_BF16 || T[l.t[i]].dim(0) != D)) return fail(MPK_ERR_INVALID, "residual_norm: weights must be bf16 [width]");
    if (l.t[3] >= 0 && l.t[4] < 0) return fail(MPK_ERR_INVALID, "residual_norm: a norm weight needs an output");
    const int bias = norm_tensor(l, 6), add = norm_tensor(l, 7), row = norm_tensor(l, 8), exps = norm_tensor(l, 9), ew = norm_tensor(l, 10), gate = norm_tensor(l, 11);
    if ((bias >= 0 && (l.t[3] < 0 || T[bias].dtype != MPK_BF16 || T[bias].dim(0) != D)) || (row >= 0 && (T[row].dtype != MPK_BF16 || T[row].dim(0) != D)) ||
        (add >= 0 && (T[add].dtype != MPK_F32 || T[add].dims.size() != 2 || T[add].dim(1) != D)))
      return fail(MPK_ERR_INVALID, "residual_norm: bf16 bias and row [width], float32 added stream [tokens, width]");
    if ((exps >= 0) != (ew >= 0) || (exps >= 0 && (T[exps].dtype != MPK_F32 || T[exps].dims.size() != 3 || T[exps].dim(2) != D || T[exps].strides[1] != D ||
                                                   T[exps].strides[0] != T[exps].dim(1) * D || T[ew].dtype != MPK_F32 || T[ew].dim(1) != T[exps].dim(1))))
      return fail(MPK_ERR_INVALID, "residual_norm: expert outputs float32 [tokens, slots, width] with weights [tokens, slots]");
    if (gate >= 0 && (l.t[1] < 0 || T[gate].dtype != MPK_F32 || l.params.size() < 4 || l.params[3] < 0 || l.params[3] >= T[gate].dim(1)))
      return fail(MPK_ERR_INVALID, "residual_norm: gate column of a float32 tensor");
    if (l.t[2] >= 0 && (gate >= 0 || (norm_flags(l) & 4) || (l.t[1] < 0 && exps < 0)))
      return fail(MPK_ERR_UNSUPPORTED, "residual_norm: a norm of y (or of the experts' sum) goes with RMS norms and without a gate");
    if (l.t[4] >= 0 && (T[l.t[4]].dtype != act_dtype() || T[l.t[4]].dim(1) < D)) return fail(MPK_ERR_INVALID, "residual_norm: output type or width");
    const int results = norm_tensor(l, 12), rw = norm_tensor(l, 13), terms = rw >= 0 ? (int)T[rw].dim(0) : 0;
    if ((results >= 0) != (rw >= 0) || (results >= 0 && (T[results].dtype != MPK_F32 || T[results].dims.size() != 3 || T[results].dim(2) != D || T[results].strides[1] != D ||
                                                         T[results].dim(1) < cfg.max_num_batched_tokens || T[rw].dtype != MPK_BF16 || terms < 2 || terms > T[results].dim(0) || l.t[1] < 0)))
      return fail(MPK_ERR_INVALID, "residual_norm: results float32 [results, tokens, width], at least two of them with bf16 weights, and a y");
    if (D > x.dim(1) || (D < x.dim(1) && resnorm_moves(l))) return fail(MPK_ERR_INVALID, "residual_norm: leading columns of x, with nothing added");
    const TensorInfo &xo = T[resnorm_out(l)];
    if (resnorm_moves(l) && (xo.dtype != MPK_F32 || xo.dim(1) != D)) return fail(MPK_ERR_INVALID, "residual_norm: the new stream must be float32 of x's width");
    const int rows = (int)std::min<int64_t>(x.dim(0), cfg.max_num_batched_tokens), nt = std::min(rows, W);
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_RESIDUAL_NORM, li);
      d.p[5] = (uint64_t)xo.ptr; d.a[8] = (int)xo.ld();
      d.p[0] = (uint64_t)x.ptr; d.p[1] = opt(1); d.p[2] = opt(2); d.p[3] = opt(3); d.p[4] = opt(4);
      d.a[0] = (int)((int64_t)rows * i / nt); d.a[1] = (int)((int64_t)rows * (i + 1) / nt); d.a[2] = D;
      d.a[3] = (int)x.ld(); d.a[4] = l.t[1] >= 0 ? (int)T[l.t[1]].ld() : 0; d.a[5] = l.t[4] >= 0 ? (int)T[l.t[4]].ld() : 0;
      d.a[6] = bits_of(l.params[0]);
      d.a[7] = (g->hybrid == HYB_F32 ? 1 : 0) | norm_flags(l);
      put_wide(&d, RN_BIAS, bias); put_wide(&d, RN_ADD, add); put_wide(&d, RN_ROW, row); put_wide(&d, RN_EXP, exps); put_wide(&d, RN_EW, ew);
      if (gate >= 0) {
        const uint64_t gp = (uint64_t)T[gate].ptr + 4ull * l.params[3];
        std::memcpy(&d.a[RN_GATE], &gp, 8);
        d.a[RN_LDGATE] = (int)T[gate].ld();
      }
      d.a[RN_LDADD] = add >= 0 ? (int)T[add].ld() : 0;
      d.a[RN_SLOTS] = exps >= 0 ? (int)T[exps].dim(1) : 0;
      d.a[RN_LDEW] = ew >= 0 ? (int)T[ew].ld() : 0;
      d.a[RN_POST] = norm_factor(l);
      if (results >= 0) {
        d.p[6] = (uint64_t)T[results].ptr; d.p[7] = (uint64_t)T[rw].ptr; d.a[RN_TERMS] = terms; d.a[RN_HSTRIDE] = (int)T[results].strides[0];
      }
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_qkv_append(int li, int ex) {
    const LayerInfo &l = L[li];
    const bool caches = l.t[2] >= 0;   // else queries only
    if (caches != (l.t[3] >= 0)) return fail(MPK_ERR_INVALID, "qkv_append: both caches or none");
    const TensorInfo &pr = T[l.t[0]], &q = T[l.t[1]], &kc = T[l.t[caches ? 2 : 1]], &vc = T[l.t[caches ? 3 : 1]];
    if (l.params.size() < 10) return fail(MPK_ERR_INVALID, "qkv_append needs 10 parameters");
    const int hq = (int)l.params[0], hkv = (int)l.params[1], dim = (int)l.params[2], vdim = (int)l.params[3], rdim = (int)l.params[7];
    const int pairs = l.params.size() > 10 ? (int)l.params[10] : 0, maps = l.params.size() > 11 ? (int)l.params[11] : 1;
    if ((l.t[4] < 0 || l.t[5] < 0) && rdim) return fail(MPK_ERR_INVALID, "qkv_append: no tables, but rotated dimensions");
    const TensorInfo &cs = T[l.t[l.t[4] >= 0 ? 4 : 0]], &sn = T[l.t[l.t[5] >= 0 ? 5 : 0]];   // (nothing to rotate: absent)
    const bool whole = l.params.size() > 12 && l.params[12];
    const int temp = l.params.size() > 13 ? bits_of(l.params[13]) : 0, every = l.params.size() > 14 ? (int)l.params[14] : 0;
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "qkv_append needs the batch meta tensors");
    if ((whole && (rdim || maps != 1 || l.params[8] || norm_tensor(l, 6) < 0 || (caches && norm_tensor(l, 7) < 0))) || (!whole && every) || every < 0)
      return fail(MPK_ERR_UNSUPPORTED, "qkv_append: norms over all heads go with q and k weights and without rotation, the query temperature with such norms");
    if (pr.dtype != MPK_F32 || q.dtype != act_dtype() || (caches && (kc.dtype != act_dtype() || vc.dtype != act_dtype())) || cs.dtype != MPK_F32 || sn.dtype != MPK_F32)
      return fail(MPK_ERR_INVALID, "qkv_append: float32 projections and tables, q and caches of the graph's activation type");
    if (hq < 1 || hkv < 1 || hq % hkv || dim < 1 || vdim < 1 || rdim < 0 || rdim > dim || rdim % 2 || maps < 1 || maps > 2)
      return fail(MPK_ERR_INVALID, "qkv_append: head counts or sizes");
    const int dimp = caches && kc.dims.size() == 4 ? (int)kc.dim(3) : (int)q.dim(1) / (hq * maps);
    for (int i : {6, 7})
      if (norm_tensor(l, i) >= 0 && (T[l.t[i]].dtype != MPK_BF16 || T[l.t[i]].dim(0) < (whole ? (int64_t)dim * (i == 6 ? hq : hkv) : dim) || l.params[8])) return fail(MPK_ERR_INVALID, "qkv_append: bf16 norm weights [dim], no unit norm beside them");
    if (!caches) {
      if (dimp < maps * dim || dimp % 8 || q.dim(1) != (int64_t)hq * maps * dimp || l.params[4] + (int64_t)hq * maps * dim > pr.dim(1)) return fail(MPK_ERR_INVALID, "qkv_append: q [tokens, heads x head size rounded up to 8], columns inside the projections");
    } else if (kc.dims.size() != 4 || vc.dims.size() != 4 || kc.dim(1) != cfg.page_size || vc.dim(1) != cfg.page_size || kc.dim(2) != hkv ||
        vc.dim(2) != hkv || kc.dim(3) < maps * dim || vc.dim(3) < vdim || kc.dim(3) % 8 || vc.dim(3) % 8 || q.dim(1) != hq * maps * kc.dim(3))
      return fail(MPK_ERR_INVALID, "qkv_append: caches [pages, page, kv_heads, head size rounded up to 8], q [tokens, heads x that]");
    else if (l.params[4] + (int64_t)hq * maps * dim > pr.dim(1) || l.params[5] + (int64_t)hkv * maps * dim > pr.dim(1) || l.params[6] + (int64_t)hkv * vdim > pr.dim(1))
      return fail(MPK_ERR_INVALID, "qkv_append: columns outside the projections");
    if (rdim > 0 && (cs.dims.size() != 2 || cs.dim(1) != rdim / 2 || sn.dim(1) != rdim / 2 || cs.dim(0) != sn.dim(0)))
      return fail(MPK_ERR_INVALID, "qkv_append: cos / sin tables [positions, rotated dims / 2]");
    const int nt = std::max(1, std::min(W, whole ? nb_max * (caches ? 2 : 1) : (nb_max * (hq + (caches ? hkv : 0)) * maps + 7) / 8));
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_QKV_APPEND, li);
      d.p[0] = (uint64_t)pr.ptr; d.p[1] = (uint64_t)q.ptr; d.p[2] = caches ? (uint64_t)kc.ptr : 0; d.p[3] = caches ? (uint64_t)vc.ptr : 0;
      d.p[4] = (uint64_t)cs.ptr; d.p[5] = (uint64_t)sn.ptr;
      for (int k : {6, 7}) d.p[k] = norm_tensor(l, k) >= 0 ? (uint64_t)T[l.t[k]].ptr : 0;
      d.a[QA_PAIRS] = pairs; d.a[QA_MAPS] = maps; d.a[QA_WHOLE] = whole ? 1 : 0; d.a[QA_TEMP] = temp; d.a[QA_EVERY] = every;
      d.a[QA_T0] = i; d.a[QA_T1] = nt; d.a[QA_LDP] = (int)pr.ld();
      d.a[QA_QOFF] = (int)l.params[4]; d.a[QA_KOFF] = (int)l.params[5]; d.a[QA_VOFF] = (int)l.params[6];
      d.a[QA_HQ] = hq; d.a[QA_HKV] = hkv; d.a[QA_DIM] = dim; d.a[QA_DIMP] = dimp; d.a[QA_VDIM] = vdim; d.a[QA_VDIMP] = caches ? (int)vc.dim(3) : 0;
      d.a[QA_ROT] = rdim; d.a[QA_NORM] = (int)l.params[8]; d.a[QA_EPS] = bits_of(l.params[9]); d.a[QA_PAGE] = cfg.page_size;
      d.a[QA_LDQ] = (int)q.ld(); d.a[QA_ROWS] = rdim > 0 ? (int)cs.dim(0) : 1;
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_ext_attention(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &q = T[l.t[0]], &kc = T[l.t[1]], &vc = T[l.t[2]], &o = T[l.t[3]];
    if (l.params.size() < 8) return fail(MPK_ERR_INVALID, "ext_attention needs 8 parameters");
    const int hq = (int)l.params[0], hkv = (int)l.params[1], vdim = (int)l.params[2], ocol = (int)l.params[3];
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "ext_attention needs the batch meta tensors");
    if (hq < 1 || hkv < 1 || hq % hkv || kc.dims.size() != 4 || vc.dims.size() != 4 || kc.dim(2) != hkv || vc.dim(2) != hkv ||
        kc.dim(1) != cfg.page_size || vc.dim(1) != cfg.page_size || kc.dim(3) % 8 || vc.dim(3) % 8 || vc.dim(3) < vdim ||
        q.dim(1) != hq * kc.dim(3) || ocol < 0 || ocol + (int64_t)hq * vdim > o.dim(1))
      return fail(MPK_ERR_INVALID, "ext_attention: shapes of q, caches and output disagree");
    if (q.dtype != act_dtype() || kc.dtype != act_dtype() || vc.dtype != act_dtype() || (o.dtype != act_dtype() && o.dtype != MPK_F32))
      return fail(MPK_ERR_INVALID, "ext_attention: q and caches of the graph's activation type, output of that or float32");
    const int64_t window = l.params.size() > 9 ? l.params[9] : 0, keep = l.params.size() > 10 ? l.params[10] : 0;
    if (window < 0 || keep < 0 || window > (1 << 30) || keep > (1 << 30)) return fail(MPK_ERR_INVALID, "ext_attention: window or kept positions");
    const bool shared = kc.storage == vc.storage, bf16 = g->hybrid == HYB_BF16;
    const int r1 = norm_tensor(l, 5), r2 = norm_tensor(l, 6);
    if ((r1 >= 0) != (r2 >= 0) || (r1 >= 0 && (T[r1].dtype != MPK_BF16 || T[r2].dtype != MPK_BF16 || T[r1].dim(0) < hq || T[r2].dim(0) < hq)))
      return fail(MPK_ERR_INVALID, "ext_attention: distance bias of two bf16 tensors [heads]");
    if (shared && (keep > 0 || r1 >= 0 || (bf16 && o.dtype == MPK_F32)))
      return fail(MPK_ERR_UNSUPPORTED, "ext_attention: no kept positions, distance bias or float32 output with shared keys and values");
    if (shared && bf16 && (hkv != 1 || vdim % 8 || (ocol | o.ld()) % 2)) return fail(MPK_ERR_UNSUPPORTED, "ext_attention: shared keys and values have one kv head and a value size of whole 16-byte pieces");
    if (bf16 && !shared ? std::max(kc.dim(3), vc.dim(3)) > 256 : kc.dim(3) > 1024 || vdim > 512)
      return fail(MPK_ERR_UNSUPPORTED, "ext_attention: head sizes up to 256 (32-bit graphs and shared keys and values: keys up to 1024, values up to 512)");
    const int sinks = l.t.size() > 4 ? l.t[4] : -1;
    if (sinks >= 0 && (T[sinks].dtype != MPK_BF16 || T[sinks].dim(0) < hq || !l.params[6])) return fail(MPK_ERR_INVALID, "ext_attention: bf16 sinks [heads], sink = 1");
    const bool merge = l.params.size() > 8 && l.params[8];
    const int slots = cfg.max_num_batched_requests, max_seq = std::max(cfg.max_seq_length, 1);
    // chunks of a (request, kv head): enough to occupy the workers, at most ~2048 keys each, at least 64
    int NC = std::max(std::max(1, W / std::max(slots * hkv, 1)), (max_seq + 2047) / 2048);
    NC = std::min(std::min(NC, std::max(1, max_seq / 64)), 32);
    LatentPlan lp{0, xattn_stages(), 0};
    if (shared && bf16) {   // row tiles of a prompt portion times key chunks of a decoded token
      lp = latent_plan(l);
      const int64_t tiles = ((int64_t)cfg.max_num_batched_tokens * hq + 15) / 16;
      NC = (int)std::min<int64_t>(std::max(1, W / slots), tiles * std::max(1, (max_seq + 63) / 64));
    }
    const int srec = round_up(vdim, 4) + kXaRecHead;
    for (int s = 0; s < slots; ++s)
      for (int h = 0; h < hkv; ++h)
        for (int ch = 0; ch < NC; ++ch) {
          TaskDesc d = blank(TASK_EXT_ATTENTION, li);
          for (int i = 0; i < 4; ++i) d.p[i] = (uint64_t)T[l.t[i]].ptr;
          d.p[4] = sinks >= 0 ? (uint64_t)T[sinks].ptr : 0;
          d.p[5] = r1 >= 0 ? (uint64_t)T[r1].ptr : 0; d.p[6] = r2 >= 0 ? (uint64_t)T[r2].ptr : 0;
          d.a[XA_WINDOW] = (int)window; d.a[XA_KEEP] = (int)keep; d.a[XA_OUTF32] = o.dtype == MPK_F32 ? 1 : 0;
          d.a[XA_SHARED] = shared && bf16 ? 1 : 0; d.a[XA_KEYS] = lp.keys; d.a[XA_MERGE] = merge ? 1 : 0;
          d.a[XA_SLOT] = s; d.a[XA_HEAD] = h; d.a[XA_CHUNK] = ch; d.a[XA_NCHUNK] = NC; d.a[XA_HQ] = hq; d.a[XA_HKV] = hkv;
          d.a[XA_DIMP] = (int)kc.dim(3); d.a[XA_VDIM] = vdim; d.a[XA_VDIMP] = (int)vc.dim(3); d.a[XA_PAGE] = cfg.page_size;
          d.a[XA_LDQ] = (int)q.ld(); d.a[XA_LDO] = (int)o.ld(); d.a[XA_OCOL] = ocol;
          d.a[XA_SCALE] = bits_of(l.params[4]); d.a[XA_CAP] = bits_of(l.params[5]); d.a[XA_SINK] = (int)l.params[6];
          d.a[XA_OSCALE] = bits_of(l.params[7]);
          d.a[XA_TICKET] = hybrid_tickets + (s * hkv + h) * NC;   // one per part of the query rows
          d.a[XA_SREC] = srec;
          d.a[XA_STAGES] = lp.stages;
          put(((s * hkv + h) * NC + ch + rot) % W, d, ex);
          xattn_task = d;
        }
    hybrid_tickets += slots * hkv * NC;
    // a (request, kv head) has at most one query tile's rows for each of its tasks in the scratch
    g->attn_scratch_floats = std::max<int64_t>(g->attn_scratch_floats, (int64_t)slots * hkv * NC * 16 * srec);
    return MPK_OK;
  }

  int emit_attn_merge(int li, int ex) {
    const LayerInfo &l = L[li];
    const int at = li - 1;
    if (at < 0 || L[at].op != MPK_OP_EXT_ATTENTION || L[at].t != l.t || L[at].params != l.params || l.params.size() < 9 || !l.params[8])
      return fail(MPK_ERR_INVALID, "attn_merge: follows an ext_attention layer of the same tensors and parameters");
    const int cols = (int)((l.params[2] + 127) / 128), nt = (int)std::max<int64_t>(1, std::min<int64_t>(W, ((int64_t)nb_max * l.params[0] * cols + 7) / 8));
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = xattn_task;
      d.type = TASK_ATTN_MERGE;
      d.layer = li;
      d.a[XA_SLOT] = i; d.a[XA_CHUNK] = nt;
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_short_conv(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]], &w = T[l.t[2]], &st = T[l.t[4]], &o = T[l.t[5]];
    if (l.params.size() < 2 || w.dims.size() != 2) return fail(MPK_ERR_INVALID, "short_conv: taps [channels, taps], params [in_col, activation]");
    const int C = (int)w.dim(0), taps = (int)w.dim(1);
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "short_conv needs the batch meta tensors");
    if (x.dtype != MPK_F32 || st.dtype != MPK_F32 || o.dtype != MPK_F32 || w.dtype != MPK_BF16 || l.params[0] + C > x.dim(1) || o.dim(1) != C ||
        (int64_t)(st.bytes / 4) < (taps > 1 ? (int64_t)cfg.max_num_batched_requests * (taps - 1) * C : 0))
      return fail(MPK_ERR_INVALID, "short_conv: float32 input, output and state [slots, taps - 1, channels], bf16 taps");
    for (int i : {1, 3})
      if (l.t[i] >= 0 && (T[l.t[i]].dtype != MPK_BF16 || T[l.t[i]].dim(0) != C)) return fail(MPK_ERR_INVALID, "short_conv: bf16 biases [channels]");
    const int copy = norm_tensor(l, 6);
    if (copy >= 0 && (T[copy].dtype != act_dtype() || T[copy].dim(1) < C)) return fail(MPK_ERR_INVALID, "short_conv: copy of the output in the graph's activation type");
    const int nt = std::max(1, std::min(W, C / 32));
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_SHORT_CONV, li);
      for (int k = 0; k < 6; ++k) d.p[k] = l.t[k] >= 0 ? (uint64_t)T[l.t[k]].ptr : 0;
      d.p[6] = copy >= 0 ? (uint64_t)T[copy].ptr : 0; d.a[8] = copy >= 0 ? (int)T[copy].ld() : 0;
      d.a[0] = (int)((int64_t)C * i / nt); d.a[1] = (int)((int64_t)C * (i + 1) / nt); d.a[2] = C; d.a[3] = taps;
      d.a[4] = (int)x.ld(); d.a[5] = (int)l.params[0]; d.a[6] = (int)o.ld(); d.a[7] = (int)l.params[1];
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_selective_scan(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &u = T[l.t[0]], &low = T[l.t[1]], &gate = T[l.t[2]], &dt = T[l.t[3]], &st = T[l.t[7]], &o = T[l.t[8]];
    if (l.params.size() < 3 || dt.dims.size() != 2) return fail(MPK_ERR_INVALID, "selective_scan: dt weight [channels, rank], params [rank, n, gate column]");
    const int C = (int)dt.dim(0), rank = (int)l.params[0], n = (int)l.params[1], np = round_up(n, 4);
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "selective_scan needs the batch meta tensors");
    if (n > 128) return fail(MPK_ERR_UNSUPPORTED, "selective_scan: state sizes up to 128");
    if (rank < 1 || n < 1 || u.dtype != MPK_F32 || low.dtype != MPK_F32 || gate.dtype != MPK_F32 || st.dtype != MPK_F32 || o.dtype != act_dtype() ||
        u.dim(1) < C || low.dim(1) < rank + 2 * n || l.params[2] < 0 || l.params[2] + C > gate.dim(1) || o.dim(1) < C || st.dims.size() != 3 ||
        st.dim(0) < cfg.max_num_batched_requests || st.dim(1) != C || st.dim(2) != np)
      return fail(MPK_ERR_INVALID, "selective_scan: float32 inputs and state [slots, channels, n rounded up to 4], output of the activation type");
    for (int i = 3; i < 7; ++i)
      if (T[l.t[i]].dtype != MPK_BF16 || (int64_t)(T[l.t[i]].bytes / 2) != (int64_t)C * (i == 3 ? rank : i == 5 ? n : 1) ||
          (T[l.t[i]].dims.size() == 2 && T[l.t[i]].strides[1] != 1))
        return fail(MPK_ERR_INVALID, "selective_scan: bf16 dt weight [channels, rank], dt bias, A_log [channels, n] and D");
    const int blocks = (C + 7) / 8, nt = std::min(W, blocks);   // eight channels: rows of whole 16-byte pieces
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_SELECTIVE_SCAN, li);
      for (int k = 0; k < 7; ++k) d.p[k] = (uint64_t)T[l.t[k]].ptr;
      d.p[7] = (uint64_t)o.ptr;
      put_wide(&d, SS_STATE, l.t[7]);
      d.a[SS_C0] = (int)((int64_t)blocks * i / nt) * 8; d.a[SS_C1] = std::min(C, (int)((int64_t)blocks * (i + 1) / nt) * 8); d.a[SS_C] = C; d.a[SS_RANK] = rank; d.a[SS_N] = n;
      d.a[SS_NP] = np; d.a[SS_LANES] = scan_lanes(n); d.a[SS_LDU] = (int)u.ld(); d.a[SS_LDL] = (int)low.ld(); d.a[SS_LDG] = (int)gate.ld();
      d.a[SS_GOFF] = (int)l.params[2]; d.a[SS_LDO] = (int)o.ld();
      put((i + rot) % W, d, ex);
    }
    g->weight_bytes += (int64_t)C * (rank + n + 2) * 2;
    return MPK_OK;
  }

  int emit_diff_combine(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &x = T[l.t[0]], &o = T[l.t[1]];
    if (l.params.size() < 5) return fail(MPK_ERR_INVALID, "diff_combine needs 5 parameters");
    const int H = (int)l.params[0], vdim = (int)l.params[1];
    if (H < 1 || vdim < 1 || x.dtype != MPK_F32 || o.dtype != act_dtype() || x.dim(1) < (int64_t)2 * H * vdim || o.dim(1) < (int64_t)H * vdim)
      return fail(MPK_ERR_INVALID, "diff_combine: float32 maps [tokens, heads x 2 x vdim], output [tokens, heads x vdim] of the activation type");
    const int nt = std::max(1, std::min(W, (nb_max * H + 7) / 8));
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_DIFF_COMBINE, li);
      d.p[0] = (uint64_t)x.ptr; d.p[1] = (uint64_t)o.ptr;
      d.a[0] = i; d.a[1] = nt; d.a[2] = H; d.a[3] = vdim; d.a[4] = (int)x.ld(); d.a[5] = (int)o.ld();
      for (int k = 0; k < 3; ++k) d.a[6 + k] = bits_of(l.params[2 + k]);
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_poly_norm(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &z = T[l.t[0]], &co = T[l.t[1]], &o = T[l.t[2]];
    const int N = (int)z.dim(1), rows = (int)std::min<int64_t>(z.dim(0), cfg.max_num_batched_tokens), nt = std::min(rows, W);
    if (l.params.empty() || z.dtype != MPK_F32 || z.dims.size() != 2 || co.dtype != MPK_BF16 || co.dim(0) != 4 || o.dtype != act_dtype() || o.dim(1) < N || o.dim(0) < rows)
      return fail(MPK_ERR_INVALID, "poly_norm: float32 values [tokens, n], four bf16 coefficients, output [tokens, >= n] of the activation type");
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(TASK_POLY_NORM, li);
      for (int k = 0; k < 3; ++k) d.p[k] = (uint64_t)T[l.t[k]].ptr;
      d.a[0] = (int)((int64_t)rows * i / nt); d.a[1] = (int)((int64_t)rows * (i + 1) / nt); d.a[2] = N; d.a[3] = (int)z.ld(); d.a[4] = (int)o.ld();
      d.a[5] = bits_of(l.params[0]);
      put((i + rot) % W, d, ex);
    }
    return MPK_OK;
  }

  int emit_rglru(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &u = T[l.t[0]], &pr = T[l.t[1]], &ra = T[l.t[3]], &st = T[l.t[8]], &o = T[l.t[9]];
    if (l.params.size() < 4 || ra.dims.size() != 3 || ra.dim(1) != ra.dim(2)) return fail(MPK_ERR_INVALID, "rglru: gates [blocks, size, size], 4 parameters");
    const int nb = (int)ra.dim(0), bs = (int)ra.dim(1);
    const int64_t width = (int64_t)nb * bs;
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "rglru needs the batch meta tensors");
    if (u.dtype != MPK_F32 || pr.dtype != MPK_F32 || st.dtype != MPK_F32 || o.dtype != act_dtype() || u.dim(1) != width ||
        l.params[0] + width > pr.dim(1) || l.params[1] + width > o.dim(1) || (int64_t)(st.bytes / 4) < (int64_t)cfg.max_num_batched_requests * width)
      return fail(MPK_ERR_INVALID, "rglru: shapes or types of u, projections, state [slots, width] and output");
    for (int i = 2; i < 8; ++i)
      if (T[l.t[i]].dtype != MPK_BF16 || (int64_t)(T[l.t[i]].bytes / 2) < (i == 3 || i == 5 ? width * bs : width) || ((uint64_t)T[l.t[i]].ptr & 3))
        return fail(MPK_ERR_INVALID, "rglru: bf16 gate weights and biases, 4-byte aligned");
    int C, TG;
    rglru_plan(l, &C, &TG);
    int i = 0;
    for (int b = 0; b < nb; ++b)
      for (int c0 = 0; c0 < bs; c0 += C, ++i) {
        TaskDesc d = blank(TASK_RGLRU, li);
        for (int k = 0; k < 8; ++k) d.p[k] = (uint64_t)T[l.t[k]].ptr;
        const uint64_t sp = (uint64_t)st.ptr, op = (uint64_t)o.ptr;
        std::memcpy(&d.a[GL_STATE], &sp, 8);
        std::memcpy(&d.a[GL_OUT], &op, 8);
        d.a[GL_BLOCK] = b; d.a[GL_C0] = c0; d.a[GL_C1] = std::min(c0 + C, bs); d.a[GL_BS] = bs; d.a[GL_WIDTH] = (int)width;
        d.a[GL_LDU] = (int)u.ld(); d.a[GL_LDP] = (int)pr.ld(); d.a[GL_YOFF] = (int)l.params[0]; d.a[GL_LDO] = (int)o.ld();
        d.a[GL_OCOL] = (int)l.params[1]; d.a[GL_OSCALE] = bits_of(l.params[2]); d.a[GL_GATE_C] = bits_of(l.params[3]); d.a[GL_TG] = TG;
        put((i + rot) % W, d, ex);
      }
    g->weight_bytes += 4 * width * bs;
    return MPK_OK;
  }

  int emit_mlstm(int li, int ex) {
    const LayerInfo &l = L[li];
    const TensorInfo &pr = T[l.t[0]], &S = T[l.t[4]], &nm = T[l.t[5]], &raw = T[l.t[6]], &o = T[l.t[7]];
    if (l.params.size() < 13) return fail(MPK_ERR_INVALID, "mlstm needs 13 parameters");
    const int H = (int)l.params[0], dim = (int)l.params[1], vdim = (int)l.params[2], chunks = (int)l.params[12];
    const int slots = cfg.max_num_batched_requests;
    if (!batch_meta_given()) return fail(MPK_ERR_INVALID, "mlstm needs the batch meta tensors");
    if (H < 1 || dim < 1 || vdim < 1) return fail(MPK_ERR_INVALID, "mlstm: head count or sizes");
    if (dim > 1024) return fail(MPK_ERR_UNSUPPORTED, "mlstm: key sizes up to 1024");
    if (pr.dtype != MPK_F32 || S.dtype != MPK_F32 || nm.dtype != MPK_F32 || raw.dtype != MPK_F32 || o.dtype != act_dtype() || S.dims.size() != 4 ||
        S.dim(0) < slots || S.dim(1) != H || S.dim(2) != dim || S.dim(3) < vdim || S.dim(3) % 4 || raw.dim(1) < (int64_t)H * vdim ||
        o.dim(1) < (int64_t)H * vdim)
      return fail(MPK_ERR_INVALID, "mlstm: state [slots, heads, dim, vdim rounded up to 4], scratch and output [tokens, heads x vdim]");
    for (int i = 3; i < 9; ++i) {
      const int64_t w = i < 5 ? (int64_t)H * dim : (i < 7 ? (int64_t)H * vdim : H);
      if (l.params[i] < 0 || l.params[i] + w > pr.dim(1)) return fail(MPK_ERR_INVALID, "mlstm: columns outside the projections");
    }
    for (int i = 1; i < 4; ++i)
      if (T[l.t[i]].dtype != MPK_BF16 || (int64_t)(T[l.t[i]].bytes / 2) < (i == 3 ? (int64_t)H * vdim : H)) return fail(MPK_ERR_INVALID, "mlstm: bf16 biases [heads] and norm [heads x vdim]");
    const int vc = MPK_MLSTM_COLUMNS(dim), nsub = (vdim + vc - 1) / vc;
    if (chunks < 1 || chunks > nsub || nm.dims.size() != 4 || nm.dim(0) < slots || nm.dim(1) != H || nm.dim(2) != chunks || nm.dim(3) != dim + 1)
      return fail(MPK_ERR_INVALID, "mlstm: chunk count or normaliser state [slots, heads, chunks, dim + 1]");
    for (int s = 0; s < slots; ++s)
      for (int h = 0; h < H; ++h)
        for (int ch = 0; ch < chunks; ++ch) {
          TaskDesc d = blank(TASK_MLSTM, li);
          for (int k = 0; k < 8; ++k) d.p[k] = (uint64_t)T[l.t[k]].ptr;
          d.a[ML_SLOT] = s; d.a[ML_HEAD] = h; d.a[ML_CHUNK] = ch; d.a[ML_NCHUNK] = chunks; d.a[ML_H] = H; d.a[ML_DIM] = dim;
          d.a[ML_VDIM] = vdim; d.a[ML_VDIMP] = (int)S.dim(3);
          d.a[ML_V0] = nsub * ch / chunks * vc; d.a[ML_V1] = std::min(nsub * (ch + 1) / chunks * vc, (int)S.dim(3));
          d.a[ML_CAP] = bits_of(l.params[9]); d.a[ML_EPS] = bits_of(l.params[10]); d.a[ML_QSCALE] = bits_of(l.params[11]);
          d.a[ML_LDP] = (int)pr.ld(); d.a[ML_QOFF] = (int)l.params[3]; d.a[ML_KOFF] = (int)l.params[4]; d.a[ML_VOFF] = (int)l.params[5];
          d.a[ML_GOFF] = (int)l.params[6]; d.a[ML_IOFF] = (int)l.params[7]; d.a[ML_FOFF] = (int)l.params[8]; d.a[ML_LDO] = (int)o.ld();
          d.a[ML_TICKET] = hybrid_tickets + s * H + h; d.a[ML_TC] = mlstm_tokens(dim); d.a[ML_LDR] = (int)raw.ld();
          put(((s * H + h) * chunks + ch + rot) % W, d, ex);
        }
    hybrid_tickets += slots * H;
    return MPK_OK;
  }

  void emit_token_rows(uint32_t type, int li, int ex, uint64_t p0, uint64_t p1, uint64_t p2, int width, int ldi,
                       int ldo, int aux, int ldi2, int rows_total) {
    const int nt = std::min(rows_total, W);
    for (int i = 0; i < nt; ++i) {
      TaskDesc d = blank(type, li);
      d.p[0] = p0; d.p[1] = p1; d.p[2] = p2;
      d.a[E_T0] = (int)((int64_t)rows_total * i / nt);
      d.a[E_T1] = (int)((int64_t)rows_total * (i + 1) / nt);
      d.a[E_WIDTH] = width; d.a[E_LDI] = ldi; d.a[E_LDO] = ldo; d.a[E_AUX] = aux; d.a[E_LDI2] = ldi2;
      put((i + rot) % W, d, ex);
    }
  }

  int emit(int li, int ex, int *attn_ordinal) {
    const LayerInfo &l = L[li];
    const int mbt = cfg.max_num_batched_tokens;
    switch (l.op) {
      case MPK_OP_LINEAR: case MPK_OP_LINEAR_RESIDUAL: case MPK_OP_SPLITK_LINEAR:
        return g->hybrid == HYB_F32 ? emit_linear_f32(li, ex) : emit_linear(li, ex);
      case MPK_OP_RESIDUAL_NORM: return emit_residual_norm(li, ex);
      case MPK_OP_QKV_APPEND: return emit_qkv_append(li, ex);
      case MPK_OP_EXT_ATTENTION: return emit_ext_attention(li, ex);
      case MPK_OP_SHORT_CONV: return emit_short_conv(li, ex);
      case MPK_OP_RGLRU: return emit_rglru(li, ex);
      case MPK_OP_SELECTIVE_SCAN: return emit_selective_scan(li, ex);
      case MPK_OP_DIFF_COMBINE: return emit_diff_combine(li, ex);
      case MPK_OP_POLY_NORM: return emit_poly_norm(li, ex);
      case MPK_OP_MLSTM: return emit_mlstm(li, ex);
      case MPK_OP_GLA: return emit_gla(li, ex);
      case MPK_OP_LATENT_APPEND: return emit_latent_append(li, ex);
      case MPK_OP_GROUPED_LINEAR: return emit_grouped_linear(li, ex);
      case MPK_OP_ATTN_MERGE: return emit_attn_merge(li, ex);
      case MPK_OP_LINEAR_FP8: case MPK_OP_LINEAR_FP8_RESIDUAL:
        return emit_linear_fp8(li, ex);
      case MPK_OP_QUANTIZE_FP8:
        return emit_quantize_fp8(li, ex);
      case MPK_OP_MOE_W13_LINEAR: case MPK_OP_MOE_W2_LINEAR: case MPK_OP_MOE_W13_FP8: case MPK_OP_MOE_W2_FP8:
        return emit_moe_gemm(li, ex);
      case MPK_OP_MOE_TOPK_SOFTMAX: {
        // the same task as the sigmoid routing with one group, no bias and scaling 1: only the score function differs
        const TensorInfo &lg = T[l.t[0]], &w = T[l.t[1]], &idx = T[l.t[2]], &mask = T[l.t[3]];
        const int E = g->hybrid ? (int)idx.dim(0) : (int)lg.dim(1), topk = (int)w.dim(1);
        if (lg.dim(1) < E || (lg.dtype != MPK_BF16 && lg.dtype != MPK_F32) || w.dtype != MPK_F32 || idx.dtype != MPK_I32 || mask.dtype != MPK_I32 ||
            E > 1024 || idx.dim(0) != E || mask.dim(0) != E + 1 || topk <= 0 || topk > std::min(E, 32) || idx.dim(1) > kMaxLinearTokens)
          return fail(MPK_ERR_UNSUPPORTED, "softmax routing: logits bf16/f32 [B, E <= 1024], weights f32 [B, topk <= 32], indices and mask int32");
        TaskDesc d = blank(TASK_MOE_ROUTING, li);
        d.p[0] = (uint64_t)lg.ptr; d.p[1] = 0; d.p[2] = (uint64_t)w.ptr; d.p[3] = (uint64_t)idx.ptr; d.p[4] = (uint64_t)mask.ptr;
        d.a[0] = E; d.a[1] = topk; d.a[2] = 1; d.a[3] = 1; d.a[4] = l.params.size() > 3 ? bits_of(l.params[3]) : float_bits(1.0f); d.a[5] = (int)lg.ld();
        d.a[6] = (int)w.ld(); d.a[7] = (int)idx.dim(1); d.a[8] = lg.dtype == MPK_F32 ? 1 : 0;
        d.a[9] = l.params.size() > 1 ? (int)l.params[0] : 0;
        d.a[10] = l.params.size() > 1 ? (int)l.params[1] : E;
        d.a[11] = 1;   // softmax scores, logits left in place
        d.a[13] = l.params.size() > 2 ? (int)l.params[2] : 0;
        if (d.a[9] < 0 || d.a[10] > E || d.a[9] >= d.a[10]) return fail(MPK_ERR_INVALID, "softmax routing: bad local expert range");
        put(rot % W, d, ex);
        return MPK_OK;
      }
      case MPK_OP_MOE_TOPK_SIGMOID: {
        const TensorInfo &lg = T[l.t[0]], &bias = T[l.t[1]], &w = T[l.t[2]], &idx = T[l.t[3]], &mask = T[l.t[4]];
        if (l.params.size() < 3) return fail(MPK_ERR_INVALID, "sigmoid routing needs [num_groups, topk_group, scaling_bits]");
        // (hybrid graphs: the router's logits may be the leading columns of a wider tensor)
        const int E = g->hybrid ? (int)idx.dim(0) : (int)lg.dim(1), topk = (int)w.dim(1), groups = (int)l.params[0], keep = (int)l.params[1];
        if (lg.dim(1) < E || (g->hybrid && !keeps_logits(l))) return fail(MPK_ERR_INVALID, "sigmoid routing: fewer logits than experts, or (hybrid graphs) logits that are not kept");
        if ((lg.dtype != MPK_BF16 && lg.dtype != MPK_F32) || bias.dtype != MPK_F32 || w.dtype != MPK_F32 ||
            idx.dtype != MPK_I32 || mask.dtype != MPK_I32)
          return fail(MPK_ERR_INVALID, "sigmoid routing: logits bf16/f32, bias and weights f32, indices and mask int32");
        if (groups <= 0 || groups > 64 || E % groups != 0 || keep <= 0 || keep > groups || E > 1024 || bias.dim(0) != E ||
            idx.dim(0) != E || mask.dim(0) != E + 1 || topk <= 0 || topk > keep * (E / groups) || idx.dim(1) > kMaxLinearTokens)
          return fail(MPK_ERR_UNSUPPORTED, "sigmoid routing: unsupported expert / group / top-k configuration");
        TaskDesc d = blank(TASK_MOE_ROUTING, li);
        d.p[0] = (uint64_t)lg.ptr; d.p[1] = (uint64_t)bias.ptr; d.p[2] = (uint64_t)w.ptr; d.p[3] = (uint64_t)idx.ptr;
        d.p[4] = (uint64_t)mask.ptr;
        d.a[0] = E; d.a[1] = topk; d.a[2] = groups; d.a[3] = keep; d.a[4] = (int)l.params[2]; d.a[5] = (int)lg.ld();
        d.a[6] = (int)w.ld(); d.a[7] = (int)idx.dim(1); d.a[8] = lg.dtype == MPK_F32 ? 1 : 0;
        // optional params [3], [4]: first and one-past-last expert this rank runs (expert parallelism)
        d.a[9] = l.params.size() > 4 ? (int)l.params[3] : 0;
        d.a[10] = l.params.size() > 4 ? (int)l.params[4] : E;
        d.a[12] = keeps_logits(l) ? 1 : 0;
        if (d.a[9] < 0 || d.a[10] > E || d.a[9] >= d.a[10] || topk > 32)
          return fail(MPK_ERR_INVALID, "sigmoid routing: bad local expert range");
        put(rot % W, d, ex);
        return MPK_OK;
      }
      case MPK_OP_MLA_KV_GATHER: {
        const TensorInfo &lat = T[l.t[0]], &pe = T[l.t[1]], &cache = T[l.t[2]];
        if (l.params.size() < 3) return fail(MPK_ERR_INVALID, "mla_kv_gather needs [d_k, d_v, page_size]");
        const int dk = (int)l.params[0], dv = (int)l.params[1], page = (int)l.params[2];
        if (dk != 576 || dv != 512 || cache.dims.size() != 3 || cache.dim(1) != page || cache.dim(2) != dk ||
            lat.dtype != MPK_BF16 || pe.dtype != MPK_BF16 || cache.dtype != MPK_BF16 || lat.dim(1) < dv || pe.dim(1) < dk - dv)
          return fail(MPK_ERR_UNSUPPORTED, "mla_kv_gather: bf16 cache [pages, page, 576], c_latent [tokens, 512], k_pe [tokens, >= 64]");
        if (!cfg.qo_indptr || !cfg.paged_kv_indptr || !cfg.paged_kv_indices || !cfg.paged_kv_last_page_len) {
          if (!cfg.dry_run) return fail(MPK_ERR_INVALID, "mla_kv_gather needs the batch meta tensors");
        }
        for (int s = 0; s < cfg.max_num_batched_requests; ++s) {
          TaskDesc d = blank(TASK_MLA_APPEND, li);
          d.p[0] = (uint64_t)lat.ptr; d.p[1] = (uint64_t)pe.ptr; d.p[2] = (uint64_t)cache.ptr;
          d.a[0] = s; d.a[1] = (int)lat.ld(); d.a[2] = (int)pe.ld(); d.a[3] = page; d.a[4] = dk; d.a[5] = dv;
          put((s + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_MLA_DECODE: {
        const TensorInfo &q = T[l.t[0]], &cache = T[l.t[1]], &po = T[l.t[2]], &lse = T[l.t[3]];
        if (l.params.size() < 6) return fail(MPK_ERR_INVALID, "mla decode needs [heads, q_len, kv_len, splits, scale, page]");
        const int H = (int)l.params[0], q_len = (int)l.params[1], kv_len = (int)l.params[2], S = (int)l.params[3];
        const int page = (int)l.params[5];
        if (H <= 0 || H % 16 != 0 || q.dim(q.dims.size() - 1) != (int64_t)H * 576 || q.dtype != MPK_BF16 ||
            cache.dtype != MPK_BF16 || po.dtype != MPK_BF16 || lse.dtype != MPK_F32 || S != (kv_len + 127) / 128)
          return fail(MPK_ERR_UNSUPPORTED, "mla decode: bf16 q [tokens, heads * 576] with heads a multiple of 16");
        if ((int64_t)(po.bytes / 2) < (int64_t)mbt * H * S * 512 || (int64_t)(lse.bytes / 4) < (int64_t)mbt * H * S)
          return fail(MPK_ERR_INVALID, "mla decode: partial buffers hold fewer than tokens x heads x splits rows");
        if (page > 0 && (cache.dims.size() != 3 || cache.dim(1) != page || cache.dim(2) != 576))
          return fail(MPK_ERR_INVALID, "mla decode: paged cache must be [pages, page, 576]");
        if (page > 0 && !cfg.dry_run && (!cfg.qo_indptr || !cfg.paged_kv_indptr || !cfg.paged_kv_indices || !cfg.paged_kv_last_page_len))
          return fail(MPK_ERR_INVALID, "mla decode on a paged cache needs the batch meta tensors");
        if (page == 0 && (q_len <= 0 || mbt % q_len != 0 || (int64_t)(cache.bytes / 2) < (int64_t)(mbt / q_len) * kv_len * 576))
          return fail(MPK_ERR_INVALID, "mla decode: dense cache must be [requests * kv_len, 576] with q_len tokens per request");
        int i = 0;
        for (int t = 0; t < mbt; ++t)
          for (int s = 0; s < S; ++s)
            for (int h0 = 0; h0 < H; h0 += 16, ++i) {
              TaskDesc d = blank(TASK_MLA_DECODE, li);
              d.p[0] = (uint64_t)q.ptr; d.p[1] = (uint64_t)cache.ptr; d.p[2] = (uint64_t)po.ptr; d.p[3] = (uint64_t)lse.ptr;
              d.a[0] = t; d.a[1] = s; d.a[2] = h0; d.a[3] = H; d.a[4] = S; d.a[5] = page; d.a[6] = (int)q.ld();
              d.a[7] = (int)l.params[4]; d.a[8] = q_len; d.a[9] = kv_len;
              put((i + rot) % W, d, ex);
            }
        return MPK_OK;
      }
      case MPK_OP_MLA_REDUCE: {
        const TensorInfo &po = T[l.t[0]], &lse = T[l.t[1]], &y = T[l.t[2]];
        if (l.params.size() < 2) return fail(MPK_ERR_INVALID, "mla reduce needs [heads, splits]");
        const int H = (int)l.params[0], S = (int)l.params[1];
        if (S > 64) return fail(MPK_ERR_UNSUPPORTED, "mla reduce handles at most 64 splits (8192 positions)");
        if (y.dtype != MPK_BF16 || (int64_t)(y.bytes / 2) < (int64_t)mbt * H * 512 || po.dtype != MPK_BF16 || lse.dtype != MPK_F32)
          return fail(MPK_ERR_INVALID, "mla reduce: bf16 output [tokens, heads * 512]");
        const int rows = mbt * H, nt = std::max(1, std::min(W, rows / 8));
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_MLA_REDUCE, li);
          d.p[0] = (uint64_t)po.ptr; d.p[1] = (uint64_t)lse.ptr; d.p[2] = (uint64_t)y.ptr;
          d.a[0] = (int)((int64_t)rows * i / nt); d.a[1] = (int)((int64_t)rows * (i + 1) / nt); d.a[2] = H; d.a[3] = S;
          d.a[4] = y.dims.size() == 2 ? (int)y.ld() : H * 512;
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_MOE_SILU_MUL: {
        const TensorInfo &m = T[l.t[0]], &y = T[l.t[1]];
        if (m.dims.size() != 3 || y.dims.size() != 3 || m.dim(2) != 2 * y.dim(2) || m.dtype != MPK_BF16)
          return fail(MPK_ERR_INVALID, "moe_silu_mul: [B, topk, 2I] -> [B, topk, I] bf16");
        const int rows = (int)(y.dim(0) * y.dim(1)), nt = std::min(rows, W);
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_MOE_SILU_MUL, li);
          d.p[0] = (uint64_t)m.ptr; d.p[2] = (uint64_t)y.ptr;
          d.a[0] = (int)((int64_t)rows * i / nt); d.a[1] = (int)((int64_t)rows * (i + 1) / nt);
          d.a[2] = (int)y.dim(2); d.a[3] = (int)m.strides[1]; d.a[4] = (int)y.strides[1]; d.a[5] = (int)y.dim(1);
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_MOE_MUL_SUM_ADD: {
        const TensorInfo &x = T[l.t[0]], &w = T[l.t[1]], &y = T[l.t[3]];
        const bool has_res = l.t[2] >= 0;
        if (x.dims.size() != 3 || w.dtype != MPK_F32 || x.dtype != MPK_BF16 || y.dim(1) != x.dim(2) || w.dim(1) != x.dim(1))
          return fail(MPK_ERR_INVALID, "moe_mul_sum_add: x [B, topk, H] bf16, weights [B, topk] f32, out [B, H]");
        const int H = (int)x.dim(2), nt = std::max(1, std::min(W, H / 64));
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_MOE_MUL_SUM_ADD, li);
          d.p[0] = (uint64_t)x.ptr; d.p[1] = (uint64_t)w.ptr; d.p[2] = (uint64_t)y.ptr;
          d.p[3] = has_res ? (uint64_t)T[l.t[2]].ptr : 0;
          d.a[0] = (int)((int64_t)H * i / nt); d.a[1] = (int)((int64_t)H * (i + 1) / nt); d.a[2] = H; d.a[3] = (int)x.dim(1);
          d.a[4] = (int)y.ld(); d.a[5] = has_res ? (int)T[l.t[2]].ld() : 0; d.a[6] = (int)w.ld(); d.a[7] = (int)x.dim(0);
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_ATTENTION: case MPK_OP_PAGED_ATTENTION:
        return emit_attention(li, ex, (*attn_ordinal)++);
      case MPK_OP_EMBED: {
        const TensorInfo &tab = T[l.t[1]], &y = T[l.t[2]];
        if (T[l.t[0]].dtype != MPK_I64) return fail(MPK_ERR_INVALID, "embed ids must be int64");
        if (g->hybrid) {
          // the table may be wider than the stream (padded to the projections' k granularity)
          if (y.dtype != MPK_F32 || tab.dtype != MPK_BF16 || tab.dim(1) < y.dim(1)) return fail(MPK_ERR_INVALID, "embed in a hybrid graph: bf16 table, float32 output");
          const int pairs = norm_tensor(l, 3), freq = norm_tensor(l, 4), copy = norm_tensor(l, 5);
          if (pairs >= 0 && (T[pairs].dtype != MPK_BF16 || T[pairs].dims.size() != 2 || T[pairs].dim(0) < 2 || T[pairs].dim(1) < y.dim(1) || l.params.size() < 4))
            return fail(MPK_ERR_INVALID, "embed: bigram table bf16 [buckets + 1, width], two multipliers");
          if (pairs >= 0 && !cfg.dry_run && !cfg.tokens) return fail(MPK_ERR_INVALID, "embed: bigrams need the token table");
          if (freq >= 0 && (T[freq].dtype != MPK_I64 || T[freq].dim(0) < (y.dim(1) + 1) / 2)) return fail(MPK_ERR_INVALID, "embed: position frequencies int64 [(width + 1) / 2]");
          if (copy >= 0 && (T[copy].dtype != MPK_F32 || T[copy].dims.size() < 2 || T[copy].dims.back() < y.dim(1) || T[copy].dim((int)T[copy].dims.size() - 2) < mbt))
            return fail(MPK_ERR_INVALID, "embed: copy of the output float32 [.., tokens, width]");
          if ((pairs >= 0 || freq >= 0) && !batch_meta_given()) return fail(MPK_ERR_INVALID, "embed: bigrams and positions need the batch meta tensors");
          const int nt = std::min(mbt, W);
          for (int i = 0; i < nt; ++i) {
            TaskDesc d = blank(TASK_EMBED_F32, li);
            for (int k = 0; k < 6; ++k) d.p[k] = norm_tensor(l, k) >= 0 ? (uint64_t)T[l.t[k]].ptr : 0;
            d.a[E_T0] = (int)((int64_t)mbt * i / nt); d.a[E_T1] = (int)((int64_t)mbt * (i + 1) / nt);
            d.a[E_WIDTH] = (int)y.dim(1); d.a[E_LDI] = (int)tab.ld(); d.a[E_LDO] = (int)y.ld(); d.a[E_AUX] = (int)tab.dim(0);
            d.a[E_LDI2] = l.params.size() > 1 ? bits_of(l.params[1]) : float_bits(1.0f);
            d.a[E_LDC] = copy >= 0 ? (int)T[copy].ld() : 0;
            if (pairs >= 0) {
              d.a[E_LDB] = (int)T[pairs].ld(); d.a[E_BUCKETS] = (int)T[pairs].dim(0) - 1;
              std::memcpy(&d.a[E_PREV], &l.params[2], 8);
              std::memcpy(&d.a[E_CUR], &l.params[3], 8);
            }
            put((i + rot) % W, d, ex);
          }
          return MPK_OK;
        }
        if (tab.dim(1) % 8 != 0) return fail(MPK_ERR_UNSUPPORTED, "embedding width must be a multiple of 8");
        emit_token_rows(TASK_EMBED, li, ex, (uint64_t)T[l.t[0]].ptr, (uint64_t)tab.ptr, (uint64_t)y.ptr,
                        (int)tab.dim(1), (int)tab.ld(), (int)y.ld(), (int)tab.dim(0), 0, mbt);
        return MPK_OK;
      }
      case MPK_OP_RMSNORM: {
        const TensorInfo &x = T[l.t[0]], &y = T[l.t[2]];
        if (x.dim(1) % 8 != 0) return fail(MPK_ERR_UNSUPPORTED, "rmsnorm width must be a multiple of 8");
        emit_token_rows(TASK_RMSNORM, li, ex, (uint64_t)x.ptr, (uint64_t)T[l.t[1]].ptr, (uint64_t)y.ptr,
                        (int)x.dim(1), (int)x.ld(), (int)y.ld(), float_bits(1e-6f), 0, (int)std::min<int64_t>(x.dim(0), mbt));
        return MPK_OK;
      }
      case MPK_OP_ELEMENTWISE_ADD: {
        const TensorInfo &a = T[l.t[0]], &b = T[l.t[1]], &y = T[l.t[2]];
        emit_token_rows(TASK_ELEMENTWISE_ADD, li, ex, (uint64_t)a.ptr, (uint64_t)b.ptr, (uint64_t)y.ptr,
                        (int)a.dim(1), (int)a.ld(), (int)y.ld(), 0, (int)b.ld(), (int)std::min<int64_t>(a.dim(0), mbt));
        return MPK_OK;
      }
      case MPK_OP_TENSOR_INIT: {
        const TensorInfo &t = T[l.t[0]];
        const int es = elt_size(t.dtype);
        const int rows = (int)t.dim(0);
        const int64_t row_bytes = (int64_t)(t.bytes / std::max(rows, 1));
        if (row_bytes % 4 != 0) return fail(MPK_ERR_UNSUPPORTED, "tensor_init rows must be a multiple of 4 bytes");
        (void)es;
        emit_token_rows(TASK_TENSOR_INIT, li, ex, 0, 0, (uint64_t)t.ptr, (int)row_bytes, 0, (int)row_bytes, 0, 0, rows);
        return MPK_OK;
      }
      case MPK_OP_SILU_MUL: {
        const TensorInfo &m = T[l.t[0]], &y = T[l.t[1]];
        const int I = (int)y.dim(1);
        const int groups = std::max(l.grid[0], 1);
        if (m.dim(1) != 2 * (int64_t)I || I % groups != 0) return fail(MPK_ERR_INVALID, "silu_mul shapes");
        // column ranges in units of 8 (one 16-byte vector); about 4096 elements of work per task at least
        const int units = I % 8 == 0 ? I / 8 : I, unit = I % 8 == 0 ? 8 : 1;
        const int nt = (int)std::max<int64_t>(1, std::min<int64_t>({(int64_t)W, (int64_t)units, (int64_t)mbt * I / 4096}));
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_SILU_MUL, li);
          d.p[0] = (uint64_t)m.ptr; d.p[2] = (uint64_t)y.ptr;
          d.a[E_T0] = 0; d.a[E_T1] = mbt; d.a[E_WIDTH] = I; d.a[E_LDI] = (int)m.ld(); d.a[E_LDO] = (int)y.ld();
          d.a[E_AUX] = groups;
          d.a[7] = (int)((int64_t)units * i / nt) * unit;
          d.a[8] = (int)((int64_t)units * (i + 1) / nt) * unit;
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_ARGMAX_PARTIAL: case MPK_OP_SAMPLING_PARTIAL: {
        const TensorInfo &lg = T[l.t[0]], &pv = T[l.t[1]], &pi = T[l.t[2]];
        const bool sampling = l.op == MPK_OP_SAMPLING_PARTIAL;
        const int n = std::max(l.grid[0], 1);
        const int V = (int)lg.dim(1);
        if (pv.dim(1) < n || pi.dim(1) < n || pi.dtype != MPK_I64)
          return fail(MPK_ERR_INVALID, "argmax partial buffers must be [tokens, >= grid.x], index int64");
        if (lg.dtype != (g->hybrid ? MPK_F32 : MPK_BF16) || pv.dtype != (g->hybrid && !sampling ? MPK_F32 : MPK_BF16))
          return fail(MPK_ERR_INVALID, "argmax / sampling: bf16 logits and values (hybrid graphs: float32 logits, float32 argmax values)");
        for (int i = 0; i < n; ++i) {
          TaskDesc d = blank(sampling ? TASK_SAMPLING_PARTIAL : TASK_ARGMAX_PARTIAL, li);
          d.p[0] = (uint64_t)lg.ptr; d.p[1] = (uint64_t)pv.ptr; d.p[2] = (uint64_t)pi.ptr;
          d.a[0] = (int)((int64_t)V * i / n); d.a[1] = (int)((int64_t)V * (i + 1) / n); d.a[2] = i;
          d.a[3] = (int)lg.ld(); d.a[4] = (int)pv.ld();
          if (sampling) {   // Gumbel-max: philox seed and the rows one reference task would see (noise repeats per task)
            const uint64_t seed = l.params.size() > 0 ? (uint64_t)l.params[0] : 42u;
            d.a[6] = (int)(uint32_t)seed; d.a[7] = (int)(uint32_t)(seed >> 32);
            d.a[8] = l.params.size() > 1 ? std::max((int)l.params[1], 1) : 1;
            d.a[9] = V;
          }
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_ARGMAX_REDUCE: case MPK_OP_SAMPLING_REDUCE: {
        const TensorInfo &pv = T[l.t[0]], &pi = T[l.t[1]], &o = T[l.t[2]];
        const int partial_op = l.op == MPK_OP_SAMPLING_REDUCE ? MPK_OP_SAMPLING_PARTIAL : MPK_OP_ARGMAX_PARTIAL;
        if (o.dtype != MPK_I64) return fail(MPK_ERR_INVALID, "argmax output must be int64");
        // number of partials = tasks of the producing partial layer
        int n = (int)pv.dim(1);
        for (int j = li - 1; j >= 0; --j)
          if (L[j].op == partial_op && T[L[j].t[1]].storage == pv.storage) { n = std::max(L[j].grid[0], 1); break; }
        TaskDesc d = blank(l.op == MPK_OP_SAMPLING_REDUCE ? TASK_SAMPLING_REDUCE : TASK_ARGMAX_REDUCE, li);
        d.p[0] = (uint64_t)pv.ptr; d.p[1] = (uint64_t)pi.ptr; d.p[2] = (uint64_t)o.ptr;
        d.a[0] = n; d.a[1] = (int)pv.ld();
        put(rot % W, d, ex);
        return MPK_OK;
      }
      case MPK_OP_ARGMAX_EXCHANGE: {
        const TensorInfo &pv = T[l.t[0]], &pi = T[l.t[1]], &o = T[l.t[2]];
        if (o.dtype != MPK_I64 || pi.dtype != MPK_I64) return fail(MPK_ERR_INVALID, "argmax output and indices must be int64");
        int n = (int)pv.dim(1);
        for (int j = li - 1; j >= 0; --j)
          if (L[j].op == MPK_OP_ARGMAX_PARTIAL && T[L[j].t[1]].storage == pv.storage) { n = std::max(L[j].grid[0], 1); break; }
        TaskDesc d = blank(TASK_ARGMAX_EXCHANGE, li);
        d.p[0] = (uint64_t)pv.ptr; d.p[1] = (uint64_t)pi.ptr; d.p[2] = (uint64_t)o.ptr;
        d.p[5] = in.inbox_base_floats + (uint64_t)exchange_base_words;
        d.a[0] = n; d.a[1] = (int)pv.ld();
        d.a[2] = l.params.empty() ? 0 : (int)l.params[0];
        d.a[L_ARIDX] = l.ar_index;
        d.a[L_NAR] = g->num_allreduce;
        d.a[L_PARSTRIDE] = (int)g->inbox_floats_per_buffer;
        put(rot % W, d, ex);
        return MPK_OK;
      }
      case MPK_OP_AR_PUSH: {
        const TensorInfo &x = T[l.t[0]];
        const int N = (int)x.dim(1);
        const int nt = std::max(1, std::min(W, N / 64));
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_AR_PUSH, li);
          d.p[0] = (uint64_t)x.ptr; d.p[5] = in.inbox_base_floats;
          d.a[0] = (int)((int64_t)N * i / nt); d.a[1] = (int)((int64_t)N * (i + 1) / nt);
          d.a[2] = (int)x.ld(); d.a[3] = mbt * N; d.a[6] = N;
          d.a[7] = l.ar_index; d.a[8] = g->num_allreduce; d.a[9] = (int)g->inbox_floats_per_buffer;
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      case MPK_OP_ALLREDUCE: {
        const LayerInfo &p = L[l.ar_producer];
        const TensorInfo &y = T[l.t[2]];
        const int N = (int)y.dim(1);
        const int nt = std::max(1, std::min(W, N / 64));
        uint64_t res = 0; int ldr = 0;
        if (p.op == MPK_OP_LINEAR_RESIDUAL) { res = (uint64_t)T[p.t[2]].ptr; ldr = (int)T[p.t[2]].ld(); }
        if (p.op == MPK_OP_SPLITK_LINEAR) { res = (uint64_t)T[p.t[2]].ptr; ldr = (int)T[p.t[2]].ld(); }
        for (int i = 0; i < nt; ++i) {
          TaskDesc d = blank(TASK_ALLREDUCE, li);
          d.p[0] = in.inbox_base_floats; d.p[1] = res; d.p[2] = (uint64_t)y.ptr;
          d.a[0] = (int)((int64_t)N * i / nt); d.a[1] = (int)((int64_t)N * (i + 1) / nt);
          d.a[2] = cfg.world_size; d.a[3] = mbt * N; d.a[4] = (int)y.ld(); d.a[5] = ldr; d.a[6] = N;
          d.a[7] = l.ar_index; d.a[8] = g->num_allreduce; d.a[9] = (int)g->inbox_floats_per_buffer;
          put((i + rot) % W, d, ex);
        }
        return MPK_OK;
      }
      default: return fail(MPK_ERR_UNSUPPORTED, "op not implemented");
    }
  }

  // output tensor a layer writes only a column range of, and that range's first column
  int sliced_output(const LayerInfo &l) const {
    switch (l.op) {
      case MPK_OP_EXT_ATTENTION: return l.t[3];
      case MPK_OP_RGLRU: return l.t[9];
      case MPK_OP_LATENT_APPEND: return l.t[2];     // the rotated columns of every head
      case MPK_OP_GROUPED_LINEAR: return l.t[2];    // N columns of every group
      default: return -1;
    }
  }
  int slice_column(const LayerInfo &l) const {
    // (a latent layer's rotated columns begin behind the latent ones, parameter 1)
    const size_t i = l.op == MPK_OP_EXT_ATTENTION ? 3 : 1;
    return l.params.size() > i ? (int)l.params[i] : 0;
  }

  int run() {
    int rc = check_arity();
    if (rc) return rc;
    rc = classify_hybrid();
    if (rc) return rc;
    for (const auto &l : L) if (l.folded) g->num_folded++;     // folded before materialisation (activation epilogue)
    fold_layers();
    fold_residual_norms();
    fold_poly_norms();
    rc = plan_allreduce();
    if (rc) return rc;
    rc = plan_smem();
    if (rc) return rc;
    // inbox sizing: widest pushed output
    int64_t nmax = 0;
    for (const auto &l : L)
      if (l.push) nmax = std::max<int64_t>(nmax, l.op == MPK_OP_AR_PUSH ? T[l.t[0]].dim(1) : T[l.t[1]].dim(0));
    g->inbox_floats_per_buffer = (int64_t)cfg.world_size * cfg.max_num_batched_tokens * nmax;
    // area of the argmax exchange behind the allreduce words: [world][tokens] x 4 words (never aliased with them, so a
    // stale pair can not be taken for an arrived partial sum or the other way round)
    exchange_base_words = g->inbox_floats_per_buffer;
    for (const auto &l : L)
      if (l.op == MPK_OP_ARGMAX_EXCHANGE) {
        g->inbox_floats_per_buffer += (int64_t)cfg.world_size * cfg.max_num_batched_tokens * 4;
        // keep the second buffer on the same 4 KB alignment as the first
        g->inbox_floats_per_buffer = (g->inbox_floats_per_buffer + 1023) / 1024 * 1024;
        break;
      }

    // ---- exec layers + dependencies ------------------------------------------------
    std::vector<int> exec_of_layer(L.size(), -1);
    // Layers that write a column range of a wider tensor (the branches of a parallel mixer) do not wait for one another:
    // every range is a storage of its own for its writers, and readers of the tensor read all of them.
    int slice_id = 1 << 24;
    for (const auto &l : L) {
      const int t = sliced_output(l);
      if (t >= 0 && !slices[T[t].storage].count(slice_column(l))) slices[T[t].storage][slice_column(l)] = slice_id++;
    }
    if (!no_batch_task()) {
      ExecLayer b;
      b.type = TASK_BATCH;
      b.reads = {ST_META_OUT};
      b.writes = {ST_META};
      g->exec.push_back(b);
    }
    for (size_t i = 0; i < L.size(); ++i) {
      if (L[i].folded) continue;
      ExecLayer e;
      e.layer = (int)i;
      std::vector<int> ins, outs;
      layer_io(L[i], &ins, &outs);
      for (int t : ins) {
        e.reads.push_back(T[t].storage);
        auto it = slices.find(T[t].storage);
        if (it != slices.end()) for (const auto &sl : it->second) e.reads.push_back(sl.second);
      }
      const int sliced = sliced_output(L[i]);
      for (int t : outs) {
        if (t == sliced) e.writes.push_back(slices[T[t].storage][slice_column(L[i])]);
        else e.writes.push_back(T[t].storage);
      }
      if (!no_batch_task()) e.reads.push_back(ST_META);
      e.remote_trigger = L[i].push && !L[i].push_ll;
      exec_of_layer[i] = (int)g->exec.size();
      g->exec.push_back(e);
    }
    const int E = (int)g->exec.size();
    std::map<int, int> last_writer;
    std::map<int, std::set<int>> readers;
    std::vector<std::set<int>> deps(E);
    for (int e = 0; e < E; ++e) {
      ExecLayer &x = g->exec[e];
      for (int s : x.reads) {
        auto it = last_writer.find(s);
        if (it != last_writer.end() && it->second != e) deps[e].insert(it->second);
      }
      for (int s : x.writes) {
        auto it = last_writer.find(s);
        if (it != last_writer.end() && it->second != e) deps[e].insert(it->second);
        for (int r : readers[s]) if (r != e) deps[e].insert(r);
      }
      if (x.layer >= 0 && L[x.layer].op == MPK_OP_ALLREDUCE) deps[e].insert(exec_of_layer[L[x.layer].ar_producer]);
      for (int s : x.writes) { last_writer[s] = e; readers[s].clear(); }
      for (int s : x.reads) readers[s].insert(e);
    }
    // transitive reduction
    std::vector<std::vector<char>> anc(E, std::vector<char>(E, 0));
    for (int e = 0; e < E; ++e)
      for (int d : deps[e]) {
        anc[e][d] = 1;
        for (int k = 0; k < E; ++k) if (anc[d][k]) anc[e][k] = 1;
      }
    for (int e = 0; e < E; ++e) {
      for (int d : deps[e]) {
        bool redundant = false;
        for (int d2 : deps[e]) if (d2 != d && anc[d2][d]) redundant = true;
        if (!redundant) g->exec[e].deps.push_back(d);
      }
      if ((int)g->exec[e].deps.size() > kMaxDeps)
        return fail(MPK_ERR_UNSUPPORTED, "a layer depends on more than 3 independent producers");
    }

    // ---- tasks ---------------------------------------------------------------------
    per_worker.assign(W, {});
    per_worker_exec.assign(W, {});
    int attn_ordinal = 0;
    for (int e = 0; e < E; ++e) {
      ExecLayer &x = g->exec[e];
      rot = (e * 37) % W;
      if (x.layer < 0) {
        TaskDesc d = blank(TASK_BATCH, -1);
        put(0, d, e);
        x.type = TASK_BATCH;
        continue;
      }
      rc = emit(x.layer, e, &attn_ordinal);
      if (rc) return rc;
      if (x.num_tasks == 0) return fail(MPK_ERR_INVALID, "layer " + std::to_string(x.layer) + " produced no task");
    }
    g->attn_tickets *= std::max(attn_ordinal, 1);
    g->attn_tickets += hybrid_tickets;
    // ---- events: one per exec layer ---------------------------------------------------
    g->num_events = E;
    for (int e = 0; e < E; ++e) {
      ExecLayer &x = g->exec[e];
      for (int d : x.deps) {
        uint32_t need = (uint32_t)g->exec[d].num_tasks;
        if (g->exec[d].remote_trigger) need *= (uint32_t)cfg.world_size;
        x.dep_need.push_back(need);
      }
    }
    g->worker_begin.assign(W + 1, 0);
    for (int w = 0; w < W; ++w) {
      g->worker_begin[w] = (int32_t)g->tasks.size();
      bool observed_batch = false;   // an earlier task of this worker waited on something downstream of the batching task
      for (size_t i = 0; i < per_worker[w].size(); ++i) {
        TaskDesc d = per_worker[w][i];
        const int e = per_worker_exec[w][i];
        const ExecLayer &x = g->exec[e];
        // The attention tasks read the page tables before their own dependency wait and therefore check the
        // batching event first; once the worker has acquired any event of this iteration (every layer is
        // downstream of the batching task), that check is redundant.
        if (d.type == TASK_ATTENTION && observed_batch) d.a[A_EARLY_EV] = -1;
        if (!x.deps.empty() && x.type != TASK_BATCH && e > 0) observed_batch = true;
        for (size_t k = 0; k < x.deps.size(); ++k) {
          d.dep_event[k] = x.deps[k];
          d.dep_need[k] = x.dep_need[k];
          if (g->exec[x.deps[k]].remote_trigger) d.flags |= (TF_DEP0_REMOTE << k);
        }
        d.trig_event = e;
        if (x.remote_trigger) d.flags |= TF_REMOTE_TRIGGER;
        if (x.type == TASK_NOP) g->exec[e].type = d.type;
        g->tasks.push_back(d);
        g->task_exec.push_back(e);
      }
    }
    g->worker_begin[W] = (int32_t)g->tasks.size();
    g->general_kernel = cfg.max_num_batched_tokens > 8;
    for (const auto &d : g->tasks)
      if (!g->hybrid && ((d.type == TASK_LINEAR && (d.flags & TF_FP8)) || d.type >= TASK_QUANTIZE_FP8)) g->general_kernel = true;
    g->num_workers = W;
    g->world_size = std::max(cfg.world_size, 1);
    // attention ticket banks: patch the ticket offset now that the bank size is known
    const int64_t bank = attn_ordinal > 0 ? g->attn_tickets / attn_ordinal : 0;
    for (auto &d : g->tasks)
      if (d.type == TASK_ATTENTION) d.a[A_TICKET] = (int)(d.a[A_TICKET] * bank);
    return simulate_task_graph(*g, err);
  }
};

}  // namespace

void plan_silu_epilogue(const mpk_config &cfg, std::vector<TensorInfo> *tensors, std::vector<LayerInfo> *layers) {
  std::vector<TensorInfo> &T = *tensors;
  std::vector<LayerInfo> &L = *layers;
  auto uses = [&](const LayerInfo &l, int t) { for (int x : l.t) if (x == t) return true; return false; };
  for (size_t i = 0; i < L.size(); ++i) {
    LayerInfo &lin = L[i];
    if (lin.op != MPK_OP_LINEAR && lin.op != MPK_OP_RMSNORM_LINEAR) continue;
    const int wi = lin.op == MPK_OP_LINEAR ? 1 : 2, yi = lin.op == MPK_OP_LINEAR ? 2 : 3;
    if ((int)lin.t.size() <= yi || lin.t[wi] < 0 || lin.t[yi] < 0) continue;
    TensorInfo &w = T[lin.t[wi]];
    const int mid = lin.t[yi];
    if (w.owner != 3 || w.shuffle_src.size() != 2 || w.dims.size() != 2 || w.dtype != MPK_BF16 || T[mid].owner == 0) continue;
    const int64_t I = T[w.shuffle_src[0]].dim(0);
    if (T[w.shuffle_src[1]].dim(0) != I || w.dim(0) != 2 * I || I % 2 != 0) continue;
    // the weight may have no other user; the intermediate (often one buffer shared by all decoder layers) must
    // be read by exactly one silu_mul layer before anything defines it again
    auto output_of = [&](const LayerInfo &l) {
      switch (l.op) {
        case MPK_OP_LINEAR: case MPK_OP_SPLITK_LINEAR: return l.t.size() > 2 ? l.t[2] : -1;
        case MPK_OP_RMSNORM_LINEAR: case MPK_OP_LINEAR_RESIDUAL: return l.t.size() > 3 ? l.t[3] : -1;
        default: return -1;
      }
    };
    int silu = -1;
    bool ok = true;
    for (size_t j = 0; j < L.size() && ok; ++j)
      if (j != i && uses(L[j], lin.t[wi])) ok = false;
    for (size_t j = i + 1; j < L.size() && ok; ++j) {
      if (output_of(L[j]) == mid) break;                       // defined again: later readers see that value
      if (!uses(L[j], mid)) continue;
      if (L[j].op == MPK_OP_SILU_MUL && L[j].t[0] == mid && silu < 0) silu = (int)j;
      else ok = false;
    }
    if (!ok || silu < 0) continue;
    LayerInfo &s = L[silu];
    const TensorInfo &act = T[s.t[1]];
    if (std::max(s.grid[0], 1) != w.shuffle_groups || act.dims.size() != 2 || act.dim(1) != I || act.dtype != MPK_BF16) continue;
    (void)cfg;
    w.shuffle_groups = (int)(I / 2);      // 2 gate rows, then 2 up rows
    lin.silu_out = s.t[1];
    s.folded = true;
  }
}

int build_task_graph(GraphInputs in, CompiledGraph *out, std::string *err) {
  *out = CompiledGraph();
  Builder b(in, out, err);
  return b.run();
}

int simulate_task_graph(const CompiledGraph &g, std::string *err) {
  const int W = g.num_workers;
  std::vector<uint64_t> counters(g.num_events, 0);
  std::vector<int> pos(W);
  for (int w = 0; w < W; ++w) pos[w] = g.worker_begin[w];
  size_t done = 0;
  bool progress = true;
  while (progress) {
    progress = false;
    for (int w = 0; w < W; ++w) {
      while (pos[w] < g.worker_begin[w + 1]) {
        const TaskDesc &d = g.tasks[pos[w]];
        bool ready = true;
        for (int k = 0; k < kMaxDeps; ++k) {
          if (d.dep_event[k] < 0) continue;
          // a remote-triggered event also receives the peers' arrivals; count ours world times
          if (counters[d.dep_event[k]] < d.dep_need[k]) ready = false;
        }
        if (!ready) break;
        if (d.trig_event >= 0)
          // every rank runs the same graph: a remote-triggered arrival is mirrored by the peers
          counters[d.trig_event] += (d.flags & TF_REMOTE_TRIGGER) ? (uint64_t)g.world_size : 1ull;
        ++pos[w];
        ++done;
        progress = true;
      }
    }
  }
  if (done != g.tasks.size()) {
    std::ostringstream os;
    os << "task graph deadlocks in host simulation: " << done << " of " << g.tasks.size() << " tasks ran";
    for (int w = 0; w < W; ++w)
      if (pos[w] < g.worker_begin[w + 1]) {
        os << "; worker " << w << " stuck at task " << pos[w] << " (layer " << g.tasks[pos[w]].layer << ")";
        break;
      }
    *err = os.str();
    return MPK_ERR_DEADLOCK;
  }
  for (int e = 0; e < g.num_events; ++e) {
    uint64_t expect = (uint64_t)g.exec[e].num_tasks;
    if (g.exec[e].remote_trigger) expect *= (uint64_t)g.world_size;
    if (counters[e] != expect) {
      *err = "event " + std::to_string(e) + " fired " + std::to_string(counters[e]) + " times, expected " +
             std::to_string(expect);
      return MPK_ERR_DEADLOCK;
    }
  }
  return MPK_OK;
}

std::string dump_task_graph(const CompiledGraph &g, const std::vector<TensorInfo> &tensors,
                            const std::vector<LayerInfo> &layers) {
  static const char *names[] = {"nop", "batch", "embed", "rmsnorm", "linear", "attention", "silu_mul",
                                "argmax_partial", "argmax_reduce", "allreduce", "elementwise_add", "tensor_init",
                                "quantize_fp8", "moe_routing", "moe_gemm", "moe_silu_mul", "moe_mul_sum_add",
                                "mla_append", "mla_decode", "mla_reduce", "sampling_partial", "sampling_reduce", "argmax_exchange", "ar_push",
                                "embed_f32", "residual_norm", "linear_f32", "qkv_append", "ext_attention", "short_conv", "rglru", "mlstm",
                                "gla", "latent_append", "moe_gemm_f32", "attn_merge", "selective_scan", "diff_combine", "poly_norm"};
  std::ostringstream os;
  os << "{\"num_workers\": " << g.num_workers << ", \"num_tasks\": " << g.tasks.size()
     << ", \"num_events\": " << g.num_events << ", \"num_layers\": " << layers.size()
     << ", \"num_folded\": " << g.num_folded << ", \"num_stages\": " << g.num_stages << ", \"stage_bytes\": " << g.stage_bytes
     << ", \"x_tile_bytes\": " << g.x_tile_bytes << ", \"weight_bytes\": " << g.weight_bytes
     << ",\n \"events\": [\n";
  for (size_t e = 0; e < g.exec.size(); ++e) {
    const ExecLayer &x = g.exec[e];
    os << "  {\"event\": " << e << ", \"type\": \"" << names[x.type < sizeof(names) / sizeof(names[0]) ? x.type : 0] << "\", \"layer\": " << x.layer
       << ", \"tasks\": " << x.num_tasks << ", \"deps\": [";
    for (size_t k = 0; k < x.deps.size(); ++k) os << (k ? ", " : "") << "[" << x.deps[k] << ", " << x.dep_need[k] << "]";
    os << "]";
    if (x.layer >= 0 && layers[x.layer].prologue != PRO_PLAIN)
      os << ", \"prologue\": \"" << (layers[x.layer].prologue == PRO_RMSNORM ? "rmsnorm" : layers[x.layer].prologue == PRO_RESNORM ? "residual_norm" : layers[x.layer].prologue == PRO_POLY ? "poly_norm" : "silu_mul") << "\"";
    if (x.layer >= 0 && layers[x.layer].silu_out >= 0) os << ", \"epilogue\": \"silu_mul\"";
    if (x.layer >= 0 && layers[x.layer].op == MPK_OP_RESIDUAL_NORM && layers[x.layer].t.size() > 12 && layers[x.layer].t[12] >= 0) os << ", \"average\": true";
    if (x.remote_trigger) os << ", \"push\": true";
    if (x.tc_rows > 0) os << ", \"tcgen05\": {\"tile_rows\": " << x.tc_rows << ", \"k_blocks_per_slot\": " << x.tc_kblocks << "}";
    if (x.layer >= 0 && !layers[x.layer].t.empty()) {
      const LayerInfo &l = layers[x.layer];
      int out = l.t.back();
      if (out >= 0) os << ", \"out\": \"" << tensors[out].name << "\"";
    }
    os << "}" << (e + 1 < g.exec.size() ? ",\n" : "\n");
  }
  os << " ]}\n";
  return os.str();
}

}  // namespace mpk
