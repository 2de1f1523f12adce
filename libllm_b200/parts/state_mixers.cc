// Mixers whose state is a matrix per head, carried through a linear recurrence (csrc/state_scan.cu), in three rules.
// With h the mixer's input, d key and dv value channels, everything from the products' 32-bit results to the input of the
// output projection in 32-bit:
//
// "gated_delta": q = W_q h, k = W_k h (G key heads; head i reads key head i / (H / G)), v = W_v h (H heads); each through a short
//   causal convolution over time per channel (`taps`; none without q_conv, k_conv, v_conv) and silu; q and k unit vectors,
//   x / sqrt(sum x^2 + key_eps), q also times d^(-1/2); beta = sigmoid(W_b h), g = exp(-exp(A_log) softplus(W_a h + dt_bias)), one
//   number per head;  S <- g S;  z = beta (v - S^T k);  S <- S + k z^T;  o = S^T q.  Result W_o (o / rms(o) * norm * silu(W_g h)), norm
//   over dv values that the heads share.  ("channel_delta" in parts/recurrent.cc has a decay per key channel.)
// "time_mixing": with h' the token before (nought at first), r, k, v, gate and decay input each read h + (h' - h) mu of their own;
//   w = exp(-exp(w0 + W_2 tanh(W_1 m_w))) per key channel;  o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T.  Result
//   W_o (o / rms(o) * norm * silu(W_g m_g)), norm over all heads' values.
// "matrix_memory": log gates i = cap tanh((W_i h + b_i) / cap), f = logsigmoid(cap tanh((W_f h + b_f) / cap)) per head; with a
//   running maximum m (0 at the start), m' = max(f + m, i): S <- exp(f + m - m') S + exp(i - m') k v^T, n likewise with k alone,
//   o = S^T q / (max(|n . q|, exp(-m')) + 1e-6), q times d^(-1/2).  Result W_o (o / rms(o) * norm * sigmoid(W_g h)).
//
// rms(o) = sqrt(mean(o^2) + eps) per head.  `out_scale` (1): the mixer's result is multiplied by it (in 32-bit, before the
// output projection's input is rounded).  A prompt step packs its tokens' vectors, scans them and norms; a step of single
// tokens is one launch between the products.  The reference has no such mixers.
#include <algorithm>
#include <cmath>

#include "config/config.h"
#include "csrc/kernels.h"
#include "parts/chain.h"
#include "parts/linear.h"
#include "parts/part.h"

namespace llm {

namespace {

// Several matrices of one width as one: rows in multiples of 8, so that rows of the 32-bit product start on 32 bytes.
void stack_rows(const Loader &l, const std::vector<TensorNeed> &needs, int64_t hidden, Weight *w) {
  const size_t es = dtype_size(l.engine);
  int64_t rows = 0;
  for (const auto &n : needs) rows += n.shape[0];
  w->dtype = l.engine;
  w->rows = (rows + 7) / 8 * 8;
  w->cols = hidden;
  w->buf.allocate((size_t)w->rows * (size_t)hidden * es, true);
  int64_t at = 0;
  for (const auto &n : needs) {
    l.fetch_into(n, l.engine, (char *)w->buf.get() + (size_t)at * (size_t)hidden * es);
    at += n.shape[0];
  }
}

void *state_of(StateView *state, const std::string &name) {
  if (state)
    for (const auto &t : *state)
      if (t.name == name) return t.data;
  return nullptr;
}

class StateMixer : public Mixer {
 public:
  StateMixer(const Json &spec, const BuildEnv &env, const char *what) : Mixer(spec, env) {
    ConfigReader r(spec, std::string(what) + " description");
    hidden_ = r.integer("hidden");
    n_heads_ = (int)r.integer("n_heads");
    n_kv_ = (int)r.integer_or("n_kv_heads", n_heads_);
    d_ = (int)r.integer("head_dim");
    dv_ = (int)r.integer_or("v_head_dim", d_);
    eps_ = (float)r.number("eps");
    out_scale_ = (float)r.number_or("out_scale", 1.0, false);
    if (n_heads_ % n_kv_) r.fail("'n_heads' must be a multiple of 'n_kv_heads'");
    if (d_ > 256) LLM_THROW(Unsupported, "%s: heads of %d key channels are not supported (up to 256)", what, d_);
    if (dv_ > 512) LLM_THROW(Unsupported, "%s: heads of %d value channels are not supported (up to 512)", what, dv_);
    q_width_ = (int64_t)n_kv_ * d_;
    v_width_ = (int64_t)n_heads_ * dv_;
    q_scale_ = (float)(1.0 / std::sqrt((double)d_));
  }
  std::vector<std::string> kernel_families() const override {
    std::vector<std::string> fams = product_families(env_.dtype);
    fams.push_back("state_scan");
    return fams;
  }

 protected:
  // room for what a step's tokens bring to the scan: `vectors` per key head, `columns` of values per head
  kernels::ScanPack pack_room(StepContext &ctx, int vectors, int columns) const {
    const size_t T = (size_t)ctx.n_tokens;
    const int per = kernels::scan_columns(d_), slices = (columns + per - 1) / per;
    kernels::ScanPack p;
    p.rec = ctx.arena->alloc_n<float>(T * (size_t)(n_kv_ * vectors * kernels::scan_padded(d_)));
    p.scal = ctx.arena->alloc_n<float>(T * (size_t)(n_heads_ * 4));
    p.vals = ctx.arena->alloc_n<float>(T * (size_t)(n_heads_ * slices * per));
    return p;
  }
  bool single_step(const StepContext &ctx, int rank) const {
    return ctx.decode_only && ctx.n_tokens == ctx.n_seqs && kernels::state_step_supported(d_, dv_, n_heads_ / n_kv_, rank);
  }
  int64_t hidden_, q_width_, v_width_;
  int n_heads_, n_kv_, d_, dv_;
  float eps_, out_scale_, q_scale_;
};

// ---------------------------------------------------------------- gated delta rule, a decay per head
class GatedDelta : public StateMixer {
 public:
  GatedDelta(const Json &spec, const BuildEnv &env) : StateMixer(spec, env, "gated_delta") {
    ConfigReader r(spec, "gated_delta description");
    key_eps_ = (float)r.number_or("key_eps", 1e-6);
    for (const char *key : {"q", "k", "v", "g", "b", "a", "dt_bias", "A_log", "norm", "o"}) names_.push_back(r.string(key));
    has_conv_ = r.present("q_conv");
    taps_ = has_conv_ ? (int)r.integer("taps") : 1;
    if (taps_ > 8) LLM_THROW(Unsupported, "gated_delta: a convolution of %d taps is not supported (1 to 8)", taps_);
    if (has_conv_)
      for (const char *key : {"q_conv", "k_conv", "v_conv"}) conv_names_.push_back(r.string(key));
    conv_width_ = 2 * q_width_ + v_width_;
  }
  enum { Q, K, V, G, B, A, DT_BIAS, A_LOG, NORM, O };

  std::vector<TensorNeed> tensor_needs() const override {
    const int64_t H = n_heads_;
    std::vector<TensorNeed> needs = {{names_[Q], {q_width_, hidden_}}, {names_[K], {q_width_, hidden_}}, {names_[V], {v_width_, hidden_}},
                                     {names_[G], {v_width_, hidden_}}, {names_[B], {H, hidden_}}, {names_[A], {H, hidden_}}};
    needs.push_back({names_[DT_BIAS], {H}, TensorRole::Vector, false});
    needs.push_back({names_[A_LOG], {H}, TensorRole::Vector, false});
    needs.push_back({names_[NORM], {(int64_t)dv_}, TensorRole::Vector, false});
    needs.push_back({names_[O], {hidden_, v_width_}});
    for (size_t i = 0; i < conv_names_.size(); ++i)
      needs.push_back({conv_names_[i], {i < 2 ? q_width_ : v_width_, (int64_t)taps_}, TensorRole::Vector, false});
    return needs;
  }
  void load(const Loader &l) override {
    const std::vector<TensorNeed> needs = tensor_needs();
    stack_rows(l, {needs[Q], needs[K], needs[V], needs[G], needs[B], needs[A]}, hidden_, &w_in_);
    dt_bias_ = l.fetch(needs[DT_BIAS]);
    a_log_ = l.fetch(needs[A_LOG]);
    norm_ = l.fetch(needs[NORM]);
    w_o_ = l.fetch(needs[O]);
    // the three convolutions' weights one behind the other, as their channels lie in a row of the product
    conv_.buf.allocate((size_t)conv_width_ * taps_ * sizeof(float), true);
    if (has_conv_) {
      int64_t at = 0;
      for (size_t i = 0; i < 3; ++i) {
        const TensorNeed &n = needs[O + 1 + i];
        l.fetch_into(n, DType::F32, conv_.buf.as<float>() + at * taps_);
        at += n.shape[0];
      }
    } else {
      kernels::add_scalar(conv_.buf.as<float>(), conv_width_, 1.f, nullptr);   // one tap of weight 1: the activation alone
    }
  }
  std::vector<std::string> kernel_families() const override {
    std::vector<std::string> fams = StateMixer::kernel_families();
    fams.push_back("elementwise");
    return fams;
  }
  std::vector<StateNeed> state_need() const override {
    std::vector<StateNeed> needs = {{"gated_delta.S", {(int64_t)n_heads_, (int64_t)dv_, (int64_t)d_}, DType::F32}};
    if (taps_ > 1) needs.push_back({"gated_delta.inputs", {(int64_t)taps_ - 1, conv_width_}, DType::F32});
    return needs;
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *, StateView *state) override {
    float *S = (float *)state_of(state, "gated_delta.S"), *inputs = (float *)state_of(state, "gated_delta.inputs");
    if (!S || (taps_ > 1 && !inputs)) LLM_THROW(InvalidArg, "gated_delta: the run has no state");
    Act proj = linear(ctx, x, w_in_, nullptr, DType::F32);
    flush_chain(ctx);
    const int T = ctx.n_tokens;
    const int off_k = (int)q_width_, off_v = 2 * off_k, off_g = off_v + (int)v_width_, off_b = off_g + (int)v_width_, off_a = off_b + n_heads_;
    Act y = ctx.arena->act(ctx.dtype, T, v_width_);
    if (single_step(ctx, 0)) {
      kernels::delta_gated_step(proj, 0, off_k, off_v, off_g, off_b, off_a, conv_.buf.as<float>(), inputs, taps_, dt_bias_.buf.as<float>(),
                                a_log_.buf.as<float>(), key_eps_, q_scale_, S, norm_.buf.as<float>(), true, kernels::GateSilu, eps_,
                                out_scale_, y, ctx.seq_slot, n_heads_, n_kv_, d_, dv_, ctx.stream);
      return linear(ctx, y, w_o_, nullptr, DType::F32, true);
    }
    const kernels::ScanPack pack = pack_room(ctx, 2, dv_);
    kernels::delta_pack(proj, off_b, off_a, conv_.buf.as<float>(), taps_, inputs, dt_bias_.buf.as<float>(), a_log_.buf.as<float>(), key_eps_,
                        q_scale_, pack, ctx.tok_seq, ctx.tok_pos, ctx.seq_start, ctx.seq_past, ctx.seq_slot, ctx.n_seqs, n_heads_, n_kv_, d_,
                        dv_, ctx.decode_only, ctx.stream);
    Act o = ctx.arena->act(DType::F32, T, v_width_);
    kernels::state_scan(kernels::ScanDelta, pack, S, o, nullptr, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, n_heads_, n_kv_, d_, dv_,
                        ctx.tc_status, ctx.stream);
    kernels::head_finish(o, nullptr, pack.scal, norm_.buf.as<float>(), true, (const float *)proj.data + off_g, proj.ld, kernels::GateSilu, eps_,
                         out_scale_, n_heads_, dv_, y, ctx.stream);
    return linear(ctx, y, w_o_, nullptr, DType::F32, true);
  }

 private:
  int64_t conv_width_;
  int taps_ = 1;
  bool has_conv_;
  float key_eps_;
  std::vector<std::string> names_, conv_names_;
  Weight w_in_, w_o_, conv_, dt_bias_, a_log_, norm_;
};

// ---------------------------------------------------------------- time mixing
class TimeMixing : public StateMixer {
 public:
  TimeMixing(const Json &spec, const BuildEnv &env) : StateMixer(spec, env, "time_mixing") {
    ConfigReader r(spec, "time_mixing description");
    if (n_kv_ != n_heads_) r.fail("'n_kv_heads' must equal 'n_heads'");
    rank_ = r.integer_or("decay_rank", -1);           // -1: the size w1 is stored with
    for (const char *key : {"mu_r", "mu_k", "mu_v", "mu_g", "mu_w", "r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o"})
      names_.push_back(r.string(key));
  }
  enum { MU, R = 5, K, V, G, W1, W2, W0, U, NORM, O };
  static constexpr int N_MIX = 5;

  std::vector<TensorNeed> tensor_needs() const override {
    std::vector<TensorNeed> needs;
    for (int i = 0; i < N_MIX; ++i) needs.push_back({names_[(size_t)(MU + i)], {hidden_}, TensorRole::Vector, false, 0.5f});
    needs.push_back({names_[R], {q_width_, hidden_}});
    needs.push_back({names_[K], {q_width_, hidden_}});
    needs.push_back({names_[V], {v_width_, hidden_}});
    needs.push_back({names_[G], {v_width_, hidden_}});
    needs.push_back({names_[W1], {rank_, hidden_}});
    needs.push_back({names_[W2], {q_width_, rank_}, TensorRole::Vector, false});
    needs.push_back({names_[W0], {q_width_}, TensorRole::Vector, false});
    needs.push_back({names_[U], {(int64_t)n_heads_, (int64_t)d_}, TensorRole::Vector, false});
    needs.push_back({names_[NORM], {v_width_}, TensorRole::Vector, false});
    needs.push_back({names_[O], {hidden_, v_width_}});
    return needs;
  }
  void load(const Loader &l) override {
    if (rank_ < 0) {
      const std::vector<int64_t> stored = l.shape_of(names_[W1]);
      rank_ = stored.size() == 2 ? stored[0] : DRAWN_FREE_SIZE;
    }
    const std::vector<TensorNeed> needs = tensor_needs();
    mu_.buf.allocate((size_t)N_MIX * (size_t)hidden_ * sizeof(float));
    for (int i = 0; i < N_MIX; ++i) l.fetch_into(needs[(size_t)i], DType::F32, mu_.buf.as<float>() + (size_t)i * hidden_);
    // the five matrices one behind the other, each but the last padded to whole tiles of the grouped product
    group_n_ = (std::max(q_width_, v_width_) + 127) / 128 * 128;
    const size_t row = (size_t)hidden_ * dtype_size(l.engine);
    w_all_.dtype = l.engine;
    w_all_.rows = (N_MIX - 1) * group_n_ + (rank_ + 7) / 8 * 8;
    w_all_.cols = hidden_;
    w_all_.buf.allocate((size_t)w_all_.rows * row, true);
    for (int i = 0; i < N_MIX; ++i) {
      const TensorNeed &n = needs[(size_t)(R + i)];
      w_[i].dtype = l.engine;
      w_[i].rows = n.shape[0];
      w_[i].cols = hidden_;
      w_[i].view = (char *)w_all_.buf.get() + (size_t)(i * group_n_) * row;
      l.fetch_into(n, l.engine, w_[i].view);
    }
    w2_ = l.fetch(needs[W2]);
    w0_ = l.fetch(needs[W0]);
    u_ = l.fetch(needs[U]);
    norm_ = l.fetch(needs[NORM]);
    w_o_ = l.fetch(needs[O]);
  }
  std::vector<StateNeed> state_need() const override {
    return {{"time_mixing.S", {(int64_t)n_heads_, (int64_t)dv_, (int64_t)d_}, DType::F32}, {"time_mixing.previous", {hidden_}, env_.dtype}};
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *, StateView *state) override {
    float *S = (float *)state_of(state, "time_mixing.S");
    void *previous = state_of(state, "time_mixing.previous");
    if (!S || !previous) LLM_THROW(InvalidArg, "time_mixing: the run has no state");
    flush_chain(ctx);
    const int T = ctx.n_tokens;
    Act mixed = ctx.arena->act(ctx.dtype, (int64_t)N_MIX * T, hidden_);
    kernels::token_shift(x, mu_.buf.as<float>(), N_MIX, mixed, previous, ctx.tok_seq, ctx.tok_pos, ctx.seq_start, ctx.seq_past,
                         ctx.seq_slot, ctx.n_seqs, ctx.decode_only, ctx.stream);
    Act in[N_MIX];
    const FastSwitches &f = fast_switches();
    if (ctx.dtype == DType::BF16 && f.gemm_tc && T <= f.tc_tokens && group_n_ * (N_MIX - 1) < w_all_.rows && w_all_.rows <= group_n_ * N_MIX &&
        hidden_ % 8 == 0) {
      // few tokens: the five products in one launch
      Act all = ctx.arena->act(DType::F32, T, w_all_.rows);
      kernels::gemm_tc_grouped(mixed, w_all_, all, N_MIX, (int)group_n_, ctx.tc_status, ctx.stream);
      for (int i = 0; i < N_MIX; ++i) {
        in[i] = all;
        in[i].cols = w_[i].rows;
        in[i].data = (float *)all.data + (size_t)(i * group_n_);
      }
    } else {
      for (int i = 0; i < N_MIX; ++i) {
        Act m = mixed;
        m.rows = T;
        m.data = (char *)mixed.data + (size_t)i * (size_t)T * (size_t)hidden_ * dtype_size(ctx.dtype);
        in[i] = linear(ctx, m, w_[i], nullptr, DType::F32);
      }
    }
    flush_chain(ctx);
    Act y = ctx.arena->act(ctx.dtype, T, v_width_);
    if (single_step(ctx, (int)rank_)) {
      kernels::bonus_step(in[0], in[1], in[2], in[3], in[4], (int)rank_, w2_.buf.as<float>(), w0_.buf.as<float>(), u_.buf.as<float>(), S,
                          norm_.buf.as<float>(), kernels::GateSilu, eps_, out_scale_, y, ctx.seq_slot, n_heads_, d_, dv_, ctx.stream);
      return linear(ctx, y, w_o_, nullptr, DType::F32, true);
    }
    const kernels::ScanPack pack = pack_room(ctx, 3, dv_);
    kernels::bonus_pack(in[0], in[1], in[2], in[4], (int)rank_, w2_.buf.as<float>(), w0_.buf.as<float>(), u_.buf.as<float>(), pack, n_heads_, d_,
                        dv_, ctx.stream);
    Act o = ctx.arena->act(DType::F32, T, v_width_);
    kernels::state_scan(kernels::ScanBonus, pack, S, o, nullptr, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, n_heads_, n_heads_, d_, dv_,
                        ctx.tc_status, ctx.stream);
    kernels::head_finish(o, nullptr, pack.scal, norm_.buf.as<float>(), false, (const float *)in[3].data, in[3].ld, kernels::GateSilu, eps_,
                         out_scale_, n_heads_, dv_, y, ctx.stream);
    return linear(ctx, y, w_o_, nullptr, DType::F32, true);
  }

 private:
  int64_t rank_, group_n_ = 0;
  std::vector<std::string> names_;
  Weight mu_, w_all_, w_[N_MIX], w2_, w0_, u_, norm_, w_o_;
};

// ---------------------------------------------------------------- matrix memory
class MatrixMemory : public StateMixer {
 public:
  MatrixMemory(const Json &spec, const BuildEnv &env) : StateMixer(spec, env, "matrix_memory") {
    ConfigReader r(spec, "matrix_memory description");
    if (n_kv_ != n_heads_) r.fail("'n_kv_heads' must equal 'n_heads'");
    cap_ = (float)r.number("gate_cap");
    for (const char *key : {"q", "k", "v", "g", "i", "f", "i_bias", "f_bias", "norm", "o"}) names_.push_back(r.string(key));
  }
  enum { Q, K, V, G, I, F, I_BIAS, F_BIAS, NORM, O };

  std::vector<TensorNeed> tensor_needs() const override {
    const int64_t H = n_heads_;
    std::vector<TensorNeed> needs = {{names_[Q], {q_width_, hidden_}}, {names_[K], {q_width_, hidden_}}, {names_[V], {v_width_, hidden_}},
                                     {names_[G], {v_width_, hidden_}}, {names_[I], {H, hidden_}}, {names_[F], {H, hidden_}}};
    needs.push_back({names_[I_BIAS], {H}, TensorRole::Vector, false});
    needs.push_back({names_[F_BIAS], {H}, TensorRole::Vector, false});
    needs.push_back({names_[NORM], {v_width_}, TensorRole::Vector, false});
    needs.push_back({names_[O], {hidden_, v_width_}});
    return needs;
  }
  void load(const Loader &l) override {
    const std::vector<TensorNeed> needs = tensor_needs();
    stack_rows(l, {needs[Q], needs[K], needs[V], needs[G], needs[I], needs[F]}, hidden_, &w_in_);
    i_bias_ = l.fetch(needs[I_BIAS]);
    f_bias_ = l.fetch(needs[F_BIAS]);
    norm_ = l.fetch(needs[NORM]);
    w_o_ = l.fetch(needs[O]);
  }
  // a head's columns of S, then n: [heads, dv + 1, d]
  std::vector<StateNeed> state_need() const override {
    return {{"matrix_memory.S", {(int64_t)n_heads_, (int64_t)dv_ + 1, (int64_t)d_}, DType::F32}, {"matrix_memory.m", {(int64_t)n_heads_}, DType::F32}};
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *, StateView *state) override {
    float *S = (float *)state_of(state, "matrix_memory.S"), *m = (float *)state_of(state, "matrix_memory.m");
    if (!S || !m) LLM_THROW(InvalidArg, "matrix_memory: the run has no state");
    Act proj = linear(ctx, x, w_in_, nullptr, DType::F32);
    flush_chain(ctx);
    const int T = ctx.n_tokens;
    const int off_k = (int)q_width_, off_v = 2 * off_k, off_g = off_v + (int)v_width_, off_i = off_g + (int)v_width_, off_f = off_i + n_heads_;
    Act y = ctx.arena->act(ctx.dtype, T, v_width_);
    if (single_step(ctx, 0)) {
      kernels::memory_step(proj, 0, off_k, off_v, off_g, off_i, off_f, i_bias_.buf.as<float>(), f_bias_.buf.as<float>(), cap_, q_scale_, m, S,
                           norm_.buf.as<float>(), kernels::GateSigmoid, eps_, out_scale_, y, ctx.seq_slot, n_heads_, d_, dv_, ctx.stream);
      return linear(ctx, y, w_o_, nullptr, DType::F32, true);
    }
    const kernels::ScanPack pack = pack_room(ctx, 2, dv_ + 1);
    float *den = ctx.arena->alloc_n<float>((size_t)T * n_heads_);
    kernels::memory_pack(proj, 0, off_k, off_v, off_i, off_f, i_bias_.buf.as<float>(), f_bias_.buf.as<float>(), cap_, q_scale_, m, pack,
                         ctx.seq_start, ctx.seq_slot, ctx.n_seqs, n_heads_, d_, dv_, ctx.stream);
    Act o = ctx.arena->act(DType::F32, T, v_width_);
    kernels::state_scan(kernels::ScanMemory, pack, S, o, den, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, n_heads_, n_heads_, d_, dv_,
                        ctx.tc_status, ctx.stream);
    kernels::head_finish(o, den, pack.scal, norm_.buf.as<float>(), false, (const float *)proj.data + off_g, proj.ld, kernels::GateSigmoid, eps_,
                         out_scale_, n_heads_, dv_, y, ctx.stream);
    return linear(ctx, y, w_o_, nullptr, DType::F32, true);
  }

 private:
  float cap_;
  std::vector<std::string> names_;
  Weight w_in_, i_bias_, f_bias_, norm_, w_o_;
};

template <typename T>
PartFactory factory_of() {
  return [](const Json &spec, const BuildEnv &env) { return std::unique_ptr<Part>(new T(spec, env)); };
}

}  // namespace

void register_part_raw(const std::string &category, const std::string &kind, PartFactory factory);   // parts/part.cc

void register_state_parts() {
  register_part_raw("mixer", "gated_delta", factory_of<GatedDelta>());
  register_part_raw("mixer", "time_mixing", factory_of<TimeMixing>());
  register_part_raw("mixer", "matrix_memory", factory_of<MatrixMemory>());
}

}  // namespace llm
