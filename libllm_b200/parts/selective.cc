// "selective_scan": a mixer with a diagonal state per channel whose decay, input and read-out depend on the token
// (csrc/selective_scan.cu).  With h the mixer's input, `inner` channels, `state` numbers per channel:
//   [x | z] = W_in h;   x <- silu(conv(x) + conv_bias), a causal convolution over time per channel (`taps`)
//   [low (dt_rank) | B (state) | C (state)] = W_x x;   dt = softplus(W_dt low + dt_bias), one number per channel
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,  A = -exp(A_log);   y_c = sum_n S[c, n] C_n + D_c x_c
//   result W_o (y * silu(z))
// State per sequence and run: S [inner, state] and the convolution's last taps - 1 inputs, both 32-bit.  Everything from the
// products' 32-bit results to the input of the output projection is 32-bit; x is rounded to the engine's type once, for the products
// and the recurrence alike.  A prompt step is the convolution, two small products and the scan; a step of single tokens makes dt in
// the kernel that moves the state.  The reference has no such mixer.
#include <algorithm>

#include "config/config.h"
#include "csrc/kernels.h"
#include "parts/chain.h"
#include "parts/linear.h"
#include "parts/part.h"

namespace llm {

namespace {

const char *const SCAN_STATE = "selective_scan.S", *const SCAN_INPUTS = "selective_scan.inputs";

class SelectiveScan : public Mixer {
 public:
  SelectiveScan(const Json &spec, const BuildEnv &env) : Mixer(spec, env) {
    ConfigReader r(spec, "selective_scan description");
    hidden_ = r.integer("hidden");
    inner_ = r.integer("inner");
    state_ = (int)r.integer("state");
    rank_ = (int)r.integer("dt_rank");
    taps_ = (int)r.integer("taps");
    if (state_ > kernels::selective_max_state())
      LLM_THROW(Unsupported, "selective_scan: %d states a channel are not supported (up to %d)", state_, kernels::selective_max_state());
    if (taps_ > 8) LLM_THROW(Unsupported, "selective_scan: a convolution of %d taps is not supported (1 to 8)", taps_);
    for (const char *key : {"in", "conv", "conv_bias", "x", "dt", "dt_bias", "a_log", "skip", "o"}) names_.push_back(r.string(key));
    // columns of W_dt: whole pieces of 16 bytes for the tensor cores
    rank_cols_ = env.dtype == DType::BF16 ? (rank_ + 7) / 8 * 8 : rank_;
    low_rows_ = ((int64_t)rank_ + 2 * state_ + 7) / 8 * 8;
  }
  enum { IN, CONV, CONV_BIAS, X, DT, DT_BIAS, A_LOG, SKIP, O };

  std::vector<TensorNeed> tensor_needs() const override {
    auto vec = [](const std::string &name, std::vector<int64_t> shape) { return TensorNeed{name, std::move(shape), TensorRole::Vector, false}; };
    return {{names_[IN], {2 * inner_, hidden_}},
            vec(names_[CONV], {inner_, (int64_t)taps_}),
            vec(names_[CONV_BIAS], {inner_}),
            {names_[X], {(int64_t)rank_ + 2 * state_, inner_}},
            {names_[DT], {inner_, (int64_t)rank_}},
            vec(names_[DT_BIAS], {inner_}),
            vec(names_[A_LOG], {inner_, (int64_t)state_}),
            vec(names_[SKIP], {inner_}),
            {names_[O], {hidden_, inner_}}};
  }
  void load(const Loader &l) override {
    const std::vector<TensorNeed> needs = tensor_needs();
    const size_t es = dtype_size(l.engine);
    w_in_ = l.fetch(needs[IN]);
    w_o_ = l.fetch(needs[O]);
    // stored [channels, taps]; the kernel reads [taps, channels]
    Weight conv = l.fetch(needs[CONV]);
    std::vector<float> a((size_t)(inner_ * taps_)), b(a.size());
    LLM_CUDA(cudaMemcpy(a.data(), conv.buf.get(), a.size() * sizeof(float), cudaMemcpyDeviceToHost));
    for (int64_t c = 0; c < inner_; ++c)
      for (int j = 0; j < taps_; ++j) b[(size_t)(j * inner_ + c)] = a[(size_t)(c * taps_ + j)];
    conv_.buf.allocate(b.size() * sizeof(float));
    LLM_CUDA(cudaMemcpy(conv_.buf.get(), b.data(), b.size() * sizeof(float), cudaMemcpyHostToDevice));
    conv_bias_ = l.fetch(needs[CONV_BIAS]);
    w_x_.dtype = l.engine;
    w_x_.rows = low_rows_;
    w_x_.cols = inner_;
    w_x_.buf.allocate((size_t)(low_rows_ * inner_) * es, true);
    l.fetch_into(needs[X], l.engine, w_x_.buf.get());
    w_dt_.dtype = l.engine;
    w_dt_.rows = inner_;
    w_dt_.cols = rank_cols_;
    w_dt_.buf.allocate((size_t)(inner_ * rank_cols_) * es, true);
    DeviceBuffer staged((size_t)(inner_ * rank_) * es);
    l.fetch_into(needs[DT], l.engine, staged.get());
    LLM_CUDA(cudaMemcpy2D(w_dt_.buf.get(), (size_t)rank_cols_ * es, staged.get(), (size_t)rank_ * es, (size_t)rank_ * es, (size_t)inner_,
                          cudaMemcpyDeviceToDevice));
    dt_bias_ = l.fetch(needs[DT_BIAS]);
    a_log_ = l.fetch(needs[A_LOG]);
    skip_ = l.fetch(needs[SKIP]);
  }
  std::vector<std::string> kernel_families() const override {
    std::vector<std::string> fams = product_families(env_.dtype);
    fams.push_back("selective_scan");
    return fams;
  }
  std::vector<StateNeed> state_need() const override {
    std::vector<StateNeed> needs = {{SCAN_STATE, {inner_, (int64_t)state_}, DType::F32}};
    if (taps_ > 1) needs.push_back({SCAN_INPUTS, {(int64_t)taps_ - 1, inner_}, DType::F32});
    return needs;
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *, StateView *state) override {
    float *S = nullptr, *inputs = nullptr;
    if (state)
      for (const auto &t : *state) {
        if (t.name == SCAN_STATE) S = (float *)t.data;
        if (t.name == SCAN_INPUTS) inputs = (float *)t.data;
      }
    if (!S || (taps_ > 1 && !inputs)) LLM_THROW(InvalidArg, "selective_scan: the run has no state");
    const int T = ctx.n_tokens;
    Act proj = linear(ctx, x, w_in_, nullptr, DType::F32);
    flush_chain(ctx);
    const float *z = (const float *)proj.data + inner_;
    Act xc = ctx.arena->act(ctx.dtype, T, inner_);
    kernels::short_conv_silu(proj, conv_.buf.as<float>(), conv_bias_.buf.as<float>(), taps_, inputs, xc, ctx.tok_seq, ctx.tok_pos, ctx.seq_start,
                             ctx.seq_past, ctx.seq_slot, ctx.n_seqs, ctx.decode_only, ctx.stream);
    const bool single = ctx.decode_only && T == ctx.n_seqs;
    // partial products where the kernel behind adds them; not the room or the stream of the block's own result
    float *const pool = ctx.parts_pool, *const sink = ctx.residual_sink;
    ctx.parts_pool = ctx.residual_sink = nullptr;
    Act low = linear(ctx, xc, w_x_, nullptr, DType::F32, single);
    ctx.parts_pool = pool;
    ctx.residual_sink = sink;
    flush_chain(ctx);
    const int off_b = rank_, off_c = rank_ + state_;
    Act y = ctx.arena->act(ctx.dtype, T, inner_);
    if (single) {
      kernels::selective_step(xc, low, rank_, w_dt_, dt_bias_.buf.as<float>(), off_b, off_c, z, proj.ld, a_log_.buf.as<float>(),
                              skip_.buf.as<float>(), S, y, ctx.seq_slot, state_, ctx.stream);
    } else {
      Act dt_in = low;                         // the product's first columns, rounded where the engine rounds
      dt_in.cols = rank_cols_;
      if (ctx.dtype == DType::BF16) {
        dt_in = ctx.arena->act(DType::BF16, T, rank_cols_);
        kernels::rows_cast(low, rank_, dt_in, ctx.stream);
      }
      Act dt = linear(ctx, dt_in, w_dt_, nullptr, DType::F32);
      flush_chain(ctx);
      kernels::selective_scan(xc, dt, dt_bias_.buf.as<float>(), low, off_b, off_c, z, proj.ld, a_log_.buf.as<float>(), skip_.buf.as<float>(), S,
                              y, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, state_, ctx.stream);
    }
    return linear(ctx, y, w_o_, nullptr, DType::F32, true);
  }

 private:
  int64_t hidden_, inner_, low_rows_;
  int state_, rank_, rank_cols_, taps_;
  std::vector<std::string> names_;
  Weight w_in_, w_x_, w_dt_, w_o_, conv_, conv_bias_, dt_bias_, a_log_, skip_;
};

}  // namespace

void register_part_raw(const std::string &category, const std::string &kind, PartFactory factory);   // parts/part.cc

void register_selective_parts() {
  register_part_raw("mixer", "selective_scan",
                    [](const Json &spec, const BuildEnv &env) { return std::unique_ptr<Part>(new SelectiveScan(spec, env)); });
}

}  // namespace llm
