// Attention whose weights stand each for itself, and a mixer that adds the results of several.
//
// "sigmoid_attention": grouped-query attention over the paged cache without a softmax.  q, k, v = W h (+ bias), each through a
// short causal convolution over time per channel (`taps`; none without q_conv, k_conv, v_conv), then a rotation of the first
// position.rotary_dim channels of every q and k head in pairs (i, i + rotary_dim/2); score s = (q . k) scale temp[head],
// bounded by softcap (s <- cap tanh(s / cap); absent: not); a visible key's weight is sigmoid(s + score_bias[head]), weights are
// not normalised over the keys; causal, or the last `window` positions.  Values have a width of their own.  The output
// projection may have a bias.  `out_scale` (1): the whole result times it.  Biases are added where the convolution is
// computed (32-bit), so that the products run on the tensor cores; the convolution's last taps - 1 inputs are state of the run.
//
// "sum": a list of mixers that all read the same input; the result is the sum of theirs.  At most one keeps keys and values;
// state of all is kept side by side.  With `norms` {weights: a name per mixer, eps, scale}, of two mixers, the result is
// scale * sum_i y_i / sqrt(mean(y_i^2) + eps) * weight_i (32-bit, in the pass that adds it to the stream).
//
// Reference counterpart of the attention: src/libllm/llama.cc:178-225 (a softmax, no convolution); none of the sum.
#include <algorithm>
#include <cmath>

#include "config/config.h"
#include "csrc/kernels.h"
#include "parts/chain.h"
#include "parts/linear.h"
#include "parts/part.h"

namespace llm {

namespace {

const char *const CONV_INPUTS = "sigmoid_attention.inputs";

class SigmoidAttention : public Mixer {
 public:
  SigmoidAttention(const Json &spec, const BuildEnv &env) : Mixer(spec, env) {
    ConfigReader r(spec, "sigmoid_attention description");
    hidden_ = r.integer("hidden");
    n_heads_ = (int)r.integer("n_heads");
    n_kv_ = (int)r.integer_or("n_kv_heads", n_heads_);
    d_ = (int)r.integer("head_dim");
    dv_ = (int)r.integer_or("v_head_dim", d_);
    if (n_heads_ % n_kv_) r.fail("'n_heads' must be a multiple of 'n_kv_heads'");
    if (d_ > 1024 || dv_ > 1024) LLM_THROW(Unsupported, "sigmoid_attention: head sizes %d / %d are not supported (up to 1024)", d_, dv_);
    window_ = (int)r.integer_or("window", 0, 0);
    scale_ = (float)r.number_or("scale", 1.0 / std::sqrt((double)d_), false);
    cap_ = (float)r.number_or("softcap", 0.0, false);
    if (cap_ < 0.f) r.fail("'softcap' must not be negative");
    out_scale_ = (float)r.number_or("out_scale", 1.0, false);
    for (const char *key : {"q", "k", "v", "o"}) names_.push_back(r.string(key));
    for (const char *key : {"q_bias", "k_bias", "v_bias"}) bias_names_.push_back(r.string_or(key, ""));
    o_bias_name_ = r.string_or("o_bias", "");
    temp_name_ = r.string_or("temp", "");
    score_bias_name_ = r.string_or("score_bias", "");
    has_conv_ = r.present("q_conv");
    taps_ = has_conv_ ? (int)r.integer("taps") : 1;
    if (taps_ > 8) LLM_THROW(Unsupported, "sigmoid_attention: a convolution of %d taps is not supported (1 to 8)", taps_);
    if (has_conv_)
      for (const char *key : {"q_conv", "k_conv", "v_conv"}) conv_names_.push_back(r.string(key));
    if (!spec.get("position").is_null()) position_ = build_as<PositionEncoding>("position", spec.get("position"), env);
    widths_[0] = (int64_t)n_heads_ * d_;
    widths_[1] = (int64_t)n_kv_ * d_;
    widths_[2] = (int64_t)n_kv_ * dv_;
    channels_ = widths_[0] + widths_[1] + widths_[2];
  }
  TensorNeed vector_need(const std::string &name, int64_t n) const { return {name, {n}, TensorRole::Vector, false}; }
  std::vector<TensorNeed> tensor_needs() const override {
    std::vector<TensorNeed> needs;
    for (int i = 0; i < 3; ++i) needs.push_back({names_[(size_t)i], {widths_[i], hidden_}});
    needs.push_back({names_[3], {hidden_, (int64_t)n_heads_ * dv_}});
    for (int i = 0; i < 3; ++i)
      if (!bias_names_[(size_t)i].empty()) needs.push_back(vector_need(bias_names_[(size_t)i], widths_[i]));
    if (!o_bias_name_.empty()) needs.push_back(vector_need(o_bias_name_, hidden_));
    if (!temp_name_.empty()) needs.push_back(vector_need(temp_name_, n_heads_));
    if (!score_bias_name_.empty()) needs.push_back(vector_need(score_bias_name_, n_heads_));
    for (size_t i = 0; i < conv_names_.size(); ++i) needs.push_back({conv_names_[i], {widths_[i], (int64_t)taps_}, TensorRole::Vector, false});
    if (position_)
      for (auto &n : position_->tensor_needs()) needs.push_back(n);
    return needs;
  }
  void load(const Loader &l) override {
    const size_t es = dtype_size(l.engine);
    w_qkv_.dtype = l.engine;
    w_qkv_.rows = (channels_ + 7) / 8 * 8;
    w_qkv_.cols = hidden_;
    w_qkv_.buf.allocate((size_t)w_qkv_.rows * (size_t)hidden_ * es, true);
    bias_.buf.allocate((size_t)channels_ * sizeof(float), true);
    std::vector<float> conv((size_t)taps_ * (size_t)channels_, 1.f), one;
    int64_t at = 0;
    for (int i = 0; i < 3; ++i) {
      l.fetch_into({names_[(size_t)i], {widths_[i], hidden_}}, l.engine, (char *)w_qkv_.buf.get() + (size_t)at * (size_t)hidden_ * es);
      if (!bias_names_[(size_t)i].empty()) l.fetch_into(vector_need(bias_names_[(size_t)i], widths_[i]), DType::F32, bias_.buf.as<float>() + at);
      if (has_conv_) {                                 // stored [channels, taps]; the kernel reads [taps, channels]
        Weight w = l.fetch({conv_names_[(size_t)i], {widths_[i], (int64_t)taps_}, TensorRole::Vector, false});
        one.resize((size_t)(widths_[i] * taps_));
        LLM_CUDA(cudaMemcpy(one.data(), w.buf.get(), one.size() * sizeof(float), cudaMemcpyDeviceToHost));
        for (int64_t c = 0; c < widths_[i]; ++c)
          for (int j = 0; j < taps_; ++j) conv[(size_t)(j * channels_ + at + c)] = one[(size_t)(c * taps_ + j)];
      }
      at += widths_[i];
    }
    conv_.buf.allocate(conv.size() * sizeof(float));
    LLM_CUDA(cudaMemcpy(conv_.buf.get(), conv.data(), conv.size() * sizeof(float), cudaMemcpyHostToDevice));
    w_o_ = l.fetch({names_[3], {hidden_, (int64_t)n_heads_ * dv_}});
    temp_ = per_head(l, temp_name_, 1.f);
    score_bias_ = per_head(l, score_bias_name_, 0.f);
    if (!o_bias_name_.empty()) {                       // the result's scale goes on its bias once, here
      o_bias_ = l.fetch(vector_need(o_bias_name_, hidden_));
      std::vector<float> host((size_t)hidden_);
      LLM_CUDA(cudaMemcpy(host.data(), o_bias_.buf.get(), host.size() * sizeof(float), cudaMemcpyDeviceToHost));
      for (auto &v : host) v *= out_scale_;
      LLM_CUDA(cudaMemcpy(o_bias_.buf.get(), host.data(), host.size() * sizeof(float), cudaMemcpyHostToDevice));
    }
    if (position_) position_->load(l);
  }
  std::vector<std::string> kernel_families() const override {
    std::vector<std::string> fams = product_families(env_.dtype);
    fams.push_back("rope");
    fams.push_back(tiled(env_.page_size) ? "attention_sigmoid" : "attention_generic");
    return fams;
  }
  bool wants_cache() const override { return true; }
  CacheNeed cache_need() const override {
    CacheNeed n;
    n.kind = window_ > 0 ? "window" : "full";
    n.n_kv_heads = n_kv_;
    n.k_dim = d_;
    n.v_dim = dv_;
    n.window = window_;
    return n;
  }
  std::vector<StateNeed> state_need() const override {
    if (taps_ < 2) return {};
    return {{CONV_INPUTS, {(int64_t)taps_ - 1, channels_}, DType::F32}};
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *cache, StateView *state) override {
    if (!cache) LLM_THROW(InvalidArg, "sigmoid_attention: the run has no cache to attend over");
    float *inputs = nullptr;
    if (state)
      for (const auto &t : *state)
        if (t.name == CONV_INPUTS) inputs = (float *)t.data;
    if (taps_ > 1 && !inputs) LLM_THROW(InvalidArg, "sigmoid_attention: the run has no state");
    int table_rows = 0, rot_dim = 0;
    const float *table = position_ ? position_->half_split_table(&table_rows, &rot_dim) : nullptr;
    if (position_ && !table) LLM_THROW(Unsupported, "sigmoid_attention: the position part has no half-split table");
    Act qkv = linear(ctx, x, w_qkv_, nullptr, DType::F32);
    flush_chain(ctx);
    Act q = ctx.arena->act(ctx.dtype, ctx.n_tokens, widths_[0]);
    kernels::conv_rope_place(qkv, bias_.buf.as<float>(), conv_.buf.as<float>(), taps_, inputs, q, n_heads_, n_kv_, d_, dv_, table, table_rows,
                             rot_dim, ctx.tok_seq, ctx.tok_pos, ctx.seq_start, ctx.seq_past, ctx.seq_slot, ctx.n_seqs, cache->page_table,
                             cache->table_width, cache->k, cache->v, cache->page_size, cache->writes, ctx.decode_only, ctx.stream);
    Act out = ctx.arena->act(ctx.dtype, ctx.n_tokens, (int64_t)n_heads_ * dv_);
    attend(ctx, q, out, *cache);
    if (o_bias_name_.empty()) return linear(ctx, out, w_o_, nullptr, DType::F32, true);
    // with a bias the product cannot add to the stream as it stores: the bias goes with the result
    float *const sink = ctx.residual_sink;
    ctx.residual_sink = nullptr;
    Act y = linear(ctx, out, w_o_, nullptr, DType::F32, true);
    ctx.residual_sink = sink;
    y.col_bias = o_bias_.buf.as<float>();
    return y;
  }

 private:
  // bfloat16 heads that both tensor-core kernels take; all else is the general kernel's
  bool tiled(int page_size) const {
    return env_.dtype == DType::BF16 && fast_switches().prefill_attention_tc && page_size == 64 && d_ % 16 == 0 && d_ <= 128 && dv_ % 16 == 0 &&
           dv_ <= 256 && n_heads_ / n_kv_ <= 16;
  }
  void attend(StepContext &ctx, const Act &q, const Act &out, LayerCache &cache) const {
    const float *temp = temp_.buf.as<float>(), *bias = score_bias_.buf.as<float>();
    if (!tiled(cache.page_size)) {
      kernels::attention_generic_sigmoid(q, out, cache.k, cache.v, ctx.tok_seq, ctx.tok_pos, cache.page_table, cache.table_width, n_heads_,
                                         n_kv_, d_, dv_, cache.page_size, window_, scale_, temp, bias, cap_, out_scale_, ctx.stream);
    } else if (ctx.decode_only) {
      // as many runs of pages as fill the GPU once, at the longest length the step's shape allows
      const int longest = window_ > 0 ? std::min(ctx.max_kv_len, window_ + cache.page_size) : ctx.max_kv_len;
      const int pages = std::max(1, (longest + cache.page_size - 1) / cache.page_size), pairs = std::max(1, ctx.n_seqs * n_kv_);
      int n_splits = std::max(1, std::min(ctx.sm_count * kernels::sigmoid_decode_ctas_per_sm(d_, dv_) / pairs, pages));
      if (pairs > ctx.n_zero_counters) n_splits = 1;
      float *ws = n_splits > 1 ? ctx.arena->alloc_n<float>((size_t)ctx.n_seqs * n_heads_ * dv_ * n_splits) : nullptr;
      kernels::sigmoid_decode(q, out, cache.k, cache.v, ctx.tok_pos, cache.page_table, cache.table_width, n_heads_, n_kv_, d_, dv_,
                              cache.page_size, window_, scale_, temp, bias, cap_, out_scale_, n_splits, ws, ctx.zero_counters, ctx.stream);
    } else {
      kernels::sigmoid_prefill(q, out, cache.k, cache.v, cache.n_pages, ctx.seq_start, ctx.seq_past, cache.page_table, cache.table_width,
                               ctx.n_seqs, ctx.max_q_len, n_heads_, n_kv_, d_, dv_, cache.page_size, window_, scale_, temp, bias, cap_,
                               out_scale_, ctx.tc_status, ctx.stream);
    }
  }
  Weight per_head(const Loader &l, const std::string &name, float fallback) const {
    if (!name.empty()) return l.fetch(vector_need(name, n_heads_));
    Weight w;
    w.rows = 1;
    w.cols = n_heads_;
    w.buf.allocate((size_t)n_heads_ * sizeof(float));
    const std::vector<float> host((size_t)n_heads_, fallback);
    LLM_CUDA(cudaMemcpy(w.buf.get(), host.data(), host.size() * sizeof(float), cudaMemcpyHostToDevice));
    return w;
  }
  int64_t hidden_, channels_, widths_[3];
  int n_heads_, n_kv_, d_, dv_, window_, taps_ = 1;
  bool has_conv_;
  float scale_, cap_, out_scale_;
  std::vector<std::string> names_, bias_names_, conv_names_;
  std::string o_bias_name_, temp_name_, score_bias_name_;
  std::unique_ptr<PositionEncoding> position_;
  Weight w_qkv_, w_o_, bias_, conv_, temp_, score_bias_, o_bias_;
};

// ---------------------------------------------------------------- the sum of several mixers
class SumMixer : public Mixer {
 public:
  SumMixer(const Json &spec, const BuildEnv &env) : Mixer(spec, env) {
    const Json &list = spec.get("mixers");
    if (!list.is_array() || list.size() == 0) LLM_THROW(Config, "sum description: 'mixers' must be a list with at least one mixer");
    int caches = 0;
    for (const auto &m : list.items()) {
      mixers_.push_back(build_as<Mixer>("mixer", m, env));
      caches += mixers_.back()->wants_cache() ? 1 : 0;
    }
    if (caches > 1) LLM_THROW(Unsupported, "sum: %d of the mixers keep keys and values (a run has one cache)", caches);
    if (!spec.get("norms").is_null()) {
      ConfigReader r(spec.get("norms"), "sum description: norms");
      hidden_ = r.integer("hidden");
      eps_ = (float)r.number("eps");
      scale_ = (float)r.number_or("scale", 1.0, false);
      const Json &names = spec.get("norms").get("weights");
      if (!names.is_array() || names.size() != mixers_.size()) r.fail("'weights' must name a vector per mixer");
      if (mixers_.size() != 2) LLM_THROW(Unsupported, "sum: results with norms of their own are of two mixers (%zu given)", mixers_.size());
      for (const auto &n : names.items()) norm_names_.push_back(n.as_string());
    }
  }
  std::vector<TensorNeed> tensor_needs() const override {
    std::vector<TensorNeed> out;
    for (const auto &m : mixers_)
      for (auto &n : m->tensor_needs()) out.push_back(n);
    for (const auto &n : norm_names_) out.push_back({n, {hidden_}, TensorRole::Vector, false});
    return out;
  }
  void load(const Loader &l) override {
    for (auto &m : mixers_) m->load(l);
    norms_.clear();
    for (const auto &n : norm_names_) norms_.push_back(l.fetch({n, {hidden_}, TensorRole::Vector, false}));
  }
  std::vector<std::string> kernel_families() const override {
    std::vector<std::string> out = {"elementwise"};
    for (const auto &m : mixers_)
      for (auto &f : m->kernel_families()) out.push_back(f);
    return out;
  }
  bool capturable() const override {
    for (const auto &m : mixers_)
      if (!m->capturable()) return false;
    return true;
  }
  bool wants_cache() const override {
    for (const auto &m : mixers_)
      if (m->wants_cache()) return true;
    return false;
  }
  CacheNeed cache_need() const override {
    for (const auto &m : mixers_)
      if (m->wants_cache()) return m->cache_need();
    return CacheNeed();
  }
  static std::string prefix(size_t i) { return std::to_string(i) + ":"; }
  std::vector<StateNeed> state_need() const override {
    std::vector<StateNeed> out;
    for (size_t i = 0; i < mixers_.size(); ++i)
      for (auto n : mixers_[i]->state_need()) {
        n.name = prefix(i) + n.name;
        out.push_back(n);
      }
    return out;
  }
  Act forward(StepContext &ctx, const Act &x, LayerCache *cache, StateView *state) override {
    // Steps of few tokens hand back partial products: room where all mixers' parts lie one behind the other, so that the next
    // norm adds them in one pass (an outer block may have given such room already).
    constexpr int POOL_PARTS = 16;
    const bool normed = !norm_names_.empty(), few = ctx.dtype == DType::BF16 && x.rows <= fast_switches().tc_tokens;
    const bool own_pool = !ctx.parts_pool && (few || normed) && !ctx.chain;
    if (own_pool) {
      ctx.parts_cap = few ? POOL_PARTS : (int)mixers_.size();
      ctx.parts_pool = ctx.arena->alloc_n<float>((size_t)ctx.parts_cap * (size_t)(x.rows * x.cols));
      ctx.parts_used = 0;
      ctx.parts_rows = x.rows;
      ctx.parts_cols = x.cols;
    }
    Act sum, added;
    if (normed) ctx.residual_sink = nullptr;             // a normed result cannot be added by the product that makes it
    float *const sink = ctx.residual_sink;
    int first_parts = 0;
    for (size_t i = 0; i < mixers_.size(); ++i) {
      StateView mine;
      const std::string p = prefix(i);
      if (state)
        for (const auto &t : *state)
          if (t.name.compare(0, p.size(), p) == 0) {
            mine.push_back(t);
            mine.back().name = t.name.substr(p.size());
          }
      Act r = mixers_[i]->forward(ctx, x, mixers_[i]->wants_cache() ? cache : nullptr, mine.empty() ? nullptr : &mine);
      if (sink && r.data == (void *)sink) {            // on the stream already
        added = r;
        continue;
      }
      if (normed && (r.col_bias || r.normed())) LLM_THROW(Unsupported, "sum: a result that is normed comes without a bias or a norm of its own");
      if (i == 0) first_parts = r.parts;
      sum = sum.data ? joined(ctx, sum, r) : r;
    }
    if (normed) {
      sum.first_parts = first_parts;
      for (int i = 0; i < 2; ++i) sum.pair_w[i] = norms_[(size_t)i].buf.as<float>();
      sum.pair_eps = eps_;
      sum.pair_scale = scale_;
    }
    if (own_pool) ctx.parts_pool = nullptr;
    return sum.data ? sum : added;
  }

 private:
  // Two results as one run of parts.
  static Act joined(StepContext &ctx, const Act &a, const Act &b) {
    if (a.dtype != DType::F32 || b.dtype != DType::F32 || a.rows != b.rows || a.cols != b.cols || a.ld != a.cols || b.ld != b.cols || a.col_scale ||
        b.col_scale || (a.col_bias && b.col_bias))
      LLM_THROW(Unsupported, "sum: the mixers' results must be dense 32-bit rows without scales, with a bias on one of them at most");
    Act s = a;
    s.parts = a.parts + b.parts;
    if (b.col_bias) s.col_bias = b.col_bias;
    const int64_t stride = a.rows * a.cols;
    const bool adjacent = (const float *)b.data == (const float *)a.data + (size_t)a.parts * (size_t)stride &&
                          (a.parts == 1 || a.part_stride == stride) && (b.parts == 1 || b.part_stride == stride);
    s.part_stride = stride;
    if (adjacent) return s;
    flush_chain(ctx);
    Act out = ctx.arena->act(DType::F32, a.rows, a.cols, s.parts);
    s.data = out.data;
    s.part_stride = out.part_stride;
    for (int p = 0; p < s.parts; ++p) {
      const Act &from = p < a.parts ? a : b;
      const int q = p < a.parts ? p : p - a.parts;
      LLM_CUDA(cudaMemcpyAsync((float *)out.data + (size_t)p * (size_t)out.part_stride, (const float *)from.data + (size_t)q * (size_t)from.part_stride,
                               sizeof(float) * (size_t)stride, cudaMemcpyDeviceToDevice, ctx.stream));
    }
    return s;
  }
  std::vector<std::unique_ptr<Mixer>> mixers_;
  std::vector<std::string> norm_names_;
  std::vector<Weight> norms_;
  int64_t hidden_ = 0;
  float eps_ = 0.f, scale_ = 1.f;
};

template <typename T>
PartFactory factory_of() {
  return [](const Json &spec, const BuildEnv &env) { return std::unique_ptr<Part>(new T(spec, env)); };
}

}  // namespace

void register_part_raw(const std::string &category, const std::string &kind, PartFactory factory);   // parts/part.cc

void register_sigmoid_parts() {
  register_part_raw("mixer", "sigmoid_attention", factory_of<SigmoidAttention>());
  register_part_raw("mixer", "sum", factory_of<SumMixer>());
}

}  // namespace llm
