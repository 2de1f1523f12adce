// The Fomodra decoder: its configuration and its description as parts.
//
// config.json (`architecture`: "Fomodra") lists the layers one by one; every size and constant is read from it.  The stream
// starts as the token's row ("embed") plus the row (previous * mul_prev + current * mul_cur) mod buckets of the table of token
// pairs ("bigram"; its last row for a sequence's first token).  Every layer norms both ends of its sublayers,
// x += norm1b(mixer(norm1 x)), x += norm2b(ff(norm2 x)) (RMS norms), and then adds the token's own slice of "side.embed" behind a
// gate the stream makes ("l<i>.side.*", parts/builtin.cc "side").  A layer names
//   type   "attention": grouped-query attention with biases on q, k, v, a rotation of the first rot.dims channels, a sliding window,
//          a learned sink per head; with kv_from it has no keys and values and reads those of the layer it names;
//          "latent_attention": queries from the input, keys and values through one normed latent plus a rotated key part that all
//          heads share (parts/latent.cc), a sliding window, a sink and a sigmoid gate per head;
//          "parallel": chunked attention ("left": visible are the keys of the query's own chunk of mask.size positions) beside a
//          selective scan ("right", parts/selective.cc), half the sum of the two results, each normed first;
//   mlp    null, or {kind "moe"}: experts with a bounded gated unit, chosen by softmax scores plus a correction, weighted by their
//          scores over their sum, the last router.identity choices giving the input back; plus a shared expert of the same form.
// Last: the norm, then logits = head x.
#include <algorithm>
#include <cmath>

#include "config/layered.h"

namespace llm {

namespace {

// What a model of this design can hold when the engine names no shorter bound: the configuration itself has no longest
// sequence.
const int64_t FOMODRA_MAX_POSITIONS = 1 << 20;
// The design's constants.
const double ROUTE_NORM_EPS = 1e-20;     // weights: s / (sum of the chosen s + this)
const double GLU_SLOPE = 1.702;          // the gated unit: g sigmoid(slope g) (u + shift)
const double GLU_SHIFT = 1.0;
const double PAIR_SCALE = 0.5;           // the parallel mixer: half the sum

Json parse_heads(const ConfigReader &r, const std::string &where) {
  Json m = Json::object();
  const int64_t heads = r.integer("heads"), dim = r.integer("dim"), kv = r.integer_or("kv_heads", heads);
  if (heads % kv) r.fail("'heads' must be a multiple of 'kv_heads'");
  m.set("heads", heads);
  m.set("kv_heads", kv);
  m.set("dim", dim);
  m.set("vdim", r.integer_or("vdim", dim));
  m.set("scale", r.number_or("scale", 1.0 / std::sqrt((double)dim), false));
  m.set("rot", r.present("rot") ? parse_rot(r.object("rot"), where + ".rot", dim) : Json());
  m.set("mask", parse_mask(r, where));
  return m;
}

Json parse_mixer(const Json &layer, const std::string &where) {
  ConfigReader lr(layer, where);
  const std::string type = lr.string("type"), mw = where + ": mixer";
  ConfigReader r(lr.object("mixer"), mw);
  if (type == "attention") {
    Json m = parse_heads(r, mw);
    m.set("kv_from", r.present("kv_from") ? Json(r.integer("kv_from", 0)) : Json());
    return m;
  }
  Json m = Json::object();
  if (type == "latent_attention") {
    const int64_t dim = r.integer("dim"), rot_dim = r.integer("rot_dim", 0);
    m.set("heads", r.integer("heads"));
    m.set("dim", dim);
    m.set("rot_dim", rot_dim);
    m.set("vdim", r.integer_or("vdim", dim));
    m.set("kv_rank", r.integer("kv_rank"));
    m.set("scale", r.number_or("scale", 1.0 / std::sqrt((double)(dim + rot_dim)), false));
    m.set("rot", Json());
    if (rot_dim > 0) {
      Json rot = parse_rot(r.object("rot"), mw + ".rot", rot_dim);
      if (rot.get("dims").as_int() != rot_dim) r.fail("'rot.dims' must equal 'rot_dim'");
      m.set("rot", rot);
    }
    m.set("mask", parse_mask(r, mw));
  } else if (type == "parallel") {
    ConfigReader l(r.object("left"), mw + ".left"), rt(r.object("right"), mw + ".right");
    Json right = Json::object();
    for (const char *key : {"inner", "state", "dt_rank", "conv"}) right.set(key, rt.integer(key));
    m.set("left", parse_heads(l, mw + ".left"));
    m.set("right", right);
  } else {
    lr.fail("mixer type '" + type + "' is not known (attention, latent_attention, parallel)");
  }
  return m;
}

// the gated unit's width and bound
Json parse_unit(const Json &raw, const std::string &where) {
  ConfigReader r(raw, where);
  Json u = Json::object();
  u.set("ff", r.integer("ff"));
  u.set("limit", r.number("limit"));
  return u;
}

Json parse_experts(const Json &raw, const std::string &where) {
  if (raw.is_null()) return Json();
  if (!raw.is_object()) LLM_THROW(Config, "%s: 'mlp' must be an object or null", where.c_str());
  const std::string mw = where + ": mlp";
  ConfigReader r(raw, mw);
  const std::string kind = r.string_or("kind", "moe");
  if (kind != "moe") r.fail("feed-forward kind '" + kind + "' is not known (moe)");
  Json m = Json::object();
  m.set("kind", kind);
  m.set("expert", parse_unit(r.object("expert"), mw + ".expert"));
  ConfigReader ro(r.object("router"), mw + ".router");
  Json router = Json::object();
  const int64_t experts = ro.integer("experts"), identity = ro.integer_or("identity", 0, 0), top = ro.integer("top");
  if (top > experts + identity) ro.fail("'top' exceeds 'experts' + 'identity'");
  router.set("experts", experts);
  router.set("identity", identity);
  router.set("top", top);
  m.set("router", router);
  m.set("shared", r.present("shared") ? parse_unit(r.object("shared"), mw + ".shared") : Json());
  return m;
}

// config.json as read -> normal form: the same layout with every optional key present.
Json parse_fomodra(const Json &data) {
  const std::string where = "config.json";
  ConfigReader r(data, where);
  Json c = Json::object();
  c.set("architecture", "Fomodra");
  c.set("vocab", r.integer("vocab"));
  c.set("width", r.integer("width"));
  Json norm = Json::object();
  norm.set("eps", ConfigReader(r.object("norm"), where + ": norm").number("eps"));
  c.set("norm", norm);
  Json embedding = Json::object();
  embedding.set("bigram", Json());
  if (r.present("embedding") && !r.object("embedding").get("bigram").is_null()) {
    ConfigReader b(r.object("embedding").get("bigram"), where + ": embedding.bigram");
    Json pair = Json::object();
    pair.set("buckets", b.integer("buckets"));
    pair.set("mul_prev", b.integer("mul_prev", 0));
    pair.set("mul_cur", b.integer("mul_cur", 0));
    embedding.set("bigram", pair);
  }
  c.set("embedding", embedding);
  Json side;
  if (r.present("token_side")) {
    side = Json::object();
    side.set("dim", ConfigReader(r.object("token_side"), where + ": token_side").integer("dim"));
  }
  c.set("token_side", side);
  const Json &layers = data.get("layers");
  if (!layers.is_array() || layers.size() == 0) r.fail("'layers' must be a list with at least one layer");
  Json ls = Json::array();
  for (size_t i = 0; i < layers.size(); ++i) {
    const std::string lw = where + ": layers[" + std::to_string(i) + "]";
    const Json &l = layers.at(i);
    if (!l.is_object()) LLM_THROW(Config, "%s must be an object", lw.c_str());
    Json o = Json::object();
    o.set("type", ConfigReader(l, lw).string("type"));
    o.set("mixer", parse_mixer(l, lw));
    o.set("mlp", parse_experts(l.get("mlp"), lw));
    const Json &from = o.get("mixer").get("kv_from");
    if (from.is_int()) {
      const int64_t j = from.as_int();
      if (j >= (int64_t)i) LLM_THROW(Config, "%s: mixer: 'kv_from' must name an earlier layer, found %lld", lw.c_str(), (long long)j);
      const Json &lender = ls.at((size_t)j);
      if (lender.get("type").as_string() != "attention" || !lender.get("mixer").get("kv_from").is_null())
        LLM_THROW(Config, "%s: mixer: 'kv_from' must name an attention layer with keys and values of its own", lw.c_str());
      for (const char *key : {"kv_heads", "dim", "vdim"})
        if (lender.get("mixer").get(key).as_int() != o.get("mixer").get(key).as_int())
          LLM_THROW(Config, "%s: mixer: '%s' differs from that of layer %lld, whose keys and values it reads", lw.c_str(), key, (long long)j);
    }
    ls.push(o);
  }
  c.set("layers", ls);
  return c;
}

// tensor names of several matrices: "<key>" -> prefix + name
void names(Json *m, const std::string &prefix, std::initializer_list<std::pair<const char *, const char *>> list) {
  for (const auto &kv : list) m->set(kv.first, prefix + kv.second);
}

Json describe_heads(const Json &m, int64_t width, const char *mask_key) {
  Json d = Json::object();
  d.set("kind", "attention");
  d.set("hidden", width);
  d.set("n_heads", m.get("heads"));
  d.set("n_kv_heads", m.get("kv_heads"));
  d.set("head_dim", m.get("dim"));
  d.set("v_head_dim", m.get("vdim"));
  d.set("scale", m.get("scale"));
  d.set("position", m.get("rot").is_null() ? Json() : rope_description(m.get("rot"), m.get("dim").as_int()));
  if (!m.get("mask").get("size").is_null()) d.set(mask_key, m.get("mask").get("size"));
  return d;
}

// cache_window: how many positions later layers read of this layer's keys and values (0: all)
Json describe_attention(const Json &m, const std::string &x, int64_t width, int64_t cache_window) {
  Json d = describe_heads(m, width, "window");
  d.set("bias", true);
  d.set("null_scores", x + "sink");
  names(&d, x, {{"q", "q"}, {"q_bias", "q.b"}, {"o", "o"}});
  if (m.get("kv_from").is_null()) {
    names(&d, x, {{"k", "k"}, {"v", "v"}, {"k_bias", "k.b"}, {"v_bias", "v.b"}});
    if (d.has("window")) d.set("cache_window", cache_window);
  }
  return d;
}

Json describe_latent(const Json &m, const std::string &x, int64_t width, double eps) {
  Json d = Json::object();
  d.set("kind", "latent_attention");
  d.set("hidden", width);
  d.set("n_heads", m.get("heads"));
  d.set("head_dim", m.get("dim"));
  d.set("rot_dim", m.get("rot_dim"));
  d.set("v_head_dim", m.get("vdim"));
  d.set("kv_rank", m.get("kv_rank"));
  d.set("scale", m.get("scale"));
  d.set("eps", eps);
  d.set("position", m.get("rot").is_null() ? Json() : rope_description(m.get("rot"), m.get("rot_dim").as_int()));
  if (!m.get("mask").get("size").is_null()) d.set("window", m.get("mask").get("size"));
  names(&d, x, {{"q", "q"}, {"kv_down", "dkv"}, {"kv_norm", "dkv.norm"}, {"k_up", "uk"}, {"v_up", "uv"}, {"null_scores", "sink"},
                {"head_gate", "g"}, {"o", "o"}});
  return d;
}

Json describe_parallel(const Json &m, const std::string &x, int64_t width, double eps) {
  Json left = describe_heads(m.get("left"), width, "block"), right = Json::object();
  names(&left, x + "left.", {{"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}});
  const Json &r = m.get("right");
  right.set("kind", "selective_scan");
  right.set("hidden", width);
  right.set("inner", r.get("inner"));
  right.set("state", r.get("state"));
  right.set("dt_rank", r.get("dt_rank"));
  right.set("taps", r.get("conv"));
  names(&right, x + "right.", {{"in", "in"}, {"conv", "conv"}, {"conv_bias", "conv.b"}, {"x", "x"}, {"dt", "dt"}, {"dt_bias", "dt.b"},
                               {"a_log", "A_log"}, {"skip", "D"}, {"o", "o"}});
  Json d = Json::object(), list = Json::array(), norms = Json::object(), weights = Json::array();
  list.push(left);
  list.push(right);
  weights.push(x + "left.out");
  weights.push(x + "right.out");
  norms.set("hidden", width);
  norms.set("eps", eps);
  norms.set("scale", PAIR_SCALE);
  norms.set("weights", weights);
  d.set("kind", "sum");
  d.set("mixers", list);
  d.set("norms", norms);
  return d;
}

Json describe_experts(const Json &f, const std::string &p, int64_t width) {
  if (f.is_null()) return Json();
  const Json &ro = f.get("router");
  Json ff = Json::object();
  ff.set("kind", "moe");
  ff.set("hidden", width);
  ff.set("experts", ro.get("experts"));
  ff.set("identity", ro.get("identity"));
  ff.set("top", ro.get("top"));
  ff.set("score", "softmax");
  ff.set("renormalize", true);
  ff.set("norm_eps", ROUTE_NORM_EPS);
  ff.set("weight_on", "output");
  ff.set("router", p + "router");
  ff.set("correction", p + "correction");
  Json e = Json::object();
  e.set("intermediate", f.get("expert").get("ff"));
  e.set("activation", "bounded_glu");
  e.set("limit", f.get("expert").get("limit"));
  e.set("slope", GLU_SLOPE);
  e.set("up_shift", GLU_SHIFT);
  names(&e, p, {{"gate", "e{}.gate"}, {"up", "e{}.up"}, {"down", "e{}.down"}});
  ff.set("expert", e);
  if (!f.get("shared").is_null()) {
    Json s = Json::object();
    s.set("kind", "clamped_glu");
    s.set("hidden", width);
    s.set("intermediate", f.get("shared").get("ff"));
    s.set("limit", f.get("shared").get("limit"));
    s.set("slope", GLU_SLOPE);
    s.set("up_shift", GLU_SHIFT);
    names(&s, p + "shared.", {{"gate", "gate"}, {"up", "up"}, {"down", "down"}});
    ff.set("shared", s);
  }
  return ff;
}

ModelSpec describe_fomodra(const Json &c) {
  const int64_t width = c.get("width").as_int();
  const double eps = c.get("norm").get("eps").as_number();
  auto norm = [&](const std::string &weight) {
    Json n = Json::object();
    n.set("kind", "rmsnorm");
    n.set("size", width);
    n.set("eps", eps);
    n.set("weight", weight);
    return n;
  };
  auto post = [&](const std::string &weight) {
    Json n = Json::object();
    n.set("weight", weight);
    n.set("eps", eps);
    return n;
  };
  ModelSpec s;
  s.name = "Fomodra";
  s.vocab_size = c.get("vocab").as_int();
  s.hidden = width;
  s.embedding = "embed";
  s.head = "head";
  s.max_positions = FOMODRA_MAX_POSITIONS;
  const Json &layers = c.get("layers"), &pair = c.get("embedding").get("bigram"), &side = c.get("token_side");
  if (!pair.is_null()) {
    s.token_pairs.table = "bigram";
    s.token_pairs.buckets = pair.get("buckets").as_int();
    s.token_pairs.mul_prev = pair.get("mul_prev").as_int();
    s.token_pairs.mul_cur = pair.get("mul_cur").as_int();
  }
  const int64_t side_dim = side.is_null() ? 0 : side.get("dim").as_int();
  if (side_dim > 0) {
    s.token_table = "side.embed";
    s.token_table_width = side_dim * (int64_t)layers.size();
  }
  // how far back each layer's keys and values are read: by itself and by the layers that borrow them (0: to the start)
  std::vector<int64_t> reach;
  for (size_t i = 0; i < layers.size(); ++i) {
    const Json &m = layers.at(i).get("mixer"), &size = m.get("mask").get("size"), &from = m.get("kv_from");
    const int64_t own = size.is_int() ? size.as_int() : 0;
    reach.push_back(own);
    if (from.is_int()) {
      int64_t &r = reach[(size_t)from.as_int()];
      r = r == 0 || own == 0 ? 0 : std::max(r, own);
    }
  }
  for (size_t i = 0; i < layers.size(); ++i) {
    const Json &l = layers.at(i), &m = l.get("mixer");
    const std::string type = l.get("type").as_string(), p = "l" + std::to_string(i) + ".", x = p + "mix.";
    const Json ff = describe_experts(l.get("mlp"), p + "mlp.", width);
    Json block = Json::object();
    block.set("kind", "prenorm");
    block.set("hidden", width);
    block.set("mixer_norm", norm(p + "norm1"));
    block.set("mixer", type == "attention" ? describe_attention(m, x, width, reach[i]) : type == "latent_attention" ? describe_latent(m, x, width, eps)
                                                                                                                     : describe_parallel(m, x, width, eps));
    block.set("mixer_post", post(p + "norm1b"));
    block.set("ff_norm", ff.is_null() ? Json() : norm(p + "norm2"));
    block.set("ff", ff);
    if (!ff.is_null()) {
      block.set("ff_post", post(p + "norm2b"));
    } else {                               // a layer without a feed-forward reads nothing of its norms
      s.ignore_tensors.push_back(p + "norm2");
      s.ignore_tensors.push_back(p + "norm2b");
    }
    if (side_dim > 0) {
      Json sd = Json::object();
      sd.set("dim", side_dim);
      sd.set("offset", side_dim * (int64_t)i);
      sd.set("eps", eps);
      names(&sd, p + "side.", {{"gate", "gate"}, {"proj", "proj"}, {"norm", "norm"}});
      block.set("side", sd);
    }
    s.layers.push_back(block);
    ScheduleEntry e;
    e.layer = (int)i;
    if (m.get("kv_from").is_int()) e.cache_from = (int)m.get("kv_from").as_int();
    s.schedule.push_back(e);
  }
  s.final_norm = norm("final.norm");
  return s;
}

}  // namespace

void register_architecture_unlocked(Architecture arch);   // config/config.cc

void register_fomodra_architecture() {
  Architecture a;
  a.name = "Fomodra";
  a.parse = parse_fomodra;
  a.describe = describe_fomodra;
  register_architecture_unlocked(std::move(a));
}

}  // namespace llm
