// The Rarelorn decoder: its configuration and its description as parts.
//
// config.json (`architecture`: "Rarelorn") lists the layers one by one; every size and constant is read from it, the rank of
// the low-rank decay input from the stored tensor's shape.  The stream starts as the token's row ("embed").  Every layer is
// pre-norm; its RMS norms have one gain for all channels, a tensor of a single number ("l<i>.norm1", "l<i>.norm2",
// "final.norm").  A layer names
//   type   "delta": the gated delta rule with a decay per head (parts/state_mixers.cc "gated_delta"), short convolutions and silu
//          on q, k and v;
//          "mlstm": a matrix memory with exponential gates ("matrix_memory");
//          "parallel": left_scale times sigmoid attention with biases, short convolutions, a rotation of part of each head,
//          a bounded score, a sliding window (parts/sigmoid_attention.cc), plus right_scale times time mixing with a bonus for the
//          current token ("time_mixing"), both on the same input;
//   mlp    null, or {kind "moe"}: experts down(silu(gate h) * up h) chosen by softmax scores among the best groups of experts (a
//          group's score: its largest), weighted by their scores times router.scale (parts/feed_forward.cc).
// `loop` {start, stop, times}: layers start .. stop-1 run `times` times in a row with the same weights, each pass with a cache
// and state of its own; before each pass but the first the token rows are added to the stream, before each pass row t of
// "loop.step" [times, width].  Last: the norm, then logits = head x.
#include <cmath>

#include "config/layered.h"

namespace llm {

namespace {

// What a model of this design can hold when the engine names no shorter bound: the configuration itself has no longest
// sequence.
const int64_t RARELORN_MAX_POSITIONS = 1 << 20;
// The design's constants.
const double UNIT_EPS = 1e-6;            // unit vectors of the delta rule: x / sqrt(sum x^2 + this)
const int64_t GROUP_TOP = 1;             // a group's score: its largest expert's

void heads_of(const ConfigReader &r, Json *m, bool groups, bool values) {
  const int64_t heads = r.integer("heads"), dim = r.integer("dim");
  m->set("heads", heads);
  m->set("dim", dim);
  if (groups) {
    const int64_t kv = r.integer_or("kv_heads", heads);
    if (heads % kv) r.fail("'heads' must be a multiple of 'kv_heads'");
    m->set("kv_heads", kv);
  }
  if (values) m->set("vdim", r.integer_or("vdim", dim));
}

Json parse_mixer(const Json &layer, const std::string &where) {
  ConfigReader lr(layer, where);
  const std::string type = lr.string("type");
  ConfigReader r(lr.object("mixer"), where + ": mixer");
  Json m = Json::object();
  if (type == "delta") {
    heads_of(r, &m, true, true);
    m.set("conv", r.integer_or("conv", 0, 0));
  } else if (type == "mlstm") {
    heads_of(r, &m, false, true);
    m.set("gate_cap", r.number("gate_cap"));
  } else if (type == "parallel") {
    ConfigReader l(r.object("left"), where + ": mixer.left"), rt(r.object("right"), where + ": mixer.right");
    Json left = Json::object(), right = Json::object();
    heads_of(l, &left, true, true);
    const int64_t dim = left.get("dim").as_int();
    left.set("conv", l.integer_or("conv", 0, 0));
    left.set("scale", l.number_or("scale", 1.0 / std::sqrt((double)dim), false));
    left.set("softcap", l.number_or("softcap", 0.0, false));
    left.set("rot", l.present("rot") ? parse_rot(l.object("rot"), where + ": mixer.left.rot", dim) : Json());
    left.set("mask", parse_mask(l, where + ": mixer.left"));
    heads_of(rt, &right, false, false);
    m.set("left", left);
    m.set("right", right);
    m.set("left_scale", r.number_or("left_scale", 1.0, false));
    m.set("right_scale", r.number_or("right_scale", 1.0, false));
  } else {
    lr.fail("mixer type '" + type + "' is not known (delta, mlstm, parallel)");
  }
  return m;
}

// config.json as read -> normal form: the same layout with every optional key present.
Json parse_rarelorn(const Json &data) {
  const std::string where = "config.json";
  ConfigReader r(data, where);
  Json c = Json::object();
  c.set("architecture", "Rarelorn");
  c.set("vocab", r.integer("vocab"));
  c.set("width", r.integer("width"));
  Json norm = Json::object();
  norm.set("eps", ConfigReader(r.object("norm"), where + ": norm").number("eps"));
  c.set("norm", norm);
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
    o.set("mlp", parse_mlp(l.get("mlp"), lw));
    if (o.get("mlp").is_object() && !o.get("mlp").get("shared").is_null())
      LLM_THROW(Config, "%s: mlp: this design has no shared expert", lw.c_str());
    ls.push(o);
  }
  c.set("layers", ls);
  c.set("loop", parse_loop(r, (int64_t)layers.size(), where));
  return c;
}

// tensor names of several matrices: "<key>" -> prefix + name
void names(Json *m, const std::string &prefix, std::initializer_list<std::pair<const char *, const char *>> list) {
  for (const auto &kv : list) m->set(kv.first, prefix + kv.second);
}

Json describe_delta(const Json &m, const std::string &x, int64_t width, double eps) {
  Json d = Json::object();
  d.set("kind", "gated_delta");
  d.set("hidden", width);
  d.set("n_heads", m.get("heads"));
  d.set("n_kv_heads", m.get("kv_heads"));
  d.set("head_dim", m.get("dim"));
  d.set("v_head_dim", m.get("vdim"));
  d.set("eps", eps);
  d.set("key_eps", UNIT_EPS);
  names(&d, x, {{"q", "q"}, {"k", "k"}, {"v", "v"}, {"g", "g"}, {"b", "b"}, {"a", "a"}, {"dt_bias", "dt_bias"}, {"A_log", "A_log"},
                {"norm", "norm"}, {"o", "o"}});
  if (m.get("conv").as_int() > 0) {
    d.set("taps", m.get("conv"));
    names(&d, x, {{"q_conv", "q.conv"}, {"k_conv", "k.conv"}, {"v_conv", "v.conv"}});
  }
  return d;
}

Json describe_mlstm(const Json &m, const std::string &x, int64_t width, double eps) {
  Json d = Json::object();
  d.set("kind", "matrix_memory");
  d.set("hidden", width);
  d.set("n_heads", m.get("heads"));
  d.set("head_dim", m.get("dim"));
  d.set("v_head_dim", m.get("vdim"));
  d.set("gate_cap", m.get("gate_cap"));
  d.set("eps", eps);
  names(&d, x, {{"q", "q"}, {"k", "k"}, {"v", "v"}, {"g", "g"}, {"i", "i"}, {"f", "f"}, {"i_bias", "i.b"}, {"f_bias", "f.b"},
                {"norm", "norm"}, {"o", "o"}});
  return d;
}

Json describe_parallel(const Json &m, const std::string &x, int64_t width, double eps) {
  const Json &l = m.get("left"), &r = m.get("right");
  Json left = Json::object(), right = Json::object();
  left.set("kind", "sigmoid_attention");
  left.set("hidden", width);
  left.set("n_heads", l.get("heads"));
  left.set("n_kv_heads", l.get("kv_heads"));
  left.set("head_dim", l.get("dim"));
  left.set("v_head_dim", l.get("vdim"));
  left.set("scale", l.get("scale"));
  left.set("softcap", l.get("softcap"));
  left.set("out_scale", m.get("left_scale"));
  if (!l.get("mask").get("size").is_null()) left.set("window", l.get("mask").get("size"));
  left.set("position", l.get("rot").is_null() ? Json() : rope_description(l.get("rot"), l.get("dim").as_int()));
  names(&left, x + "left.", {{"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}, {"q_bias", "q.b"}, {"k_bias", "k.b"}, {"v_bias", "v.b"},
                             {"o_bias", "o.b"}, {"temp", "temp"}, {"score_bias", "pb"}});
  if (l.get("conv").as_int() > 0) {
    left.set("taps", l.get("conv"));
    names(&left, x + "left.", {{"q_conv", "q.conv"}, {"k_conv", "k.conv"}, {"v_conv", "v.conv"}});
  }
  right.set("kind", "time_mixing");
  right.set("hidden", width);
  right.set("n_heads", r.get("heads"));
  right.set("head_dim", r.get("dim"));
  right.set("eps", eps);
  right.set("out_scale", m.get("right_scale"));
  names(&right, x + "right.", {{"mu_r", "mu.r"}, {"mu_k", "mu.k"}, {"mu_v", "mu.v"}, {"mu_g", "mu.g"}, {"mu_w", "mu.w"}, {"r", "r"}, {"k", "k"},
                               {"v", "v"}, {"g", "g"}, {"w1", "w1"}, {"w2", "w2"}, {"w0", "w0"}, {"u", "u"}, {"norm", "norm"}, {"o", "o"}});
  Json d = Json::object(), list = Json::array();
  list.push(left);
  list.push(right);
  d.set("kind", "sum");
  d.set("mixers", list);
  return d;
}

Json describe_experts(const Json &f, const std::string &p, int64_t width) {
  if (f.is_null()) return Json();
  const Json &ro = f.get("router");
  Json ff = Json::object();
  ff.set("kind", "moe");
  ff.set("hidden", width);
  ff.set("experts", ro.get("experts"));
  ff.set("top", ro.get("top"));
  ff.set("score", "softmax");
  ff.set("renormalize", false);
  ff.set("route_scale", ro.get("scale"));
  ff.set("weight_on", "output");
  ff.set("router", p + "router");
  if (!ro.get("groups").is_null()) {
    Json g = Json::object();
    g.set("count", ro.get("groups").get("count"));
    g.set("keep", ro.get("groups").get("keep"));
    g.set("top", GROUP_TOP);
    ff.set("groups", g);
  }
  Json e = Json::object();
  e.set("intermediate", f.get("expert").get("ff"));
  e.set("activation", "silu");
  e.set("gate", p + "e{}.gate");
  e.set("up", p + "e{}.up");
  e.set("down", p + "e{}.down");
  ff.set("expert", e);
  return ff;
}

ModelSpec describe_rarelorn(const Json &c) {
  const int64_t width = c.get("width").as_int();
  const double eps = c.get("norm").get("eps").as_number();
  auto norm = [&](const std::string &weight) {
    Json n = Json::object();
    n.set("kind", "rmsnorm");
    n.set("size", width);
    n.set("eps", eps);
    n.set("weight", weight);
    n.set("one_gain", true);                         // a single number for all channels
    return n;
  };
  ModelSpec s;
  s.name = "Rarelorn";
  s.vocab_size = c.get("vocab").as_int();
  s.hidden = width;
  s.embedding = "embed";
  s.head = "head";
  s.max_positions = RARELORN_MAX_POSITIONS;
  const Json &layers = c.get("layers");
  for (size_t i = 0; i < layers.size(); ++i) {
    const Json &l = layers.at(i);
    const Json &m = l.get("mixer");
    const std::string type = l.get("type").as_string(), p = "l" + std::to_string(i) + ".", x = p + "mix.";
    const Json ff = describe_experts(l.get("mlp"), p + "mlp.", width);
    Json block = Json::object();
    block.set("kind", "prenorm");
    block.set("hidden", width);
    block.set("mixer_norm", norm(p + "norm1"));
    block.set("mixer", type == "delta" ? describe_delta(m, x, width, eps) : type == "mlstm" ? describe_mlstm(m, x, width, eps)
                                                                                             : describe_parallel(m, x, width, eps));
    block.set("ff_norm", ff.is_null() ? Json() : norm(p + "norm2"));
    block.set("ff", ff);
    s.layers.push_back(block);
  }
  // the order of runs: the layers before the loop, the looped ones `times` times, the rest; what a pass adds to the
  // stream comes before its first layer
  const Json &loop = c.get("loop");
  const int64_t n = (int64_t)layers.size(), start = loop.get("start").as_int(), stop = loop.get("stop").as_int(),
                times = loop.get("times").as_int();
  for (int64_t i = 0; i < start; ++i) s.schedule.push_back({(int)i});
  for (int64_t t = 0; t < times; ++t)
    for (int64_t i = start; i < stop; ++i) {
      ScheduleEntry e;
      e.layer = (int)i;
      if (i == start) {
        e.add_tokens = t > 0;
        e.add_vector = "loop.step";
        e.add_row = (int)t;
      }
      s.schedule.push_back(e);
    }
  for (int64_t i = stop; i < n; ++i) s.schedule.push_back({(int)i});
  if (start == stop || times == 0) s.ignore_tensors.push_back("loop.step");    // an empty loop reads nothing of it
  s.final_norm = norm("final.norm");
  return s;
}

}  // namespace

void register_architecture_unlocked(Architecture arch);   // config/config.cc

void register_rarelorn_architecture() {
  Architecture a;
  a.name = "Rarelorn";
  a.parse = parse_rarelorn;
  a.describe = describe_rarelorn;
  register_architecture_unlocked(std::move(a));
}

}  // namespace llm
