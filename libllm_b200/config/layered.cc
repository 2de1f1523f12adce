#include "config/layered.h"

#include <cmath>

namespace llm {

Json parse_rot(const Json &raw, const std::string &where, int64_t head_dim) {
  ConfigReader r(raw, where);
  Json rot = Json::object();
  const int64_t dims = r.integer("dims");
  if (dims % 2 || dims > head_dim) r.fail("'dims' must be even and at most the rotated head's size");
  rot.set("dims", dims);
  rot.set("base", r.number("base"));
  if (r.present("scaling")) {
    ConfigReader s(r.object("scaling"), where + ".scaling");
    Json sc = Json::object();
    sc.set("factor", s.number("factor"));
    sc.set("original", s.number("original"));
    if (s.present("low") || s.present("high")) {
      sc.set("low", s.number("low"));
      sc.set("high", s.number("high"));
    } else {
      sc.set("fast", s.number("fast"));
      sc.set("slow", s.number("slow"));
    }
    rot.set("scaling", sc);
  } else {
    rot.set("scaling", Json());
  }
  return rot;
}

Json parse_mask(const ConfigReader &r, const std::string &where) {
  Json mask = Json::object();
  mask.set("size", r.present("mask") ? Json(ConfigReader(r.object("mask"), where + ".mask").integer("size")) : Json());
  return mask;
}

Json parse_mlp(const Json &raw, const std::string &where) {
  if (raw.is_null()) return Json();
  if (!raw.is_object()) LLM_THROW(Config, "%s: 'mlp' must be an object or null", where.c_str());
  ConfigReader r(raw, where + ": mlp");
  const std::string kind = r.string_or("kind", "moe");
  if (kind != "moe") r.fail("feed-forward kind '" + kind + "' is not known (moe)");
  Json m = Json::object();
  m.set("kind", kind);
  Json expert = Json::object();
  expert.set("ff", ConfigReader(r.object("expert"), where + ": mlp.expert").integer("ff"));
  m.set("expert", expert);
  ConfigReader ro(r.object("router"), where + ": mlp.router");
  Json router = Json::object();
  const int64_t experts = ro.integer("experts"), top = ro.integer("top");
  if (top > experts) ro.fail("'top' exceeds 'experts'");
  router.set("experts", experts);
  router.set("top", top);
  router.set("scale", ro.number_or("scale", 1.0, false));
  if (ro.present("groups")) {
    ConfigReader g(ro.object("groups"), where + ": mlp.router.groups");
    Json groups = Json::object();
    const int64_t count = g.integer("count"), keep = g.integer("keep");
    if (experts % count) g.fail("'count' must divide 'experts'");
    if (keep > count) g.fail("'keep' exceeds 'count'");
    if (keep * (experts / count) < top) g.fail("the kept groups hold fewer experts than 'top'");
    groups.set("count", count);
    groups.set("keep", keep);
    router.set("groups", groups);
  } else {
    router.set("groups", Json());
  }
  m.set("router", router);
  if (r.present("shared")) {
    Json shared = Json::object();
    shared.set("ff", ConfigReader(r.object("shared"), where + ": mlp.shared").integer("ff"));
    m.set("shared", shared);
  } else {
    m.set("shared", Json());
  }
  return m;
}

Json parse_loop(const ConfigReader &r, int64_t n, const std::string &where) {
  Json loop = Json::object();
  if (r.present("loop")) {
    ConfigReader lp(r.object("loop"), where + ": loop");
    const int64_t start = lp.integer("start", 0), stop = lp.integer("stop", 0), times = lp.integer_or("times", 1, 0);
    if (start > stop || stop > n) lp.fail("'start' <= 'stop' <= the number of layers");
    loop.set("start", start);
    loop.set("stop", stop);
    loop.set("times", times);
  } else {
    loop.set("start", (int64_t)0);
    loop.set("stop", (int64_t)0);
    loop.set("times", (int64_t)1);
  }
  return loop;
}

Json rope_description(const Json &rot, int64_t head_dim) {
  Json p = Json::object();
  p.set("kind", "rope");
  p.set("head_dim", head_dim);
  p.set("rotary_dim", rot.get("dims"));
  p.set("theta", rot.get("base"));
  p.set("pairing", "half");                         // channel i goes with channel i + dims/2
  const Json &sc = rot.get("scaling");
  if (sc.is_null()) {
    p.set("scaling", Json());
  } else {
    Json y = Json::object();
    if (sc.has("low")) {
      y.set("rope_type", "llama3");
      y.set("factor", sc.get("factor"));
      y.set("original_max_position_embeddings", sc.get("original"));
      y.set("low_freq_factor", sc.get("low"));
      y.set("high_freq_factor", sc.get("high"));
      p.set("scaling", y);
      return p;
    }
    y.set("rope_type", "yarn");
    y.set("factor", sc.get("factor"));
    y.set("original_max_position_embeddings", sc.get("original"));
    y.set("beta_fast", sc.get("fast"));
    y.set("beta_slow", sc.get("slow"));
    y.set("magnitude", 0.1 * std::log(sc.get("factor").as_number()) + 1.0);   // on cosines and sines alike
    p.set("scaling", y);
  }
  return p;
}

}  // namespace llm
