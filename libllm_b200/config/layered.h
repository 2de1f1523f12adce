// Pieces of config.json that designs which list their layers one by one have in common (config/tazizen.cc,
// config/rarelorn.cc, config/fomodra.cc): each checks what it reads and returns it in normal form, every key present.
#pragma once
#include "config/config.h"

namespace llm {

// {dims, base, scaling {factor, original, fast, slow} (a ramp over the pairs), {factor, original, low, high} (by wavelength) or
// absent}; dims even and at most head_dim
Json parse_rot(const Json &raw, const std::string &where, int64_t head_dim);
// the mixer's `mask` {size}, or no key at all -> {size: number or null}
Json parse_mask(const ConfigReader &r, const std::string &where);
// null, or {kind "moe", expert {ff}, router {experts, top, scale, groups {count, keep}}, shared {ff}}
Json parse_mlp(const Json &raw, const std::string &where);
// `loop` {start, stop, times} of the configuration r reads; without the key an empty loop run once
Json parse_loop(const ConfigReader &r, int64_t n_layers, const std::string &where);
// parse_rot's result as the description of a "rope" position part (pairs i, i + dims/2)
Json rope_description(const Json &rot, int64_t head_dim);

}  // namespace llm
