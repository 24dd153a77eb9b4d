// Small pieces the readers of layered designs share.
#pragma once

#include <algorithm>
#include <cmath>
#include <string>
#include <utility>

#include "json.h"
#include "layered.h"

namespace hb {

inline int64_t int_of(const Json* j, const char* key) {
  const double v = j ? j->number_or(key, 0) : 0;
  return v > -1e15 && v < 1e15 ? (int64_t)v : 0;
}
inline const Json* object_of(const Json& j, const char* key) {
  const Json* o = j.get(key);
  return o && o->kind == Json::Obj ? o : nullptr;
}
// The next rows of the layer's input projection (parts begin at multiples of 8).
inline void place(ProjPart* p, std::string tensor, int64_t rows, int64_t* offset) {
  p->tensor = std::move(tensor);
  p->rows = rows;
  p->offset = *offset;
  *offset = (*offset + rows + 7) / 8 * 8;
}
// Frequencies base^(-2i / dims) of the channel pairs (i, i + dims / 2), or (not halves) (2i, 2i + 1).
// Scaling by a factor alone divides them all.  `ramped` (YaRN): pairs that turn more than `fast` times
// within `original` positions keep theirs, those that turn less than `slow` times are divided, a ramp over
// the pair's number lies between them, and sines and cosines grow with the logarithm of the factor.
inline int read_rotation(const Json* rot, const std::string& t, int width, bool ramped, bool halves, AttentionSpec* a) {
  const double pi = 3.14159265358979323846;
  const double base = rot->number_or("base", 0);
  const int64_t dims = int_of(rot, "dims");
  if (base <= 0 || dims < 0 || dims % 2 || dims > width) return fail(HB_ERR_INVALID_ARG, "%s: bad rotation", t.c_str());
  const Json* s = object_of(*rot, "scaling");
  const double factor = s ? s->number_or("factor", 0) : 1;
  if (!(factor > 0)) return fail(HB_ERR_INVALID_ARG, "%s: bad rotation scaling", t.c_str());
  a->rotation_halves = halves;
  double lo = 0, hi = 0;
  const bool ramp = ramped && s;
  if (ramp) {
    const double original = s->number_or("original", 0), fast = s->number_or("fast", 0), slow = s->number_or("slow", 0);
    if (!(original > 0) || !(fast > 0) || !(slow > 0) || base == 1) return fail(HB_ERR_INVALID_ARG, "%s: bad rotation scaling", t.c_str());
    auto pair_of = [&](double turns) { return (double)dims * std::log(original / (2.0 * pi * turns)) / (2.0 * std::log(base)); };
    lo = std::max(std::floor(pair_of(fast)), 0.0);
    hi = std::min(std::ceil(pair_of(slow)), (double)dims - 1.0);
    a->rotation_gain = (float)(0.1 * std::log(factor) + 1.0);
  }
  for (int64_t i = 0; i < dims / 2; ++i) {
    const double f = std::pow(base, -2.0 * (double)i / (double)dims);
    const double slowed = ramp ? std::min(1.0, std::max(0.0, ((double)i - lo) / std::max(hi - lo, 0.001))) : 1.0;
    a->rotation.push_back(f / factor * slowed + f * (1.0 - slowed));
  }
  return HB_OK;
}

}  // namespace hb
