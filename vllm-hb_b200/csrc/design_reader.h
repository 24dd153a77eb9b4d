// Small pieces the readers of layered designs share.
#pragma once

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

}  // namespace hb
