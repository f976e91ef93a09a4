// Tables of a routed feed-forward pass, shared by its kernels.
#pragma once
#include <stdint.h>

namespace zse {

// One token tile of the grouped products: rows [row0, row0 + rows) of the rows sorted by expert belong to `group`.
struct MoeTile {
  int group, row0, rows, pad;
};

}  // namespace zse
