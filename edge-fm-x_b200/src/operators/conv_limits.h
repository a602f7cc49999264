// Input convolutions: rows a thread of the many-row form walks, and the widest filter (a filter reaches back kConvRows rows at most, so
// that only an entry's first chunk of rows needs what the sequence keeps).
#pragma once

namespace efm {
constexpr int kConvRows = 16, kMaxConvTaps = 16;
}  // namespace efm
