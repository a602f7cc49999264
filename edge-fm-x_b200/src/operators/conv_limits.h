// Input convolutions: rows a thread of the many-row form walks, and the widest filter (a filter reaches back as many rows at most, so
// that only an entry's first chunk of rows needs what the sequence keeps).
#pragma once

namespace efm {
constexpr int kConvRows = 16, kMaxConvTaps = 16;
constexpr int kConvShortRows = 4;     // the same for filters of up to four taps
}  // namespace efm
