// Shape heuristic of the decode GEMV.
#pragma once
#include "../operators/gemv.cuh"

namespace efm {

// How many of a block's 16 warps share one row pair (ks).  The serial length of a warp's work is
// waves x units per item; the shortest wins, ties go to the smaller split (less reduction).
inline int plan_gemv_ksplit(int n_items, int K, int n_blocks) {
    const int nch = K / 8;
    int best = 1;
    long best_cost = -1;
    for (int ks = 1; ks <= kGemvWarps; ks *= 2) {
        const long slots = (long)n_blocks * (kGemvWarps / ks);
        const long waves = (n_items + slots - 1) / slots;
        const long cpl = (nch + 32 * ks - 1) / (32 * ks);
        const long units = (cpl + kGemvU - 1) / kGemvU;
        const long cost = waves * units * 64 + ks;
        if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = ks; }
    }
    return best;
}

}  // namespace efm
