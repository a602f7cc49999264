// Routed experts: limits, the router's shape and where a pass keeps the rows' choices.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace efm {

constexpr int kMaxExperts = 512, kMaxExpertTop = 32, kMaxExpertGroups = 64;
constexpr int kExpertTile = 128;      // rows of an expert start at multiples of this

enum : int { kSharedNone = 0, kSharedGated = 1, kSharedPlain = 2 };
struct RouteShape {
    int experts, top, groups, keep;
    int sigmoid;                      // scores: 0 softmax of the logits, 1 sigmoid of each
    int shared;                       // a shared expert: gated by logit `experts`, or as it is
    float scale;                      // of the choices' weights
};

struct ExpertRows {
    int32_t* id;                      // [rows][top]
    float* weight;                    // [rows][top]
    int32_t* place;                   // [rows][top]: place among the expert's rows, then row of the sorted order
    int32_t* count;                   // [experts], zero between passes
    int4* tile;                       // [tiles]: expert, its first tile, its number of tiles
    int32_t* n_tiles;                 // tiles in use
    float* shared;                    // [rows]: gate of the shared expert
};

}  // namespace efm
