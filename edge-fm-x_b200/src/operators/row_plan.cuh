// How the rows of one batched step map onto sequences.  A step concatenates the new tokens of every entry (portions of
// prompts and single decoded tokens alike) into rows [0, T); the row kernels find a row's sequence, position and cache
// pages here.  Passed by value; a step of one entry needs no device arrays (and can be captured in a graph).
#pragma once
#include <stdint.h>

namespace efm {

constexpr int kPageTokens = 64;       // cache rows per page
constexpr int kLinearChunk = 64, kLinearChunkTc = 128;      // tokens per chunk of linear attention: CUDA cores, tensor cores
constexpr int kLinearPowers = kLinearChunkTc;               // powers of a decay at hand

struct RowEntry {
    int32_t row0, n, pos0;            // rows [row0, row0 + n) hold positions [pos0, pos0 + n) of the sequence
    int32_t table;                    // row of the page table
    int32_t state;                    // recurrent-state slot
    int32_t ws0;                      // workspace row of position 0 (may be negative: only the positions a pass needs have one)
};

// One block's share of attention rows: rows [row, row + tile) of an entry.
struct RowTile { int32_t entry, row; };

struct RowPlan {
    RowEntry one;                     // the entry, when entries == nullptr
    const RowEntry* entries;
    const int32_t* row_entry;         // [T]
    const int32_t* page_table;        // [tables][max_pages] pool page of each 64-token page of a sequence
    int32_t max_pages, n_entries, rows;
#ifdef __CUDACC__
    __device__ __forceinline__ RowEntry entry(int e) const { return entries != nullptr ? entries[e] : one; }
    __device__ __forceinline__ RowEntry of_row(int row) const { return entries != nullptr ? entries[row_entry[row]] : one; }
    // pool row of a position
    __device__ __forceinline__ size_t cache_row(const RowEntry& e, int pos) const {
        return (size_t)page_table[(size_t)e.table * max_pages + pos / kPageTokens] * kPageTokens + pos % kPageTokens;
    }
#endif
};

#ifdef __CUDACC__
// Chunk `idx` of the pass, entries cut into chunks of C tokens each -> entry, first token; false past the last chunk.
template <int C>
__device__ __forceinline__ bool locate_chunk(const RowPlan& plan, int idx, RowEntry& e, int& t0) {
    int at = 0;
    for (int i = 0; i < plan.n_entries; ++i) {
        e = plan.entry(i);
        const int n = (e.n + C - 1) / C;
        if (idx < at + n) { t0 = (idx - at) * C; return true; }
        at += n;
    }
    return false;
}
#endif
// chunks of a pass, at most
inline int max_chunks(const RowPlan& plan, int C) { return plan.n_entries == 1 ? (plan.rows + C - 1) / C : plan.rows / C + plan.n_entries; }

}  // namespace efm
