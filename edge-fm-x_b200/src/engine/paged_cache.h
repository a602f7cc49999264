// Page and state bookkeeping of models on the paged cache: a pool of 64-token pages (the same page number in every
// attention layer's pool) and a pool of recurrent-state slots, given to sequences on demand and taken back when they end.
// The device side only sees the resulting page lists (PageMapper).
#pragma once
#include <cstdint>
#include <unordered_map>
#include <vector>

namespace edge_fm {

constexpr int32_t kCachePageTokens = 64;

// Where a sequence's page list goes.  The engine plugs in the device backend; tests plug in a recorder.
class PageMapper {
public:
    virtual ~PageMapper() = default;
    virtual void map(int32_t slot, const std::vector<int32_t>& pages, int32_t state_slot) = 0;
    virtual void unmap(int32_t slot) = 0;
};

class PagedCache {
public:
    PagedCache(int32_t pages, int32_t state_slots, PageMapper* mapper);
    // Makes room for `tokens` tokens of the sequence (its first call opens it).  false: not enough free pages or state
    // slots; nothing changed then.
    bool reserve(int32_t slot, int32_t tokens);
    void release(int32_t slot);
    // A state slot outside any sequence (the copy of a fixed prefix); -1: none free.
    int32_t take_state();
    int32_t free_pages() const { return (int32_t)free_.size(); }
    int32_t free_states() const { return (int32_t)states_.size(); }
    int32_t pages_held(int32_t slot) const {
        auto it = seqs_.find(slot);
        return it == seqs_.end() ? 0 : (int32_t)it->second.pages.size();
    }
    bool holds(int32_t slot) const { return seqs_.count(slot) > 0; }
    static int32_t pages_for(int32_t tokens) { return (tokens + kCachePageTokens - 1) / kCachePageTokens; }

private:
    struct Seq { std::vector<int32_t> pages; int32_t state = -1; };
    std::vector<int32_t> free_, states_;
    bool has_state_;
    PageMapper* mapper_;
    std::unordered_map<int32_t, Seq> seqs_;
};

}  // namespace edge_fm
