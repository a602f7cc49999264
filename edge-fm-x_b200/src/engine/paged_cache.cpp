#include "paged_cache.h"

#include <algorithm>

namespace edge_fm {

PagedCache::PagedCache(int32_t pages, int32_t state_slots, PageMapper* mapper) : has_state_(state_slots > 0), mapper_(mapper) {
    for (int32_t i = pages - 1; i >= 0; --i) free_.push_back(i);
    for (int32_t i = state_slots - 1; i >= 0; --i) states_.push_back(i);
}

bool PagedCache::reserve(int32_t slot, int32_t tokens) {
    auto it = seqs_.find(slot);
    const bool fresh = it == seqs_.end();
    const int32_t have = fresh ? 0 : (int32_t)it->second.pages.size(), need = std::max(1, pages_for(tokens));
    if (!fresh && need <= have) return true;
    if (need - have > (int32_t)free_.size() || (fresh && has_state_ && states_.empty())) return false;
    Seq& s = fresh ? seqs_[slot] : it->second;
    for (int32_t i = have; i < need; ++i) {
        s.pages.push_back(free_.back());
        free_.pop_back();
    }
    if (fresh && has_state_) {
        s.state = states_.back();
        states_.pop_back();
    }
    mapper_->map(slot, s.pages, s.state);
    return true;
}

void PagedCache::release(int32_t slot) {
    auto it = seqs_.find(slot);
    if (it == seqs_.end()) return;
    mapper_->unmap(slot);
    for (size_t i = it->second.pages.size(); i > 0; --i) free_.push_back(it->second.pages[i - 1]);
    if (it->second.state >= 0) states_.push_back(it->second.state);
    seqs_.erase(it);
}

int32_t PagedCache::take_state() {
    if (states_.empty()) return -1;
    const int32_t s = states_.back();
    states_.pop_back();
    return s;
}

}  // namespace edge_fm
