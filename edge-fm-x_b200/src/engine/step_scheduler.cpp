#include "step_scheduler.h"

#include <algorithm>
#include <set>

namespace edge_fm {

StepScheduler::StepScheduler(std::shared_ptr<PagedCache> cache, int32_t first_slot, int32_t max_live)
    : cache_(std::move(cache)), max_live_(max_live) {
    for (int32_t i = max_live - 1; i >= 0; --i) free_slots_.push_back(first_slot + i);
}

int32_t StepScheduler::length(const std::string& id) const {
    auto it = live_.find(id);
    return it == live_.end() ? 0 : it->second.len;
}

bool StepScheduler::try_admit(const std::string& id, int32_t tokens) {
    auto it = live_.find(id);
    if (it != live_.end()) return cache_->reserve(it->second.slot, tokens);
    if (free_slots_.empty() || !cache_->reserve(free_slots_.back(), tokens)) return false;
    Live l;
    l.slot = free_slots_.back();
    free_slots_.pop_back();
    live_.emplace(id, l);
    return true;
}

std::vector<PlannedEntry> StepScheduler::plan(const std::vector<StepEntry>& entries) {
    if (entries.empty()) throw InvalidRequestError("a step needs at least one entry");
    std::set<std::string> seen;
    for (const StepEntry& e : entries) {
        if (e.tokens.empty()) throw InvalidRequestError("step entry without tokens: " + e.id);
        if (!seen.insert(e.id).second) throw InvalidRequestError("request appears twice in one step: " + e.id);
    }
    int32_t pages = 0, fresh = 0;
    for (const StepEntry& e : entries) {
        auto it = live_.find(e.id);
        const int32_t have = it == live_.end() ? 0 : cache_->pages_held(it->second.slot);
        pages += std::max(0, PagedCache::pages_for(length(e.id) + (int32_t)e.tokens.size()) - have);
        fresh += it == live_.end() ? 1 : 0;
    }
    if (fresh > (int32_t)free_slots_.size()) throw InvalidRequestError("no free slot for the step's new requests");
    if (pages > cache_->free_pages()) throw InvalidRequestError("the cache pool has no room for the step's tokens");
    std::vector<PlannedEntry> out;
    for (const StepEntry& e : entries) {
        const int32_t len = length(e.id);
        if (!try_admit(e.id, len + (int32_t)e.tokens.size()))
            throw InvalidRequestError("no cache pages or state slot for request " + e.id);
        PlannedEntry p;
        p.slot = live_.at(e.id).slot;
        p.kv_offset = len;
        out.push_back(p);
    }
    return out;
}

void StepScheduler::commit(const std::vector<StepEntry>& entries) {
    for (const StepEntry& e : entries) live_.at(e.id).len += (int32_t)e.tokens.size();
}

void StepScheduler::finish(const std::string& id) {
    auto it = live_.find(id);
    if (it == live_.end()) throw InvalidRequestError("finish: request is not live: " + id);
    cache_->release(it->second.slot);
    free_slots_.push_back(it->second.slot);
    live_.erase(it);
}

}  // namespace edge_fm
