// Batched steps: which sequences are live, where each of them stands, and what a step's entries become for the device.
// A request is admitted at its first entry and ends with finish(); it may be left out of steps in between, and its tokens
// may arrive in portions of any size.
#pragma once
#include <edge-fm/edge-fm.h>

#include <cstdint>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "paged_cache.h"

namespace edge_fm {

struct PlannedEntry {
    int32_t slot = 0;
    int32_t kv_offset = 0;               // tokens of the sequence before this step
};

class StepScheduler {
public:
    // Sequences get the slot numbers first_slot, first_slot + 1, ...; max_live of them at a time.
    StepScheduler(std::shared_ptr<PagedCache> cache, int32_t first_slot, int32_t max_live);
    // Admits and places every entry of one step, or throws InvalidRequestError and changes nothing.
    std::vector<PlannedEntry> plan(const std::vector<StepEntry>& entries);
    // The step has run: the entries' tokens are in the cache.
    void commit(const std::vector<StepEntry>& entries);
    void finish(const std::string& id);
    bool is_live(const std::string& id) const { return live_.count(id) > 0; }
    int32_t live() const { return (int32_t)live_.size(); }
    int32_t max_live() const { return max_live_; }
    int32_t length(const std::string& id) const;
    // Room for `tokens` tokens of a request ahead of its steps (admits it); false: not now.
    bool try_admit(const std::string& id, int32_t tokens);

private:
    struct Live { int32_t slot = 0, len = 0; };
    std::shared_ptr<PagedCache> cache_;
    int32_t max_live_;
    std::vector<int32_t> free_slots_;
    std::map<std::string, Live> live_;
};

}  // namespace edge_fm
