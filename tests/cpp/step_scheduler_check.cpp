// Test driver for the paged cache and the step scheduler (host logic only, no GPU): random admissions, portions, pauses and
// endings against a recorder in the device's place.  Prints "ok" or what went wrong.
//   step_scheduler_check <pages> <state slots> <max live> <seed> <steps>
#include <cstdio>
#include <cstdlib>
#include <map>
#include <random>
#include <set>
#include <string>

#include "step_scheduler.h"

using namespace edge_fm;

namespace {
struct Recorder : PageMapper {
    std::map<int32_t, std::vector<int32_t>> pages;
    std::map<int32_t, int32_t> state;
    const char* bad = nullptr;
    void map(int32_t slot, const std::vector<int32_t>& p, int32_t s) override {
        auto it = pages.find(slot);
        if (it != pages.end()) {                       // a sequence keeps the pages it has, in order, and its state
            if (p.size() <= it->second.size() || !std::equal(it->second.begin(), it->second.end(), p.begin())) bad = "pages of a live sequence moved";
            if (state[slot] != s) bad = "state of a live sequence moved";
        }
        for (const auto& kv : pages)
            if (kv.first != slot) {
                for (int32_t a : p)
                    for (int32_t b : kv.second)
                        if (a == b) bad = "page given twice";
                if (s >= 0 && state[kv.first] == s) bad = "state given twice";
            }
        pages[slot] = p;
        state[slot] = s;
    }
    void unmap(int32_t slot) override {
        if (pages.erase(slot) == 0) bad = "unmapping an unknown slot";
        state.erase(slot);
    }
};
}  // namespace

int main(int argc, char** argv) {
    if (argc != 6) return 2;
    const int pages = std::atoi(argv[1]), states = std::atoi(argv[2]), live_max = std::atoi(argv[3]), steps = std::atoi(argv[5]);
    std::mt19937 rng((unsigned)std::atoi(argv[4]));
    Recorder rec;
    auto cache = std::make_shared<PagedCache>(pages, states, &rec);
    StepScheduler sched(cache, 1000, live_max);
    std::map<std::string, int32_t> len;
    int refused = 0, next = 0;
    for (int i = 0; i < steps; ++i) {
        std::vector<StepEntry> entries;
        for (const auto& kv : len)
            if (rng() % 3) entries.push_back(StepEntry{kv.first, std::vector<int32_t>(1 + rng() % 90, 7), {}});
        if (rng() % 2) entries.push_back(StepEntry{"r" + std::to_string(next++), std::vector<int32_t>(1 + rng() % 200, 7), {0}});
        if (!entries.empty()) {
            try {
                const std::vector<PlannedEntry> plan = sched.plan(entries);
                for (size_t e = 0; e < entries.size(); ++e) {
                    const int32_t before = len.count(entries[e].id) ? len[entries[e].id] : 0;
                    if (plan[e].kv_offset != before) { std::puts("wrong offset"); return 1; }
                    if ((int)rec.pages[plan[e].slot].size() != PagedCache::pages_for(before + (int32_t)entries[e].tokens.size())) { std::puts("wrong page count"); return 1; }
                    len[entries[e].id] = before + (int32_t)entries[e].tokens.size();
                }
                sched.commit(entries);
            } catch (const InvalidRequestError&) {
                ++refused;                              // and nothing has changed
                for (const StepEntry& e : entries)
                    if (sched.is_live(e.id) != (len.count(e.id) > 0)) { std::puts("a refused step admitted a request"); return 1; }
            }
        }
        if (rec.bad != nullptr) { std::puts(rec.bad); return 1; }
        if (!len.empty() && rng() % 3 == 0) {
            auto it = len.begin();
            std::advance(it, (long)(rng() % len.size()));
            sched.finish(it->first);
            len.erase(it);
        }
    }
    while (!len.empty()) { sched.finish(len.begin()->first); len.erase(len.begin()); }
    if (cache->free_pages() != pages || cache->free_states() != states || sched.live() != 0) { std::puts("something was not given back"); return 1; }
    if (refused == 0) { std::puts("the pool was never full: the case tests nothing"); return 1; }
    std::puts("ok");
    return 0;
}
