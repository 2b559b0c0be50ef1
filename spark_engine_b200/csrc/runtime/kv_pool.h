// KV pool: one pool of token rows per GPU, leased to sequence slots in granules.
// Contiguous first-fit placement (a sequence never moves; its region can grow in place while the following
// granules are free) with LRU eviction candidates for idle stores.  The same bookkeeping drives the CUDA-VMM
// backend (vmm.cpp), where a region keeps its virtual address and physical granules are mapped behind it.
// Reference: engine-rs/src/kv_pool.rs:1-19,53-241 (pool, leases, per-array {div,width,kind} layout),
// shim/vmm.cpp:28-86.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace spark_rt {

struct Lease {
  int id = -1;
  int64_t base = 0;      // first token row
  int64_t cap = 0;       // rows reserved (multiple of the granule)
  int64_t used = 0;      // rows holding committed tokens
  uint64_t last_use = 0; // LRU stamp
  bool pinned = false;   // running sequences cannot be evicted
};

struct ArrayLayout {     // one cached array of a layer: rows = tokens / div, row width in bytes
  std::string name;
  int div = 1;
  int width = 0;
  int kind = 0;
};

class KvPool {
 public:
  KvPool(int64_t total_tokens, int64_t granule);
  // Reserve room for `tokens` rows.  Returns lease id or -1 (nothing is modified on failure: capacity checks
  // fail before any state is written).
  int acquire(int64_t tokens);
  bool grow(int id, int64_t tokens);          // in place; false if the following granules are taken
  void shrink(int id, int64_t tokens);
  void release(int id);
  void touch(int id);
  void pin(int id, bool on);
  void set_used(int id, int64_t used);
  const Lease* get(int id) const;
  int lru_victim() const;                     // idle lease with the oldest stamp, -1 if none
  int64_t free_tokens() const;
  int64_t largest_free_run() const;
  int64_t allocated_tokens() const;
  int64_t active_tokens() const;
  int64_t total() const { return total_; }
  int64_t granule() const { return granule_; }
  int64_t bytes_per_token(const std::vector<ArrayLayout>& arrays, int layers) const;

 private:
  int64_t round_up(int64_t t) const { return (t + granule_ - 1) / granule_ * granule_; }
  int64_t total_, granule_;
  std::map<int64_t, int> by_base_;            // base -> lease id
  std::map<int, Lease> leases_;
  int next_id_ = 0;
  uint64_t clock_ = 0;
};

// Page pool: the same leases over fixed-size pages instead of one contiguous run per sequence.  A lease grows by any free
// pages, so a pool that is exactly as large as what its sequences hold never fails by fragmentation; a sequence's rows
// are found through its page list (models whose cache kernels take a page table).
struct PageLease {
  int id = -1;
  std::vector<int32_t> pages;
  int64_t cap = 0, used = 0;
  uint64_t last_use = 0;
  bool pinned = false;
};

class PagePool {
 public:
  PagePool(int64_t total_tokens, int64_t page);
  int acquire(int64_t tokens);                // lease id or -1 (nothing changes on failure)
  bool grow(int id, int64_t tokens);
  void release(int id);                       // pages go back; the one given back last is handed out next
  void touch(int id);
  void pin(int id, bool on);
  void set_used(int id, int64_t used);
  const PageLease* get(int id) const;
  int lru_victim() const;
  int64_t total() const { return total_; }
  int64_t granule() const { return page_; }
  int64_t free_tokens() const { return static_cast<int64_t>(free_.size()) * page_; }
  int64_t largest_free_run() const { return free_tokens(); }
  int64_t allocated_tokens() const { return total_ - free_tokens(); }
  int64_t active_tokens() const;

 private:
  int64_t total_, page_;
  std::vector<int32_t> free_;
  std::map<int, PageLease> leases_;
  int next_id_ = 0;
  uint64_t clock_ = 0;
};

}  // namespace spark_rt
