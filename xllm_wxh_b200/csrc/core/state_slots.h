// Slots of recurrent state: the fixed-size counterpart of the KV blocks for layers that carry a state from token to token.
//
// A sequence holds one slot from its first step until it ends or is preempted; every recurrent layer run keeps one record
// per slot.  Slot 0 belongs to the padding rows of a step and is never handed out.  A slot is not cleared when it changes
// hands: a sequence whose step starts at position 0 starts from zero, whatever its slot holds.
#pragma once
#include <queue>
#include <stdexcept>
#include <vector>

namespace xl {

class StateSlots {
 public:
  explicit StateSlots(int n) : used_(n + 1, 0) {
    if (n < 1) throw std::invalid_argument("StateSlots needs at least one slot");
    for (int i = 1; i <= n; ++i) free_.push(i);
  }
  int num_slots() const { return static_cast<int>(used_.size()) - 1; }
  int num_free() const { return static_cast<int>(free_.size()); }
  int acquire() {  // smallest free slot; 0 when there is none
    if (free_.empty()) return 0;
    const int id = free_.top();
    free_.pop();
    used_[id] = 1;
    return id;
  }
  void release(int id) {
    if (id <= 0 || id >= static_cast<int>(used_.size()) || !used_[id]) throw std::logic_error("release of a state slot not in use");
    used_[id] = 0;
    free_.push(id);
  }

 private:
  std::priority_queue<int, std::vector<int>, std::greater<int>> free_;
  std::vector<char> used_;
};

}  // namespace xl
