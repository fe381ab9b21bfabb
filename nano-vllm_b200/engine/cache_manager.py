"""Host bookkeeping of what live sequences hold on the device: blocks of the paged KV cache and slots of recurrent state."""
from __future__ import annotations

from collections import deque


class CacheManager:

    def __init__(self, num_blocks: int, block_size: int, num_state_slots: int = 0):
        self.block_size = block_size
        self.free_blocks = deque(range(num_blocks))
        self.free_slots = deque(range(num_state_slots))
        self.uses_state = num_state_slots > 0

    def blocks_missing(self, seq, num_tokens: int) -> int:
        """Blocks `seq` still needs before its first num_tokens tokens have a place."""
        return max(0, -(-num_tokens // self.block_size) - len(seq.block_table))

    def can_hold(self, seq, num_tokens: int) -> bool:
        if self.uses_state and seq.state_slot < 0 and not self.free_slots:
            return False
        return self.blocks_missing(seq, num_tokens) <= len(self.free_blocks)

    def hold(self, seq, num_tokens: int) -> None:
        """Give `seq` blocks for its first num_tokens tokens, and a state slot."""
        if not self.can_hold(seq, num_tokens):
            raise RuntimeError("no free KV block or state slot")
        if self.uses_state and seq.state_slot < 0:
            seq.state_slot = self.free_slots.popleft()
        for _ in range(self.blocks_missing(seq, num_tokens)):
            seq.block_table.append(self.free_blocks.popleft())

    def release(self, seq) -> None:
        """Take back everything `seq` holds; it would have to be computed again from its first token.  The state slot is not
        cleared: a sequence at position 0 starts from zero whatever its slot holds."""
        self.free_blocks.extend(seq.block_table)
        seq.block_table = []
        if seq.state_slot >= 0:
            self.free_slots.append(seq.state_slot)
            seq.state_slot = -1
        seq.num_cached_tokens = 0
