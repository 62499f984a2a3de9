"""A prompt store: what the caches of a decoder hold for prompts already prefilled, kept in pinned host memory and copied
back into a slot instead of prefilling the same prompt again.

The reference keeps prompts in registered host memory as bf16 rows [L][n][C], copied with one 2-D memcpy per cache
(model/kernels/decode.cu:933-946,1055-1075), keyed by the prompt's token tuple, stored once and never evicted
(inference/decoder.py:172-175,193-232). Here the unit of copy is a cache's page: 64 positions of an attention layer's
cache, or the whole state of a recurrent layer (which after prefill is the state at exactly the prompt's positions). A
prompt of n positions (all but its last token) occupies pages_for(n) pages of every cache and head; positions past n
inside the last page are whatever the source slot held there, which the attention kernels never read (they mask by
length) and the next append overwrites."""

import torch

from .kv_cache import PAGE_TOKENS


class PromptStore:
    def __init__(self, caches: list, store_positions: int):
        """Room for `store_positions` positions (rounded up to pages) of every layer's cache in `caches`; a recurrent
        layer gets one state per page of that room, which is as many as there can be prompts."""
        self.caches = caches
        self.pages = (store_positions + PAGE_TOKENS - 1) // PAGE_TOKENS
        self.buffers = []
        for cache in caches:
            _, heads, _, page_bytes = cache.pages.shape
            buffer = torch.empty((heads, self.pages, page_bytes), dtype=torch.uint8)
            if torch.cuda.is_available() and cache.device.type == "cuda":
                buffer = buffer.pin_memory()
            self.buffers.append(buffer)
        self.taken = [0] * len(caches)  # store pages in use, per cache
        self.stored: dict[tuple[int, ...], list[tuple[int, int]]] = {}  # prompt -> (first store page, pages) per cache

    @property
    def used(self) -> int:
        """Store pages in use (of the cache that uses most)."""
        return max(self.taken, default=0)

    def save(self, slot: int, input_ids: list[int]) -> bool:
        """Keep slot's pages for the prompt's positions 0 .. len - 2, unless already stored or out of room (a
        prompt is stored once and never evicted). Stream-ordered on the current stream."""
        key, n = tuple(input_ids), len(input_ids) - 1
        need = [cache.pages_for(n) for cache in self.caches]
        if key in self.stored or n <= 0 or any(u + k > self.pages for u, k in zip(self.taken, need)):
            return False
        for cache, buffer, at, k in zip(self.caches, self.buffers, self.taken, need):
            buffer[:, at:at + k].copy_(cache.pages[slot, :, :k], non_blocking=True)
        self.stored[key] = list(zip(self.taken, need))
        self.taken = [u + k for u, k in zip(self.taken, need)]
        return True

    def load(self, slot: int, input_ids: list[int]) -> bool:
        """Copy a stored prompt's pages into `slot`; False if the prompt is not in the store."""
        hit = self.stored.get(tuple(input_ids))
        if hit is None:
            return False
        for cache, buffer, (at, k) in zip(self.caches, self.buffers, hit):
            cache.pages[slot, :, :k].copy_(buffer[:, at:at + k], non_blocking=True)
        return True
