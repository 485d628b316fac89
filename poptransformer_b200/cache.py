"""Sequence slots and cache pages for decoders whose sequences have positions of their own.

A slot is a row of the page table and the place of a sequence's recurrent state; pages hold `page_size` positions of every
attention layer's keys and values (the pools of all layers share one page numbering).  Slots and pages are handed out on demand
and returned when a sequence ends.  Nothing is cleared on return: kernels read no key beyond a sequence's own position and
ignore a slot's old recurrent state at position 0.
"""
import torch

from ._lib import PtError


class SequenceSlots:
    def __init__(self, max_seqs, max_len, page_size=64, n_pages=None, device="cuda"):
        self.max_seqs, self.max_len, self.page_size, self.device = max_seqs, max_len, page_size, device
        self.max_pages = -(-max_len // page_size)
        self.n_pages = max_seqs * self.max_pages if n_pages is None else n_pages
        self._free_slots = list(range(max_seqs - 1, -1, -1))
        self._free_pages = list(range(self.n_pages - 1, -1, -1))
        self._pages = {}                       # slot -> pages in position order
        self.length = {}                       # slot -> positions cached so far
        self.page_table = torch.zeros((max_seqs, self.max_pages), dtype=torch.int32, device=device)

    @property
    def free_slots(self):
        return len(self._free_slots)

    @property
    def free_pages(self):
        return len(self._free_pages)

    def open(self):
        """A slot for a new sequence (length 0, no pages yet)."""
        if not self._free_slots:
            raise PtError(f"all {self.max_seqs} sequence slots are in use")
        slot = self._free_slots.pop()
        self._pages[slot], self.length[slot] = [], 0
        return slot

    def extend(self, slot, n):
        """Makes room for `n` more positions and counts them as cached; returns the first of them."""
        start = self.length[slot]
        if start + n > self.max_len:
            raise PtError(f"a sequence of {start} + {n} tokens exceeds max_len={self.max_len}")
        pages = self._pages[slot]
        need = -(-(start + n) // self.page_size) - len(pages)
        if need > len(self._free_pages):
            raise PtError(f"{need} more cache pages needed, {len(self._free_pages)} of {self.n_pages} are free")
        if need > 0:
            first = len(pages)
            pages.extend(self._free_pages.pop() for _ in range(need))
            self.page_table[slot, first:len(pages)] = torch.tensor(pages[first:], dtype=torch.int32).to(self.device)
        self.length[slot] = start + n
        return start

    def close(self, slot):
        """Ends a sequence: its slot and pages can be used by the next one."""
        self._free_pages.extend(reversed(self._pages.pop(slot)))
        del self.length[slot]
        self._free_slots.append(slot)

    def close_all(self):
        for slot in list(self._pages):
            self.close(slot)
        self._free_slots.sort(reverse=True)    # the next open() calls return 0, 1, 2, ...
