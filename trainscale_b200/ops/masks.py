"""Which earlier positions of a sequence a position sees."""
from __future__ import annotations

from dataclasses import dataclass


UNBOUNDED = 1 << 30       # size of a window that no sequence outgrows


@dataclass(frozen=True)
class KeyMask:
    """Itself and the `size` - 1 positions before it, or (`chunked`) the positions before it in its chunk of `size`, chunks
    counted from position 0; besides, the first `keep` positions of the sequence."""
    size: int
    keep: int = 0
    chunked: bool = False

    def first(self, position: int) -> int:
        """First position of the window or chunk."""
        return position // self.size * self.size if self.chunked else max(0, position - self.size + 1)

    def most(self, length: int) -> int:
        """Upper bound of the keys that a position of a sequence of `length` sees."""
        return min(length, self.size + self.keep)

    def positions(self, position: int) -> list[int]:
        lo = self.first(position)
        return [*range(min(self.keep, lo)), *range(lo, position + 1)]
