"""What a mixer asks of the cache manager.

A mixer with a growing cache asks for paged keys and values (`PagedKVNeed`); a
mixer with state of fixed size asks for a per-request slot (`SlotStateNeed`); a
mixer without memory asks for nothing; a mixer that needs several of these asks
with a dictionary and gets a dictionary of handles.  The reference's counterpart of the first
is `DecodeStateConfig` (simply/utils/ragged_paged_attention.py:113-173); it has no
counterpart of the second (its per-request rows hold tokens and positions only,
:1451-1461).

Caches whose needs have the same `group_key()` share one pool of page ids and one block table
per request; the need itself says which of a request's pages may be given back
(`first_needed_page`) and how large its group's pool has to be (`pool_pages`), and which of its first pages stay whatever
the window (`kept_pages`).  A mixer with
another rule (a dilated window, a pool of its own) subclasses `PagedKVNeed` and overrides these;
the cache manager calls them and knows no rule of its own.
"""

from __future__ import annotations

import dataclasses

import numpy as np


@dataclasses.dataclass(frozen=True)
class PagedKVNeed:
  """Keys and values of every cached token, in pages.

  window: None keeps every token; an integer W keeps only what a query can still
    see, i.e. pages that lie wholly more than W-1 tokens behind the next query
    are given back.
  """

  num_kv_heads: int
  head_dim: int
  window: int | None = None
  # Size of a value head where it differs from a key head's (None: the same).
  value_dim: int | None = None
  # One entry per `stride` tokens instead of one per token (a cache of block summaries): the entry
  # of the tokens b*stride .. b*stride + stride - 1 lives in the page of token b*stride.
  stride: int = 1
  # Storage type where it is not the activations' ("float32").
  dtype: str | None = None
  # True: an entry has one row of head_dim numbers, whose first value_dim are its value as well
  # (a cache of latents that are key and value at once); a page then holds key rows only.
  values_in_keys: bool = False
  # With a window: the request's first `keep_first` tokens stay visible to every query, so their
  # pages are never given back while the request lives.
  keep_first: int = 0

  @property
  def v_dim(self) -> int:
    return self.head_dim if self.value_dim is None else self.value_dim

  def entries_per_page(self, page_size: int) -> int:
    return -(-page_size // self.stride)

  def storage_shape(self, num_pages: int, page_size: int) -> tuple[int, ...]:
    """Per page all key rows `[num_kv_heads, entries, head_dim]`, then all value rows
    `[num_kv_heads, entries, v_dim]`; with equal sizes that is `[2, heads, entries, head_dim]`."""
    entries = self.entries_per_page(page_size)
    if self.values_in_keys:
      return (num_pages, self.num_kv_heads * entries * self.head_dim)
    if self.v_dim == self.head_dim:
      return (num_pages, 2, self.num_kv_heads, entries, self.head_dim)
    return (num_pages, self.num_kv_heads * entries * (self.head_dim + self.v_dim))

  def group_key(self) -> tuple:
    """Needs with equal keys share page ids: the same pages are held, and given back together."""
    if self.window is not None and self.keep_first > 0:
      return ("window", self.window, "first", self.keep_first)
    return ("window", self.window)

  def kept_pages(self, page_size: int) -> int:
    """A request's first pages that are never given back although the window has left them."""
    return 0 if self.window is None else -(-self.keep_first // page_size)

  def first_needed_page(self, lengths: np.ndarray, page_size: int) -> np.ndarray:
    """Per request, the first page that the query after `lengths` cached tokens can still see;
    pages before it may be given back.  The reference's rule,
    `max(kv_len - window_size, 0) // page_size` with its window_size = window - 1
    (simply/utils/ragged_paged_attention.py:437-443)."""
    lengths = np.asarray(lengths, dtype=np.int64)
    if self.window is None:
      return np.zeros_like(lengths)
    return np.maximum(lengths - (self.window - 1), 0) // page_size

  def first_needed_page_of(self, length: int, page_size: int) -> int:
    """`first_needed_page` for one request, in plain integers (the books' inner loops use it)."""
    if type(self).first_needed_page is PagedKVNeed.first_needed_page:
      return 0 if self.window is None else max(length - (self.window - 1), 0) // page_size
    return int(self.first_needed_page(np.array([length], dtype=np.int64), page_size)[0])

  def release_length(self, first_page: int, page_size: int) -> int | None:
    """The smallest number of cached tokens at which a request whose first held page is
    `first_page` has a page to give back (`first_needed_page` exceeds `first_page`), or None when
    this need cannot say (the books then ask `first_needed_page` every time).  A very large
    number means never."""
    if type(self).first_needed_page is not PagedKVNeed.first_needed_page:
      return None
    if self.window is None:
      return 1 << 62
    return (first_page + 1) * page_size + (self.window - 1)

  def covers(self, reader: "PagedKVNeed") -> bool:
    """True if a cache with this need still holds, at every length, all that `reader` can see."""
    if self.window is None:
      return True
    return (type(reader) is PagedKVNeed and reader.window is not None and reader.window <= self.window
            and reader.keep_first <= self.keep_first)

  def pool_pages(self, *, page_size: int, max_slots: int, max_seq_len: int, all_pages: int,
                 step_tokens: int, burst_tokens: int) -> int:
    """Pages the group's pool needs so that it never runs out before a pool that keeps every
    token does (`all_pages`): every live request holds at most its window plus what one burst of
    decode steps adds, rounded up to pages with one page of slack at either end, and one step's
    prompt portions (`step_tokens` over all requests) come on top.  The reference sizes its local
    pool as batch * (ceil(window_size / page) + 1) and clips each portion to the room left
    (simply/serving/page_server.py:175-196, simply/utils/ragged_paged_attention.py:95-110, :418-434)."""
    if self.window is None:
      return all_pages
    per_slot = -(-(self.window - 1 + max(burst_tokens, 1)) // page_size) + 2 + self.kept_pages(page_size)
    per_slot = min(per_slot, -(-max_seq_len // page_size))
    return min(all_pages, max_slots * per_slot + -(-step_tokens // page_size))


@dataclasses.dataclass(frozen=True)
class ChunkedKVNeed(PagedKVNeed):
  """Keys and values of the query's own chunk: with chunks of C tokens, counted from position 0,
  position i sees the tokens from (i // C) * C on, so everything before the chunk of the next query
  is given back.  `chunks` names the chunk sizes of all layers that read the cache; a page goes
  when none of them can see it any more."""

  chunks: tuple[int, ...] = ()

  def group_key(self) -> tuple:
    return ("chunks", tuple(sorted(set(self.chunks))))

  def first_needed_page(self, lengths: np.ndarray, page_size: int) -> np.ndarray:
    lengths = np.asarray(lengths, dtype=np.int64)
    first = lengths
    for size in self.chunks:
      first = np.minimum(first, lengths // size * size)
    return first // page_size

  def first_needed_page_of(self, length: int, page_size: int) -> int:
    return min(length // size * size for size in self.chunks) // page_size

  def release_length(self, first_page: int, page_size: int) -> int | None:
    # every reader's chunk has to start at or behind the end of the page
    end = (first_page + 1) * page_size
    return max(-(-end // size) * size for size in self.chunks)

  def covers(self, reader: PagedKVNeed) -> bool:
    return isinstance(reader, ChunkedKVNeed) and set(reader.chunks) <= set(self.chunks)

  def pool_pages(self, *, page_size: int, max_slots: int, max_seq_len: int, all_pages: int,
                 step_tokens: int, burst_tokens: int) -> int:
    per_slot = -(-(max(self.chunks) + max(burst_tokens, 1)) // page_size) + 2
    per_slot = min(per_slot, -(-max_seq_len // page_size))
    return min(all_pages, max_slots * per_slot + -(-step_tokens // page_size))


@dataclasses.dataclass(frozen=True)
class SlotStateNeed:
  """A tensor of fixed shape per live request, zeroed when the request starts."""

  shape: tuple[int, ...]
  dtype: str = "float32"


def flatten_needs(name: str, need) -> list[tuple[str, object]]:
  """A mixer may ask for several caches at once as a dictionary `{key: need}` (nested ones too: a
  mixer made of mixers).  Returns `[(name.key..., need)]` for every single need inside."""
  if isinstance(need, dict):
    out = []
    for key, sub in need.items():
      out += flatten_needs(f"{name}.{key}", sub)
    return out
  return [(name, need)]
