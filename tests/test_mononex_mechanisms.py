"""Each mechanism of the Mononex layers alone: one call of the kernel table (the CUDA kernels on a
GPU, their plain PyTorch statements on the CPU) against the function of the plain NumPy model, and
the books of a cache with chunks."""

import types

import numpy as np
import pytest
import torch

from simply_b200.cache import CacheManager
from simply_b200.cache.needs import ChunkedKVNeed, PagedKVNeed
from simply_b200.parts.position import scaled_frequencies
from tests.plain import mononex_plain as plain
from tests.test_sapivik_mechanisms import close, context, held, table

CPU = pytest.param(("float32", "cpu"), id="cpu")
GPU32 = pytest.param(("float32", "cuda"), id="gpu-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param(("bfloat16", "cuda"), id="gpu-bf16", marks=pytest.mark.gpu)
WHERE = [CPU, GPU32, GPU16]


def f32(x, device):
  return torch.from_numpy(np.ascontiguousarray(x, np.float32)).to(device)


def f64(t):
  return t.float().cpu().numpy().astype(np.float64)


# ---- two norms of one stream and the token shift ---------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width,rows", [(32, 0), (32, 2), (200, 3), (37, 0), (1030, 0), (2048, 3), (8192, 0), (8200, 0)])
def test_two_norms_and_the_shift_carry_a_row_between_steps(width, rows, where):
  ops, dtype = table(where)
  device = where[1]
  if device == "cuda":
    ops.two_norms_rows = rows
  rng = np.random.default_rng(0)
  lengths = [23, 9, 40]
  total = sum(lengths)
  h = f32(rng.standard_normal((total, width)) * 3.0, device)
  b1, b1_64 = held(rng.standard_normal((total, width)), dtype, device)
  b2, b2_64 = held(rng.standard_normal((total, width)), dtype, device)
  w1, w1_64 = held(rng.standard_normal(width) * 0.3, dtype, device)
  w2, w2_64 = held(rng.standard_normal(width) * 0.3, dtype, device)
  shift = f32(rng.uniform(0, 1, width), device)
  norm = types.SimpleNamespace(weight=w1, eps=1e-3, plus_one=True)
  norm2 = types.SimpleNamespace(weight=w2.float(), eps=0.5, plus_one=True)
  state = torch.full((5, width), float("nan"), device=device)
  slots, starts = [3, 0, 4], np.concatenate([[0], np.cumsum(lengths)[:-1]])
  for s in slots:
    state[s].zero_()
  x = f64(h) + b1_64 + b2_64
  done = [0, 0, 0]
  for portions in ([5, 9, 20], [1, 0, 2], [17, 0, 1], [0, 0, 17]):
    who = [i for i, p in enumerate(portions) if p]
    pick = np.concatenate([np.arange(starts[i] + done[i], starts[i] + done[i] + portions[i]) for i in who])
    at = torch.from_numpy(pick).to(device)
    ctx = context(ops, device, [done[i] for i in who], [portions[i] for i in who], slots=[slots[i] for i in who])
    out, y, y2 = ops.residual_two_norms(h[at].contiguous(), b1[at].contiguous(), b2[at].contiguous(), norm, norm2, shift, state, ctx)
    close(f64(out), x[pick], torch.float32, "the stream")
    close(f64(y2), plain.zero_centred_norm(x[pick], w2_64, 0.5), dtype, "the second norm")
    want = np.concatenate([
        plain.token_shift(plain.zero_centred_norm(x[starts[i]:starts[i] + lengths[i]], w1_64, 1e-3), f64(shift))[done[i]:done[i] + portions[i]]
        for i in who])
    close(f64(y), want, dtype, f"the shifted norm, portions {portions}")
    for i in who:
      done[i] += portions[i]
  assert torch.isnan(state[1]).all() and torch.isnan(state[2]).all(), "a slot no request holds was written"
  # without a shift, without branches, without a second norm
  ctx = context(ops, device, [0, 0], [10, 4], slots=[1, 2])
  out, y, y2 = ops.residual_two_norms(h[:14].contiguous(), None, None, norm, None, None, None, ctx)
  assert y2 is None and torch.equal(out, h[:14])
  close(f64(y), plain.zero_centred_norm(f64(h[:14]), w1_64, 1e-3), dtype, "one norm alone")
  out, y, y2 = ops.residual_two_norms(h[:14].contiguous(), b1[:14].contiguous(), None, norm, norm2, None, None, ctx)
  close(f64(out), (f64(h) + b1_64)[:14], torch.float32, "one branch")
  close(f64(y2), plain.zero_centred_norm((f64(h) + b1_64)[:14], w2_64, 0.5), dtype, "two norms without a shift")
  if device == "cuda":
    ops.check_errors()


def test_a_shift_of_nothing_and_of_all():
  ops, _ = table(("float32", "cpu"))
  h = f32(np.random.default_rng(1).standard_normal((6, 8)), "cpu")
  norm = types.SimpleNamespace(weight=torch.zeros(8), eps=1e-6, plus_one=True)
  normed = plain.unit_rms(f64(h), 1e-6)
  for s, want in ((0.0, normed), (1.0, np.concatenate([np.zeros((1, 8)), normed[:-1]]))):
    ctx = context(ops, "cpu", [0], [6])
    _, y, _ = ops.residual_two_norms(h, None, None, norm, None, torch.full((8,), s), torch.zeros(1, 8), ctx)
    close(f64(y), want, torch.float32, f"shift {s}")


# ---- gated linear attention -----------------------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("sizes", [(2, 12, 8, 5, 8.0), (3, 16, 24, 16, 1.0), (1, 40, 5, 3, 0.5), (2, 128, 64, 64, 16.0), (1, 300, 3, 1, 2.0),
                                   (5, 1, 1, 7, 16.0), (3, 7, 9, 33, 4.0)])
def test_the_gated_linear_scan_carries_its_state_between_steps(sizes, where):
  heads, d, dv, rank, tau = sizes
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(0)
  lengths = [23, 9, 300]
  total, n = sum(lengths), heads * d
  low_at = 2 * n + 2 * heads * dv
  pre, pre64 = held(rng.standard_normal((total, low_at + rank + 3)), dtype, device)
  w_t, bias_t = f32(rng.standard_normal((rank, n)) / rank ** 0.5, device), f32(rng.standard_normal(n) + 1.0, device)
  want, start = [], 0
  for length in lengths:
    x = pre64[start:start + length]
    keep = plain.sigmoid(x[:, low_at:low_at + rank] @ f64(w_t) + f64(bias_t)) ** (1.0 / tau)
    q, k = x[:, :n].reshape(length, heads, d) * d ** -0.5, x[:, n:2 * n].reshape(length, heads, d)
    v = x[:, 2 * n:2 * n + heads * dv].reshape(length, heads, dv)
    out, s = np.zeros((length, heads, dv)), np.zeros((heads, d, dv))
    for i in range(length):
      s = keep[i].reshape(heads, d)[:, :, None] * s + k[i][:, :, None] * v[i][:, None, :]
      out[i] = np.einsum("hdv,hd->hv", s, q[i])
    want.append(out)
    start += length
  state = torch.full((5, heads, d, dv), float("nan"), device=device)
  slots = [3, 0, 4]
  for s in slots:
    state[s].zero_()
  done, got = [0, 0, 0], [[] for _ in lengths]
  starts = np.concatenate([[0], np.cumsum(lengths)[:-1]])
  for portions in ([5, 9, 270], [1, 0, 2], [17, 0, 28]):
    who = [i for i, p in enumerate(portions) if p]
    rows = np.concatenate([np.arange(starts[i] + done[i], starts[i] + done[i] + portions[i]) for i in who])
    ctx = context(ops, device, [done[i] for i in who], [portions[i] for i in who], slots=[slots[i] for i in who])
    out = f64(ops.gated_linear_scan(pre[torch.from_numpy(rows).to(device)].contiguous(), low_at, w_t, bias_t, tau, state, ctx,
                                    num_heads=heads, head_dim=d, value_dim=dv))
    at = 0
    for i in who:
      got[i].append(out[at:at + portions[i]])
      at += portions[i]
      done[i] += portions[i]
  for i in range(len(lengths)):
    g = np.concatenate(got[i])
    close(g, want[i][:len(g)], torch.float32, f"sequence {i} of sizes {sizes}")
  assert torch.isnan(state[1]).all() and torch.isnan(state[2]).all(), "a slot no request holds was written"


@pytest.mark.gpu
@pytest.mark.parametrize("copies", [1, 3])
def test_rows_that_repeat_a_request_get_what_its_first_row_gets(copies):
  """A decode graph pads its batch with copies of the last request's row: every copy's result is the
  first row's, and the state moves on by one token."""
  ops, _ = table(("float32", "cuda"))
  rng = np.random.default_rng(3)
  heads, d, dv, rank, width = 2, 16, 24, 4, 64
  slots = [2, 0] + [1] * copies
  state = f32(rng.standard_normal((3, heads, d, dv)), "cuda")
  base = rng.standard_normal((3, 2 * heads * d + 2 * heads * dv + rank))
  pre = f32(base[[0, 1] + [2] * copies], "cuda")
  w, bias = f32(rng.standard_normal((rank, heads * d)), "cuda"), f32(rng.standard_normal(heads * d), "cuda")
  ctx = context(ops, "cuda", [7, 3] + [5] * copies, [1] * len(slots), slots=slots)
  run = lambda p, c, st: ops.gated_linear_scan(p, 2 * heads * d + 2 * heads * dv, w, bias, 4.0, st, c, num_heads=heads, head_dim=d, value_dim=dv)
  alone_state = state.clone()
  alone = run(pre[:3].contiguous(), context(ops, "cuda", [7, 3, 5], [1, 1, 1], slots=[2, 0, 1]), alone_state)
  out = run(pre, ctx, state)
  assert torch.equal(out[:3], alone) and torch.equal(state, alone_state)
  for c in range(copies):
    assert torch.equal(out[2 + c], alone[2])
  h, branch = f32(rng.standard_normal((3, width)), "cuda"), f32(rng.standard_normal((3, width)), "cuda")
  pick = [0, 1] + [2] * copies
  shift, st = f32(rng.uniform(0, 1, width), "cuda"), f32(rng.standard_normal((3, width)), "cuda")
  norm = types.SimpleNamespace(weight=torch.zeros(width, device="cuda"), eps=1e-6, plus_one=True)
  st_alone = st.clone()
  alone = ops.residual_two_norms(h, branch, None, norm, norm, shift, st_alone, context(ops, "cuda", [7, 3, 5], [1, 1, 1], slots=[2, 0, 1]))
  both = ops.residual_two_norms(h[pick].contiguous(), branch[pick].contiguous(), None, norm, norm, shift, st, ctx)
  assert torch.equal(st, st_alone)
  for a, b in zip(alone, both):
    assert torch.equal(a, b[:3]) and all(torch.equal(a[2], b[2 + c]) for c in range(copies))
  ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,dv", [(3, 20), (1, 7), (12, 64)])
def test_head_norm_with_a_silu_gate(heads, dv, where):
  ops, dtype = table(where)
  rng = np.random.default_rng(1)
  o, w = f32(rng.standard_normal((7, heads, dv)), where[1]), f32(rng.uniform(0.5, 1.5, dv), where[1])
  gate, gate64 = held(rng.standard_normal((7, 5 + heads * dv)) * 2.0, dtype, where[1])
  g = gate64[:, 5:]
  want = (plain.unit_rms(f64(o), 1e-5) * f64(w)).reshape(7, -1)
  close(f64(ops.gated_head_norm(o, gate, 5, w, 1e-5, heads, dv, gate="silu")), want * g * plain.sigmoid(g), dtype, "silu")
  close(f64(ops.gated_head_norm(o, gate, 5, w, 1e-5, heads, dv)), want * plain.sigmoid(g), dtype, "sigmoid")


# ---- the feed-forward ---------------------------------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("rows,width,hidden", [(1, 32, 64), (9, 64, 24), (20, 64, 48), (200, 64, 96), (5, 36, 18), (40, 20, 7)])
def test_squared_relu_on_the_products_sums(rows, width, hidden, where):
  ops, dtype = table(where)
  rng = np.random.default_rng(2)
  x, x64 = held(rng.standard_normal((rows, width)), dtype, where[1])
  w, w64 = held(rng.standard_normal((hidden, width)) / width ** 0.5, dtype, where[1])
  close(f64(ops.linear_relu_squared(x, w)), np.maximum(x64 @ w64.T, 0.0) ** 2, dtype, "relu squared")


# ---- rotations over latents -------------------------------------------------------------------------------

@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, dict(factor=4.0, original=512, fast=32.0, slow=1.0)), (8, 500.0, dict(factor=1.0, original=100, fast=4.0, slow=0.5)),
    (64, 1e6, dict(factor=40.0, original=4096, fast=32.0, slow=1.0)), (2, 100.0, dict(factor=8.0, original=64, fast=2.0, slow=1.0)),
    (12, 50.0, dict(factor=2.5, original=7, fast=30.0, slow=20.0)), (10, 3000.0, None)])
def test_scaled_frequencies(dims, base, scaling):
  freq, amplitude = scaled_frequencies(dims, base, scaling)
  want, want_amplitude = plain.yarn_frequencies(dims, base, scaling)
  np.testing.assert_allclose(freq, want, rtol=1e-6)
  assert abs(amplitude - want_amplitude) < 1e-12
  if scaling and scaling["factor"] > 1.0 and dims >= 16:  # the fastest pairs keep their frequency, the slowest lose the factor
    assert freq[0] == np.float32(1.0) and abs(freq[-1] * scaling["factor"] / base ** (-2.0 * (dims // 2 - 1) / dims) - 1.0) < 1e-3


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("rot_dim,dims,amplitude", [(8, 8, 1.3), (12, 4, 1.0), (6, 6, 0.7)])
def test_neighbours_turn_in_keys_and_queries_over_latents(rot_dim, dims, amplitude, where):
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(4)
  q_rank, kv_rank, heads, d, page = 9, 14, 3, 5, 8
  before, counts = [13, 0], [6, 11]
  t = sum(counts)
  manager = CacheManager({"c": PagedKVNeed(1, kv_rank + rot_dim, None, value_dim=kv_rank, values_in_keys=True)}, page_size=page,
                         max_slots=2, max_seq_len=64, max_cache_tokens=128, dtype=dtype, device=device)
  for n in before:
    slot = manager.acquire_slot(n)
    if n:
      manager.extend([(slot, n)])
  manager.extend([(i, n) for i, n in enumerate(counts)])
  ctx = context(ops, device, before, counts, tables=[g.tables for g in manager.groups], page_size=page)
  storage = manager.paged["c"].storage
  freq64 = rng.uniform(0.1, 1.0, dims // 2)
  freq = f32(freq64, device)
  down, down64 = held(rng.standard_normal((t, q_rank + kv_rank + rot_dim + 2)), dtype, device)
  n_q, n_kv = f32(rng.uniform(0.5, 1.5, q_rank), device), f32(rng.uniform(0.5, 1.5, kv_rank), device)
  cq = ops.latent_prepare(down, n_q, n_kv, 1e-5, freq, query_rank=q_rank, kv_rank=kv_rank, rotated_dim=rot_dim, storage=storage,
                          block_table=ctx.block_tables[0], ctx=ctx, interleaved=True, amplitude=amplitude)
  close(f64(cq), plain.unit_rms(down64[:, :q_rank], 1e-5) * f64(n_q), dtype, "the queries' latent")
  pos = np.concatenate([np.arange(b, b + n) for b, n in zip(before, counts)]).astype(np.float64)
  rows = np.concatenate([plain.unit_rms(down64[:, q_rank:q_rank + kv_rank], 1e-5) * f64(n_kv),
                         plain.turn_neighbours(down64[:, q_rank + kv_rank:q_rank + kv_rank + rot_dim], pos, f64(freq), amplitude)], axis=1)
  cached = f64(storage.view(storage.shape[0], page, kv_rank + rot_dim))
  for i in range(t):
    b = 0 if i < counts[0] else 1
    p = int(pos[i])
    close(cached[manager.groups[0].tables[b, p // page], p % page], rows[i], dtype, f"the cached row of token {i}")
  q, q64 = held(rng.standard_normal((t, heads * (d + rot_dim))), dtype, device)
  up, up64 = held(rng.standard_normal((heads, kv_rank, d)) / d ** 0.5, dtype, device)
  asked = f64(ops.latent_queries(q, up, freq, 0.37, ctx, num_heads=heads, head_dim=d, rotated_dim=rot_dim, interleaved=True,
                                 amplitude=amplitude)).reshape(t, heads, kv_rank + rot_dim)
  qh = q64.reshape(t, heads, d + rot_dim)
  close(asked[..., :kv_rank], np.einsum("thd,hrd->thr", qh[..., :d], up64) * 0.37, dtype, "the plain part")
  close(asked[..., kv_rank:], plain.turn_neighbours(qh[..., d:], pos, f64(freq), amplitude) * 0.37, dtype, "the turned part")


# ---- attention: chunks, slopes, sinks, two sizes ------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,kv_heads,d,dv,chunk,slopes,sinks", [
    (4, 2, 16, 16, 10, True, True), (4, 1, 64, 64, 24, True, True), (8, 2, 128, 128, 50, True, False), (6, 3, 64, 32, 33, False, True),
    (4, 2, 96, 48, 100, True, True), (4, 4, 32, 112, 64, True, True), (2, 1, 7, 5, 9, True, True), (2, 1, 12, 20, 1, True, True),
    (4, 2, 64, 64, None, True, True), (4, 2, 192, 128, None, False, True), (16, 1, 32, 16, 40, True, True), (32, 1, 64, 64, 40, True, True),
    (2, 2, 256, 256, 37, True, True), (4, 2, 16, 240, 21, True, True)])
def test_attention_by_chunks_with_slopes_and_sinks(heads, kv_heads, d, dv, chunk, slopes, sinks, where):
  """Portions of a prompt beside single tokens; what lies before a query's chunk was given back and
  is poisoned."""
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(5)
  page = 16
  before, counts = [131, 0, 40, 99, 100], [1, 70, 9, 1, 2]
  need = (PagedKVNeed(kv_heads, d, None, value_dim=None if dv == d else dv) if chunk is None
          else ChunkedKVNeed(kv_heads, d, value_dim=None if dv == d else dv, chunks=(chunk,)))
  manager = CacheManager({"c": need}, page_size=page, max_slots=len(before), max_seq_len=256, max_cache_tokens=5 * 256, dtype=dtype,
                         device=device, poison_freed_pages=True)
  keys = [held(rng.standard_normal((b + n, kv_heads, d)), dtype, device) for b, n in zip(before, counts)]
  values = [held(rng.standard_normal((b + n, kv_heads, dv)), dtype, device) for b, n in zip(before, counts)]
  storage = manager.paged["c"].storage
  storage.fill_(float("nan"))
  flat = storage.view(storage.shape[0], -1)
  k_view = flat[:, :kv_heads * page * d].view(-1, kv_heads, page, d)
  v_view = flat[:, kv_heads * page * d:].view(-1, kv_heads, page, dv)

  def write(b, lo, hi):
    for p in range(lo, hi):
      row = manager.groups[0].tables[b, p // page]
      k_view[row, :, p % page], v_view[row, :, p % page] = keys[b][0][p], values[b][0][p]

  for b, n in enumerate(before):
    slot = manager.acquire_slot(b)
    assert slot == b
    for lo in range(0, n, 30):
      manager.extend([(b, min(30, n - lo))])
      write(b, lo, min(lo + 30, n))
  manager.extend(list(enumerate(counts)))
  for b, n in enumerate(before):
    write(b, n, n + counts[b])
  ctx = context(ops, device, before, counts, tables=[g.tables for g in manager.groups], page_size=page)
  ctx.older_keys_settled = True
  t = sum(counts)
  q, q64 = held(rng.standard_normal((t, heads, d)) / d ** 0.5, dtype, device)
  slope = 2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)
  sink = rng.standard_normal(heads) * 2.0
  opts = {}
  if slopes:
    opts["distance_bias"] = f32(slope[None], device)
  if sinks:
    opts["sink"] = f32(sink, device)
  got = f64(ops.paged_attention(q, storage, ctx.block_tables[0], ctx, num_heads=heads, num_kv_heads=kv_heads, head_dim=d,
                                logit_softcap=0.0, window=None, value_dim=dv, key_chunk=chunk, **opts)).reshape(t, heads, dv)
  row = 0
  for b, n in enumerate(before):
    for i in range(n, n + counts[b]):
      lo = i // chunk * chunk if chunk else 0
      for a in range(heads):
        g = a // (heads // kv_heads)
        s = keys[b][1][lo:i + 1, g] @ q64[row, a] - (slope[a] * (i - np.arange(lo, i + 1)) if slopes else 0.0)
        s = np.append(s, sink[a] if sinks else -np.inf)
        e = np.exp(s - s.max())
        want = e[:-1] / e.sum() @ values[b][1][lo:i + 1, g]
        assert np.abs(got[row, a] - want).max() <= (3e-5 if dtype == torch.float32 else 3e-2), (b, i, a)
      row += 1
  if device == "cuda":
    ops.check_errors()


# ---- the books of a cache with chunks ---------------------------------------------------------------------

@pytest.mark.parametrize("chunks,page", [((12,), 8), ((7, 12), 4), ((64,), 64), ((1,), 4), ((100, 30), 16), ((5,), 16)])
def test_pages_go_when_no_chunk_needs_them(chunks, page):
  need = ChunkedKVNeed(2, 8, chunks=chunks)
  for length in range(0, 300):
    first = min(length // c * c for c in chunks)  # the lowest key that the next query sees
    assert need.first_needed_page_of(length, page) == first // page == int(need.first_needed_page(np.array([length]), page)[0])
  for first_page in range(6):
    at = need.release_length(first_page, page)
    assert need.first_needed_page_of(at, page) > first_page >= need.first_needed_page_of(at - 1, page)
  manager = CacheManager({"c": need}, page_size=page, max_slots=2, max_seq_len=400, max_cache_tokens=800, device=None)
  rng = np.random.default_rng(0)
  slots = [manager.acquire_slot(i) for i in range(2)]
  for _ in range(60):
    for s in slots:
      n = int(rng.integers(1, 6))
      if manager.length(s) + n <= 400:
        before = manager.length(s)
        manager.extend([(s, n)])
        held_from = int(manager.groups[0].first_page[s]) * page
        lowest = min(before // c * c for c in chunks)
        assert held_from <= lowest < held_from + page
    manager.check_invariants()
  for s in slots:
    manager.release_slot(s)
  assert manager.all_pages_free()


def test_needs_of_equal_chunks_share_pages_and_readers_are_checked():
  a, b, c = ChunkedKVNeed(2, 8, chunks=(7, 12)), ChunkedKVNeed(4, 16, chunks=(12, 7)), ChunkedKVNeed(2, 8, chunks=(12,))
  assert a.group_key() == b.group_key() != c.group_key() != PagedKVNeed(2, 8).group_key()
  assert a.covers(c) and not c.covers(a) and not a.covers(PagedKVNeed(2, 8)) and PagedKVNeed(2, 8).covers(a)
  manager = CacheManager({"a": a, "b": b, "c": c}, page_size=4, max_slots=1, max_seq_len=64, max_cache_tokens=64, device=None)
  assert len(manager.groups) == 2
  pages = a.pool_pages(page_size=4, max_slots=2, max_seq_len=640, all_pages=1000, step_tokens=16, burst_tokens=8)
  assert pages == 2 * (-(-20 // 4) + 2) + 4
