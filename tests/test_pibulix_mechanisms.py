"""Each mechanism of the Pibulix layers alone: one call of the kernel table (the CUDA kernels on a
GPU, their plain PyTorch statements on the CPU) against the function of the plain NumPy model, and
the books of a cache that keeps first tokens beside a window."""

import types

import numpy as np
import pytest
import torch

from simply_b200.cache import CacheManager, PagedKVNeed
from simply_b200.parts.normed_attention import rotation_frequencies
from tests.plain import pibulix_plain as plain
from tests.test_sapivik_mechanisms import close, context, held, table

CPU = pytest.param(("float32", "cpu"), id="cpu")
GPU32 = pytest.param(("float32", "cuda"), id="gpu-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param(("bfloat16", "cuda"), id="gpu-bf16", marks=pytest.mark.gpu)
WHERE = [CPU, GPU32, GPU16]


def f32(x, device):
  return torch.from_numpy(np.ascontiguousarray(x, np.float32)).to(device)


def f64(t):
  return t.float().cpu().numpy().astype(np.float64)


# ---- the norm behind the sum ------------------------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width", [32, 200, 37, 1030, 2048, 4100, 8192, 12296])
def test_the_norm_of_a_sum(width, where):
  ops, dtype = table(where)
  rng = np.random.default_rng(0)
  for rows, alpha, eps in ((1, 2.25, 1e-4), (9, 0.75, 0.5), (70, 1.0, 1e-3)):
    h = f32(rng.standard_normal((rows, width)) * 3.0, where[1])
    b, b64 = held(rng.standard_normal((rows, width)), dtype, where[1])
    w, w64 = held(rng.standard_normal(width) * 0.3, dtype, where[1])
    want = plain.normed_sum(f64(h), b64, alpha, w64, eps)
    y = ops.norm_of_sum(h, b, alpha, types.SimpleNamespace(weight=w, eps=eps, plus_one=True))
    close(f64(h), want, torch.float32, "the stream")
    close(f64(y), want, dtype, "what the next sublayer reads")
    h = f32(rng.standard_normal((rows, width)), where[1])
    want = plain.unit_rms(alpha * f64(h) + b64, eps) * w64
    ops.norm_of_sum(h, b, alpha, types.SimpleNamespace(weight=w.float(), eps=eps, plus_one=False))
    close(f64(h), want, torch.float32, "a plain scale")


# ---- convolution, norm, rotation, store -------------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,kv_heads,d,dv,taps,dims,extra", [
    (4, 2, 16, 16, 3, 8, 0), (6, 1, 64, 64, 4, 32, 3), (2, 2, 128, 96, 2, 128, 0), (3, 1, 7, 5, 3, 6, 0), (2, 1, 256, 40, 4, 64, 0),
    (4, 4, 12, 20, 6, 12, 1), (2, 1, 16, 16, 1, 0, 0), (2, 1, 32, 64, 0, 16, 0), (5, 5, 10, 6, 2, 2, 0), (1, 1, 300, 12, 3, 20, 0)])
def test_convolved_heads_are_normed_turned_and_stored(heads, kv_heads, d, dv, taps, dims, extra, where):
  """Portions of prompts beside single tokens, then a step of single tokens alone (whose kernel moves the
  convolution's state on itself)."""
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(1)
  page, total = 8, [70, 23, 40]
  nq, nk, nv = heads * d, kv_heads * d, kv_heads * dv
  channels = nq + nk + nv
  manager = CacheManager({"c": PagedKVNeed(kv_heads, d, None, value_dim=None if dv == d else dv)}, page_size=page, max_slots=5,
                         max_seq_len=128, max_cache_tokens=5 * 128, dtype=dtype, device=device)
  slots = [manager.acquire_slot(i) for i in range(4)][1:]
  storage = manager.paged["c"].storage
  pre = [held(rng.standard_normal((n, channels + extra)), dtype, device) for n in total]
  conv = rng.standard_normal((taps, channels)) * 0.5 if taps else None
  conv_t = f32(conv, device) if taps else None
  q_scale_w, k_scale_w = rng.uniform(0.5, 1.5, d), rng.uniform(0.5, 1.5, d)
  freq = rotation_frequencies(dims, 5000.0) if dims else None
  want = []
  for x, x64 in pre:
    u = x64[:, :channels]
    u = plain.short_convolution(u, f64(conv_t).T) if taps else u
    parts = []
    for lo, n, scale in ((0, heads, f64(f32(q_scale_w, "cpu"))), (nq, kv_heads, f64(f32(k_scale_w, "cpu")))):
      z = plain.unit_rms(u[:, lo:lo + n * d].reshape(-1, n, d), 1e-4) * scale
      parts.append(plain.turn_halves(z, np.arange(len(z), dtype=np.float64), dims, 5000.0) if dims else z)
    want.append((parts[0] * 0.37, parts[1], u[:, nq + nk:].reshape(-1, kv_heads, dv)))
  state = torch.full((5, max(taps - 1, 1), channels), float("nan"), device=device)
  for s in slots:
    state[s].zero_()
  done = [0, 0, 0]
  # (the interleaving of portions, and at the end single tokens only, with requests left out)
  for portions in ([30, 1, 2], [1, 0, 2], [2, 7, 1], [1, 1, 1], [0, 1, 1], [1, 0, 0], [30, 3, 0], [1, 1, 20], [1, 1, 1]):
    who = [i for i, p in enumerate(portions) if p]
    manager.extend([(slots[i], portions[i]) for i in who])
    ctx = context(ops, device, [done[i] for i in who], [portions[i] for i in who], slots=[slots[i] for i in who],
                  tables=[g.tables for g in manager.groups], page_size=page)
    x = torch.cat([pre[i][0][done[i]:done[i] + portions[i]] for i in who]).contiguous()
    q = ops.conv_headnorm_rotate_store(
        x, conv_t, state if taps > 1 else None, f32(q_scale_w, device), f32(k_scale_w, device), 1e-4, 0.37,
        torch.from_numpy(freq).to(device) if dims else None, interleaved=False, num_heads=heads, num_kv_heads=kv_heads, head_dim=d,
        value_dim=dv, storage=storage, block_table=ctx.block_tables[0], ctx=ctx)
    close(f64(q).reshape(-1, heads, d), np.concatenate([want[i][0][done[i]:done[i] + portions[i]] for i in who]), dtype, f"queries {portions}")
    for i in who:
      done[i] += portions[i]
  flat = storage.view(storage.shape[0], -1)
  keys = f64(flat[:, :kv_heads * page * d]).reshape(-1, kv_heads, page, d)
  values = f64(flat[:, kv_heads * page * d:]).reshape(-1, kv_heads, page, dv)
  for i, s in enumerate(slots):
    at = [(manager.groups[0].tables[s, p // page], p % page) for p in range(done[i])]
    close(np.stack([keys[r, :, o] for r, o in at]), want[i][1][:done[i]], dtype, f"keys of request {i}")
    close(np.stack([values[r, :, o] for r, o in at]), want[i][2][:done[i]], dtype, f"values of request {i}")
    if taps > 1:
      close(f64(state[s]), pre[i][1][done[i] - taps + 1:done[i], :channels], torch.float32, f"state of request {i}")
  assert torch.isnan(state[0]).all() and torch.isnan(state[4]).all(), "a slot no request of the step holds was written"
  if device == "cuda":
    ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,kv_heads,d,dv,taps", [(5, 1, 64, 64, 3), (4, 2, 128, 128, 4), (2, 1, 24, 40, 2), (2, 1, 256, 192, 4),
                                                      (3, 1, 32, 16, 0), (2, 2, 7, 9, 3), (2, 1, 16, 16, 5)])
def test_convolved_heads_of_a_long_step(heads, kv_heads, d, dv, taps, where):
  """Well over a thousand tokens in one step, where a block serves several: requests begin and end inside one."""
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(2)
  counts, before, page = [7, 1061, 1, 2, 70, 1, 3], [5, 9, 0, 1, 0, 4, 2], 64
  dims = d // 4 * 2 if d % 4 == 0 else 2
  channels = heads * d + kv_heads * (d + dv)
  manager = CacheManager({"c": PagedKVNeed(kv_heads, d, None, value_dim=None if dv == d else dv)}, page_size=page, max_slots=7,
                         max_seq_len=1152, max_cache_tokens=7 * 1152, dtype=dtype, device=device)
  conv = rng.standard_normal((taps, channels)) * 0.5 if taps else None
  conv_t = f32(conv, device) if taps else None
  scale, freq = rng.uniform(0.5, 1.5, d), rotation_frequencies(dims, 5000.0)
  pre = [held(rng.standard_normal((b + n, channels)), dtype, device) for b, n in zip(before, counts)]
  state = torch.zeros((7, max(taps - 1, 1), channels), device=device)
  for i, b in enumerate(before):
    assert manager.acquire_slot(i) == i
    if b:
      manager.extend([(i, b)])
    for r in range(taps - 1):
      if b - (taps - 1) + r >= 0:
        state[i, r] = pre[i][0][b - (taps - 1) + r].float()
  manager.extend(list(enumerate(counts)))
  ctx = context(ops, device, before, counts, tables=[g.tables for g in manager.groups], page_size=page)
  x = torch.cat([pre[i][0][b:] for i, b in enumerate(before)]).contiguous()
  storage = manager.paged["c"].storage
  q = f64(ops.conv_headnorm_rotate_store(
      x, conv_t, state if taps > 1 else None, f32(scale, device), f32(scale, device), 1e-4, 0.5, torch.from_numpy(freq).to(device),
      interleaved=False, num_heads=heads, num_kv_heads=kv_heads, head_dim=d, value_dim=dv, storage=storage,
      block_table=ctx.block_tables[0], ctx=ctx)).reshape(-1, heads, d)
  flat = storage.view(storage.shape[0], -1)
  keys = f64(flat[:, :kv_heads * page * d]).reshape(-1, kv_heads, page, d)
  values = f64(flat[:, kv_heads * page * d:]).reshape(-1, kv_heads, page, dv)
  at, scale64 = 0, f64(f32(scale, "cpu"))
  for i, (b, n) in enumerate(zip(before, counts)):
    u = plain.short_convolution(pre[i][1], f64(conv_t).T) if taps else pre[i][1]
    pos = np.arange(b + n, dtype=np.float64)
    turned = lambda lo, hh: plain.turn_halves(plain.unit_rms(u[:, lo:lo + hh * d].reshape(-1, hh, d), 1e-4) * scale64, pos, dims, 5000.0)[b:]
    close(q[at:at + n], turned(0, heads) * 0.5, dtype, f"queries of request {i}", f32=1e-4)
    rows = [(manager.groups[0].tables[i, p // page], p % page) for p in range(b, b + n)]
    close(np.stack([keys[r, :, o] for r, o in rows]), turned(heads * d, kv_heads), dtype, f"keys of request {i}", f32=1e-4)
    close(np.stack([values[r, :, o] for r, o in rows]), u[b:, (heads + kv_heads) * d:].reshape(n, kv_heads, dv), dtype, f"values of request {i}")
    if taps > 1:
      tail = np.concatenate([np.zeros((taps, channels)), pre[i][1]])[-(taps - 1):]
      close(f64(state[i]), tail, torch.float32, f"state of request {i}")
    at += n
  if device == "cuda":
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("copies", [1, 3])
def test_rows_that_repeat_a_request_get_what_its_first_row_gets(copies):
  ops, _ = table(("float32", "cuda"))
  rng = np.random.default_rng(3)
  heads, kv_heads, d, dv, taps, page = 3, 1, 16, 24, 3, 8
  channels = heads * d + kv_heads * (d + dv)
  manager = CacheManager({"c": PagedKVNeed(kv_heads, d, None, value_dim=dv)}, page_size=page, max_slots=3, max_seq_len=64,
                         max_cache_tokens=192, dtype=torch.float32, device="cuda")
  for i, n in enumerate((4, 6, 8)):
    manager.acquire_slot(i)
    manager.extend([(i, n)])
  storage = manager.paged["c"].storage
  before, slots = [7, 3] + [5] * copies, [2, 0] + [1] * copies
  base = f32(rng.standard_normal((3, channels)), "cuda")
  conv, norm_w = f32(rng.standard_normal((taps, channels)), "cuda"), f32(rng.uniform(0.5, 1.5, d), "cuda")
  state = f32(rng.standard_normal((3, taps - 1, channels)), "cuda")

  def run(rows, st):
    ctx = context(ops, "cuda", [before[r] for r in rows], [1] * len(rows), slots=[slots[r] for r in rows],
                  tables=[g.tables for g in manager.groups], page_size=page)
    q = ops.conv_headnorm_rotate_store(
        base[[min(r, 2) for r in rows]].contiguous(), conv, st, norm_w, norm_w, 1e-5, 0.5, None, interleaved=False, num_heads=heads,
        num_kv_heads=kv_heads, head_dim=d, value_dim=dv, storage=storage, block_table=ctx.block_tables[0], ctx=ctx)
    return q, storage.clone()

  st_alone, st_both = state.clone(), state.clone()
  alone, cached = run([0, 1, 2], st_alone)
  both, cached_both = run(list(range(2 + copies)), st_both)
  assert torch.equal(st_alone, st_both) and torch.equal(cached, cached_both)
  assert torch.equal(both[:3], alone) and all(torch.equal(both[2 + c], alone[2]) for c in range(copies))
  ops.check_errors()


# ---- attention: a window with kept first keys, the cap, the one ---------------------------------------------

def _fill(manager, need, rng, before, counts, dtype, device, page):
  """Random keys and values of every request, written as a request's own steps would; what a window has left
  was given back and is poisoned."""
  g, d, dv = need.num_kv_heads, need.head_dim, need.v_dim
  keys = [held(rng.standard_normal((b + n, g, d)), dtype, device) for b, n in zip(before, counts)]
  values = [held(rng.standard_normal((b + n, g, dv)), dtype, device) for b, n in zip(before, counts)]
  storage = manager.paged["c"].storage
  storage.fill_(float("nan"))
  flat = storage.view(storage.shape[0], -1)
  k_view = flat[:, :g * page * d].view(-1, g, page, d)
  v_view = flat[:, g * page * d:].view(-1, g, page, dv)

  def write(b, lo, hi):
    for p in range(lo, hi):
      row = manager.groups[0].tables[b, p // page]
      k_view[row, :, p % page], v_view[row, :, p % page] = keys[b][0][p], values[b][0][p]

  for b, n in enumerate(before):
    assert manager.acquire_slot(b) == b
    for lo in range(0, n, 30):
      manager.extend([(b, min(30, n - lo))])
      write(b, lo, min(lo + 30, n))
  manager.extend(list(enumerate(counts)))
  for b, n in enumerate(before):
    write(b, n, n + counts[b])
  manager.check_invariants()
  return keys, values, storage


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,kv_heads,d,dv,window,keep,cap,page", [
    (4, 2, 16, 16, 20, 3, 5.0, 16), (4, 1, 64, 64, 40, 4, 20.0, 16), (8, 2, 128, 128, 50, 17, 8.0, 16), (6, 3, 64, 32, 33, 70, 0.0, 16),
    (10, 2, 64, 64, 36, 5, 18.0, 64), (4, 2, 96, 48, 100, 1, 3.0, 16), (2, 1, 7, 5, 9, 4, 6.0, 16), (2, 1, 12, 20, 1, 1, 5.0, 16),
    (4, 2, 64, 64, None, 0, 10.0, 16), (4, 4, 32, 112, 30, 0, 10.0, 16), (32, 1, 64, 64, 40, 5, 10.0, 16), (2, 2, 256, 256, 37, 40, 15.0, 64),
    (16, 1, 32, 16, 64, 64, 10.0, 64), (4, 1, 64, 64, 10, 90, 2.0, 8)])
def test_attention_over_a_window_with_kept_first_keys(heads, kv_heads, d, dv, window, keep, cap, page, where):
  ops, dtype = table(where)
  device = where[1]
  rng = np.random.default_rng(5)
  before, counts = [131, 0, 40, 99, 100, 230], [1, 70, 9, 1, 2, 20]
  need = PagedKVNeed(kv_heads, d, window, value_dim=None if dv == d else dv, keep_first=keep)
  manager = CacheManager({"c": need}, page_size=page, max_slots=len(before), max_seq_len=256, max_cache_tokens=6 * 256, dtype=dtype,
                         device=device, poison_freed_pages=True)
  keys, values, storage = _fill(manager, need, rng, before, counts, dtype, device, page)
  ctx = context(ops, device, before, counts, tables=[g.tables for g in manager.groups], page_size=page)
  ctx.older_keys_settled = True
  q, q64 = held(rng.standard_normal((sum(counts), heads, d)) * 2.0 / d ** 0.5, dtype, device)
  m = {"heads": heads, "kv_heads": kv_heads, "scale": 1.0, "softcap": cap, "mask": {"size": window, "keep_first": keep} if window else None}
  starts = np.concatenate([[0], np.cumsum(counts)])
  want = np.concatenate([plain.attend(q64[starts[b]:starts[b + 1]], keys[b][1], values[b][1], m, first=n) for b, n in enumerate(before)])
  more = {"keep_first": keep} if keep else {}
  call = lambda c, qq: f64(ops.paged_attention(
      qq, storage, c.block_tables[0], c, num_heads=heads, num_kv_heads=kv_heads, head_dim=d, logit_softcap=cap, window=window, value_dim=dv,
      sink=torch.zeros(heads, device=device), **more)).reshape(-1, heads, dv)
  got = call(ctx, q)
  bound = 3e-5 if dtype == torch.float32 else 2.5e-2
  assert np.abs(got - want).max() <= bound, np.abs(got - want).max()
  if device == "cuda":
    # the kernels that these shapes do not take by themselves
    for setting, value in (("prefill_tcgen05", False), ("decode_variant", 1), ("decode_variant", 2), ("decode_variant", 16), ("decode_chunk", 64),
                           ("tensor_core_attention", False)):
      kept = getattr(ops, setting)
      setattr(ops, setting, value)
      ctx.memo.clear()
      again = call(ctx, q)
      setattr(ops, setting, kept)
      assert np.abs(again - want).max() <= bound, (setting, value, np.abs(again - want).max())
    ops.check_errors()


@pytest.mark.gpu
def test_the_caps_curve_in_16_bits():
  """Scores from far below to far above the cap in one row: the weights follow the exact tanh on both branches
  of the kernels' own (small arguments, and large ones)."""
  ops, dtype = table(("bfloat16", "cuda"))
  rng = np.random.default_rng(6)
  page, d, n = 16, 64, 200
  for size in (0.3, 3.0):
    need = PagedKVNeed(1, d, 150, keep_first=4)
    manager = CacheManager({"c": need}, page_size=page, max_slots=2, max_seq_len=256, max_cache_tokens=512, dtype=dtype, device="cuda")
    before, counts = [0, n - 1], [n, 1]
    keys, values, storage = _fill(manager, need, rng, before, counts, dtype, "cuda", page)
    ctx = context(ops, "cuda", before, counts, tables=[g.tables for g in manager.groups], page_size=page)
    q, q64 = held(rng.standard_normal((n + 1, 4, d)) * size, dtype, "cuda")
    m = {"heads": 4, "kv_heads": 1, "scale": 1.0, "softcap": 10.0, "mask": {"size": 150, "keep_first": 4}}
    want = np.concatenate([plain.attend(q64[:n], keys[0][1], values[0][1], m), plain.attend(q64[n:], keys[1][1], values[1][1], m, first=n - 1)])
    got = f64(ops.paged_attention(q, storage, ctx.block_tables[0], ctx, num_heads=4, num_kv_heads=1, head_dim=d, logit_softcap=10.0, window=150,
                                  sink=torch.zeros(4, device="cuda"), keep_first=4)).reshape(-1, 4, d)
    assert np.abs(got - want).max() <= 2e-2, (size, np.abs(got - want).max())
  ops.check_errors()


# ---- the router -------------------------------------------------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("experts,top,groups,shift", [
    (12, 4, (2, 1), 0.0), (8, 3, (4, 2), -1.2), (8, 2, (8, 3), 0.0), (64, 6, (8, 4), -0.7), (6, 6, (3, 3), 0.5), (9, 2, (3, 1), -2.0),
    (40, 1, (20, 1), -0.5), (16, 4, None, -0.6), (1, 1, None, 0.0), (96, 12, (2, 1), -0.5)])
def test_experts_of_the_best_groups(experts, top, groups, shift, where):
  ops, dtype = table(where)
  rng = np.random.default_rng(experts)
  width, tokens = 64, 300
  x, x64 = held(rng.standard_normal((tokens, width)), dtype, where[1])
  router = f32(rng.standard_normal((experts, width)) / 6.0, where[1])
  correction = f32(rng.standard_normal(experts) * 0.3 + shift, where[1])  # choice scores below zero among them
  sg = f32(rng.standard_normal(width) / 8.0, where[1])
  r = {"experts": experts, "top": top, "scale": 2.5}
  more = {}
  if groups:
    r["groups"] = {"count": groups[0], "keep": groups[1]}
    if groups[1] < groups[0]:
      more["groups"] = groups
  chosen, weight, gate = ops.route_tokens(x, router, correction, sg, top=top, scale=2.5, score=1, renormalize=True, **more)
  scores = plain.sigmoid(x64 @ f64(router).T)
  for t in range(tokens):
    best, w = plain.choose(scores[t], f64(correction), r)
    assert chosen[t].tolist() == best, t
    close(f64(weight[t]), w, torch.float32, f"weights of token {t}")
  close(f64(gate), plain.sigmoid(x64 @ f64(sg)), torch.float32, "the shared expert's gate")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("tau,rank", [(0.5, 1), (16.0, 12)])
def test_key_decays_and_the_recurrence(tau, rank, where):
  """The whole mixer over one sequence (the scan's own tests stand beside Mononex)."""
  from simply_b200.parts.linear_attention import GatedLinearAttention
  ops, dtype = table(where)
  width, m = 24, {"heads": 3, "dim": 8, "vdim": 16, "tau": tau}
  mixer = GatedLinearAttention("m", width, 3, 8, 16, tau, 1e-3, rank)
  rng = np.random.default_rng(2)
  w, w64 = {}, {}
  for s in mixer.tensor_specs():
    w[s.name], w64[s.name] = held(rng.standard_normal(s.shape) / width ** 0.5 + (1.0 if s.name.endswith("norm") else 0.0), dtype, where[1])
  mixer.bind(w, ops)
  x, x64 = held(rng.standard_normal((50, width)), dtype, where[1])
  state = torch.zeros((2, 3, 8, 16), device=where[1])
  got, at = [], 0
  for n in (20, 1, 2, 1, 26):
    ctx = context(ops, where[1], [at], [n], slots=[1])
    got.append(f64(mixer.forward(x[at:at + n].contiguous(), ctx, types.SimpleNamespace(storage=state))))
    at += n
  close(np.concatenate(got), plain.gated_linear_attention(x64, m, w64, "m", 1e-3), dtype, "the mixer", f32=5e-5)


# ---- the books of a cache that keeps first tokens -----------------------------------------------------------

@pytest.mark.parametrize("window,keep,page", [(12, 3, 8), (7, 5, 4), (64, 4, 64), (1, 1, 4), (100, 30, 16), (5, 70, 16), (9, 0, 4)])
def test_kept_pages_stay_and_windowed_pages_go(window, keep, page):
  need = PagedKVNeed(2, 8, window, keep_first=keep)
  assert need.kept_pages(page) == -(-keep // page)
  manager = CacheManager({"c": need}, page_size=page, max_slots=3, max_seq_len=400, max_cache_tokens=1200, device=None)
  g = manager.groups[0]
  rng = np.random.default_rng(0)
  slots = [manager.acquire_slot(i) for i in range(2)]
  for step in range(120):
    for s in slots:
      n = int(rng.integers(1, 9))
      if manager.length(s) + n <= 400 and rng.random() < 0.9:
        before = manager.length(s)
        manager.extend([(s, n)])
        # a key is held if a query of this step sees it
        for q in (before, before + n - 1):
          for j in {0, max(keep - 1, 0), max(q - window + 1, 0), q}:
            if j <= q and (q - j < window or j < keep):
              assert g.tables[s, j // page] >= 0, (q, j)
        held_pages = len(g.held_pages(s))
        most = -(-keep // page) + -(-(window + n) // page) + 2
        assert held_pages <= most, (held_pages, most)
    manager.check_invariants()
    if step % 40 == 39:  # a slot is freed and used again
      manager.release_slot(slots[0])
      slots[0] = manager.acquire_slot(step)
  for s in slots:
    manager.release_slot(s)
  assert manager.all_pages_free()


def test_needs_with_kept_tokens_share_pages_only_with_their_like():
  a, b, c = PagedKVNeed(2, 8, 16, keep_first=4), PagedKVNeed(4, 16, 16, keep_first=4), PagedKVNeed(2, 8, 16)
  assert a.group_key() == b.group_key() != c.group_key() and PagedKVNeed(2, 8, None, keep_first=4).group_key() == PagedKVNeed(2, 8).group_key()
  assert a.covers(c) and not c.covers(a) and PagedKVNeed(2, 8).covers(a)
  pages = dict(page_size=4, max_slots=2, max_seq_len=640, all_pages=1000, step_tokens=16, burst_tokens=8)
  assert a.pool_pages(**pages) == c.pool_pages(**pages) + 2 * 1
