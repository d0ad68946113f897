"""The Pibulix decoder through the engine against the plain NumPy model.

Each scenario runs on the CPU with the plain PyTorch kernel statements (this checks the parts,
the configuration, the cache manager and the step function) and, marked `gpu`, with the CUDA
kernels in float32 and bfloat16."""

import copy
import json
import os

import numpy as np
import pytest
import torch

from simply_b200 import Engine, EngineConfig, SamplingParams, StepEntry
from simply_b200.config import ConfigError, config_from_dict, load_config
from simply_b200.parts.model import DecoderModel
from simply_b200.weights import write_model_folder
from tests import pibulix_cases as px
from tests.plain import pibulix_plain as plain
from tests.reference_ops import ReferenceOps

CPU = pytest.param(("float32", "cpu"), id="cpu")
GPU32 = pytest.param(("float32", "cuda"), id="gpu-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param(("bfloat16", "cuda"), id="gpu-bf16", marks=pytest.mark.gpu)
WHERE = [CPU, GPU32, GPU16]
CONFIGS = {"a": px.CONFIG_A, "b": px.CONFIG_B, "c": px.CONFIG_C, "d": px.CONFIG_D}


def engine_for(cfg_dict, where, seed=0, tensors=None, **kw):
  dtype, device = where
  cfg, t = px.weights(cfg_dict, seed)
  if tensors is not None:
    t = tensors
  ops = ReferenceOps(torch.float32) if device == "cpu" else None
  return px.build_engine(cfg, t, dtype, device, ops, **kw), t


def random_tokens(cfg_dict, n, seed):
  return np.random.default_rng(seed).integers(0, cfg_dict["vocab"], n).tolist()


# ---- whole prompts, portions, decoding, batches -------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_whole_portions_and_decoding(which, where):
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, where, seed=3, poison=True)
  toks = px.tokens(cfg_dict, t, 61, 1)
  want = plain.forward(cfg_dict, px.as_numpy(t), toks)
  n = len(toks)
  for what, cuts in [
      ("whole", [n]),
      ("token by token", [1] * n),
      ("prompt then decoding", [n - 40] + [1] * 40),
      ("portions down to two tokens", px.cuts_of(n, [7, 2, 5, 3, 11, 2, 13, 4, 2, 9])),
      ("portions that end at the pages' and the windows' borders", px.cuts_of(n, [8, 4, 8, 1, 7, 9, 16, 2])),
      ("portions of two", [2] * (n // 2) + [1]),
      ("one token, then the rest", [1, n - 1]),
      ("the kept tokens, then the rest", [3, n - 3]),
  ]:
    px.check_close(px.run_cuts(engine, toks, cuts), want, where[0], f"{which}: {what}")
  engine.cache.check_invariants()
  assert engine.cache.all_pages_free()
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b"])
def test_the_stream_after_every_layer(which, where):
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, where, seed=5)
  toks = px.tokens(cfg_dict, t, 30, 2)
  want = []
  plain.forward(cfg_dict, px.as_numpy(t), toks, want)
  slot = engine.open_request()
  at, got = 0, [[] for _ in want]
  for n in (11, 2, 1, 16):
    ctx = engine._prepare([StepEntry(slot, toks[at:at + n], ())])
    streams = ctx.memo["layer_outputs"] = []
    engine.model.forward(ctx, engine.caches)
    for layer, s in enumerate(streams):
      got[layer].append(s.float().cpu().numpy())
    at += n
  engine.close_request(slot)
  for layer, parts in enumerate(got):
    px.check_close(np.concatenate(parts), want[layer], where[0], f"{which}: stream after layer {layer}")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b", "c"])
def test_unequal_requests_side_by_side_with_pages_and_slots_used_again(which, where):
  cfg_dict = CONFIGS[which]
  # room for three live requests of these lengths, not for all six: pages and slots come back
  engine, t = engine_for(cfg_dict, where, seed=5, slots=3, max_cache_tokens=3 * 80, poison=True)
  lengths = [70, 9, 33, 1, 58, 21]
  requests = [px.tokens(cfg_dict, t, n, 10 + i) for i, n in enumerate(lengths)]
  w = px.as_numpy(t)
  want = [plain.forward(cfg_dict, w, r) for r in requests]
  got = px.run_mixed(engine, requests, seed=2)
  for i, (g, x) in enumerate(zip(got, want)):
    px.check_close(g, x, where[0], f"request {i} in a mixed batch")
  # the same requests once more through the used slots and pages, each alone
  for i in (0, 4):
    px.check_close(px.run_cuts(engine, requests[i], [len(requests[i])]), want[i], where[0], f"request {i} again")
  engine.cache.check_invariants()
  assert engine.cache.all_pages_free()
  engine.ops.check_errors()


@pytest.mark.gpu
def test_a_batch_gives_the_same_numbers_every_time():
  """Short requests beside longer ones in steps of a few tokens, three times over: bit for bit."""
  cfg_dict = px.config([px.attention(dim=64, vdim=64, window=20), px.gla(), px.attention(dim=32, vdim=16, window=9, keep_first=2)],
                       [px.dense(32), px.dense(32), px.dense(32)], width=64, vocab=90)
  engine, t = engine_for(cfg_dict, ("bfloat16", "cuda"), seed=1, page_size=16)
  requests = [random_tokens(cfg_dict, n, 60 + i) for i, n in enumerate((5, 40, 17, 9))]
  want = [plain.forward(cfg_dict, px.as_numpy(t), r) for r in requests]
  runs = [px.run_mixed(engine, requests, seed=6, max_live=4, portions=(2, 3)) for _ in range(3)]
  for i, x in enumerate(want):
    px.check_close(runs[0][i], x, "bfloat16", f"request {i}")
    assert np.array_equal(runs[0][i], runs[1][i]) and np.array_equal(runs[0][i], runs[2][i]), f"request {i} differs between runs"


@pytest.mark.parametrize("where", WHERE)
def test_long_decoding_past_many_pages(where):
  """150 tokens over pages of 4: windows of 12 and 7 tokens pass over decoded tokens, the pages they
  leave are given back on the way, those of the kept first tokens stay."""
  cfg_dict = px.CONFIG_A
  engine, t = engine_for(cfg_dict, where, seed=7, page_size=4, poison=True)
  toks = px.tokens(cfg_dict, t, 150, 4)
  want = plain.forward(cfg_dict, px.as_numpy(t), toks)
  px.check_close(px.run_cuts(engine, toks, [3] + [1] * 147), want, where[0], "long decoding")
  engine.cache.check_invariants()
  engine.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_pages_of_64_and_sizes_of_the_tensor_core_kernels(dtype):
  """500 tokens over pages of 64: the tcgen05 prefill kernel (groups that divide 128), the mma.sync kernels
  (a group of three, two sizes), the split-key kernels with and without TMA; kept tokens within a page,
  across pages and across a tile of 64; a recurrence of 128 channels; experts for a long portion."""
  cfg_dict = px.config(
      [px.attention(heads=8, kv_heads=2, dim=64, vdim=64, window=150, keep_first=5, dims=32, base=1e4, softcap=12.0, scale=0.2),
       px.attention(heads=4, kv_heads=1, dim=128, vdim=128, window=90, keep_first=70, dims=128, base=1e5, conv=4, scale=0.12),
       px.attention(heads=6, kv_heads=2, dim=96, vdim=48, window=70, keep_first=130, dims=48, softcap=None, conv=2, scale=0.15),
       px.gla(heads=2, dim=128, vdim=64, tau=12.0),
       px.attention(heads=3, kv_heads=1, dim=32, vdim=32, window=33, keep_first=4, scale=0.25), 1],
      [px.dense(192), None, px.moe(ff=64, experts=8, top=2, groups=(2, 1), shared=32), px.dense(128), px.dense(64), None],
      width=128, vocab=300, rank=16)
  cfg, t = px.weights(cfg_dict, seed=3)
  engine = px.build_engine(cfg, t, dtype, "cuda", None, page_size=64, slots=2, max_seq_len=512, poison=True)
  toks = px.tokens(cfg_dict, t, 500, 1)
  want = plain.forward(cfg_dict, px.as_numpy(t), toks)
  for what, cuts in [("whole", [500]), ("portions", px.cuts_of(500, [100, 2, 37, 64, 3, 129, 200])),
                     ("decoding", [440] + [1] * 60)]:
    px.check_close(px.run_cuts(engine, toks, cuts), want, dtype, what)
  engine.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_step_of_more_than_a_thousand_tokens(dtype):
  """Enough tokens for blocks that serve several tokens and for experts one by one; two requests in one step, then
  single tokens and a second long portion."""
  cfg_dict = px.config(
      [px.attention(heads=8, kv_heads=2, dim=64, vdim=64, window=300, keep_first=5, dims=32, base=1e4, softcap=12.0, scale=0.2),
       px.gla(heads=2, dim=64, vdim=32), px.attention(heads=3, kv_heads=1, dim=32, vdim=48, window=90, keep_first=70, dims=16, conv=4), 1],
      [px.moe(ff=64, experts=4, top=4, groups=(2, 2), shared=32), px.dense(64), px.moe(ff=32, experts=3, top=3, groups=None), None],
      width=64, vocab=300, max_context=4096)  # (every expert is chosen: no close calls)
  cfg, t = px.weights(cfg_dict, seed=3)
  engine = px.build_engine(cfg, t, dtype, "cuda", None, page_size=64, slots=2, max_seq_len=2560, poison=True)
  requests = [random_tokens(cfg_dict, n, i) for i, n in enumerate((2450, 143))]
  w = px.as_numpy(t)
  want = [plain.forward(cfg_dict, w, r) for r in requests]
  slots, got, at = [engine.open_request() for _ in requests], [[], []], [0, 0]
  for portions in ((1301, 61), (2, 1), (1, 1), (1, 80), (1145, 0)):
    entries = [StepEntry(slots[i], requests[i][at[i]:at[i] + n], tuple(range(n))) for i, n in enumerate(portions) if n]
    rows = engine.step_raw(entries).float().cpu().numpy()
    for i, n in enumerate(portions):
      got[i].append(rows[:n])
      rows, at[i] = rows[n:], at[i] + n
  for i in range(2):
    px.check_close(np.concatenate(got[i]), want[i], dtype, f"request {i}")
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
def test_many_query_heads_per_kv_head(where):
  """32 and 12 query heads per kv head: a single token's rows no longer fit the split-key kernel's
  16, so decoded tokens take the tile kernels too."""
  cfg_dict = px.config(
      [px.attention(heads=32, kv_heads=1, dim=64, vdim=64, window=50, keep_first=6, scale=0.2),
       px.attention(heads=24, kv_heads=2, dim=32, vdim=16, window=31, keep_first=2, scale=0.25)],
      [px.dense(64), px.dense(64)], width=64, vocab=90)
  engine, t = engine_for(cfg_dict, where, seed=8, page_size=16, max_seq_len=128, poison=True)
  toks = random_tokens(cfg_dict, 90, 2)
  want = plain.forward(cfg_dict, px.as_numpy(t), toks)
  for what, cuts in [("whole", [90]), ("decoding", [60] + [1] * 30), ("portions", px.cuts_of(90, [17, 2, 40, 3]))]:
    px.check_close(px.run_cuts(engine, toks, cuts), want, where[0], what)
  engine.ops.check_errors()


# ---- a key that stands out -----------------------------------------------------------------------------

NEEDLES = [(4, 16, 16, 8, 4), (2, 64, 64, 64, 4), (6, 32, 48, 16, 20), (2, 12, 10, 8, 1), (8, 128, 128, 64, 70)]


@pytest.mark.parametrize("where,sizes", [
    pytest.param(w.values[0], sizes, id=f"{w.id}-{sizes[1]}-{sizes[2]}", marks=w.marks)
    for w in WHERE for sizes in (NEEDLES[:1] if w is CPU else NEEDLES)])
def test_a_key_that_stands_out_at_every_edge(where, sizes):
  """A query answered by one key among many: the last kept token and the next one, the window's oldest
  key and the one just behind it, keys at pages' borders; asked in portions of prompts and by a token
  decoded alone."""
  heads, dim, vdim, page, keep = sizes
  window, n = (40, 110) if where[1] == "cpu" else (100, 330)
  layer = px.attention(heads=heads, kv_heads=2, dim=dim, vdim=vdim, window=window, keep_first=keep, dims=dim // 4 * 2, softcap=20.0,
                       scale=1.2 * (16 / dim) ** 0.5)
  cfg_dict = px.config([layer], [px.dense(32)], width=32, vocab=50, alpha=0.5)
  cfg, t = px.weights(cfg_dict, seed=11)
  px.plant_needle(cfg_dict, t, 0, needle=2, asker=1, strength=14.0 * (dim / 16) ** 0.5)
  w = px.as_numpy(t)
  engine, _ = engine_for(cfg_dict, where, tensors=t, page_size=page, max_seq_len=512, poison=True)
  rng = np.random.default_rng(0)
  mid = n - window // 2
  cases = {(0, 1), (0, n - 1), (keep - 1, n - 1), (keep, n - 1), (keep - 1, mid), (keep, mid), (n - window, n - 1),
           (n - 1 - window, n - 1), (64, 63 + window), (63, 63 + window), (mid - 1, mid)}
  if where[1] == "cuda":
    cases |= {(127, 226), (128, 228), (160, 191), (100, 200), (101, 200)}
  for needle_at, ask_at in sorted(c for c in cases if c[0] < c[1]):
    toks = rng.integers(3, cfg_dict["vocab"], n).tolist()
    toks[needle_at], toks[ask_at] = 2, 1
    want = plain.forward(cfg_dict, w, toks)
    without = list(toks)
    without[needle_at] = 5
    decides = np.abs(plain.forward(cfg_dict, w, without)[ask_at] - want[ask_at]).max() > 0.03 * np.abs(want).max()
    assert decides == (ask_at - needle_at < window or needle_at < keep), (needle_at, ask_at)
    for cuts in ([n], [ask_at, 1, n], [max(ask_at - 1, 1), 2, n], [needle_at + 1, ask_at - needle_at - 1] + [1] * 4 + [n]):
      got = px.run_cuts(engine, toks, [c for c in cuts if c > 0])
      px.check_close(got, want, where[0], f"needle at {needle_at}, asked at {ask_at}, cuts {cuts[:3]}")
  engine.cache.check_invariants()
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
def test_the_one_in_the_denominator_and_the_cap_decide(where):
  """Few keys, whose scores the cap brings down: the one in the denominator takes a good part of the weight."""
  def attend_without_the_one(q, k, v, m):
    out = np.zeros(q.shape[:2] + (v.shape[2],))
    for i in range(q.shape[0]):
      seen = [j for j in range(i + 1) if plain.sees(i, j, m["mask"])]
      for a in range(m["heads"]):
        e = np.exp(m["softcap"] * np.tanh((k[seen, 0] @ q[i, a]) * m["scale"] / m["softcap"]))
        out[i, a] = (e / e.sum()) @ v[seen, 0]
    return out

  toks = np.random.default_rng(2).integers(0, 50, 60).tolist()
  wants = {}
  for cap in (1.0, 6.0):
    cfg_dict = px.config([px.attention(heads=2, kv_heads=1, dim=16, vdim=16, window=4, keep_first=1, softcap=cap, scale=0.8)], [None],
                         width=32, vocab=50, alpha=0.5)
    engine, t = engine_for(cfg_dict, where, seed=4, page_size=8, max_seq_len=256)
    w = px.as_numpy(t)
    want = wants[cap] = plain.forward(cfg_dict, w, toks)
    for cuts in ([60], [55, 1, 4], px.cuts_of(60, [9, 2, 31]), [1] * 60):
      px.check_close(px.run_cuts(engine, toks, cuts), want, where[0], f"cap {cap}, cuts {cuts[:3]}")
    real = plain.attend
    try:
      plain.attend = attend_without_the_one
      other = plain.forward(cfg_dict, w, toks)
    finally:
      plain.attend = real
    assert np.abs(other - want).max() > 0.1 * np.abs(want).max()
  assert np.abs(wants[1.0] - wants[6.0]).max() > 0.1 * np.abs(wants[1.0]).max()


@pytest.mark.parametrize("where", WHERE)
def test_a_convolutions_state_crosses_portions(where):
  """Taps that look back as far as they can and hardly at the token itself: a lost or stale row shows."""
  for taps in (2, 3, 4, 6):
    cfg_dict = px.config([px.attention(conv=taps, window=30), px.gla()], [px.dense(24), px.dense(24)], width=32, vocab=40)
    cfg, t = px.weights(cfg_dict, seed=taps)
    for name in t:
      if name.endswith(".conv"):
        t[name] = t[name].clone()
        t[name][:, 0], t[name][:, -1] = 1.0, 0.1
    engine, _ = engine_for(cfg_dict, where, tensors=t, slots=2, poison=True)
    w = px.as_numpy(t)
    requests = [random_tokens(cfg_dict, n, taps + i) for i, n in enumerate((31, 12, 2, 1, 25))]
    want = [plain.forward(cfg_dict, w, r) for r in requests]
    for cuts in ([1] * 31, px.cuts_of(31, [2, 1, 3]), [taps - 1, 31], px.cuts_of(31, [1, 2])):
      px.check_close(px.run_cuts(engine, requests[0], cuts), want[0], where[0], f"{taps} taps, cuts {cuts[:3]}")
    got = px.run_mixed(engine, requests, seed=taps, max_live=2, portions=(2, 3))
    for i, x in enumerate(want):
      px.check_close(got[i], x, where[0], f"{taps} taps, request {i}")
    engine.ops.check_errors()


# ---- generation through the entry point and the scheduler -----------------------------------------

def _greedy(cfg_dict, w, prompt, n):
  toks = list(prompt)
  for _ in range(n):
    toks.append(int(np.argmax(plain.forward(cfg_dict, w, toks)[-1])))
  return toks[len(prompt):]


@pytest.mark.parametrize("where", [CPU, GPU32])
def test_greedy_generation_through_the_scheduler(where):
  cfg_dict = px.CONFIG_B
  engine, t = engine_for(cfg_dict, where, seed=9, slots=2)
  w = px.as_numpy(t)
  prompts = [random_tokens(cfg_dict, n, 30 + i) for i, n in enumerate((5, 17, 1, 26))]
  results = engine.generate(prompts, SamplingParams(temperature=0.0, max_decode_steps=12))
  for prompt, r in zip(prompts, results):
    assert r.output_token_ids == _greedy(cfg_dict, w, prompt, 12)
  assert engine.cache.all_pages_free()


@pytest.mark.parametrize("where", [CPU, GPU32])
def test_generation_in_a_pool_that_makes_requests_wait(where):
  """The step's budget cuts prompts into portions and the pool has no room for all requests at once."""
  cfg_dict = px.CONFIG_A
  cfg, t = px.weights(cfg_dict, 21)
  dtype, device = where
  ec = EngineConfig(activation_dtype=dtype, page_size=4, batch_size=3, max_seq_len=64, max_cache_tokens=96, max_num_issue_tokens=9,
                    poison_freed_pages=True, use_cuda_graphs=False)
  ops = ReferenceOps(torch.float32) if device == "cpu" else None
  engine = Engine(cfg, {k: v.to(device=device, dtype=getattr(torch, dtype)) for k, v in t.items()}, ec, ops=ops, device=device)
  w = px.as_numpy(t)
  prompts = [random_tokens(cfg_dict, n, 70 + i) for i, n in enumerate((30, 3, 22, 11))]
  results = engine.generate(prompts, SamplingParams(temperature=0.0, max_decode_steps=10))
  for prompt, r in zip(prompts, results):
    assert r.output_token_ids == _greedy(cfg_dict, w, prompt, 10)
  engine.cache.check_invariants()
  assert engine.cache.all_pages_free()


@pytest.mark.gpu
@pytest.mark.parametrize("which,burst", [("a", 1), ("b", 5)])
def test_decoding_from_cuda_graphs(which, burst):
  """Three live requests decode from the graph of four rows (the fourth repeats the third),
  several steps per replay burst."""
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, ("float32", "cuda"), seed=13, slots=4, graphs=True, burst=burst)
  assert engine._decode_runner is not None, "the model's parts must all allow graph capture"
  w = px.as_numpy(t)
  prompts = [random_tokens(cfg_dict, n, 40 + i) for i, n in enumerate((9, 3, 14))]
  results = engine.generate(prompts, SamplingParams(temperature=0.0, max_decode_steps=17))
  assert engine._decode_runner.bursts > 0
  for prompt, r in zip(prompts, results):
    assert r.output_token_ids == _greedy(cfg_dict, w, prompt, 17)
  engine.ops.check_errors()


@pytest.mark.gpu
def test_bfloat16_generation_runs_and_samples():
  engine, _ = engine_for(px.CONFIG_A, ("bfloat16", "cuda"), seed=2, slots=3)
  prompts = [random_tokens(px.CONFIG_A, n, i) for i, n in enumerate((4, 30, 11, 2, 19))]
  results = engine.generate(prompts, SamplingParams(temperature=0.8, top_k=20, max_decode_steps=20, seed=4))
  assert all(len(r.output_token_ids) == 20 for r in results)
  again = engine.generate(prompts, SamplingParams(temperature=0.8, top_k=20, max_decode_steps=20, seed=4))
  assert [r.output_token_ids for r in results][0] == [r.output_token_ids for r in again][0]
  engine.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_tokens_replayed_from_cuda_graphs(dtype):
  """Past the edges of windows of 50 and 33 tokens with kept ones before them (some further than a chunk of
  the split-key kernel), with a row that repeats the last request."""
  cfg_dict = px.config(
      [px.attention(heads=4, kv_heads=2, dim=64, vdim=64, window=50, keep_first=4, scale=0.2), px.gla(heads=2, dim=32, vdim=32),
       px.attention(heads=4, kv_heads=1, dim=48, vdim=32, window=33, keep_first=20, scale=0.25, conv=2), 0],
      [px.dense(64), px.dense(64), px.moe(experts=4, top=2, groups=(2, 1)), None], width=64, vocab=120)
  engine, t = engine_for(cfg_dict, (dtype, "cuda"), seed=6, slots=4, graphs=True, page_size=16, max_seq_len=512)
  assert engine._decode_runner is not None
  engine._decode_runner.keep_logits = True
  w = px.as_numpy(t)
  requests = [px.tokens(cfg_dict, t, n, 50 + i) for i, n in enumerate((120, 71, 345))]
  want = [plain.forward(cfg_dict, w, r) for r in requests]
  slots = [engine.open_request() for _ in requests]
  heads = [len(r) - 60 for r in requests]
  engine.step_raw([StepEntry(s, r[:h], ()) for s, r, h in zip(slots, requests, heads)])
  got = [[] for _ in requests]
  for step in range(60):
    entries = [StepEntry(s, [r[h + step]], (0,)) for s, r, h in zip(slots, requests, heads)]
    logits = engine.step_raw(entries, from_graph=True).float().cpu().numpy()
    for i in range(len(requests)):
      got[i].append(logits[i])
  for i, h in enumerate(heads):
    px.check_close(np.stack(got[i]), want[i][h:], dtype, f"request {i}, replayed steps")
  engine.ops.check_errors()


# ---- configuration, model folders, the preset ---------------------------------------------------------

def test_config_round_trip_caches_and_errors():
  for d in CONFIGS.values():
    cfg = config_from_dict(d)
    assert config_from_dict(cfg.to_dict()) == cfg
  spec = config_from_dict(px.CONFIG_A).model_spec()
  assert [c.layer for c in spec.run_order] == ["l0", "l1", "l0", "l3", "l1", "l5"]
  needs = DecoderModel(spec).cache_needs()
  assert set(needs) == {"l0#0", "l1#1", "l0#2", "l3#3", "l1#4", "l5#5"}  # a cache or state per layer, shared tensors or not
  assert needs["l0#0"]["kv"].window == 12 and needs["l0#0"]["kv"].keep_first == 3 and needs["l0#0"]["conv"].shape == (2, 128)
  names = {s.name for s in DecoderModel(spec).tensor_specs()}
  assert "l0.mix.q.conv" in names and "l3.mix.k.norm" in names and not any(n.startswith(("l2.", "l4.")) for n in names)
  specs_b = {s.name: s for s in DecoderModel(config_from_dict(px.CONFIG_B).model_spec()).tensor_specs()}
  assert specs_b["l1.norm2"].optional and not specs_b["l0.norm2"].optional  # no feed-forward: its norm may be absent
  for change, text in [
      (lambda d: d["layers"][0].update(type="conv"), "unknown type"),
      (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
      (lambda d: d["layers"][2].update(weights_of=9), "weights_of"),
      (lambda d: d["layers"][2].update(weights_of=2), "weights_of"),
      (lambda d: d["layers"][2]["mixer"].update(dim=32), "mixer differs from layer 0"),
      (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=5), "rot.dims"),
      (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
      (lambda d: d["layers"][1]["mixer"].pop("tau"), "tau"),
      (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
      (lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
      (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups.count"),
      (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "fewer experts"),
      (lambda d: d["layers"][3]["mlp"].update(kind="sparse"), "unknown mlp kind"),
      (lambda d: d.pop("postln_alpha"), "postln_alpha"),
      (lambda d: d.pop("norm"), "norm"),
  ]:
    d = copy.deepcopy(px.CONFIG_A)
    change(d)
    with pytest.raises(ConfigError, match=text):
      config_from_dict(d)


def test_model_folder_and_the_step_function_on_it(tmp_path):
  cfg = config_from_dict(px.CONFIG_B)
  folder = write_model_folder(cfg, 4, str(tmp_path / "m"), matrix_std=0.2, scale_std=0.1)
  assert load_config(folder) == cfg
  with open(os.path.join(folder, "config.json")) as f:
    assert json.load(f)["architecture"] == "Pibulix"
  ec = EngineConfig(activation_dtype="float32", page_size=8, batch_size=2, max_seq_len=64, use_cuda_graphs=False)
  engine = Engine.from_folder(folder, ec, ops=ReferenceOps(torch.float32), device="cpu")
  from simply_b200.weights import safetensors_io as st
  entries = st.index_files(st.model_files(folder))
  reader = st.TensorReader(entries)
  w = {n: reader.read(n).float().numpy().astype(np.float64) for n in entries}
  toks = random_tokens(px.CONFIG_B, 19, 3)
  slot = engine.open_request()
  got = engine.step_raw([StepEntry(slot, toks, tuple(range(len(toks))))]).numpy()
  engine.close_request(slot)
  px.check_close(got, plain.forward(px.CONFIG_B, w, toks), "float32", "a written folder")


def test_the_preset_generates_from_random_weights():
  from simply_b200.config import preset
  cfg = preset("pibulix-tiny")
  assert cfg.architecture == "Pibulix" and {l["type"] for l in cfg.layers} == {"attention", "gla"}
  ec = EngineConfig(activation_dtype="float32", page_size=8, batch_size=2, max_seq_len=64, use_cuda_graphs=False)
  engine = Engine.from_config(cfg, 1, ec, matrix_std=0.2, ops=ReferenceOps(torch.float32), device="cpu")
  results = engine.generate([[1, 2, 3], [7]], SamplingParams(temperature=0.0, max_decode_steps=5))
  assert [len(r.output_token_ids) for r in results] == [5, 5]
