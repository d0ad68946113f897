"""The Mononex decoder through the engine against the plain NumPy model.

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
from tests import mononex_cases as mx
from tests.plain import mononex_plain as plain
from tests.reference_ops import ReferenceOps

CPU = pytest.param(("float32", "cpu"), id="cpu")
GPU32 = pytest.param(("float32", "cuda"), id="gpu-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param(("bfloat16", "cuda"), id="gpu-bf16", marks=pytest.mark.gpu)
WHERE = [CPU, GPU32, GPU16]
CONFIGS = {"a": mx.CONFIG_A, "b": mx.CONFIG_B, "c": mx.CONFIG_C, "d": mx.CONFIG_D}


def engine_for(cfg_dict, where, seed=0, tensors=None, **kw):
  dtype, device = where
  cfg, t = mx.weights(cfg_dict, seed)
  if tensors is not None:
    t = tensors
  ops = ReferenceOps(torch.float32) if device == "cpu" else None
  return mx.build_engine(cfg, t, dtype, device, ops, **kw), t


def tokens_for(cfg_dict, n, seed):
  return np.random.default_rng(seed).integers(0, cfg_dict["vocab"], n).tolist()


# ---- whole prompts, portions, decoding, batches -------------------------------------------------

@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_whole_portions_and_decoding(which, where):
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, where, seed=3)
  toks = tokens_for(cfg_dict, 61, 1)
  want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
  n = len(toks)
  for what, cuts in [
      ("whole", [n]),
      ("token by token", [1] * n),
      ("prompt then decoding", [n - 40] + [1] * 40),
      ("portions down to two tokens", mx.cuts_of(n, [7, 2, 5, 3, 11, 2, 13, 4, 2, 9])),
      ("portions that end at the pages' and the chunks' borders", mx.cuts_of(n, [8, 4, 8, 1, 7, 9, 16, 2])),
      ("portions of two", [2] * (n // 2) + [1]),
      ("one token, then the rest", [1, n - 1]),
  ]:
    mx.check_close(mx.run_cuts(engine, toks, cuts), want, where[0], f"{which}: {what}")
  engine.cache.check_invariants()
  assert engine.cache.all_pages_free()
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b"])
def test_the_stream_after_every_layer(which, where):
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, where, seed=4)
  toks = tokens_for(cfg_dict, 30, 2)
  want = []
  plain.forward(cfg_dict, mx.as_numpy(t), toks, want)
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
    mx.check_close(np.concatenate(parts), want[layer], where[0], f"{which}: stream after layer {layer}")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("which", ["a", "b", "c"])
def test_unequal_requests_side_by_side_with_pages_and_slots_used_again(which, where):
  cfg_dict = CONFIGS[which]
  # room for three live requests of these lengths, not for all six: pages and slots come back
  engine, t = engine_for(cfg_dict, where, seed=5, slots=3, max_cache_tokens=3 * 80, poison=True)
  lengths = [70, 9, 33, 1, 58, 21]
  requests = [tokens_for(cfg_dict, n, 10 + i) for i, n in enumerate(lengths)]
  w = mx.as_numpy(t)
  want = [plain.forward(cfg_dict, w, r) for r in requests]
  got = mx.run_mixed(engine, requests, seed=2)
  for i, (g, x) in enumerate(zip(got, want)):
    mx.check_close(g, x, where[0], f"request {i} in a mixed batch")
  # the same requests once more through the used slots and pages, each alone
  for i in (0, 4):
    mx.check_close(mx.run_cuts(engine, requests[i], [len(requests[i])]), want[i], where[0], f"request {i} again")
  engine.cache.check_invariants()
  assert engine.cache.all_pages_free()
  engine.ops.check_errors()


@pytest.mark.gpu
def test_a_batch_gives_the_same_numbers_every_time():
  """Short requests beside longer ones in steps of a few tokens, three times over: bit for bit."""
  cfg_dict = mx.config([mx.latent(heads=8, dim=16, rot_dim=16, vdim=16, q_rank=32, kv_rank=64), mx.gla(), mx.attention(dim=32, vdim=16)],
                       [32, 32, 32], width=64, vocab=90)
  engine, t = engine_for(cfg_dict, ("bfloat16", "cuda"), seed=1, page_size=16)
  requests = [tokens_for(cfg_dict, n, 60 + i) for i, n in enumerate((5, 40, 17, 9))]
  want = [plain.forward(cfg_dict, mx.as_numpy(t), r) for r in requests]
  runs = [mx.run_mixed(engine, requests, seed=6, max_live=4, portions=(2, 3)) for _ in range(3)]
  for i, x in enumerate(want):
    mx.check_close(runs[0][i], x, "bfloat16", f"request {i}")
    assert np.array_equal(runs[0][i], runs[1][i]) and np.array_equal(runs[0][i], runs[2][i]), f"request {i} differs between runs"


@pytest.mark.parametrize("where", WHERE)
def test_long_decoding_past_many_pages_and_chunks(where):
  """150 tokens over pages of 4: chunks of 12 and 7 tokens begin many times in decoded tokens and
  the pages before them are given back on the way."""
  cfg_dict = mx.CONFIG_A
  engine, t = engine_for(cfg_dict, where, seed=7, page_size=4)
  toks = tokens_for(cfg_dict, 150, 4)
  want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
  mx.check_close(mx.run_cuts(engine, toks, [3] + [1] * 147), want, where[0], "long decoding")
  engine.cache.check_invariants()
  engine.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_pages_of_64_and_sizes_of_the_tensor_core_kernels(dtype):
  """500 tokens over pages of 64: the tcgen05 prefill kernel (equal sizes of 64 and 128), the mma.sync
  kernels (two sizes, and sizes that are no multiple of 64), the kernel over latents; chunks that end
  inside a page and that span several, one without chunks, a recurrence of 128 channels."""
  cfg_dict = mx.config(
      [mx.attention(heads=8, kv_heads=2, dim=64, vdim=64, chunk=150, scale=0.1),
       mx.attention(heads=8, kv_heads=2, dim=64, vdim=64, chunk=90, scale=0.12, kv_from=0),
       mx.attention(heads=4, kv_heads=1, dim=128, vdim=128, chunk=None, scale=0.08),
       mx.latent(heads=8, dim=32, rot_dim=16, vdim=32, q_rank=64, kv_rank=64, base=10000.0, original=128, fast=8.0, slow=1.0, scale=0.15),
       mx.attention(heads=6, kv_heads=2, dim=96, vdim=48, chunk=70, scale=0.1),
       mx.gla(heads=2, dim=128, vdim=64, tau=12.0),
       mx.attention(heads=4, kv_heads=4, dim=32, vdim=80, chunk=200, scale=0.15)],
      [192, None, 96, 128, 64, 64, 64], width=128, vocab=300, rank=16)
  cfg, t = mx.weights(cfg_dict, seed=3)
  engine = mx.build_engine(cfg, t, dtype, "cuda", None, page_size=64, slots=2, max_seq_len=512)
  toks = tokens_for(cfg_dict, 500, 1)
  want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
  for what, cuts in [("whole", [500]), ("portions", mx.cuts_of(500, [100, 2, 37, 64, 3, 129, 200])),
                     ("decoding", [440] + [1] * 60)]:
    mx.check_close(mx.run_cuts(engine, toks, cuts), want, dtype, what)
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
def test_many_query_heads_per_kv_head(where):
  """32 and 12 query heads per kv head: a single token's rows no longer fit the split-key kernel's
  16, so decoded tokens take the tile kernels too; and 40 heads over one latent."""
  cfg_dict = mx.config(
      [mx.attention(heads=32, kv_heads=1, dim=64, vdim=64, chunk=50, scale=0.12),
       mx.attention(heads=24, kv_heads=2, dim=32, vdim=16, chunk=31, scale=0.2),
       mx.latent(heads=40, dim=8, rot_dim=16, vdim=8, q_rank=16, kv_rank=32)],
      [64, None, 32], width=64, vocab=90)
  engine, t = engine_for(cfg_dict, where, seed=8, page_size=16, max_seq_len=128)
  toks = tokens_for(cfg_dict, 90, 2)
  want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
  for what, cuts in [("whole", [90]), ("decoding", [60] + [1] * 30), ("portions", mx.cuts_of(90, [17, 2, 40, 3]))]:
    mx.check_close(mx.run_cuts(engine, toks, cuts), want, where[0], what)
  engine.ops.check_errors()


# ---- a key that stands out -----------------------------------------------------------------------------

def _needle_runs(cfg_dict, where, cases, sees, seed=11):
  cfg, t = mx.weights(cfg_dict, seed=seed)
  mx.plant_needle(cfg_dict, t, 0, needle=2, asker=1)
  w = mx.as_numpy(t)
  engine, _ = engine_for(cfg_dict, where, tensors=t, page_size=8, max_seq_len=512)
  rng = np.random.default_rng(0)
  decides = {}
  for n, needle_at, ask_at in cases:
    toks = rng.integers(3, cfg_dict["vocab"], n).tolist()
    toks[needle_at], toks[ask_at] = 2, 1
    want = plain.forward(cfg_dict, w, toks)
    without = list(toks)
    without[needle_at] = 5
    decides[(needle_at, ask_at)] = np.abs(plain.forward(cfg_dict, w, without)[ask_at] - want[ask_at]).max() > 0.1 * np.abs(want).max()
    for cuts in ([n], [ask_at, 1, n], [max(ask_at - 1, 1), 2, n], mx.cuts_of(n, [5, 2, 3, 64]),
                 [needle_at + 1, ask_at - needle_at - 1] + [1] * 8 + [n]):
      got = mx.run_cuts(engine, toks, [c for c in cuts if c > 0])
      mx.check_close(got, want, where[0], f"needle at {needle_at}, asked at {ask_at}, cuts {cuts[:3]}")
  for at, seen in decides.items():
    assert seen == sees(*at), (at, seen)
  engine.ops.check_errors()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("sizes", [(16, 16), (16, 32), (12, 10)])
def test_a_key_that_stands_out_inside_and_outside_its_chunk(sizes, where):
  """A query answered by one key among hundreds while both are in one chunk: at the first tokens,
  either side of a page's border, as the first and the last key of the chunk, and as the last key of
  the chunk before; in portions of prompts and asked for by a token decoded alone."""
  chunk = 100
  # (one head: its slope is 2^-8, so that a key at the chunk's far end still stands out)
  layer = mx.attention(heads=1, kv_heads=1, dim=sizes[0], vdim=sizes[1], chunk=chunk, scale=0.5)
  cfg_dict = mx.config([layer], [32], width=32, vocab=50)
  cases = [(40, 0, 1), (40, 0, 39), (75, 7, 8), (75, 8, 71), (110, 0, 99), (110, 99, 100), (230, 100, 199),
           (230, 199, 200), (230, 99, 101), (230, 104, 103 + 8), (330, 200, 299), (330, 199, 299), (330, 300, 329)]
  _needle_runs(cfg_dict, where, cases, lambda needle, asked: needle // chunk == asked // chunk)


@pytest.mark.parametrize("where", WHERE)
def test_a_key_that_stands_out_far_back_over_latents(where):
  cfg_dict = mx.config([mx.latent(heads=4, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=32, scale=0.5)], [32], width=32, vocab=50)
  cases = [(40, 0, 1), (75, 7, 8), (75, 8, 71), (330, 0, 329), (330, 63, 300), (330, 64, 128), (330, 250, 320)]
  _needle_runs(cfg_dict, where, cases, lambda needle, asked: True)


@pytest.mark.parametrize("where", WHERE)
def test_sink_and_slopes_decide(where):
  """Logits differ clearly without the sink, with another sink, and with flat slopes; the engine
  follows the model in each case."""
  cfg_dict = mx.config([mx.attention(heads=2, kv_heads=1, dim=16, vdim=16, chunk=64, scale=0.5)], [None], width=32, vocab=50)
  cfg, t = mx.weights(cfg_dict, seed=4)
  mx.plant_needle(cfg_dict, t, 0, needle=2, asker=1, strength=3.0)
  toks = np.random.default_rng(2).integers(3, 50, 60).tolist()
  toks[5], toks[40], toks[55] = 2, 2, 1
  wants = []
  for sink in ([2.5, 1.0], [-30.0, -30.0], [30.0, 0.0]):
    t["l0.mix.sink"] = torch.tensor(sink).to(torch.bfloat16)
    want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
    wants.append(want)
    engine, _ = engine_for(cfg_dict, where, tensors=t, page_size=8, max_seq_len=256)
    for cuts in ([60], [55, 1, 4], mx.cuts_of(60, [9, 2, 31])):
      mx.check_close(mx.run_cuts(engine, toks, cuts), want, where[0], f"sink {sink}, cuts {cuts[:3]}")
  for other in wants[1:]:
    assert np.abs(wants[0] - other)[10:].max() > 0.05 * np.abs(wants[0]).max()


@pytest.mark.parametrize("where", WHERE)
def test_a_readers_chunks_are_its_own(where):
  """A layer that reads another's keys through larger chunks sees keys the owner no longer sees; the
  cache keeps them for it."""
  for owner, reader in ((10, 25), (25, 10), (10, None), (9, 9)):
    cfg_dict = mx.config([mx.attention(chunk=owner), mx.attention(chunk=reader, kv_from=0), mx.gla()], [24, 24, 24])
    engine, t = engine_for(cfg_dict, where, seed=2, page_size=4, poison=True)
    toks = tokens_for(cfg_dict, 70, 3)
    want = plain.forward(cfg_dict, mx.as_numpy(t), toks)
    for cuts in ([70], [30] + [1] * 40, mx.cuts_of(70, [3, 2, 11])):
      mx.check_close(mx.run_cuts(engine, toks, cuts), want, where[0], f"chunks {owner}, {reader}, cuts {cuts[:3]}")
    engine.cache.check_invariants()
    engine.ops.check_errors()


# ---- generation through the entry point and the scheduler -----------------------------------------

@pytest.mark.parametrize("where", [CPU, GPU32])
def test_greedy_generation_through_the_scheduler(where):
  cfg_dict = mx.CONFIG_B
  engine, t = engine_for(cfg_dict, where, seed=9, slots=2)
  w = mx.as_numpy(t)
  prompts = [tokens_for(cfg_dict, n, 30 + i) for i, n in enumerate((5, 17, 1, 26))]
  results = engine.generate(prompts, SamplingParams(temperature=0.0, max_decode_steps=12))
  for prompt, r in zip(prompts, results):
    toks = list(prompt)
    for _ in range(12):
      toks.append(int(np.argmax(plain.forward(cfg_dict, w, toks)[-1])))
    assert r.output_token_ids == toks[len(prompt):], (r.output_token_ids, toks[len(prompt):])
  assert engine.cache.all_pages_free()


@pytest.mark.gpu
@pytest.mark.parametrize("which,burst", [("a", 1), ("b", 5)])
def test_decoding_from_cuda_graphs(which, burst):
  """Three live requests decode from the graph of four rows (the fourth repeats the third),
  several steps per replay burst."""
  cfg_dict = CONFIGS[which]
  engine, t = engine_for(cfg_dict, ("float32", "cuda"), seed=13, slots=4, graphs=True, burst=burst)
  assert engine._decode_runner is not None, "the model's parts must all allow graph capture"
  w = mx.as_numpy(t)
  prompts = [tokens_for(cfg_dict, n, 40 + i) for i, n in enumerate((9, 3, 14))]
  results = engine.generate(prompts, SamplingParams(temperature=0.0, max_decode_steps=17))
  assert engine._decode_runner.bursts > 0
  for prompt, r in zip(prompts, results):
    toks = list(prompt)
    for _ in range(17):
      toks.append(int(np.argmax(plain.forward(cfg_dict, w, toks)[-1])))
    assert r.output_token_ids == toks[len(prompt):], (r.output_token_ids, toks[len(prompt):])
  engine.ops.check_errors()


@pytest.mark.gpu
def test_bfloat16_generation_runs_and_samples():
  engine, _ = engine_for(mx.CONFIG_A, ("bfloat16", "cuda"), seed=2, slots=3)
  prompts = [tokens_for(mx.CONFIG_A, n, i) for i, n in enumerate((4, 30, 11, 2, 19))]
  results = engine.generate(prompts, SamplingParams(temperature=0.8, top_k=20, max_decode_steps=20, seed=4))
  assert all(len(r.output_token_ids) == 20 for r in results)
  again = engine.generate(prompts, SamplingParams(temperature=0.8, top_k=20, max_decode_steps=20, seed=4))
  assert [r.output_token_ids for r in results][0] == [r.output_token_ids for r in again][0]
  engine.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_tokens_replayed_from_cuda_graphs(dtype):
  """Past the edges of chunks of 50 and 33 tokens, with a row that repeats the last request."""
  cfg_dict = mx.config(
      [mx.attention(heads=4, kv_heads=2, dim=64, vdim=64, chunk=50, scale=0.12), mx.gla(heads=2, dim=32, vdim=32),
       mx.attention(heads=4, kv_heads=1, dim=48, vdim=32, chunk=33, scale=0.2),
       mx.latent(heads=4, dim=16, rot_dim=16, vdim=16, q_rank=32, kv_rank=48)],
      [64, 64, None, 64], width=64, vocab=120)
  engine, t = engine_for(cfg_dict, (dtype, "cuda"), seed=6, slots=4, graphs=True, page_size=16)
  assert engine._decode_runner is not None
  engine._decode_runner.keep_logits = True
  w = mx.as_numpy(t)
  requests = [tokens_for(cfg_dict, n, 50 + i) for i, n in enumerate((120, 71, 105))]
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
    mx.check_close(np.stack(got[i]), want[i][h:], dtype, f"request {i}, replayed steps")
  engine.ops.check_errors()


# ---- configuration, model folders, the preset ---------------------------------------------------------

def test_config_round_trip_caches_and_errors():
  for d in CONFIGS.values():
    cfg = config_from_dict(d)
    assert config_from_dict(cfg.to_dict()) == cfg
  spec = config_from_dict(mx.CONFIG_A).model_spec()
  assert [c.mixer_cache for c in spec.run_order] == [None, None, None, "l0#0", None, None]
  needs = DecoderModel(spec).cache_needs()
  assert set(needs["l0#0"]) == {"mixer", "shift"} and set(needs["l3#3"]) == {"shift"}  # the reader's state is its own
  assert needs["l0#0"]["mixer"].chunks == (7, 12)
  names = {s.name for s in DecoderModel(spec).tensor_specs()}
  assert "l0.mix.k" in names and "l3.mix.k" not in names and "l3.mix.v" not in names and "l3.shift" in names
  specs_b = {s.name: s for s in DecoderModel(config_from_dict(mx.CONFIG_B).model_spec()).tensor_specs()}
  assert specs_b["l1.norm2"].optional and not specs_b["l0.norm2"].optional  # no feed-forward: its norm may be absent
  for change, text in [
      (lambda d: d["layers"][0].update(type="conv"), "unknown type"),
      (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
      (lambda d: d["layers"][3]["mixer"].update(kv_from=3), "kv_from must name an earlier layer"),
      (lambda d: d["layers"][3]["mixer"].update(kv_from=1), "keys and values of its own"),
      (lambda d: d["layers"][3]["mixer"].update(vdim=16), "vdim differs"),
      (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
      (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
      (lambda d: d["layers"][2]["mixer"].pop("tau"), "tau"),
      (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
      (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "unknown mlp kind"),
      (lambda d: d.pop("norm"), "norm"),
  ]:
    d = copy.deepcopy(mx.CONFIG_A)
    change(d)
    with pytest.raises(ConfigError, match=text):
      config_from_dict(d)


def test_model_folder_and_the_step_function_on_it(tmp_path):
  cfg = config_from_dict(mx.CONFIG_B)
  folder = write_model_folder(cfg, 4, str(tmp_path / "m"), matrix_std=0.2, scale_std=0.1)
  assert load_config(folder) == cfg
  with open(os.path.join(folder, "config.json")) as f:
    assert json.load(f)["architecture"] == "Mononex"
  ec = EngineConfig(activation_dtype="float32", page_size=8, batch_size=2, max_seq_len=64, use_cuda_graphs=False)
  engine = Engine.from_folder(folder, ec, ops=ReferenceOps(torch.float32), device="cpu")
  from simply_b200.weights import safetensors_io as st
  entries = st.index_files(st.model_files(folder))
  reader = st.TensorReader(entries)
  w = {n: reader.read(n).float().numpy().astype(np.float64) for n in entries}
  toks = tokens_for(mx.CONFIG_B, 19, 3)
  slot = engine.open_request()
  got = engine.step_raw([StepEntry(slot, toks, tuple(range(len(toks))))]).numpy()
  engine.close_request(slot)
  mx.check_close(got, plain.forward(mx.CONFIG_B, w, toks), "float32", "a written folder")


def test_the_preset_generates_from_random_weights():
  from simply_b200.config import preset
  cfg = preset("mononex-tiny")
  assert cfg.architecture == "Mononex" and {l["type"] for l in cfg.layers} == {"attention", "latent_attention", "gla"}
  ec = EngineConfig(activation_dtype="float32", page_size=8, batch_size=2, max_seq_len=64, use_cuda_graphs=False)
  engine = Engine.from_config(cfg, 1, ec, matrix_std=0.2, ops=ReferenceOps(torch.float32), device="cpu")
  results = engine.generate([[1, 2, 3], [7]], SamplingParams(temperature=0.0, max_decode_steps=5))
  assert [len(r.output_token_ids) for r in results] == [5, 5]
