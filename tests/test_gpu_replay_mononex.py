"""bin/trace_run on the GPU with Mononex model folders, as a user runs it, against the plain model:
every request whole; most of it in one step and the last 32 tokens one by one; in portions of
changing size; and mixed with other requests in a pool so small that pages and slots are used again."""

import json
import os

import numpy as np
import pytest

from simply_b200.weights import safetensors_io as st
from tests import mononex_cases as mx
from tests import replay_cases as cases
from tests import trace_util
from tests.plain import mononex_plain as plain

pytestmark = pytest.mark.gpu

# A model of middling size (head sizes for the tcgen05 kernel, the mma.sync kernels of two sizes and the
# kernel over latents; chunks shorter and longer than a page of 64, a reader with chunks of its own),
# and the small one without whole 16-byte groups.
MIDDLING = mx.config(
    [mx.attention(heads=8, kv_heads=4, dim=64, vdim=64, chunk=40, scale=0.18),
     mx.gla(heads=3, dim=32, vdim=48, tau=10.0),
     mx.attention(heads=8, kv_heads=4, dim=64, vdim=64, chunk=100, scale=0.15, kv_from=0),
     mx.latent(heads=6, dim=24, rot_dim=16, vdim=32, q_rank=48, kv_rank=80, base=5000.0, original=64, fast=8.0, slow=1.0, scale=0.2),
     mx.attention(heads=6, kv_heads=2, dim=48, vdim=80, chunk=64, scale=0.15)],
    [192, 96, None, 160, 64], width=160, vocab=384, rank=12)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
  root = tmp_path_factory.mktemp("mononex_models")
  out = {}
  for which, cfg_dict in (("a", MIDDLING), ("b", mx.CONFIG_C)):
    cfg, t = mx.weights(cfg_dict, seed=17)
    folder = str(root / which)
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
      json.dump(cfg.to_dict(), f)
    st.write_file(os.path.join(folder, "model.safetensors"), t)
    requests = cases.make_requests(which, cfg_dict["vocab"])
    w = mx.as_numpy(t)
    expected = {rid: plain.forward(cfg_dict, w, toks) for rid, toks in requests.items()}
    out[which] = (folder, cfg_dict["vocab"], requests, expected)
  return out


def compare(got, requests, expected, dtype):
  assert got, "no logits came back"
  for key, rows in sorted(got.items()):
    rid = key.split(":")[1]
    assert sorted(rows) == list(range(len(requests[rid]))), f"{key}: positions missing"
    mx.check_close(np.stack([rows[p] for p in sorted(rows)]), expected[rid], dtype, key)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["a", "b"])
def test_trace_run_four_ways(models, tmp_path, which, dtype):
  folder, vocab, requests, expected = models[which]
  steps = cases.combined_trace(requests)
  out_dir = str(tmp_path / "out")
  trace_util.run_tool(folder, dtype, steps, out_dir, trace_util.tokens_needed(steps, 64))
  compare(trace_util.collect(steps, out_dir, vocab), requests, expected, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_small_pages_poisoned(models, tmp_path, dtype):
  """Pages of 8 tokens, freed pages filled with NaN, the pool exactly as large as the trace needs."""
  folder, vocab, requests, expected = models["a"]
  steps = cases.combined_trace(requests, modes=("mixed", "portions"))
  out_dir = str(tmp_path / "out")
  trace_util.run_tool(folder, dtype, steps, out_dir, trace_util.tokens_needed(steps, 8),
                      extra=("--page-size", "8", "--poison-freed-pages"))
  compare(trace_util.collect(steps, out_dir, vocab), requests, expected, dtype)
