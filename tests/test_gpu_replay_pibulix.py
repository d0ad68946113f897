"""bin/trace_run on the GPU with Pibulix model folders, as a user runs it, against the plain model:
every request whole; most of it in one step and the last 32 tokens one by one; in portions of
changing size; and mixed with other requests in a pool so small that pages and slots are used again."""

import json
import os

import numpy as np
import pytest

from simply_b200.weights import safetensors_io as st
from tests import pibulix_cases as px
from tests import replay_cases as cases
from tests import trace_util
from tests.plain import pibulix_plain as plain

pytestmark = pytest.mark.gpu

# A model of middling size (groups of query heads for the tcgen05 and for the mma.sync kernels, two sizes;
# windows shorter and longer than a page of 64 and kept tokens of less and of more than a page), and the
# small one without whole 16-byte groups.
MIDDLING = px.config(
    [px.attention(heads=8, kv_heads=4, dim=64, vdim=64, window=40, keep_first=5, dims=48, base=2e4, softcap=15.0, scale=0.18),
     px.gla(heads=3, dim=32, vdim=48, tau=10.0),
     px.attention(heads=5, kv_heads=1, dim=48, vdim=80, window=75, keep_first=67, dims=16, softcap=9.0, conv=4, scale=0.2), 1, 0,
     px.gla(heads=2, dim=64, vdim=32, tau=3.0)],
    [px.dense(192), px.moe(ff=48, experts=10, top=3, groups=(5, 3), shared=56, scale=1.8), None, None, None,
     px.moe(ff=32, experts=6, top=2, groups=(2, 1), shared=24)], width=160, vocab=384, rank=12)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
  root = tmp_path_factory.mktemp("pibulix_models")
  out = {}
  for which, cfg_dict in (("a", MIDDLING), ("b", px.CONFIG_C)):
    cfg, t = px.weights(cfg_dict, seed=17)
    folder = str(root / which)
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
      json.dump(cfg.to_dict(), f)
    st.write_file(os.path.join(folder, "model.safetensors"), t)
    requests = {rid: px.tokens(cfg_dict, t, len(toks), i) for i, (rid, toks) in
                enumerate(cases.make_requests(which, cfg_dict["vocab"]).items())}
    w = px.as_numpy(t)
    expected = {rid: plain.forward(cfg_dict, w, toks) for rid, toks in requests.items()}
    out[which] = (folder, cfg_dict["vocab"], requests, expected)
  return out


def compare(got, requests, expected, dtype):
  assert got, "no logits came back"
  for key, rows in sorted(got.items()):
    rid = key.split(":")[1]
    assert sorted(rows) == list(range(len(requests[rid]))), f"{key}: positions missing"
    px.check_close(np.stack([rows[p] for p in sorted(rows)]), expected[rid], dtype, key)


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
