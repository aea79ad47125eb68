"""Tipidra on the PyTorch definitions: every mechanism, the cache and state, batching, the scheduler, model folders and the command lines."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import tipidra_models as M
import tipidra_oracle as O
from helpers import BASE_YML, ROOT
from tipidra_suite import Suite


class TestTipidraCpu(Suite):
  device = "cpu"
  dtypes = ("float32",)
  len_ = 50


# ------------------------------------------------------------------------------------------ single operations
def _param(t):
  return type("P", (), {"data": t, "leaf": lambda s: t})()


def test_streams_match_their_definition():
  from maxtext_b200.ops import functional as F
  g = torch.Generator().manual_seed(0)
  for k in (1, 2, 3, 5):
    x, y = torch.randn(2, 7, k, 24, generator=g), torch.randn(2, 7, 24, generator=g)
    hc = type("H", (), {n: _param(torch.randn(*s, generator=g)) for n, s in (("read", (k,)), ("write", (k,)), ("mix", (k, k)))})()
    w, b, eps = torch.randn(24, generator=g), torch.randn(24, generator=g), 0.03
    norm = type("N", (), {"scale": _param(w), "bias": _param(b), "eps": eps})()
    with torch.no_grad():
      h = F.stream_read(x, F.StreamReader(hc, norm), torch.float32)
      got, nxt = F.stream_mix(x.clone(), y, hc, F.StreamReader(None, norm))
    streams = [x[:, :, s].double() for s in range(k)]
    seen = []
    want = O.hyper_sublayer(streams, {"in": hc.read.data.double(), "mix": hc.mix.data.double(), "out": hc.write.data.double()},
                            lambda u: O.layer_norm(u, w.double(), b.double(), eps), lambda u: seen.append(u) or y.double())
    assert torch.allclose(h.double(), seen[0], atol=1e-5)
    assert torch.allclose(got.double(), torch.stack(want, 2), atol=1e-5)
    assert torch.allclose(nxt.double(), O.layer_norm(sum(want), w.double(), b.double(), eps), atol=1e-5)


def test_selective_scan_matches_its_definition():
  from maxtext_b200.layers.ssm import selective_scan
  g = torch.Generator().manual_seed(1)
  T, c, n = 40, 6, 10
  x, dt = torch.randn(T, c, generator=g), torch.rand(T, c, generator=g)
  A, B, C, D = -torch.rand(c, n, generator=g), torch.randn(T, n, generator=g), torch.randn(T, n, generator=g), torch.randn(c, generator=g)
  want = O.selective_scan(*(t.double() for t in (x, dt, A, B, C, D)))
  got, state = selective_scan(x[None], dt[None], A, B[None], C[None], D)
  assert torch.allclose(got[0].double(), want, atol=1e-5)
  first, s1 = selective_scan(x[None, :13], dt[None, :13], A, B[None, :13], C[None, :13], D)
  rest, s2 = selective_scan(x[None, 13:], dt[None, 13:], A, B[None, 13:], C[None, 13:], D, s1)
  assert torch.allclose(torch.cat([first, rest], 1), got, atol=1e-6) and torch.allclose(s2, state, atol=1e-6)


def test_oracle_attention_by_hand():
  """Two keys, one head: the sink enters the denominator only, unscaled and uncapped; the cap bounds the scores."""
  q = torch.tensor([[[1.0]], [[2.0]]], dtype=torch.float64)
  k = torch.tensor([[[3.0]], [[-1.0]]], dtype=torch.float64)
  v = torch.tensor([[[10.0]], [[20.0]]], dtype=torch.float64)
  out = O.sink_attention(q, k, v, 0.5, 2.0, torch.tensor([1.0], dtype=torch.float64))
  t = torch.tanh(torch.tensor([2 * 3 * 0.5 / 2, 2 * -1 * 0.5 / 2], dtype=torch.float64)) * 2
  e, s = torch.exp(t), torch.exp(torch.tensor(1.0, dtype=torch.float64))
  assert torch.allclose(out[1, 0, 0], (10 * e[0] + 20 * e[1]) / (e.sum() + s))


# ------------------------------------------------------------------------------------------ configuration and weights
def test_folder_becomes_configuration(tmp_path):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  c = M.config(path, "float32", "cpu")
  assert (c.decoder_block, c.emb_dim, c.vocab_size, c.num_decoder_layers) == ("tipidra", 60, 93, 5)
  assert (c.mhc_expansion_rate, c.embedding_multiplier, c.final_logits_soft_cap) == (3, 3.0, 6.0)
  from maxtext_b200.config import pyconfig
  with pytest.raises(pyconfig.ConfigError, match="vocab_size"):
    pyconfig.initialize(["t", BASE_YML, f"model_dir={path}", "vocab_size=7"], num_devices=1)


@pytest.mark.parametrize("break_it, message", [
    (lambda s: s["layers"][0].update(type="delta"), "delta"), (lambda s: s["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda s: s["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"), (lambda s: s["layers"][1]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda s: s["layers"][0]["mlp"].update(kind="gated"), "gated"), (lambda s: s["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda s: s.update(streams=0), "stream"), (lambda s: s["layers"][0]["mixer"].update(conv=0), "tap")])
def test_what_a_folder_may_not_say(tmp_path, break_it, message):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  s = json.load(open(os.path.join(path, "config.json")))
  break_it(s)
  json.dump(s, open(os.path.join(path, "config.json"), "w"))
  with pytest.raises(ValueError, match=message):
    M.config(path, "float32", "cpu")


def test_missing_tensor_and_wrong_shape_are_errors(tmp_path):
  sp = M.SPECS["scan"]
  W = M.weights(sp)
  for gone in ("l0.mix.D", "l0.hc1.mix", "final.norm.b"):
    with pytest.raises(KeyError, match=gone):
      M.engine(M.write_folder(tmp_path / gone, sp, {k: v for k, v in W.items() if k != gone}))
  with pytest.raises(ValueError, match="mix.x"):
    M.engine(M.write_folder(tmp_path / "b", sp, dict(W, **{"l0.mix.x": torch.zeros(7, 40)})))


def test_equal_layers_share_a_stack(tmp_path):
  a, s = M.attention(2, 1, 8, 8, 4, 0.4, 5.0), M.scan(16, 4, 2, 2)
  sp = M.spec([(s, M.dense(8)), (a, None), (s, M.dense(8)), (s, M.dense(12))], 32)
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)))
  assert eng.model.stack_sizes == {"mamba1_layers": 2, "attention_layers": 1, "mamba1_layers_1": 1}


def test_catalog_entry_builds_and_counts_flops():
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models.transformer import Transformer
  from maxtext_b200.utils import flops
  c = pyconfig.initialize(["t", BASE_YML, "model_name=tipidra-1b", "log_config=false", "hardware=cpu"], num_devices=1)
  m = Transformer(c, None, "meta", build_store=False)
  n = sum(p.pdef.numel for p in m.all_params())
  idle = 0                                                               # experts that a token does not use
  for lay in c.layer_specs:
    if lay["mlp"]["kind"] == "moe":
      idle += 3 * c.emb_dim * lay["mlp"]["expert"]["ff"] * (lay["mlp"]["router"]["experts"] - lay["mlp"]["router"]["top"])
  total, weight, attention = flops.training_tflops_per_device(c, 1)
  body = n - idle - c.vocab_size * c.emb_dim                             # the embedding is a lookup
  assert 0.8e9 < body < 1.6e9
  assert weight == pytest.approx(6 * body * c.max_target_length / 1e12, rel=0.02) and attention > 0 and total == pytest.approx(weight + attention)


# ------------------------------------------------------------------------------------------ engine behaviour
def test_padding_may_run_past_the_end_of_the_cache(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  eng = M.engine(M.write_folder(tmp_path / "m", sp, W), max_len=24)
  st = eng.init_decode_state(2)
  a, b = M.prompt(24, sp, 1), M.prompt(24, sp, 2)
  eng.extend(st, [0, 1], [a[:2], b[:20]])
  lg = eng.extend(st, [0, 1], [a[2:22], b[20:22]], [[19], [1]])          # row 1 is padded to 20 tokens behind its 20 cached ones
  assert M.rel(lg, torch.stack([M.oracle_logits(sp, W, a[:22])[-1], M.oracle_logits(sp, W, b[:22])[-1]])) < 2e-5


def test_training_step_on_the_definitions(tmp_path):
  from maxtext_b200.config import pyconfig
  from maxtext_b200.train.engine import TrainEngine
  from helpers import batch_of
  sp = M.spec([(M.scan(16, 4, 2, 2), M.dense(24)), (M.attention(2, 1, 8, 8, 4, 0.4, 5.0), M.moe(3, 2, 16, 1.0))], 32)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype="float32", max_target_length=16, per_device_batch_size=2,
                            dataset_type="synthetic", hardware="cpu", enable_checkpointing=False, log_config=False, steps=4, learning_rate=5e-3,
                            warmup_steps_fraction=0.0)
  eng = TrainEngine(cfg, None, torch.device("cpu"))
  batch = batch_of(cfg)
  losses = [float(eng.train_step(batch)["learning/loss"]) for _ in range(4)]
  assert losses[-1] < losses[0] and all(x == x for x in losses)


# ------------------------------------------------------------------------------------------ command lines
def test_trace_replay(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  path = M.write_folder(tmp_path / "m", sp, W)
  a, b, c = M.prompt(12, sp, 1), M.prompt(5, sp, 2), M.prompt(9, sp, 3)
  steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": [0, 9]}, {"id": "b", "tokens": b[:4], "want": [3]}], "end": []},
           {"step": 1, "entries": [{"id": "b", "tokens": b[4:], "want": [0]}, {"id": "a", "tokens": a[10:11], "want": []}], "end": ["b"]},
           {"step": 2, "entries": [{"id": "a", "tokens": a[11:], "want": []}], "end": ["a"]},
           {"step": 3, "entries": [{"id": "c", "tokens": c, "want": [8, 2]}], "end": ["c"]}]
  out = tmp_path / "out"
  out.mkdir()
  r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "17",
                      "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
  assert r.returncode == 0, r.stderr[-2000:]
  assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32"]

  def read(i):
    return torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").copy()).view(-1, sp["vocab"])
  la, lb, lc = (M.oracle_logits(sp, W, t) for t in (a, b, c))
  for got, want in ((read(0), torch.stack([la[0], la[9], lb[3]])), (read(1), lb[4:5]), (read(3), torch.stack([lc[8], lc[2]]))):
    assert M.rel(got, want) < 2e-5


def test_decode_command_line(tmp_path):
  from maxtext_b200.inference.decode import decode
  sp = M.spec([(M.scan(16, 4, 2, 2), M.dense(24)), (M.attention(2, 1, 8, 8, 4, 0.4, 5.0), M.moe(3, 1, 16, 1.0))], 32, vocab=300)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  assert isinstance(decode(M.config(path, "float32", "cpu", max_len=24, tokenizer_type="byte"), prompt="hello"), str)
