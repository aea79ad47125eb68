"""Silinex on the PyTorch definitions: every mechanism, the cache and state, batching, the scheduler, model folders and the replay tool."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import silinex_models as M
import silinex_oracle as O
from helpers import BASE_YML, ROOT
from silinex_suite import Suite


class TestSilinexCpu(Suite):
  device = "cpu"
  dtypes = ("float32",)
  len_ = 60


# ------------------------------------------------------------------------------------------ single operations
def test_fp32_stream_norms():
  from maxtext_b200.ops import functional as F

  class N:                                        # what `layers.blocks.Norm` exposes
    def __init__(self, w, eps):
      self.eps, self.offset = eps, 1.0
      self.scale = type("P", (), {"data": w, "leaf": lambda s: w})()
  g = torch.Generator().manual_seed(0)
  x, b = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g) * 3
  w1, w2 = torch.randn(24, generator=g) * 0.3, torch.randn(24, generator=g) * 0.3
  with torch.no_grad():
    got_x, got_y = F.residual_norm(x.clone(), b, N(w1, 0.01), 0.4, N(w2, 0.2))
  want_x = x.double() + 0.4 * O.zero_centred_norm(b.double(), w1.double(), 0.01)
  assert torch.allclose(got_x.double(), want_x, atol=1e-5)
  assert torch.allclose(got_y.double(), O.zero_centred_norm(want_x, w2.double(), 0.2), atol=1e-5)


def test_recurrences_match_their_definitions():
  from maxtext_b200.layers.gdn import gated_delta_chunked, gated_delta_recurrent
  from maxtext_b200.layers.gla import gla_recurrent
  g = torch.Generator().manual_seed(1)
  T, H, dk, dv = 50, 3, 6, 10
  q, k, v = torch.randn(T, H, dk, generator=g), torch.randn(T, H, dk, generator=g), torch.randn(T, H, dv, generator=g)
  lg, beta = -torch.rand(T, H, generator=g), torch.rand(T, H, generator=g)
  want = O.delta_recurrence(O.unit(q.double()) * dk ** -0.5, O.unit(k.double()), v.double(), torch.exp(lg.double()), beta.double())
  for fn in (gated_delta_recurrent, lambda *a: gated_delta_chunked(*a, chunk=16)):
    assert torch.allclose(fn(q[None], k[None], v[None], lg[None], beta[None])[0][0].double(), want, atol=1e-5)
  la = -torch.rand(T, H, dk, generator=g)
  want = O.gated_linear_recurrence(q.double(), k.double(), v.double(), torch.exp(la.double()))
  assert torch.allclose(gla_recurrent(q[None], k[None], v[None], la[None])[0][0].double(), want, atol=1e-4)


# ------------------------------------------------------------------------------------------ configuration and weights
def test_folder_becomes_configuration(tmp_path):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  c = M.config(path, "float32", "cpu")
  assert (c.decoder_block, c.emb_dim, c.vocab_size, c.num_decoder_layers) == ("silinex", 60, 93, 6)
  assert c.layer_specs[0]["mixer"]["decay_rank"] == 12 and c.residual_multiplier == 0.8
  from maxtext_b200.config import pyconfig
  with pytest.raises(pyconfig.ConfigError, match="vocab_size"):
    pyconfig.initialize(["t", BASE_YML, f"model_dir={path}", "vocab_size=7"], num_devices=1)


@pytest.mark.parametrize("break_it, message", [
    (lambda s: s["layers"][0].update(type="mamba"), "mamba"), (lambda s: s["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda s: s["layers"][1]["mixer"]["rot"].update(dims=4), "rot.dims"), (lambda s: s["layers"][0]["mlp"].update(kind="routed"), "routed"),
    (lambda s: s.update(architecture="Other"), "Other"), (lambda s: s["layers"][1]["mixer"]["mask"].update(size=0), "window")])
def test_what_a_folder_may_not_say(tmp_path, break_it, message):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  s = json.load(open(os.path.join(path, "config.json")))
  break_it(s)
  json.dump(s, open(os.path.join(path, "config.json"), "w"))
  with pytest.raises(ValueError, match=message):
    M.config(path, "float32", "cpu")


def test_missing_tensor_and_wrong_shape_are_errors(tmp_path):
  sp = M.SPECS["gla"]
  W = M.weights(sp)
  short = {k: v for k, v in W.items() if k != "l0.mix.norm"}
  with pytest.raises(KeyError, match="l0.mix.norm"):
    M.engine(M.write_folder(tmp_path / "a", sp, short))
  bad = dict(W, head=torch.zeros(3, sp["width"]))
  with pytest.raises(ValueError, match="logits_dense"):
    M.engine(M.write_folder(tmp_path / "b", sp, bad))


def test_equal_layers_share_a_stack(tmp_path):
  sp = M.spec([M.delta(2, 1, 8, 8, 2), M.gla(2, 8, 8, 2.0, 4), M.delta(2, 1, 8, 8, 2), M.delta(2, 2, 8, 8, 2)], 32)
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)))
  assert eng.model.stack_sizes == {"delta_layers": 2, "gla_layers": 1, "delta_layers_1": 1}


def test_catalog_entry_builds_and_counts_flops():
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models.transformer import Transformer
  from maxtext_b200.utils import flops
  c = pyconfig.initialize(["t", BASE_YML, "model_name=silinex-1b", "log_config=false", "hardware=cpu"], num_devices=1)
  m = Transformer(c, None, "meta", build_store=False)
  n = sum(p.pdef.numel for p in m.all_params())
  assert 0.8e9 < n < 1.6e9
  total, weight, attention = flops.training_tflops_per_device(c, 1)
  tokens = c.max_target_length
  body = n - c.vocab_size * c.emb_dim                                   # the embedding is a lookup
  assert weight == pytest.approx(6 * body * tokens / 1e12, rel=0.02) and attention > 0 and total == pytest.approx(weight + attention)


# ------------------------------------------------------------------------------------------ engine behaviour
def test_extend_refuses_what_does_not_fit(tmp_path):
  sp = M.SPECS["latent"]
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)), max_len=20)
  st = eng.init_decode_state(2)
  for slots, toks in (([0], [[1] * 21]), ([0, 0], [[1], [2]]), ([2], [[1]]), ([0], [[]])):
    with pytest.raises((ValueError, IndexError)):
      eng.extend(st, slots, toks)
  eng.extend(st, [0], [[1] * 20])                                       # exactly full


def test_padding_may_run_past_the_end_of_the_cache(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  eng = M.engine(M.write_folder(tmp_path / "m", sp, W), max_len=24)
  st = eng.init_decode_state(2)
  a, b = M.prompt(24, sp, 1), M.prompt(24, sp, 2)
  eng.extend(st, [0, 1], [a[:2], b[:20]])
  lg = eng.extend(st, [0, 1], [a[2:22], b[20:22]], [[19], [1]])          # row 1 is padded to 20 tokens behind its 20 cached ones
  assert M.rel(lg, torch.stack([M.oracle_logits(sp, W, a[:22])[-1], M.oracle_logits(sp, W, b[:22])[-1]])) < 2e-5


def test_extend_serves_the_other_families_too():
  from helpers import tiny_config
  from maxtext_b200.inference.maxengine import MaxEngine
  for model in ("llama3-8b", "deepseek3-tiny", "qwen3-next-80b-a3b"):
    cfg = tiny_config(model, extra=["max_prefill_predict_length=24"])
    eng = MaxEngine(cfg, device="cpu")
    eng.load_params()
    g = torch.Generator().manual_seed(0)
    seqs = [torch.randint(0, 256, (n,), generator=g).tolist() for n in (20, 3, 11)]
    st = eng.init_decode_state(3)
    lg = [eng.extend(st, [0, 1, 2], [s[:-2] for s in seqs])]
    for j in (-2, -1):
      lg.append(eng.extend(st, [0, 1, 2], [[s[j]] for s in seqs]))
    for i, s in enumerate(seqs):
      full = eng.model.forward(torch.tensor([s]), None, None)[0]
      for j in range(3):
        assert torch.allclose(lg[j][i], full[len(s) - 3 + j], atol=2e-3), (model, i, j)


def test_training_step_on_the_definitions(tmp_path):
  from maxtext_b200.config import pyconfig
  from maxtext_b200.train.engine import TrainEngine
  from helpers import batch_of
  sp = M.spec([M.delta(2, 1, 8, 8, 2), M.gla(2, 8, 8, 2.0, 4), M.latent(2, 8, 4, 8, 12, 16, 6, 0.3)], 32)
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
  assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
  assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32"]

  def read(i):
    return torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").copy()).view(-1, sp["vocab"])
  la, lb, lc = (M.oracle_logits(sp, W, t) for t in (a, b, c))
  for got, want in ((read(0), torch.stack([la[0], la[9], lb[3]])), (read(1), lb[4:5]), (read(3), torch.stack([lc[8], lc[2]]))):
    assert M.rel(got, want) < 2e-5


def test_decode_command_line(tmp_path):
  from maxtext_b200.inference.decode import decode
  sp = M.spec([M.delta(2, 1, 8, 8, 2), M.latent(2, 8, 4, 8, 12, 16, 6, 0.3)], 32, vocab=300)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  text = decode(M.config(path, "float32", "cpu", max_len=24, tokenizer_type="byte"), prompt="hello")
  assert isinstance(text, str)
