"""Sitivik on the PyTorch definitions: every mechanism, the cache and state, batching, the scheduler, model folders and the command lines."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import sitivik_models as M
import sitivik_oracle as O
from helpers import BASE_YML, ROOT
from sitivik_suite import Suite


class TestSitivikCpu(Suite):
  device = "cpu"
  dtypes = ("float32",)
  len_ = 50


# ------------------------------------------------------------------------------------------ single operations
def _param(t):
  return type("P", (), {"data": t, "leaf": lambda s: t})()


def test_residual_join_matches_its_definition():
  from maxtext_b200.ops import functional as F
  g = torch.Generator().manual_seed(0)
  x, a, b = (torch.randn(2, 7, 24, generator=g) for _ in range(3))
  bias, w1, w2, w3, lanes = (torch.randn(24, generator=g) for _ in range(5))
  norm = lambda w: type("N", (), {"scale": _param(w), "eps": 0.03, "offset": 0.0})()  # noqa: E731
  with torch.no_grad():
    got, nxt = F.residual_join(x.clone(), F.Branches([F.Branch(a, _param(bias), norm(w1), 0.5), F.Branch(b, None, norm(w2), -2.0)]), _param(lanes), norm(w3))
    want = x + lanes * (0.5 * O.rms(a + bias, 0.03) * w1 - 2.0 * O.rms(b, 0.03) * w2)
    assert torch.allclose(got, want, atol=1e-5) and torch.allclose(nxt, O.rms(want, 0.03) * w3, atol=1e-5)
    got, nxt = F.residual_join(x.clone(), a, None, F.AS_IS)
    assert torch.allclose(got, x + a) and torch.equal(nxt, got)


def test_recurrences_match_their_definitions():
  from maxtext_b200.layers.channel_delta import channel_delta_recurrent
  from maxtext_b200.layers.gla import gla_recurrent
  g = torch.Generator().manual_seed(1)
  T, H, D, Dv = 40, 3, 10, 6
  q, k, v = torch.randn(T, H, D, generator=g), O.unit(torch.randn(T, H, D, generator=g)), torch.randn(T, H, Dv, generator=g)
  lg, beta = -torch.rand(T, H, D, generator=g), torch.rand(T, H, generator=g)
  want = O.delta_scan(*(t.double() for t in (q, k, v, torch.exp(lg), beta)))
  got, state = channel_delta_recurrent(q[None], k[None], v[None], lg[None], beta[None])
  assert torch.allclose(got[0].double(), want, atol=1e-5)
  first, s1 = channel_delta_recurrent(*(t[None, :13] for t in (q, k, v, lg, beta)))
  rest, s2 = channel_delta_recurrent(*(t[None, 13:] for t in (q, k, v, lg, beta)), s1)
  assert torch.allclose(torch.cat([first, rest], 1), got, atol=1e-6) and torch.allclose(s2, state, atol=1e-6)
  decay = torch.tensor([0.5, 0.9, 0.999])
  want = O.retention_scan(*(t.double() for t in (q, k, v, decay)))
  got, _ = gla_recurrent(q[None], k[None], v[None], torch.log(decay).view(1, 1, H, 1).expand(1, T, H, D))
  assert torch.allclose(got[0].double(), want, atol=1e-4)


def test_stretched_frequencies():
  """One wavelength in each of the three ranges, by hand."""
  from maxtext_b200.ops import reference as ref
  rot = {"base": 10000.0, "dims": 24, "scaling": {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 128}}
  got = ref.rope_inv_timescale(24, 1.0, 10000.0, stretch=rot["scaling"])
  assert torch.allclose(got.double(), torch.tensor(O.frequencies(rot), dtype=torch.float64), rtol=1e-6)
  plain = [10000.0 ** (-i / 12) for i in range(12)]
  kinds = ["short" if 2 * math.pi / f < 32 else "long" if 2 * math.pi / f > 128 else "between" for f in plain]
  assert {"short", "long", "between"} <= set(kinds)
  for f, k, x in zip(plain, kinds, got.tolist()):
    assert {"short": x == pytest.approx(f), "long": x == pytest.approx(f / 5), "between": f / 5 < x < f}[k]


def test_oracle_attention_by_hand():
  """Two keys, one head: the added one has no value; a window of one token sees itself; chunks of two start anew at token two."""
  q = torch.tensor([[[1.0]], [[2.0]], [[1.0]]], dtype=torch.float64)
  k = torch.tensor([[[3.0]], [[-1.0]], [[0.5]]], dtype=torch.float64)
  v = torch.tensor([[[10.0]], [[20.0]], [[30.0]]], dtype=torch.float64)
  e = [math.exp(2 * 3 * 0.5), math.exp(2 * -1 * 0.5)]
  out = O.attention(q, k, v, 0.5, O.visible(3, chunk=2), True)
  assert float(out[1, 0, 0]) == pytest.approx((10 * e[0] + 20 * e[1]) / (e[0] + e[1] + 1))
  assert float(out[2, 0, 0]) == pytest.approx(30 * math.exp(0.25) / (math.exp(0.25) + 1))
  out = O.attention(q, k, v, 0.5, O.visible(3, window=1))
  assert out.flatten().tolist() == [10.0, 20.0, 30.0]


def test_pair_cache_hands_names_to_its_parts():
  from maxtext_b200.inference.kvcache import LayerKVCache, PairCache
  from maxtext_b200.layers.gdn import RecurrentState
  c = PairCache(LayerKVCache(2, 8, 1, 4, 6, torch.float32, "cpu"), RecurrentState(2, 3, 4, 5, "cpu", 7, 3))
  c.bind(torch.tensor([1]), torch.tensor([0]))
  assert c.k is c.left.k and c.rec is c.right.rec and c.recurrent_buffers == ("conv", "rec") and c.rows_for(5) == 5 and c.right.slot_ids.tolist() == [1]
  assert not hasattr(c, "latent")
  with pytest.raises(NotImplementedError):
    PairCache(LayerKVCache(2, 8, 1, 4, 6, torch.float32, "cpu"), LayerKVCache(2, 8, 1, 4, 6, torch.float32, "cpu"))


# ------------------------------------------------------------------------------------------ configuration and weights
def test_folder_becomes_configuration(tmp_path):
  sp = M.SPECS["mixed"]
  path = M.folder(tmp_path / "m", sp, M.weights(sp))
  c = M.config(path, "float32", "cpu")
  assert (c.decoder_block, c.emb_dim, c.vocab_size, c.num_decoder_layers) == ("sitivik", 60, 93, 5)
  assert (c.token_side_dim, c.embedding_multiplier, c.logits_via_embedding, c.normalize_embedding_logits) == (9, 3.0, True, False)
  assert c.layer_specs[2]["mixer"]["right"]["decay_rank"] == 6 and c.layer_specs[2]["mixer"]["right"]["gate_rank"] == 10
  from maxtext_b200.config import pyconfig
  with pytest.raises(pyconfig.ConfigError, match="vocab_size"):
    pyconfig.initialize(["t", BASE_YML, f"model_dir={path}", "vocab_size=7"], num_devices=1)


@pytest.mark.parametrize("break_it, message", [
    (lambda s: s["layers"][0].update(type="delta"), "delta"), (lambda s: s["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda s: s["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "rot.dims"), (lambda s: s["layers"][0]["mixer"]["right"]["rot"].update(dims=18), "rot.dims"),
    (lambda s: s["layers"][0]["mlp"].update(kind="moe"), "moe"), (lambda s: s["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda s: s["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]), "decay"), (lambda s: s["layers"][2]["mixer"]["right"].update(conv=0), "tap"),
    (lambda s: s["layers"][2]["mixer"]["left"]["mask"].update(size=0), "mask"), (lambda s: s["token_side"].update(dim=0), "token_side"),
    (lambda s: s["layers"][1]["mixer"]["q_temp"].update(every=0), "q_temp")])
def test_what_a_folder_may_not_say(tmp_path, break_it, message):
  sp = M.SPECS["mixed"]
  path = M.folder(tmp_path / "m", sp, M.weights(sp))
  s = json.load(open(os.path.join(path, "config.json")))
  break_it(s)
  json.dump(s, open(os.path.join(path, "config.json"), "w"))
  with pytest.raises(ValueError, match=message):
    M.config(path, "float32", "cpu")


def test_missing_tensor_and_wrong_shape_are_errors(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  for gone in ("l0.mix.left.o.b", "l1.mix.lq2", "l2.mix.right.dt_bias", "l3.side.norm", "l4.ls1"):
    with pytest.raises(KeyError, match=gone):
      M.engine(M.folder(tmp_path / gone, sp, {k: v for k, v in W.items() if k != gone}))
  with pytest.raises(ValueError, match="side.embed"):
    M.engine(M.folder(tmp_path / "b", sp, dict(W, **{"side.embed": torch.zeros(93, 11)})))


def test_equal_layers_share_a_stack(tmp_path):
  a, d = M.parallel(M.window(2, 1, 8, 8, 4, 5, 0.4), M.retention(8, 8, 4, (0.9,))), M.differential(2, 1, 8, 8, 0.4)
  p = M.parallel_2(M.window(2, 1, 8, 8, 4, 5, 0.4), M.delta(2, 1, 8, 8, 2, 2, 2))
  sp = M.spec([(a, 8), (d, None), (p, 8), (a, 8), (a, 12)], 32)
  eng = M.engine(M.folder(tmp_path / "m", sp, M.weights(sp)))
  assert eng.model.stack_sizes == {"parallel_layers": 2, "attention_layers": 1, "parallel_2_layers": 1, "parallel_layers_1": 1}


def test_input_projections_are_one_operand():
  """What reads the common input of a pair sits back to back in its unit."""
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models.transformer import Transformer
  c = pyconfig.initialize(["t", BASE_YML, "model_name=sitivik-1b", "log_config=false", "hardware=cpu", "base_num_decoder_layers=4", "override_model_config=true",
                           "base_emb_dim=64", "vocab_size=64"] + [f"layer_specs={json.dumps(pyconfig_layers())}"], num_devices=1, dtype="float32")
  m = Transformer(c, None, "cpu")
  pairs = [b.attn for l in m.layers for b in l.blocks if b.plan.attention == "parallel"]
  assert len(pairs) == 3 and all(p.fused is not None and p.fused.fusable() and p.fused.data is not None for p in pairs)


def pyconfig_layers():
  sp = M.spec([(M.parallel(M.window(4, 2, 16, 16, 8, 5, 0.3), M.retention(16, 16, 8, (0.9, 0.5))), 32), (M.differential(2, 1, 16, 32, 0.3), 32),
               (M.parallel_2(M.window(4, 2, 16, 16, 8, 5, 0.3), M.delta(4, 2, 16, 16, 4, 8, 8)), 32),
               (M.parallel(M.window(4, 2, 16, 16, 8, 5, 0.3), M.retention(16, 16, 8, (0.9, 0.5))), 32)], 64)
  layers = copy.deepcopy(sp["layers"])
  right = layers[2]["mixer"]["right"]
  right["decay_rank"], right["gate_rank"] = right.pop("_ranks")
  return layers


def test_catalog_entry_builds_and_counts_flops():
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models.transformer import Transformer
  from maxtext_b200.utils import flops
  c = pyconfig.initialize(["t", BASE_YML, "model_name=sitivik-1b", "log_config=false", "hardware=cpu"], num_devices=1)
  m = Transformer(c, None, "meta", build_store=False)
  n = sum(p.pdef.numel for p in m.all_params())
  total, weight, attention = flops.training_tflops_per_device(c, 1)
  body = n - c.vocab_size * c.token_side_dim * c.num_decoder_layers      # the narrow tables are lookups; the wide one is also the head
  assert 0.8e9 < body < 1.6e9
  assert weight == pytest.approx(6 * body * c.max_target_length / 1e12, rel=0.02) and attention > 0 and total == pytest.approx(weight + attention)


# ------------------------------------------------------------------------------------------ engine behaviour
def test_padding_may_run_past_the_end_of_the_cache(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  eng = M.engine(M.folder(tmp_path / "m", sp, W), max_len=24)
  st = eng.init_decode_state(2)
  a, b = M.prompt(24, sp, 1), M.prompt(24, sp, 2)
  eng.extend(st, [0, 1], [a[:2], b[:20]])
  lg = eng.extend(st, [0, 1], [a[2:22], b[20:22]], [[19], [1]])          # row 1 is padded to 20 tokens behind its 20 cached ones
  assert M.rel(lg, torch.stack([M.oracle_logits(sp, W, a[:22])[-1], M.oracle_logits(sp, W, b[:22])[-1]])) < 2e-5


def test_training_step_on_the_definitions(tmp_path):
  from maxtext_b200.config import pyconfig
  from maxtext_b200.train.engine import TrainEngine
  from helpers import batch_of
  sp = M.spec([(M.parallel(M.window(2, 1, 8, 8, 4, 5, 0.4), M.retention(8, 8, 4, (0.9, 0.8))), 24), (M.differential(2, 1, 8, 8, 0.4), 16),
               (M.parallel_2(M.window(2, 1, 8, 8, 4, 5, 0.4), M.delta(2, 1, 8, 8, 2, 2, 2)), None)], 32)
  path = M.folder(tmp_path / "m", sp, M.weights(sp))
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype="float32", max_target_length=16, per_device_batch_size=2,
                            dataset_type="synthetic", hardware="cpu", enable_checkpointing=False, log_config=False, steps=4, learning_rate=5e-3,
                            warmup_steps_fraction=0.0)
  eng = TrainEngine(cfg, None, torch.device("cpu"))
  batch = batch_of(cfg)
  before = {n: p.data.clone() for n, p in eng.model.store.params.items()}
  losses = [float(eng.train_step(batch)["learning/loss"]) for _ in range(4)]
  assert losses[-1] < losses[0] and all(x == x for x in losses)
  still = [n for n, p in eng.model.store.params.items() if torch.equal(p.data, before[n])]
  assert not still, f"no gradient reached {still}"


# ------------------------------------------------------------------------------------------ command lines
def test_trace_replay(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  path = M.folder(tmp_path / "m", sp, W)
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
  sp = M.spec([(M.parallel(M.window(2, 1, 8, 8, 4, 5, 0.4), M.retention(8, 8, 4, (0.9,))), 24), (M.differential(2, 1, 8, 8, 0.4), None)], 32, vocab=300)
  path = M.folder(tmp_path / "m", sp, M.weights(sp))
  assert isinstance(decode(M.config(path, "float32", "cpu", max_len=24, tokenizer_type="byte"), prompt="hello"), str)
