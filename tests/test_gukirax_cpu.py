"""Gukirax on the PyTorch definitions: every mechanism, the caches of a loop, batching, the scheduler, model folders and the command lines."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gukirax_models as M
import gukirax_oracle as O
from gukirax_suite import Suite
from helpers import BASE_YML, ROOT


class TestGukiraxCpu(Suite):
  device = "cpu"
  dtypes = ("float32",)
  len_ = 50


# ------------------------------------------------------------------------------------------ single operations
def _param(t):
  return type("P", (), {"data": t, "leaf": lambda s: t})()


def _norm(w, eps, kind="layernorm_scale"):
  return type("N", (), {"scale": _param(w), "bias": None, "eps": eps, "kind": kind, "offset": 0.0})()


def test_gated_residual_matches_its_definition():
  from maxtext_b200.ops import functional as F
  g = torch.Generator().manual_seed(0)
  x, b, logits = (torch.randn(2, 7, 24, generator=g) + 0.5 for _ in range(3))
  bias, w1, w2 = (torch.randn(24, generator=g) for _ in range(3))
  eps = 0.03
  want = O.gated_sublayer(x.double(), lambda t: t, lambda h: b.double(), torch.zeros(24, 24).double(), bias.double(), lambda t: O.layer_norm(t, w1.double(), eps))
  ungated = x.double() + O.layer_norm(b.double(), w1.double(), eps)
  with torch.no_grad():
    got, nxt = F.residual_gate(x.clone(), b, torch.zeros_like(b), _param(bias), _norm(w1, eps), _norm(w2, eps))
    assert torch.allclose(got.double(), want, atol=1e-5) and torch.allclose(nxt.double(), O.layer_norm(want, w2.double(), eps), atol=1e-5)
    got, none = F.residual_gate(x.clone(), b, None, None, _norm(w1, eps))
    assert none is None and torch.allclose(got.double(), ungated, atol=1e-5)
    got, _ = F.residual_gate(x.clone(), b, logits, _param(bias), _norm(w1, eps, "rms"))
    gated = b.double() * O.sigmoid(logits.double() + bias.double())
    assert torch.allclose(got.double(), x.double() + O.rms(gated, eps) * w1.double(), atol=1e-5)
    buf = torch.cat([torch.zeros(2, 7, 24), logits], -1)
    got, side = F.residual_gate(x.clone(), b, None, None, _norm(w1, eps), F.Beside(buf))
    assert torch.equal(side, torch.cat([got, logits], -1))


def test_xielu_matches_its_definition():
  from maxtext_b200.ops import functional as F
  z = torch.cat([torch.linspace(-30, 30, 401), torch.tensor([0.0, -0.0, 1e-4, -1e-4])])
  for p, q in ((0.3, -0.7), (-4.0, 5.0), (12.0, -12.0)):
    want = O.xielu(z.double(), torch.tensor(p).double(), torch.tensor(q).double())
    with torch.no_grad():
      assert torch.allclose(F.act(z[None], "xielu", _param(torch.tensor([p, q])))[0].double(), want, rtol=1e-5, atol=1e-7)


def test_oracle_attention_by_hand():
  """Two heads over two keys: the mixing adds the other head's score, the sink enters the denominator only, unscaled."""
  q = torch.tensor([[[1.0], [0.5]], [[2.0], [-1.0]]], dtype=torch.float64)
  k = torch.tensor([[[3.0]], [[-1.0]]], dtype=torch.float64)
  v = torch.tensor([[[10.0]], [[20.0]]], dtype=torch.float64)
  talk = torch.tensor([[1.0, 0.25], [0.0, 1.0]], dtype=torch.float64)
  out = O.talking_attention(q, k, v, 0.5, talk, torch.tensor([1.0, -30.0], dtype=torch.float64))
  e = torch.exp(torch.tensor([3.0 + 0.25 * -1.5, -1.0 + 0.25 * 0.5], dtype=torch.float64))
  s = torch.exp(torch.tensor(1.0, dtype=torch.float64))
  assert torch.allclose(out[1, 0, 0], (10 * e[0] + 20 * e[1]) / (e.sum() + s))
  e = torch.exp(torch.tensor([-1.5, 0.5], dtype=torch.float64))
  assert torch.allclose(out[1, 1, 0], (10 * e[0] + 20 * e[1]) / e.sum())


# ------------------------------------------------------------------------------------------ configuration and weights
def test_folder_becomes_configuration(tmp_path):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  c = M.config(path, "float32", "cpu")
  assert (c.decoder_block, c.emb_dim, c.vocab_size, c.num_decoder_layers) == ("gukirax", 60, 93, 5)
  assert (dict(c.layer_loop), c.final_logits_scale, c.final_logits_soft_cap) == ({"start": 1, "stop": 4, "times": 2}, 0.7, 6.0)
  from maxtext_b200.models import families
  assert families.layer_runs(c) == [0, 1, 2, 3, 1, 2, 3, 4] == [i for i, _ in O.layer_runs(sp)]
  from maxtext_b200.config import pyconfig
  with pytest.raises(pyconfig.ConfigError, match="vocab_size"):
    pyconfig.initialize(["t", BASE_YML, f"model_dir={path}", "vocab_size=7"], num_devices=1)


@pytest.mark.parametrize("break_it, message", [
    (lambda s: s["layers"][0].update(type="delta"), "delta"), (lambda s: s["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda s: s["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"), (lambda s: s["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda s: s["layers"][0]["mlp"].update(kind="gated"), "gated"), (lambda s: s["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda s: s["layers"][0]["mixer"].update(vdim=25), "vdim"), (lambda s: s["loop"].update(stop=6), "layer_loop"),
    (lambda s: s["loop"].update(times=0), "layer_loop")])
def test_what_a_folder_may_not_say(tmp_path, break_it, message):
  sp = M.SPECS["mixed"]
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  s = json.load(open(os.path.join(path, "config.json")))
  break_it(s)
  json.dump(s, open(os.path.join(path, "config.json"), "w"))
  with pytest.raises(ValueError, match=message):
    M.config(path, "float32", "cpu")


def test_missing_tensor_and_wrong_shape_are_errors(tmp_path):
  sp = M.SPECS["mixed"]
  W = M.weights(sp)
  for gone in ("l0.mix.talk", "l2.rg1.b", "loop.in", "embed.norm", "l1.mlp.shared.down"):
    with pytest.raises(KeyError, match=gone):
      M.engine(M.write_folder(tmp_path / gone, sp, {k: v for k, v in W.items() if k != gone}))
  with pytest.raises(ValueError, match="talk"):
    M.engine(M.write_folder(tmp_path / "b", sp, dict(W, **{"l0.mix.talk": torch.zeros(4, 3)})))


def test_equal_layers_share_a_stack(tmp_path):
  a = M.attention(2, 1, 8, 4, 0.4)
  sp = M.spec([(a, M.dense(8)), (a, None), (a, M.dense(8)), (a, M.dense(12))], 32, loop=(1, 3, 2))
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)))
  assert eng.model.stack_sizes == {"attention_layers": 2, "attention_layers_1": 1, "attention_layers_2": 1}
  assert [layer.index for layer in eng.model.runs] == [0, 1, 2, 1, 2, 3] and [layer.entry is not None for layer in eng.model.layers] == [False, True, False, False]


def test_what_reads_one_input_is_one_operand(tmp_path):
  sp = M.SPECS["mixed_even"]
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)))
  for layer in eng.model.layers:
    blk = layer.blocks[0]
    assert blk.mixer_in.fusable() and blk.mlp_in.fusable()
    assert torch.equal(blk.mixer_in.data, torch.cat([p.data for p in (blk.attn.q, blk.attn.k, blk.rg1[0])]))


def test_catalog_entry_builds_and_counts_flops():
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models import families
  from maxtext_b200.models.transformer import Transformer
  from maxtext_b200.utils import flops
  c = pyconfig.initialize(["t", BASE_YML, "model_name=gukirax-1b", "log_config=false", "hardware=cpu"], num_devices=1)
  m = Transformer(c, None, "meta", build_store=False)
  per_layer = []
  for lay, layer in zip(c.layer_specs, m.layers):
    n = sum(p.pdef.numel for p in layer.params)
    if lay["mlp"]["kind"] == "moe":                                      # experts that a token does not use
      n -= 2 * c.emb_dim * lay["mlp"]["expert"]["ff"] * (lay["mlp"]["router"]["experts"] - lay["mlp"]["router"]["top"])
    per_layer.append(n)
  body = sum(per_layer[i] for i in families.layer_runs(c)) + c.vocab_size * c.emb_dim
  total, weight, attention = flops.training_tflops_per_device(c, 1)
  assert 0.5e9 < body < 1.6e9 and len(m.runs) > len(m.layers)
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


TRAIN = dict(dtype="float32", max_target_length=16, per_device_batch_size=2, dataset_type="synthetic", enable_checkpointing=False, log_config=False, steps=4,
             learning_rate=5e-3, warmup_steps_fraction=0.0)


def train_losses(path, device, steps=4, **kw):
  from helpers import batch_of
  from maxtext_b200.config import pyconfig
  from maxtext_b200.models import registry
  from maxtext_b200.train.engine import TrainEngine
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, hardware="gpu" if device == "cuda" else "cpu", **{**TRAIN, **kw})
  eng = TrainEngine(cfg, None, torch.device(device, 0) if device == "cuda" else torch.device(device))
  registry.load_weights(path, eng.model.store, cfg)
  batch = batch_of(cfg)
  return [float(eng.train_step(batch)["learning/loss"]) for _ in range(steps)], eng


def train_spec():
  return M.spec([(M.attention(2, 1, 8, 4, 0.4), M.dense(24)), (M.attention(4, 2, 16, 8, 0.3), M.moe(3, 2, 16, 12)), (M.attention(2, 2, 8, 8, 0.4), None)], 32,
                loop=(0, 2, 2))


def test_training_step_on_the_definitions(tmp_path):
  path = M.write_folder(tmp_path / "m", train_spec(), M.weights(train_spec()))
  losses, _ = train_losses(path, "cpu")
  assert losses[-1] < losses[0] and all(x == x for x in losses)


def test_gradients_of_a_loop(tmp_path):
  """The gradient of a layer that runs twice, of the pass input and of the embedding (which every pass reads) against autograd through the oracle."""
  from helpers import batch_of
  from maxtext_b200.config import pyconfig
  from maxtext_b200.train.engine import TrainEngine
  sp = train_spec()
  W = M.weights(sp)
  path = M.write_folder(tmp_path / "m", sp, W)
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, hardware="cpu", **TRAIN)
  eng = TrainEngine(cfg, None, torch.device("cpu"))
  from maxtext_b200.models import registry
  registry.load_weights(path, eng.model.store, cfg)
  batch = batch_of(cfg)
  eng.fwd_bwd(batch)
  leaves = {k: v.double().requires_grad_(True) for k, v in W.items()}
  loss = 0.0
  for row, tgt, seg in zip(batch["inputs"], batch["targets"], batch["targets_segmentation"]):
    lg = O.forward(leaves, sp, row.tolist())
    loss = loss + (torch.nn.functional.cross_entropy(lg, tgt.long(), reduction="none") * (seg != 0)).sum()
  loss.backward()
  params = eng.model.store.params
  for ours, theirs in (("attention_layers_0/pass_input/kernel", "loop.in"), ("token_embedder/embedding", "embed"), ("decoder/embedding_norm/scale", "embed.norm"),
                       ("attention_layers_1_0/mixer/talk/kernel", "l1.mix.talk"), ("attention_layers_0/mlp/act", "l0.mlp.act"),
                       ("attention_layers_1_0/residual_gate/mlp/kernel", "l1.rg2"), ("attention_layers_2_0/mixer/key/kernel", "l2.mix.k")):
    got = params[ours].main_grad
    assert M.rel(got.reshape(leaves[theirs].shape)[None], leaves[theirs].grad[None]) < 1e-4, theirs


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
  sp = M.spec([(M.attention(2, 1, 8, 4, 0.4), M.dense(24)), (M.attention(4, 2, 8, 8, 0.4), M.moe(3, 1, 16, 8))], 32, loop=(1, 2, 2), vocab=300)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  assert isinstance(decode(M.config(path, "float32", "cpu", max_len=24, tokenizer_type="byte"), prompt="hello"), str)
