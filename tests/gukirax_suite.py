"""Checks of the Gukirax family that hold on every device: the CPU and the GPU test files run them with their own tolerance."""
import random

import pytest
import torch

import gukirax_models as M


class Suite:
  device = "cpu"
  dtypes = ("float32",)
  # worst row; and the middle row, which rounding cannot move far. In bf16 a close call of a router may choose another expert, so models with
  # experts are held to the middle row there, on prompts whose first tokens choose clearly (the fp32 run and the kernel tests hold every row).
  tol = {"float32": 5e-5, "bfloat16": 0.15}
  mid = {"float32": 1e-5, "bfloat16": 0.04}
  len_ = 90

  def build(self, tmp_path, name, dtype, seed=0, **kw):
    sp = M.SPECS[name]
    W = M.weights(sp, seed)
    path = M.write_folder(tmp_path / name, sp, W)
    return sp, W, M.engine(path, dtype, self.device, **kw)

  def check(self, got, want, dtype, what="", routed=False):
    e = M.rel_rows(got, want)
    worst, middle = float(e.max()), float(e.median())
    loose = routed and dtype == "bfloat16"
    assert (loose or worst < self.tol[dtype]) and (len(e) < 8 or middle < self.mid[dtype]), f"{what}: worst {worst}, middle {middle}"

  # ---- every mechanism alone and together, whole prompts
  @pytest.mark.parametrize("name", sorted(M.SPECS))
  def test_prompt(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.clear_prompt(self.len_, sp, W)
      self.check(M.run_pieces(eng, toks, [len(toks)]), M.oracle_logits(sp, W, toks), dtype, name, M.has_experts(sp))

  # ---- token by token from the first token, and a prompt followed by decoding
  @pytest.mark.parametrize("name", ["heads", "heads_one_key", "heads_odd", "heads_single", "heads_64", "heads_20", "heads_many_keys", "heads_wide", "experts",
                                    "experts_all", "loop_all", "loop_one", "loop_once", "mixed", "mixed_even"])
  def test_decode(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.clear_prompt(40, sp, W)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [1]), want, dtype, "token by token", M.has_experts(sp))
      for first in (1, 2, 3, 17):
        self.check(M.run_pieces(eng, toks, [first, 1]), want, dtype, f"prompt of {first}", M.has_experts(sp))

  # ---- portions
  @pytest.mark.parametrize("name", ["heads", "heads_128", "heads_many_keys", "heads_wide", "experts", "loop_all", "mixed"])
  def test_portions(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.clear_prompt(75, sp, W)
      want = M.oracle_logits(sp, W, toks)
      for sizes in ([2], [7], [33], [1, 40, 1, 5], [70, 2]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"portions {sizes}", M.has_experts(sp))

  # ---- requests of unequal lengths in one batch, then decoded together while the shorter ones end
  @pytest.mark.parametrize("name", ["mixed", "mixed_even"])
  def test_batch(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      lens = [1, 40, 2, 23, 77]
      seqs = [M.clear_prompt(n + 6, sp, W, seed=n) for n in lens]
      want = [M.oracle_logits(sp, W, s) for s in seqs]
      state = eng.init_decode_state(len(lens))
      lg = eng.extend(state, [0, 1, 2, 3, 4], [s[:n] for s, n in zip(seqs, lens)], [list(range(n)) for n in lens])
      at = 0
      for n, w in zip(lens, want):
        self.check(lg[at:at + n], w[:n], dtype, f"prompt of {n}", True)
        at += n
      for step in range(6):
        live = [i for i in range(5) if step < 6 - i]
        lg = eng.extend(state, live, [[seqs[i][lens[i] + step]] for i in live])
        for row, i in zip(lg, live):
          self.check(row[None], want[i][lens[i] + step][None], dtype, f"request {i}, decoded {step}", True)

  def test_a_request_does_not_see_its_neighbours(self, tmp_path):
    """Each of a batch against itself alone, on the same device and number format."""
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "mixed", dtype)
      lens = [5, 31, 12]
      seqs = [M.clear_prompt(n + 3, sp, W, seed=50 + n) for n in lens]
      state = eng.init_decode_state(3)
      both = [eng.extend(state, [2, 0, 1], [s[:n] for s, n in zip(seqs, lens)])]
      for j in range(3):
        both.append(eng.extend(state, [2, 0, 1], [[s[n + j]] for s, n in zip(seqs, lens)]))
      for i, (s, n) in enumerate(zip(seqs, lens)):
        alone = M.run_pieces(eng, s, [n, 1])
        for j in range(4):
          e = M.rel(both[j][i][None], alone[n - 1 + j][None].double().cpu())
          assert e < (1e-4 if dtype == "float32" else 0.15), (dtype, i, j, e)

  # ---- every pass of a loop has keys of its own; a slot that is used again starts from nothing
  def test_slot_reuse(self, tmp_path):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "mixed", dtype)
      state = eng.init_decode_state(3)
      assert len(state.caches) == len(M.O.layer_runs(sp)) and len({id(c) for layer in state.caches for c in layer}) == len(state.caches)
      a, b = M.prompt(60, sp, 5), M.clear_prompt(12, sp, W, 6, 12)
      M.run_pieces(eng, a, [30, 1], state, 1)
      eng.free_slot(state, 1)
      want = M.oracle_logits(sp, W, b)
      for sizes in ([12], [1], [2, 1]):
        self.check(M.run_pieces(eng, b, sizes, state, 1), want, dtype, f"reused slot, pieces {sizes}", True)
        eng.free_slot(state, 1)
      # a dirty slot must not change its neighbours either
      M.run_pieces(eng, a, [60], state, 0)
      self.check(M.run_pieces(eng, b, [5, 1], state, 2), want, dtype, "neighbour of a dirty slot", True)

  # ---- one key among many stands out: every position back to the first token is reached, in prompts and in decoding
  @pytest.mark.parametrize("name", ["heads_64", "heads_20", "heads_many_keys"])
  def test_far_key_stands_out(self, tmp_path, name):
    sp = M.SPECS[name]
    sp = {**sp, "layers": [{**lay, "mixer": {**lay["mixer"], "scale": 16.0 / lay["mixer"]["dim"], "rot": {"base": 1e9, "dims": 4}}} for lay in sp["layers"]],
          "vocab": 300}
    W = M.matching_heads(sp, M.weights(sp, 3), 298, 299)
    path = M.write_folder(tmp_path / "sharp", sp, W)
    n = 150
    base = torch.randperm(298, generator=torch.Generator().manual_seed(1))[:n].tolist()
    base[-1] = 298
    other = M.oracle_logits(sp, W, base)
    engines = {dtype: M.engine(path, dtype, self.device, max_len=200) for dtype in self.dtypes}
    for j in (0, 1, 15, 16, 63, 64, 127, 128, 145):
      toks = list(base)
      toks[j] = 299                                                            # what the last token looks for
      want = M.oracle_logits(sp, W, toks)
      assert M.rel(want[-1:], other[-1:]) > 0.05, f"{M.rel(want[-1:], other[-1:])}: the key at place j does not matter in this model"
      for dtype, eng in engines.items():
        for sizes in ([n], [n - 1, 1], [60, 30, 1]):
          e = M.rel(M.run_pieces(eng, toks, sizes)[-1:], want[-1:])
          assert e < (self.tol[dtype] if dtype == "float32" else 0.03), (dtype, j, sizes, e)

  # ---- what a fault would hide behind: each of these must change the result, and the framework must follow
  @pytest.mark.parametrize("change", ["sink", "talk", "gate", "gate_bias", "xielu_p", "xielu_q", "shared", "embed_norm", "pass_input", "times", "logit_scale", "logit_softcap",
                                      "scale", "rotation", "eps"])
  def test_every_constant_counts(self, tmp_path, change):
    sp = M.SPECS["mixed"]
    W = M.weights(sp)
    before = (sp, dict(W))
    sp = {**sp, "loop": dict(sp["loop"]), "layers": [{**lay, "mixer": dict(lay["mixer"])} for lay in sp["layers"]]}
    if change == "sink":
      W["l2.mix.sink"] = W["l2.mix.sink"] + 5.0
    elif change == "talk":
      W["l1.mix.talk"] = W["l1.mix.talk"].t().contiguous() * 2.0
    elif change == "gate":
      W["l3.rg1"] = -2.0 * W["l3.rg1"]
    elif change == "gate_bias":
      W["l4.rg2.b"] = torch.linspace(-3, 3, sp["width"])
    elif change == "xielu_p":
      W["l0.mlp.act"] = W["l0.mlp.act"] + torch.tensor([4.0, 0.0])
    elif change == "xielu_q":
      W["l4.mlp.act"] = W["l4.mlp.act"] + torch.tensor([0.0, 4.0])
    elif change == "shared":
      W["l1.mlp.shared.down"] = -3.0 * W["l1.mlp.shared.down"]
    elif change == "embed_norm":
      W["embed.norm"] = W["embed.norm"].flip(0)
    elif change == "pass_input":
      d = sp["width"]
      W["loop.in"] = torch.cat([W["loop.in"][:, d:], W["loop.in"][:, :d]], 1)
    elif change == "times":
      sp["loop"]["times"] = 3
    elif change == "logit_scale":
      sp["logit_scale"] = 1.9
    elif change == "logit_softcap":
      sp["logit_softcap"] = 0.8
    elif change == "scale":
      sp["layers"][2]["mixer"]["scale"] = 0.6
    elif change == "rotation":
      sp["layers"][4]["mixer"]["rot"] = {"base": 3.0, "dims": 32}
    else:
      sp["norm"] = {"eps": 0.2}
    W = {k: v.bfloat16().float() for k, v in W.items()}
    toks = M.clear_prompt(30, sp, W)
    want = M.oracle_logits(sp, W, toks)
    assert M.rel(want, M.oracle_logits(*before, toks)) > 1e-2
    path = M.write_folder(tmp_path / "m", sp, W)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for sizes in ([30], [9, 1]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"{change}, pieces {sizes}", True)

  # ---- long decoding: hundreds of keys, every pass of a loop with its own
  def test_long_decode(self, tmp_path):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "loop_all", dtype, max_len=300)
      toks = M.prompt(260, sp, 9)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [4, 1]), want, dtype, "long decode")
      self.check(M.run_pieces(eng, toks, [260]), want, dtype, "long prompt")

  # ---- greedy generation through the engine's own entry points and scheduler
  @pytest.mark.parametrize("packed", [False, True])
  @pytest.mark.parametrize("name", ["mixed", "heads_128"])
  def test_greedy_through_the_scheduler(self, tmp_path, name, packed):
    from maxtext_b200.inference.offline_engine import OfflineEngine
    sp, W, eng = self.build(tmp_path, name, "float32", max_len=64)
    prompts = [M.prompt(n, sp, 20 + n) for n in (3, 17, 1, 9, 26)]
    want = [M.greedy_oracle(sp, W, p, 7) for p in prompts]
    off = OfflineEngine(eng, slots=3 if packed else 2, enable_batch_prefill=packed)
    assert off.batch_inference(prompts, max_new_tokens=7) == want

  @pytest.mark.parametrize("name", ["mixed", "mixed_even"])
  def test_prefill_entry_points_agree(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = torch.tensor(M.clear_prompt(37, sp, W, 3))
      want = M.oracle_logits(sp, W, toks.tolist())[-1][None]
      self.check(eng.prefill(toks, 37)[0].logits, want, dtype, "prefill")
      self.check(eng.prefill_chunked(toks, 10)[0].logits, want, dtype, "prefill_chunked")
      other = torch.tensor(M.clear_prompt(8, sp, W, 4))
      both = eng.prefill_concat([toks, other])
      self.check(both[0].logits, want, dtype, "prefill_concat")
      self.check(both[1].logits, M.oracle_logits(sp, W, other.tolist())[-1][None], dtype, "prefill_concat, second prompt")
      if dtype != "float32":
        continue
      state = eng.init_decode_state(2)
      state = eng.insert(both[1], eng.insert(both[0], state, 1), 0)
      ref = [M.greedy_oracle(sp, W, p, 4) for p in (other.tolist(), toks.tolist())]
      got = [[int(both[1].first_token)], [int(both[0].first_token)]]
      for _ in range(3):
        state, res = eng.generate(state)
        for s in range(2):
          got[s].append(int(res.data[s, 0]))
      assert got == ref

  def test_results_do_not_depend_on_the_cut(self, tmp_path):
    sp, W, eng = self.build(tmp_path, "mixed_even", "float32")
    rng = random.Random(0)
    toks = M.prompt(90, sp)
    base = M.run_pieces(eng, toks, [90])
    for _ in range(3):
      sizes = [rng.choice([1, 2, 3, 5, 8, 16, 31]) for _ in range(60)]
      self.check(M.run_pieces(eng, toks, sizes), base.double().cpu(), "float32", f"pieces {sizes[:8]} ...")
