"""Checks of the Tipidra family that hold on every device: the CPU and the GPU test files run them with their own tolerance."""
import random

import pytest
import torch

import tipidra_models as M


class Suite:
  device = "cpu"
  dtypes = ("float32",)
  # worst row; and the middle row, which rounding cannot move far. In bf16 a close call of a router may choose another expert, so models with
  # experts are held to the middle row there (the fp32 run and the kernel tests hold every row).
  tol = {"float32": 5e-5, "bfloat16": 0.3}
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
      toks = M.prompt(self.len_, sp)
      self.check(M.run_pieces(eng, toks, [len(toks)]), M.oracle_logits(sp, W, toks), dtype, name, M.has_experts(sp))

  # ---- token by token from the first token, and a prompt followed by decoding
  @pytest.mark.parametrize("name", ["attention", "attention_one_kv_head", "attention_odd", "attention_64", "attention_wide_keys", "attention_beyond_flash", "scan",
                                    "scan_smallest", "scan_16", "scan_64", "scan_many_states", "experts", "experts_all", "mixed", "mixed_even"])
  def test_decode(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(40, sp)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [1]), want, dtype, "token by token", M.has_experts(sp))
      for first in (1, 2, 3, 17):
        self.check(M.run_pieces(eng, toks, [first, 1]), want, dtype, f"prompt of {first}", M.has_experts(sp))

  # ---- portions
  @pytest.mark.parametrize("name", ["attention", "attention_128", "attention_narrow_values", "attention_beyond_flash", "scan", "scan_16", "experts", "mixed"])
  def test_portions(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(75, sp)
      want = M.oracle_logits(sp, W, toks)
      for sizes in ([2], [7], [33], [1, 40, 1, 5], [70, 2]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"portions {sizes}", M.has_experts(sp))

  # ---- requests of unequal lengths in one batch, then decoded together while the shorter ones end
  @pytest.mark.parametrize("name", ["mixed", "mixed_even"])
  def test_batch(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      lens = [1, 40, 2, 23, 77]
      seqs = [M.prompt(n + 6, sp, seed=n) for n in lens]
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
      seqs = [M.prompt(n + 3, sp, seed=50 + n) for n in lens]
      state = eng.init_decode_state(3)
      both = [eng.extend(state, [2, 0, 1], [s[:n] for s, n in zip(seqs, lens)])]
      for j in range(3):
        both.append(eng.extend(state, [2, 0, 1], [[s[n + j]] for s, n in zip(seqs, lens)]))
      for i, (s, n) in enumerate(zip(seqs, lens)):
        alone = M.run_pieces(eng, s, [n, 1])
        for j in range(4):
          e = M.rel(both[j][i][None], alone[n - 1 + j][None].double().cpu())
          assert e < (1e-4 if dtype == "float32" else 0.15), (dtype, i, j, e)

  # ---- a slot that is used again starts from nothing
  def test_slot_reuse(self, tmp_path):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "mixed", dtype)
      state = eng.init_decode_state(3)
      a, b = M.prompt(60, sp, 5), M.prompt(12, sp, 6)
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
  @pytest.mark.parametrize("name", ["attention_narrow_values", "attention_64"])
  def test_far_key_stands_out(self, tmp_path, name):
    sp = M.SPECS[name]
    sp = {**sp, "layers": [{**lay, "mixer": {**lay["mixer"], "scale": 16.0 / lay["mixer"]["dim"], "softcap": 40.0, "rot": {"base": 1e9, "dims": 4}}}
                           for lay in sp["layers"]], "vocab": 200}
    W = M.matching_heads(sp, M.weights(sp, 3), 198, 199)
    path = M.write_folder(tmp_path / "sharp", sp, W)
    n = 100
    base = torch.randperm(198, generator=torch.Generator().manual_seed(1))[:n].tolist()
    base[-1] = 198
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for j in (0, 1, 15, 16, 63, 64, 95):
        toks = list(base)
        toks[j] = 199                                                          # what the last token looks for
        want, other = M.oracle_logits(sp, W, toks), M.oracle_logits(sp, W, base)
        assert M.rel(want[-1:], other[-1:]) > 0.05, f"{M.rel(want[-1:], other[-1:])}: the key at place j does not matter in this model"
        for sizes in ([n], [n - 1, 1], [60, 30, 1]):
          e = M.rel(M.run_pieces(eng, toks, sizes)[-1:], want[-1:])
          assert e < (self.tol[dtype] if dtype == "float32" else 0.05), (dtype, j, sizes, e)

  # ---- what a fault would hide behind: each of these must change the result, and the framework must follow
  @pytest.mark.parametrize("change", ["sink", "softcap", "embedding", "logit_softcap", "limit", "mix", "bias", "skip", "rotation"])
  def test_every_constant_counts(self, tmp_path, change):
    sp = M.SPECS["mixed"]
    W = M.weights(sp)
    toks = M.prompt(30, sp)
    before = M.oracle_logits(sp, W, toks)
    sp = {**sp, "layers": [{**lay, "mixer": dict(lay["mixer"]), "mlp": dict(lay["mlp"]) if lay["mlp"] else None} for lay in sp["layers"]]}
    if change == "sink":
      W["l1.mix.sink"] = W["l1.mix.sink"] + 5.0
    elif change == "softcap":
      sp["layers"][1]["mixer"]["softcap"] = 0.5
    elif change == "embedding":
      sp["embedding"] = {"scale": 0.75}
    elif change == "logit_softcap":
      sp["logit_softcap"] = 0.8
    elif change == "limit":
      sp["layers"][1]["mlp"]["expert"] = {"ff": 28, "limit": 0.05}
    elif change == "mix":
      W["l2.hc1.mix"] = W["l2.hc1.mix"].t().contiguous()
    elif change == "bias":
      W["l3.norm1.b"] = W["l3.norm1.b"] + 0.5
    elif change == "skip":
      W["l0.mix.D"] = -W["l0.mix.D"]
    else:
      sp["layers"][3]["mixer"]["rot"] = {"base": 90.0, "dims": 20}
    W = {k: v.bfloat16().float() for k, v in W.items()}
    want = M.oracle_logits(sp, W, toks)
    assert M.rel(want, before) > 1e-2
    path = M.write_folder(tmp_path / "m", sp, W)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for sizes in ([30], [9, 1]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"{change}, pieces {sizes}", True)

  # ---- long decoding: the state neither drifts nor is lost
  def test_long_decode(self, tmp_path):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "scan_16", dtype, max_len=300)
      W = dict(W, **{"l0.mix.dt.b": torch.full_like(W["l0.mix.dt.b"], -5.0)})          # slow decays: hundreds of tokens stay in the state
      eng = M.engine(M.write_folder(tmp_path / "slow", sp, W), dtype, self.device, max_len=300)
      toks = M.prompt(260, sp, 9)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [4, 1]), want, dtype, "long decode")
      self.check(M.run_pieces(eng, toks, [260]), want, dtype, "long prompt")

  # ---- greedy generation through the engine's own entry points and scheduler
  @pytest.mark.parametrize("packed", [False, True])
  @pytest.mark.parametrize("name", ["mixed", "attention_128"])
  def test_greedy_through_the_scheduler(self, tmp_path, name, packed):
    from maxtext_b200.inference.offline_engine import OfflineEngine
    sp, W, eng = self.build(tmp_path, name, "float32", max_len=64)
    prompts = [M.prompt(n, sp, 20 + n) for n in (3, 17, 1, 9, 26)]
    want = [M.greedy_oracle(sp, W, p, 7) for p in prompts]
    off = OfflineEngine(eng, slots=3 if packed else 2, enable_batch_prefill=packed)
    assert off.batch_inference(prompts, max_new_tokens=7) == want

  def test_prefill_entry_points_agree(self, tmp_path):
    sp, W, eng = self.build(tmp_path, "mixed", "float32")
    toks = torch.tensor(M.prompt(37, sp, 3))
    want = M.oracle_logits(sp, W, toks.tolist())[-1][None]
    self.check(eng.prefill(toks, 37)[0].logits, want, "float32", "prefill")
    self.check(eng.prefill_chunked(toks, 10)[0].logits, want, "float32", "prefill_chunked")
    other = torch.tensor(M.prompt(8, sp, 4))
    both = eng.prefill_concat([toks, other])
    self.check(both[0].logits, want, "float32", "prefill_concat")
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
