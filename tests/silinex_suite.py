"""Checks of the Silinex family that hold on every device: the CPU and the GPU test files run them with their own tolerance."""
import random

import pytest
import torch

import silinex_models as M


class Suite:
  device = "cpu"
  dtypes = ("float32",)
  # worst row; and the middle row, which rounding cannot move far (the first tokens' rows may stand on almost cancelled sums)
  tol = {"float32": 5e-5, "bfloat16": 0.4}
  mid = {"float32": 1e-5, "bfloat16": 0.04}
  len_ = 90

  def build(self, tmp_path, name, dtype, seed=0, **kw):
    sp = M.SPECS[name]
    W = M.weights(sp, seed)
    path = M.write_folder(tmp_path / name, sp, W)
    return sp, W, M.engine(path, dtype, self.device, **kw)

  def check(self, got, want, dtype, what=""):
    e = M.rel_rows(got, want)
    assert float(e.max()) < self.tol[dtype] and (len(e) < 8 or float(e.median()) < self.mid[dtype]), f"{what}: worst {float(e.max())}, middle {float(e.median())}"

  # ---- every mechanism alone and together, whole prompts
  @pytest.mark.parametrize("name", sorted(M.SPECS))
  def test_prompt(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(self.len_, sp)
      self.check(M.run_pieces(eng, toks, [len(toks)]), M.oracle_logits(sp, W, toks), dtype, name)

  # ---- token by token from the first token, and a prompt followed by decoding
  @pytest.mark.parametrize("name", ["delta", "delta_six_taps", "gla", "latent", "latent_tc", "mixed", "mixed_even"])
  def test_decode(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(40, sp)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [1]), want, dtype, "token by token")
      for first in (1, 2, 3, 17):
        self.check(M.run_pieces(eng, toks, [first, 1]), want, dtype, f"prompt of {first}")

  # ---- portions
  @pytest.mark.parametrize("name", ["delta", "gla", "latent", "latent_window_1", "latent_tc", "mixed"])
  def test_portions(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(75, sp)
      want = M.oracle_logits(sp, W, toks)
      for sizes in ([2], [7], [33], [1, 40, 1, 5], [70, 2]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"portions {sizes}")

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
        self.check(lg[at:at + n], w[:n], dtype, f"prompt of {n}")
        at += n
      for step in range(6):
        live = [i for i in range(5) if step < 6 - i]
        lg = eng.extend(state, live, [[seqs[i][lens[i] + step]] for i in live])
        for row, i in zip(lg, live):
          self.check(row[None], want[i][lens[i] + step][None], dtype, f"request {i}, decoded {step}")

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
        self.check(M.run_pieces(eng, b, sizes, state, 1), want, dtype, f"reused slot, pieces {sizes}")
        eng.free_slot(state, 1)
      # a dirty slot must not change its neighbours either
      M.run_pieces(eng, a, [60], state, 0)
      self.check(M.run_pieces(eng, b, [5, 1], state, 2), want, dtype, "neighbour of a dirty slot")

  # ---- exactly the window: a token at distance window - 1 matters, one at distance window does not
  @pytest.mark.parametrize("name", ["latent", "latent_window_1", "latent_tc", "latent_tc_wide"])
  @pytest.mark.parametrize("sizes", [[200], [64, 1], [1], [50, 13]])
  def test_window_edges(self, tmp_path, name, sizes):
    sp = M.SPECS[name]
    path = M.write_folder(tmp_path / name, sp, M.weights(sp, sharp=0.4))               # flat scores: every key of the window counts
    win = sp["layers"][0]["mixer"]["mask"]["size"]
    n = 100
    toks = M.prompt(n, sp)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      base = M.run_pieces(eng, toks, sizes)
      for j in (0, 3, 20):
        other = list(toks)
        other[j] = (toks[j] + 1) % sp["vocab"]
        moved = (M.run_pieces(eng, other, sizes) - base).abs().amax(-1).cpu()
        inside, outside = moved[j:min(n, j + win)], torch.cat([moved[:j], moved[j + win:]])
        assert float(inside[0]) > 1e-3 and float(inside.min()) > 0, f"{dtype}, token {j}: a key inside the window of {win} is not seen"
        assert outside.numel() == 0 or float(outside.max()) == 0, f"{dtype}, token {j}: a key outside the window of {win} is seen"

  # ---- one key that stands out, anywhere in the window
  def test_far_key_stands_out(self, tmp_path):
    for dtype in self.dtypes:
      sp, W0, _ = self.build(tmp_path, "latent_tc", dtype)
      W = M.weights(sp, 3, sharp=12.0)
      eng = M.engine(M.write_folder(tmp_path / "sharp", sp, W), dtype, self.device)
      toks = M.prompt(100, sp)
      want = M.oracle_logits(sp, W, toks)
      for sizes in ([100], [30, 1]):
        e = M.rel_rows(M.run_pieces(eng, toks, sizes), want)
        assert float(e.median()) < 4 * self.mid[dtype] and float(e.max()) < 10 * self.tol[dtype], e.max()

  # ---- long decoding: the state neither drifts nor is lost
  def test_long_decode(self, tmp_path):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, "mixed", dtype, max_len=300)
      toks = M.prompt(260, sp, 9)
      got = M.run_pieces(eng, toks, [4, 1])
      self.check(got, M.oracle_logits(sp, W, toks), dtype, "long decode")

  # ---- greedy generation through the engine's own entry points and scheduler
  @pytest.mark.parametrize("packed", [False, True])
  def test_greedy_through_the_scheduler(self, tmp_path, packed):
    from maxtext_b200.inference.offline_engine import OfflineEngine
    sp, W, eng = self.build(tmp_path, "mixed", "float32", max_len=64)
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
