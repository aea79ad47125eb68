"""Checks of the Sitivik family that hold on every device: the CPU and the GPU test files run them with their own tolerance."""
import copy
import random

import pytest
import torch

import sitivik_models as M


class Suite:
  device = "cpu"
  dtypes = ("float32",)
  tol = {"float32": 5e-5, "bfloat16": 0.3}        # worst row
  mid = {"float32": 1e-5, "bfloat16": 0.04}       # middle row, which rounding cannot move far
  len_ = 90

  def build(self, tmp_path, name, dtype, seed=0, **kw):
    sp = M.SPECS[name]
    W = M.weights(sp, seed)
    return sp, W, M.engine(M.folder(tmp_path / name, sp, W), dtype, self.device, **kw)

  def check(self, got, want, dtype, what=""):
    e = M.rel_rows(got, want)
    worst, middle = float(e.max()), float(e.median())
    assert worst < self.tol[dtype] and (len(e) < 8 or middle < self.mid[dtype]), f"{what}: worst {worst}, middle {middle}"

  # ---- every mechanism alone and together, whole prompts
  @pytest.mark.parametrize("name", sorted(M.SPECS))
  def test_prompt(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(self.len_, sp)
      self.check(M.run_pieces(eng, toks, [len(toks)]), M.oracle_logits(sp, W, toks), dtype, name)

  # ---- token by token from the first token, and a prompt followed by decoding
  @pytest.mark.parametrize("name", sorted(M.SPECS))
  def test_decode(self, tmp_path, name):
    for dtype in self.dtypes:
      sp, W, eng = self.build(tmp_path, name, dtype)
      toks = M.prompt(40, sp)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [1]), want, dtype, "token by token")
      for first in (1, 2, 3, 17):
        self.check(M.run_pieces(eng, toks, [first, 1]), want, dtype, f"prompt of {first}")

  # ---- portions
  @pytest.mark.parametrize("name", ["window", "window_128", "window_beyond_flash", "chunk", "chunk_64", "differential_one_kv_head", "differential_128",
                                    "differential_apart", "differential_widest", "mixed"])
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
        self.check(M.run_pieces(eng, b, sizes, state, 1), want, dtype, f"reused slot, pieces {sizes}")
        eng.free_slot(state, 1)
      # a dirty slot must not change its neighbours either
      M.run_pieces(eng, a, [60], state, 0)
      self.check(M.run_pieces(eng, b, [5, 1], state, 2), want, dtype, "neighbour of a dirty slot")

  # ---- one key among many stands out, just inside and just outside every window and chunk, and far away
  def sharp(self, tmp_path, name, places, n, clear, change=None):
    """The last of n tokens looks for the one at each place. `clear`: the places at which seeing it or not must show; `change(spec)`: the mask
    off by one, which must give another result at some of them."""
    base_spec = {**M.SPECS[name], "vocab": 200}
    sp, W = M.sharpened(base_spec, M.weights(base_spec, 3), 198, 199)
    path = M.folder(tmp_path / "sharp", sp, W)
    base = torch.randperm(198, generator=torch.Generator().manual_seed(1))[:n].tolist()
    base[-1] = 198
    wants, shows = {}, 0
    for j in places:
      toks = list(base)
      toks[j] = 199
      wants[j] = toks, M.oracle_logits(sp, W, toks)[-1:]
      if change is not None:
        for off in (-1, 1):
          other = change(copy.deepcopy(sp), off)
          shows += M.rel(M.oracle_logits(other, W, toks)[-1:], wants[j][1]) > 0.05
      elif j in clear:
        shows += M.rel(M.oracle_logits(sp, W, base)[-1:], wants[j][1]) > 0.05
    assert shows >= len(clear), (shows, clear)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for j, (toks, want) in wants.items():
        for sizes in ([n], [n - 1, 1], [n // 2, n - n // 2 - 3, 1], [n - 2, 2]):
          e = M.rel(M.run_pieces(eng, toks, sizes)[-1:], want)
          assert e < (self.tol[dtype] if dtype == "float32" else 0.06), (dtype, j, sizes, e)

  @pytest.mark.parametrize("name", ["window_stretched", "window_64", "window_128", "window_beyond_flash"])
  def test_window_edges(self, tmp_path, name):
    size, n = M.SPECS[name]["layers"][0]["mixer"]["left"]["mask"]["size"], 100

    def change(sp, off):
      sp["layers"][0]["mixer"]["left"]["mask"]["size"] += off
      return sp
    self.sharp(tmp_path, name, [n - size - 2, n - size - 1, n - size, n - size + 1, 0], n, [n - size - 1, n - size], change)

  @pytest.mark.parametrize("name, n", [("chunk", 88), ("chunk_64", 93), ("chunk_64", 94), ("chunk_wide", 100), ("chunk_wide", 101), ("delta_unaligned", 85)])
  def test_chunk_edges(self, tmp_path, name, n):
    """The last token at a chunk's end, start or middle; keys on both sides of the chunk's start, which counts from the first token whatever the
    prompt's portions are."""
    size = M.SPECS[name]["layers"][0]["mixer"]["left"]["mask"]["size"]
    start = (n - 1) // size * size

    def change(sp, off):
      sp["layers"][0]["mixer"]["left"]["mask"]["size"] += off
      return sp
    places = sorted({j for j in (0, start - 2, start - 1, start, start + 1, n - 2) if 0 <= j < n - 1})
    self.sharp(tmp_path, name, places, n, [start - 1, start][: 1 if start == n - 1 else 2], change)

  @pytest.mark.parametrize("name", ["differential_one_kv_head", "differential_64", "differential_128", "differential_apart"])
  def test_far_keys(self, tmp_path, name):
    places = [0, 1, 15, 16, 63, 64, 97]
    self.sharp(tmp_path, name, places, 100, places)

  # ---- what a fault would hide behind: each of these must change the result, and the framework must follow
  @pytest.mark.parametrize("change", ["embedding", "bias", "out_bias", "out_norm", "lane_factor", "decay", "stretch", "temperature", "diff", "lambda", "gate",
                                      "scales", "convolution", "dt_bias", "side_table", "side_norm", "qk_norm", "rotation", "vdim_gate"])
  def test_every_constant_counts(self, tmp_path, change):
    sp = copy.deepcopy(M.SPECS["mixed"])
    W = M.weights(sp)
    toks = M.prompt(30, sp)
    before = M.oracle_logits(sp, W, toks)
    mix = [lay["mixer"] for lay in sp["layers"]]
    if change == "embedding":
      sp["embedding"] = {"scale": 0.75}
    elif change == "bias":
      W["l2.mix.left.k.b"] = W["l2.mix.left.k.b"] + 1.0
    elif change == "out_bias":
      W["l0.mix.left.o.b"] = -2.0 * W["l0.mix.left.o.b"]
    elif change == "out_norm":
      W["l3.mix.left.out"] = W["l3.mix.left.out"] + 1.0
    elif change == "lane_factor":
      W["l4.ls1"] = -W["l4.ls1"]
    elif change == "decay":
      mix[0]["right"]["decay"] = [0.3, 0.9, 0.99]
    elif change == "stretch":
      mix[0]["left"]["rot"]["scaling"] = {"factor": 8.0, "low": 1.0, "high": 3.0, "original": 50}
    elif change == "temperature":
      mix[1]["q_temp"] = {"coef": 3.0, "every": 2}
    elif change == "diff":
      mix[1]["diff"] = 0.9
    elif change == "lambda":
      W["l1.mix.lk1"], W["l1.mix.lq1"] = torch.full_like(W["l1.mix.lk1"], 0.3), torch.full_like(W["l1.mix.lq1"], 0.4)
    elif change == "gate":
      W["l1.mix.g"] = -4.0 * W["l1.mix.g"]
    elif change == "scales":
      mix[2]["left_scale"], mix[4]["right_scale"] = -0.5, 0.3
    elif change == "convolution":
      W["l2.mix.right.k.conv"] = W["l2.mix.right.k.conv"].flip(1).contiguous()
    elif change == "dt_bias":
      W["l4.mix.right.dt_bias"] = W["l4.mix.right.dt_bias"] + 3.0
    elif change == "side_table":
      W["side.embed"] = W["side.embed"].roll(sp["token_side"]["dim"], 1).contiguous()
    elif change == "side_norm":
      W["l2.side.norm"] = -W["l2.side.norm"]
    elif change == "qk_norm":
      W["l2.mix.left.q.norm"], W["l0.mix.left.k.norm"] = W["l2.mix.left.q.norm"] * -2.0, W["l0.mix.left.k.norm"] * 3.0
    elif change == "rotation":
      mix[4]["left"]["rot"] = {"base": 20.0, "dims": 18}
      mix[0]["right"]["rot"] = {"base": 5.0, "dims": 16}
    else:
      W["l3.mix.left.g"], W["l3.mix.right.g"] = -2.0 * W["l3.mix.left.g"], W["l3.mix.right.g"] * 3.0
    W = {k: v.bfloat16().float() for k, v in W.items()}
    want = M.oracle_logits(sp, W, toks)
    assert M.rel(want, before) > 1e-2
    path = M.folder(tmp_path / "m", sp, W)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for sizes in ([30], [9, 1]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"{change}, pieces {sizes}")

  # ---- strong and vanishing decays: the prompt's chunks against the token recurrence
  @pytest.mark.parametrize("rate", [-6.0, 3.0])
  def test_extreme_decays(self, tmp_path, rate):
    sp = M.SPECS["chunk_64"]
    W = M.weights(sp, 4)
    W["l0.mix.right.A_log"] = torch.full_like(W["l0.mix.right.A_log"], rate)
    path = M.folder(tmp_path / "m", sp, W)
    toks = M.prompt(140, sp, 2)
    want = M.oracle_logits(sp, W, toks)
    for dtype in self.dtypes:
      eng = M.engine(path, dtype, self.device)
      for sizes in ([140], [100, 30, 1]):
        self.check(M.run_pieces(eng, toks, sizes), want, dtype, f"rate {rate}, pieces {sizes}")

  # ---- long decoding: the states neither drift nor are lost
  @pytest.mark.parametrize("name", ["window_64", "chunk_64"])
  def test_long_decode(self, tmp_path, name):
    for dtype in self.dtypes:
      sp = copy.deepcopy(M.SPECS[name])
      W = M.weights(sp, 6)
      if name == "chunk_64":
        W["l0.mix.right.dt_bias"] = torch.full_like(W["l0.mix.right.dt_bias"], -6.0)       # hundreds of tokens stay in the state
      else:
        sp["layers"][0]["mixer"]["right"]["decay"] = [0.999, 0.9999, 1.0]
      W = {k: v.bfloat16().float() for k, v in W.items()}
      eng = M.engine(M.folder(tmp_path / "slow", sp, W), dtype, self.device, max_len=300)
      toks = M.prompt(260, sp, 9)
      want = M.oracle_logits(sp, W, toks)
      self.check(M.run_pieces(eng, toks, [4, 1]), want, dtype, "long decode")
      self.check(M.run_pieces(eng, toks, [260]), want, dtype, "long prompt")

  # ---- greedy generation through the engine's own entry points and scheduler
  @pytest.mark.parametrize("packed", [False, True])
  @pytest.mark.parametrize("name", ["mixed", "differential_128"])
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
