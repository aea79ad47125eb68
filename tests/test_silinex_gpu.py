"""Silinex on the CUDA kernels: the shared suite in fp32 and bf16, the decode graph, and the kernels on shapes of their own."""
import pytest
import torch

import silinex_models as M
import silinex_oracle as O
from silinex_suite import Suite

pytestmark = pytest.mark.gpu


class TestSilinexGpu(Suite):
  device = "cuda"
  dtypes = ("float32", "bfloat16")


def _status():
  from maxtext_b200.ops import backend
  return backend.ext(required=True).kernel_status(True)


def test_graph_decode_equals_eager(tmp_path):
  """The captured decode step must leave recurrent states as if its warm-up had not happened."""
  for dtype in ("float32", "bfloat16"):
    sp = M.SPECS["mixed_even"]
    path = M.write_folder(tmp_path / dtype, sp, M.weights(sp))
    got = []
    for graphs in (False, True):
      eng = M.engine(path, dtype, "cuda", cuda_graphs=graphs)
      state = eng.init_decode_state(3)
      for s, n in enumerate((21, 2, 40)):
        state = eng.insert(eng.prefill(torch.tensor(M.prompt(n, sp, n)), n)[0], state, s)
      toks = [state.tokens.tolist()]
      for _ in range(12):
        state, res = eng.generate(state)
        toks.append(res.data[:, 0].tolist())
      if graphs:
        assert eng._graphs and all(g is not False for g in eng._graphs.values()), "the decode step was not captured"
      got.append(toks)
    assert got[0] == got[1]
  assert _status() == 0


def test_graph_decode_of_a_gated_delta_family():
  """The same for the released gated-delta configuration, whose states the warm-up used to advance."""
  from helpers import tiny_config
  from maxtext_b200.inference.maxengine import MaxEngine
  got = []
  for graphs in ("false", "true"):
    cfg = tiny_config("qwen3-next-80b-a3b", extra=["dtype=bfloat16", "weight_dtype=bfloat16", "hardware=gpu", "max_prefill_predict_length=24", f"cuda_graphs={graphs}",
                                                   "head_dim=64", "base_emb_dim=128"])
    eng = MaxEngine(cfg, device="cuda")
    eng.load_params()
    state = eng.insert(eng.prefill(torch.arange(3, 15), 12)[0], eng.init_decode_state(1), 0)
    toks = []
    for _ in range(8):
      state, res = eng.generate(state)
      toks.append(int(res.data[0, 0]))
    got.append(toks)
  assert got[0] == got[1]


def _delta_inputs(B, S, hk, r, dk, dv, dtype, seed=0):
  g = torch.Generator().manual_seed(seed)
  mixed = torch.randn(B * S, 2 * hk * dk + hk * r * dv, generator=g)
  ba = torch.randn(B * S, hk * 2 * r, generator=g)
  A, dt = torch.randn(hk * r, generator=g) - 1.0, torch.randn(hk * r, generator=g) - 1.0
  return [t.to(dtype).cuda() for t in (mixed, ba, A, dt)]


def _delta_want(mixed, ba, A, dt, B, S, hk, r, dk, dv, b, n):
  m, ba, A, dt = (t.double().cpu() for t in (mixed, ba, A, dt))
  m, ba = m.view(B, S, -1)[b, :n], ba.view(B, S, hk, 2, r)[b, :n]
  q, k, v = m[:, :hk * dk].view(n, hk, dk), m[:, hk * dk:2 * hk * dk].view(n, hk, dk), m[:, 2 * hk * dk:].view(n, hk * r, dv)
  q, k = O.unit(q).repeat_interleave(r, 1) * dk ** -0.5, O.unit(k).repeat_interleave(r, 1)
  beta, a = O.sigmoid(ba[:, :, 0].reshape(n, -1)), ba[:, :, 1].reshape(n, -1)
  return O.delta_recurrence(q, k, v, torch.exp(-torch.exp(A) * O.softplus(a + dt)), beta)


SCAN_CASES = [(2, 150, 2, 1, 128, 128, None), (1, 300, 1, 2, 64, 128, None), (3, 70, 2, 2, 96, 48, [70, 1, 65]), (2, 200, 1, 1, 128, 64, [64, 129]),
              (1, 90, 2, 1, 20, 12, None), (2, 33, 1, 3, 256, 32, [2, 33])]


@pytest.mark.parametrize("B, S, hk, r, dk, dv, lens", SCAN_CASES)
def test_delta_scan(B, S, hk, r, dk, dv, lens):
  from maxtext_b200.ops import backend
  E = backend.ext(required=True)
  for dtype, scan, tol in ((torch.float32, E.delta_scan, 2e-5), (torch.bfloat16, E.delta_scan, 1e-2), (torch.bfloat16, E.delta_chunks, 1e-2)):
    if scan is E.delta_chunks and not E.chunk_supported(dk, dv):
      continue
    args = _delta_inputs(B, S, hk, r, dk, dv, dtype)
    rec = torch.full((B + 1, hk * r, dk, dv), 7.0, device="cuda")             # row 0 unused, dirty states elsewhere
    slots, lengths = torch.arange(B, device="cuda") + 1, torch.zeros(B, dtype=torch.long, device="cuda")
    n = torch.tensor(lens, device="cuda") if lens else None
    o = torch.empty(B * S, hk * r * dv, dtype=dtype, device="cuda")
    scan(*args, hk, hk * r, dk, dv, S, rec, slots, lengths, n, o)
    for b in range(B):
      m = lens[b] if lens else S
      want = _delta_want(*args, B, S, hk, r, dk, dv, b, m)
      got = o.view(B, S, hk * r, dv)[b, :m].double().cpu()
      assert (got - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), (dtype, b)
      assert (got - want).abs().max() < 40 * tol * want.pow(2).mean().sqrt(), (dtype, b)
    assert float((rec[0] - 7.0).abs().max()) == 0.0
    # the second half continued from the state that the first half left
    half = S // 2
    if half >= 2 and lens is None:
      cut = [t.view(B, S, -1) for t in args[:2]]
      rec2 = torch.zeros_like(rec)
      outs = []
      for lo, hi, done in ((0, half, 0), (half, S, half)):
        oo = torch.empty(B * (hi - lo), hk * r * dv, dtype=dtype, device="cuda")
        scan(*[t[:, lo:hi].reshape(B * (hi - lo), -1).contiguous() for t in cut], *args[2:], hk, hk * r, dk, dv, hi - lo, rec2, slots,
                     torch.full_like(lengths, done), None, oo)
        outs.append(oo.view(B, hi - lo, -1))
      both = torch.cat(outs, 1).view(B * S, -1)
      assert (both.double() - o.double()).pow(2).mean().sqrt() < tol * o.double().pow(2).mean().sqrt()
      assert (rec2[1:] - rec[1:]).pow(2).mean().sqrt() < tol * rec[1:].pow(2).mean().sqrt()
  assert _status() == 0


@pytest.mark.parametrize("decay", ["slow", "fast", "mixed"])
@pytest.mark.parametrize("B, S, H, dk, dv, lens", [(2, 150, 2, 64, 128, None), (1, 260, 3, 128, 64, None), (3, 70, 2, 96, 48, [70, 1, 65]), (1, 90, 2, 20, 12, None),
                                                   (2, 130, 1, 128, 128, [17, 130])])
def test_gla_scan(B, S, H, dk, dv, lens, decay):
  from maxtext_b200.ops import backend
  E = backend.ext(required=True)
  g = torch.Generator().manual_seed(3)
  ld = 2 * H * (dk + dv)
  x = torch.randn(B * S, ld, generator=g)
  z = torch.rand(B * S, H * dk, generator=g)
  la = {"slow": -0.01 * z, "fast": -30.0 * z, "mixed": -10.0 ** (4 * z - 3)}[decay].cuda()
  for dtype, scan, tol in ((torch.float32, E.gla_scan, 2e-5), (torch.bfloat16, E.gla_scan, 1e-2), (torch.bfloat16, E.gla_chunks, 1e-2)):
    if scan is E.gla_chunks and not E.chunk_supported(dk, dv):
      continue
    xd = x.to(dtype).cuda()
    rec = torch.full((B, H, dk, dv), 3.0, device="cuda")
    slots, lengths = torch.arange(B, device="cuda"), torch.zeros(B, dtype=torch.long, device="cuda")
    o = torch.empty(B * S, H * dv, dtype=dtype, device="cuda")
    scan(xd, la, H, dk, dv, S, rec, slots, lengths, torch.tensor(lens, device="cuda") if lens else None, o)
    for b in range(B):
      n = lens[b] if lens else S
      xb = xd.double().cpu().view(B, S, -1)[b, :n]
      q, k, v = xb[:, :H * dk].view(n, H, dk) * dk ** -0.5, xb[:, H * dk:2 * H * dk].view(n, H, dk), xb[:, 2 * H * dk:2 * H * dk + H * dv].view(n, H, dv)
      want = O.gated_linear_recurrence(q, k, v, torch.exp(la.double().cpu().view(B, S, H, dk)[b, :n]))
      got = o.view(B, S, H, dv)[b, :n].double().cpu()
      assert torch.isfinite(got).all()
      assert (got - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), (dtype, b)
      if n == S:                                     # the state that is left: feed one more token with decay 1 and look at the read-out
        one = xd.view(B, S, -1)[:, :1].contiguous().view(B, -1)
        oo = torch.empty(B, H * dv, dtype=dtype, device="cuda")
        rec1 = rec.clone()
        E.gla_scan(one, torch.zeros(B, H * dk, device="cuda"), H, dk, dv, 1, rec1, slots, lengths + S, None, oo)
        more = O.gated_linear_recurrence(torch.cat([q, q[:1]]), torch.cat([k, k[:1]]), torch.cat([v, v[:1]]),
                                         torch.cat([torch.exp(la.double().cpu().view(B, S, H, dk)[b]), torch.ones(1, H, dk, dtype=torch.float64)]))[-1]
        assert (oo.view(B, H, dv)[b].double().cpu() - more).pow(2).mean().sqrt() < 2 * tol * more.pow(2).mean().sqrt()
  assert _status() == 0


@pytest.mark.parametrize("N, C, rank, at", [(70, 96, 32, 64), (5, 30, 8, 13), (129, 128, 24, 16), (64, 66, 40, 8)])
def test_gla_decay(N, C, rank, at):
  from maxtext_b200.ops import backend
  E = backend.ext(required=True)
  g = torch.Generator().manual_seed(5)
  for dtype in (torch.float32, torch.bfloat16):
    x, w, b = ((torch.randn(*s, generator=g) * 3).to(dtype).cuda() for s in ((N, at + rank + 8), (C, rank), (C,)))
    out = torch.empty(N, C, device="cuda")
    E.gla_decay(x, at, w, b, 8.0, out)
    want = torch.nn.functional.logsigmoid(x[:, at:at + rank].double() @ w.double().T + b.double()) / 8.0
    assert torch.allclose(out.double(), want, rtol=2e-5, atol=1e-6), dtype


@pytest.mark.parametrize("H, R, dr, window, lens", [(5, 128, 32, 0, [1, 300, 64]), (16, 512, 64, 100, [101, 100, 700]), (33, 64, 16, 65, [65, 66, 1]),
                                                    (3, 40, 6, 9, [9, 10, 30]), (4, 448, 48, 0, [65, 128, 129])])
def test_latent_decode_attention(H, R, dr, window, lens):
  from maxtext_b200.ops import backend
  E = backend.ext(required=True)
  g = torch.Generator().manual_seed(2)
  B, L, scale = len(lens), 768, 0.2
  for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-3)):
    lat, kr = (torch.randn(B + 2, L, n, generator=g).to(dtype).cuda() for n in (R, dr))
    qa = (torch.randn(B, H, R + dr, generator=g) * 1.5).to(dtype).cuda()
    slots, lengths = torch.tensor([4, 0, 2], device="cuda"), torch.tensor(lens, device="cuda") - 1
    for splits in (1, 3, 7):
      part, ml = torch.empty(B, H, splits, R, device="cuda"), torch.empty(B, H, splits, 2, device="cuda")
      E.mla_decode_attn(qa, lat, kr, slots, lengths, scale, window, splits, part, ml)
      m = ml[..., 0].max(-1, keepdim=True).values
      w = torch.where(ml[..., 1] > 0, torch.exp(ml[..., 0] - m), torch.zeros_like(m))
      got = (torch.nan_to_num(part) * w[..., None]).sum(2) / (w * ml[..., 1]).sum(2)[..., None]
      for b in range(B):
        lo = max(0, lens[b] - window) if window else 0
        c, k = lat[slots[b], lo:lens[b]].double(), kr[slots[b], lo:lens[b]].double()
        s = qa[b].double() @ torch.cat([c, k], -1).T * scale
        want = torch.softmax(s, -1) @ c
        assert (got[b].double() - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), (dtype, splits, b)
  assert _status() == 0


@pytest.mark.parametrize("B, H, nope, dr, vd, R", [(3, 2, 20, 6, 14, 36), (1, 5, 32, 16, 48, 64), (8, 3, 48, 16, 40, 128), (70, 2, 128, 64, 128, 512), (33, 4, 16, 8, 80, 320)])
def test_latent_decode_products(B, H, nope, dr, vd, R):
  from maxtext_b200.ops import backend
  E = backend.ext(required=True)
  g = torch.Generator().manual_seed(4)
  for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 6e-3)):
    q, w = (torch.randn(*s, generator=g).to(dtype).cuda() for s in ((B, H, nope + dr), (H * (nope + vd), R)))
    pos = torch.randint(0, 5000, (B,), generator=g).cuda()
    inv = (10000.0 ** (-torch.arange(dr // 2, dtype=torch.float64) * 2 / dr)).float().cuda()
    wd = w.double().view(H, nope + vd, R)
    for inter in (True, False):
      qa = torch.empty(B, H, R + dr, dtype=dtype, device="cuda")
      E.mla_absorb(q, w, pos, inv, inter, nope, vd, qa)
      qd = q.double()
      ang = pos.double()[:, None, None] * inv.double()
      u, v = (qd[..., nope::2], qd[..., nope + 1::2]) if inter else (qd[..., nope:nope + dr // 2], qd[..., nope + dr // 2:])
      a, b = u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()
      rot = torch.stack([a, b], -1).flatten(-2) if inter else torch.cat([a, b], -1)
      want = torch.cat([torch.einsum("bhd,hdr->bhr", qd[..., :nope], wd[:, :nope]), rot], -1)
      for part in (slice(0, R), slice(R, R + dr)):
        assert (qa.double() - want)[..., part].pow(2).mean().sqrt() < max(tol, 2e-4 if part.start else 0) * want[..., part].pow(2).mean().sqrt(), (dtype, inter, part)
    for splits in (1, 3):
      part, ml = torch.randn(B, H, splits, R, generator=g).cuda(), torch.rand(B, H, splits, 2, generator=g).cuda() + 0.1
      if splits > 1:
        ml[:, :, 1] = torch.tensor([float("-inf"), 0.0])                   # a split without keys
        part[:, :, 1] = float("nan")
      out = torch.empty(B, H, vd, dtype=dtype, device="cuda")
      E.mla_value_up(part, ml, w, nope, out)
      m = ml[..., 0].double().max(-1, keepdim=True).values
      f = torch.where(ml[..., 1] > 0, torch.exp(ml[..., 0].double() - m), torch.zeros_like(m))
      ctx = (torch.nan_to_num(part.double()) * f[..., None]).sum(2) / (f * ml[..., 1].double()).sum(2)[..., None]
      want = torch.einsum("bhr,her->bhe", ctx, wd[:, nope:])
      assert (out.double() - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), (dtype, splits)
  assert _status() == 0


def test_fp32_stream_kernels():
  from maxtext_b200.ops import functional as F
  g = torch.Generator().manual_seed(0)
  for rows, D in ((3, 60), (5, 2048), (2, 4100), (4, 33)):
    for dtype in (torch.float32, torch.bfloat16):
      x = torch.randn(rows, D, generator=g).cuda()
      b = (torch.randn(rows, D, generator=g) * 3).to(dtype).cuda()
      w1, w2 = ((torch.randn(D, generator=g) * 0.3).to(dtype).cuda() for _ in range(2))

      def norm(w, eps):
        return type("N", (), {"eps": eps, "offset": 1.0, "scale": type("P", (), {"data": w})()})()
      with torch.no_grad():
        want_x = x.double() + 0.4 * O.zero_centred_norm(b.double(), w1.double(), 0.01)
        y0 = F.stream_norm(x, norm(w2, 0.2), dtype)
        got_x, got_y = F.residual_norm(x.clone(), b, norm(w1, 0.01), 0.4, norm(w2, 0.2))
      tol = 1e-5 if dtype == torch.float32 else 2e-2
      assert torch.allclose(got_x.double(), want_x, atol=1e-5)
      assert torch.allclose(got_y.double(), O.zero_centred_norm(want_x, w2.double(), 0.2), atol=tol, rtol=tol)
      assert torch.allclose(y0.double(), O.zero_centred_norm(x.double(), w2.double(), 0.2), atol=tol, rtol=tol)
      h = (torch.randn(rows * D + 3, generator=g) * 2).to(dtype).cuda()
      with torch.no_grad():
        assert torch.allclose(F.act(h, "gelu_exact").double(), O.gelu_erf(h.double()), atol=tol, rtol=tol)


def test_every_kernel_path_is_taken_in_bf16(tmp_path):
  """No attention call of a bf16 model falls back to PyTorch operations, in prompts, portions or decoding."""
  from maxtext_b200.ops import functional as F
  sp = M.SPECS["mixed_even"]
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)), "bfloat16", "cuda")
  before = F.attention_fallbacks()
  M.run_pieces(eng, M.prompt(60, sp), [30, 20, 1])
  assert F.attention_fallbacks() == before


def test_training_step_in_bf16(tmp_path):
  """The layers train through their differentiable forms, with the fp32 stream crossing units."""
  from helpers import BASE_YML
  from maxtext_b200.config import pyconfig
  from maxtext_b200.input_pipeline.synthetic import SyntheticDataIterator
  from maxtext_b200.train.engine import TrainEngine
  sp = M.spec([M.delta(4, 2, 32, 32, 2), M.gla(2, 32, 32, 2.0, 8), M.latent(4, 32, 32, 64, 64, 64, 40, 0.15)], 256, vocab=512)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype="bfloat16", max_target_length=64, per_device_batch_size=2,
                            dataset_type="synthetic", hardware="gpu", enable_checkpointing=False, log_config=False, steps=5, learning_rate=5e-3,
                            warmup_steps_fraction=0.0)
  eng = TrainEngine(cfg, None, torch.device("cuda", 0))
  batch = next(SyntheticDataIterator(cfg))
  losses = [float(eng.train_step(batch)["learning/loss"]) for _ in range(5)]
  assert losses[-1] < losses[0] and all(x == x for x in losses)
