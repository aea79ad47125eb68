"""Gukirax on the CUDA kernels: the shared suite in fp32 and bf16, the decode graph, training, and the kernels on shapes of their own."""
import pytest
import torch

import gukirax_models as M
import gukirax_oracle as O
from gukirax_suite import Suite

pytestmark = pytest.mark.gpu


class TestGukiraxGpu(Suite):
  device = "cuda"
  dtypes = ("float32", "bfloat16")


def _ext():
  from maxtext_b200.ops import backend
  return backend.ext(required=True)


def _rel(got, want):
  got, want = got.double().cpu(), want.double().cpu()
  assert torch.isfinite(got).all()
  return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-30))


def _rows(got, want):
  """Worst row (last dimension), relative to its own size or the typical row's, whichever is larger."""
  got, want = got.double().cpu(), want.double().cpu()
  assert torch.isfinite(got).all()
  size = want.pow(2).mean(-1).sqrt()
  return float(((got - want).pow(2).mean(-1).sqrt() / size.clamp_min(float(want.pow(2).mean().sqrt()) + 1e-30)).max())


TOL = {torch.float32: 1e-5, torch.bfloat16: 1.2e-2}
DTYPES = (torch.float32, torch.bfloat16)


def test_graph_decode_equals_eager(tmp_path):
  for dtype in ("float32", "bfloat16"):
    for name in ("mixed", "mixed_even"):
      sp = M.SPECS[name]
      path = M.write_folder(tmp_path / (dtype + name), sp, M.weights(sp))
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
      assert got[0] == got[1], (dtype, name)
  assert _ext().kernel_status(True) == 0


def test_the_flash_and_decode_kernels_run(tmp_path, monkeypatch):
  """Prompts and single tokens of a bf16 model run the tensor-core kernels, not the plain one."""
  from maxtext_b200.ops import backend
  sp = M.SPECS["mixed_even"]
  eng = M.engine(M.write_folder(tmp_path / "m", sp, M.weights(sp)), "bfloat16", "cuda")
  E, seen = _ext(), []

  class Spy:
    def __getattr__(self, name):
      seen.append(name)
      return getattr(E, name)
  monkeypatch.setattr(backend, "_EXT", Spy())
  M.run_pieces(eng, M.prompt(40, sp), [30, 5, 1])
  assert {"wide_flash", "wide_decode", "residual_gate", "act_rows", "expert_up"} <= set(seen) and "wide_attention" not in seen


# ------------------------------------------------------------------------------------------ gated residual step
@pytest.mark.parametrize("D, per, padded, extra, gate, centred", [
    (64, 1, False, False, True, True), (388, 2, True, True, True, True), (2048, 1, False, False, True, False), (516, 3, False, True, False, True),
    (4096, 2, True, True, True, True), (33, 1, False, False, True, True), (21, 2, False, True, True, False), (8192, 1, False, True, True, True), (1032, 2, True, False, True, True)])
def test_residual_gate(D, per, padded, extra, gate, centred):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  N, eps = 37, 0.05

  def norm(t, w):
    return O.layer_norm(t, w.double(), eps) if centred else O.rms(t, eps) * w.double()
  for dtype in DTYPES:
    x = torch.randn(N, D, generator=g) + 3.0
    rows = (torch.randn(N * per + 20, D, generator=g) + 1.0).to(dtype)
    dest = torch.randperm(N * per + 20, generator=g)[:N * per].int()
    if not padded:
      rows, dest = rows[:N * per], torch.arange(N * per).int()
    ex = torch.randn(N, D, generator=g).to(dtype) if extra else None
    wide = torch.randn(N, D + 24, generator=g).to(dtype)                       # the gate is part of a wider product
    bias, w1, w2 = (torch.randn(D, generator=g).to(dtype) for _ in range(3))
    b = rows.double()[dest.long()].view(N, per, D).sum(1) + (ex.double() if extra else 0.0)
    if gate:
      b = b * O.sigmoid(wide[:, 16:16 + D].double() + bias.double())
    want = x.double() + norm(b, w1)

    def cuda(t):
      return t.cuda() if t is not None else None
    for fresh in (False, True):
      gx, gy = x.cuda(), torch.empty(N, D, dtype=dtype, device="cuda")
      wg = wide.cuda()
      args = (rows.cuda(), dest.cuda() if padded else None, per, cuda(ex), wg[:, 16:16 + D] if gate else None, cuda(bias) if gate else None, w1.cuda())
      full = want - x.double() if fresh else want
      E.residual_gate(gx, *args, w2.cuda(), gy, eps, centred, fresh)
      assert _rel(gx, full) < 2e-6
      assert _rows(gy, norm(full, w2)) < TOL[dtype]
      only = torch.empty_like(gy)
      E.residual_gate(gx, None, None, 1, None, None, None, None, w2.cuda(), only, eps, centred, False)       # reads what is there
      assert torch.equal(only, gy)
      gx, buf = x.cuda(), torch.full((N, 2 * D), 7.0, dtype=dtype, device="cuda")
      E.residual_gate(gx, *args, None, buf[:, :D], eps, centred, fresh)        # the stream as it is, in the first half of wider rows
      assert torch.equal(buf[:, :D], gx.to(dtype)) and float((buf[:, D:] - 7.0).abs().max()) == 0


@pytest.mark.parametrize("F, off", [(64, 0), (40, 8), (33, 5), (1, 3)])
def test_activations_of_wider_rows(F, off):
  E = _ext()
  g = torch.Generator().manual_seed(F)
  for dtype in DTYPES:
    z = (torch.randn(50, F + off + 8, generator=g) * 3).to(dtype)
    z[0, off] = 0.0
    par = torch.tensor([0.4, -0.9]).to(dtype)
    zc = z.cuda()[:, off:off + F]
    out = torch.empty(50, F, dtype=dtype, device="cuda")
    E.act_rows(zc, out, 6, par.cuda())
    assert _rows(out, O.xielu(z[:, off:off + F].double(), *par.double())) < TOL[dtype]
    E.act_rows(zc, out, 5, None)
    assert _rows(out, O.relu_squared(z[:, off:off + F].double())) < TOL[dtype]


# ------------------------------------------------------------------------------------------ attention
def _attend(q, k, v, n, s, scale, sink, window=0, chunk=0, seg=None):
  """The s last of n cached tokens of one sequence, wide queries q [s, H, G * D], k [n, G, D], v [n, G, Dv] -> [s, H, Dv] in fp64."""
  H, G = q.shape[1], k.shape[1]
  p = torch.arange(n - s, n)[:, None]
  j = torch.arange(n)[None]
  see = j <= p
  if window:
    see &= j > p - window
  if chunk:
    see &= j // chunk == p // chunk
  if seg is not None:
    see &= (seg[None] == seg[n - s:, None]) & (seg[None] != 0)
  out = []
  for h in range(H):
    x = (q[:, h] @ k.flatten(1).T * scale).masked_fill(~see, float("-inf"))
    top = x.max(-1, keepdim=True).values.clamp_min(-1e30)
    e = torch.exp(x - top)
    den = e.sum(-1, keepdim=True) + (torch.exp(sink[h] - top) if sink is not None else 0.0)
    out.append((e @ v[:, h // (H // G)]) / den.clamp_min(1e-300))
  return torch.stack(out, 1)


# (heads, key heads, width): one key head to many, widths that are no multiple of 64, contractions that stay in shared memory and that do not
SHAPES = [(4, 2, 64), (6, 3, 24), (16, 4, 128), (20, 5, 40), (5, 1, 8), (12, 12, 56), (16, 16, 64), (2, 1, 128), (34, 2, 72)]


@pytest.mark.parametrize("H, G, D", SHAPES)
def test_wide_flash(H, G, D):
  """A prompt from the first token, with the key that stands out at tile borders; rows of k and v inside wider matrices."""
  E = _ext()
  g = torch.Generator().manual_seed(H * D)
  bf, B, S = torch.bfloat16, 2, 300
  q = torch.randn(B, S, H, G * D, generator=g).to(bf)
  wide = torch.randn(B, S, 2 * G * D + 16, generator=g).to(bf)
  scale = 2.0 / (G * D) ** 0.5
  k, v = wide[..., 8:8 + G * D].unflatten(2, (G, D)), wide[..., 8 + G * D:8 + 2 * G * D].unflatten(2, (G, D))
  for i, j in ((129, 128), (200, 0), (299, 127), (255, 255), (140, 140)):
    wide[0, j, 8:8 + G * D] = (q[0, i, 0].double() * 3).to(bf)
  wc = wide.cuda()
  kc, vc = (wc[..., o:o + G * D].unflatten(2, (G, D)) for o in (8, 8 + G * D))
  for sink, window, chunk in ((torch.randn(H, generator=g).to(bf), 0, 0), (None, 0, 0), (torch.randn(H, generator=g).to(bf), 70, 0), (None, 0, 96)):
    out = torch.full((B, S, H * D), 9.0, dtype=bf, device="cuda")
    E.wide_flash(q.cuda(), kc, vc, out, None, None, None, None, sink.cuda() if sink is not None else None, scale, window, chunk, 0)
    for b in range(B):
      want = _attend(q[b].double(), k[b].double(), v[b].double(), S, S, scale, sink.double() if sink is not None else None, window, chunk)
      assert _rows(out.view(B, S, H, D)[b], want) < 2e-2, (window, chunk)
  assert E.kernel_status(True) == 0


@pytest.mark.parametrize("H, G, D", [(8, 4, 128), (12, 12, 56)])
def test_wide_flash_over_many_tiles(H, G, D):
  """Rings and score buffers that go around many times; the last keys of a row outgrow the first, so that its reference maximum moves."""
  E = _ext()
  g = torch.Generator().manual_seed(3)
  bf, S = torch.bfloat16, 1500
  q, k, v = torch.randn(1, S, H, G * D, generator=g).to(bf), torch.randn(1, S, G, D, generator=g), torch.randn(1, S, G, D, generator=g).to(bf)
  k = (k * torch.linspace(0.2, 4.0, S)[None, :, None, None]).to(bf)
  sink = torch.randn(H, generator=g).to(bf)
  scale = 2.0 / (G * D) ** 0.5
  out = torch.empty(1, S, H * D, dtype=bf, device="cuda")
  E.wide_flash(q.cuda(), k.cuda(), v.cuda(), out, None, None, None, None, sink.cuda(), scale, 0, 0, 0)
  assert _rows(out.view(S, H, D), _attend(q[0].double(), k[0].double(), v[0].double(), S, S, scale, sink.double())) < 2e-2
  assert E.kernel_status(True) == 0


@pytest.mark.parametrize("H, G, D", [(4, 2, 64), (20, 5, 40), (16, 16, 64)])
def test_wide_flash_segments_and_positions(H, G, D):
  """Several prompts in one row; and portions that follow cached tokens of unequal number."""
  E = _ext()
  g = torch.Generator().manual_seed(7)
  bf, S = torch.bfloat16, 290
  scale = 2.0 / (G * D) ** 0.5
  sink = torch.randn(H, generator=g).to(bf)
  seg = torch.cat([torch.full((n,), i + 1) for i, n in enumerate((1, 130, 60, 90))] + [torch.zeros(9)]).int()
  q, k, v = torch.randn(1, S, H, G * D, generator=g).to(bf), torch.randn(1, S, G, D, generator=g).to(bf), torch.randn(1, S, G, D, generator=g).to(bf)
  out = torch.empty(1, S, H * D, dtype=bf, device="cuda")
  E.wide_flash(q.cuda(), k.cuda(), v.cuda(), out, seg[None].cuda(), seg[None].cuda(), None, None, sink.cuda(), scale, 0, 0, 0)
  want = _attend(q[0].double(), k[0].double(), v[0].double(), S, S, scale, sink.double(), seg=seg)
  assert _rows(out.view(S, H, D)[:281], want[:281]) < 2e-2
  begin, n = [0, 250, 37], 130
  K = max(begin) + n
  q = torch.randn(3, n, H, G * D, generator=g).to(bf)
  k, v = torch.randn(3, K, G, D, generator=g).to(bf), torch.randn(3, K, G, D, generator=g).to(bf)
  pos = torch.tensor(begin)[:, None] + torch.arange(n)[None]
  kp = torch.arange(K)[None].expand(3, K).clone()
  for b, s in enumerate(begin):
    kp[b, s + n:] = 1 << 30
  out = torch.empty(3, n, H * D, dtype=bf, device="cuda")
  E.wide_flash(q.cuda(), k.cuda(), v.cuda(), out, None, None, pos.int().cuda(), kp.int().cuda(), sink.cuda(), scale, 0, 0, 0)
  for b, s in enumerate(begin):
    want = _attend(q[b].double(), k[b, :s + n].double(), v[b, :s + n].double(), s + n, n, scale, sink.double())
    assert _rows(out.view(3, n, H, D)[b], want) < 2e-2, b
  assert E.kernel_status(True) == 0


@pytest.mark.parametrize("H, G, D, window", [(4, 2, 64, 0), (6, 3, 24, 0), (16, 4, 128, 33), (20, 5, 40, 0), (5, 1, 8, 1), (12, 12, 56, 64), (32, 4, 128, 0), (34, 2, 72, 0),
                                             (2, 1, 200, 0), (3, 3, 256, 17)])
def test_wide_decode(H, G, D, window):
  E = _ext()
  g = torch.Generator().manual_seed(H + D)
  max_len, lens = 220, [1, 2, 16, 17, 33, 34, 64, 65, 100, 101, 210, 220]
  B, slots_n, bf = len(lens), len(lens) + 2, torch.bfloat16
  q = torch.randn(B, H, G * D, generator=g).to(bf)
  k, v = torch.randn(slots_n, max_len, G, D, generator=g).to(bf), torch.randn(slots_n, max_len, G, D, generator=g).to(bf)
  sink = torch.randn(H, generator=g).to(bf)
  slots = torch.randperm(slots_n, generator=g)[:B]
  scale = 3.0 / (G * D) ** 0.5
  for i, n in enumerate(lens):                       # what is beyond a sequence's end must not be read as a value
    k[slots[i], n:], v[slots[i], n:] = float("nan"), float("nan")
    if window and n > window:                        # a key just outside the window would win if it were seen; one just inside wins
      k[slots[i], n - window - 1] = (q[i, 0].double() * 9).to(bf).view(G, D)
      k[slots[i], n - window] = (q[i, 0].double() * 4 / (G * D) ** 0.5).to(bf).view(G, D)
  for sk in (sink, None):
    want = torch.stack([_attend(q[i:i + 1].double(), k[s, :n].double(), v[s, :n].double(), n, 1, scale, sk.double() if sk is not None else None, window)[0]
                        for i, (n, s) in enumerate(zip(lens, slots.tolist()))])
    length = torch.tensor(lens, device="cuda") - 1
    for splits in (1, 3, E.cached_decode_splits(B, H, 1, max_len), 16):
      part, ml = torch.empty(B, H, splits, D, device="cuda"), torch.empty(B, H, splits, 2, device="cuda")
      out = torch.empty(B, H * D, dtype=bf, device="cuda")
      E.wide_decode(q.cuda(), k.cuda(), v.cuda(), slots.cuda(), length, scale, window, 0, sk.cuda() if sk is not None else None, splits, part, ml, out)
      assert _rows(out.view(B, H, D), want) < 1.5e-2, splits


@pytest.mark.parametrize("H, G, D, window", [(4, 2, 20, 0), (3, 1, 33, 7), (6, 6, 64, 32), (2, 1, 300, 0), (10, 5, 128, 0)])
def test_wide_attention(H, G, D, window):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  max_len, S = 90, 37
  begin = [0, 5, 53, 40]
  B = len(begin)
  for dtype in DTYPES:
    q = torch.randn(B * S, H, G * D, generator=g).to(dtype)
    k, v = torch.randn(B + 1, max_len, G, D, generator=g).to(dtype), torch.randn(B + 1, max_len, G, D, generator=g).to(dtype)
    for b, n in enumerate(begin):
      k[b + 1, n + S:], v[b + 1, n + S:] = float("nan"), float("nan")
    sink = torch.randn(H, generator=g).to(dtype)
    out = torch.empty(B * S, H * D, dtype=dtype, device="cuda")
    scale = 2.0 / (G * D) ** 0.5
    E.wide_attention(q.cuda(), k.cuda(), v.cuda(), torch.arange(B, device="cuda") + 1, torch.tensor(begin, device="cuda"), S, scale, window, 0, sink.cuda(), out)
    for b, n in enumerate(begin):
      want = _attend(q.view(B, S, H, G * D)[b].double(), k[b + 1, :n + S].double(), v[b + 1, :n + S].double(), n + S, S, scale, sink.double(), window)
      assert _rows(out.view(B, S, H, D)[b], want) < TOL[dtype], (dtype, b)


@pytest.mark.parametrize("H, G, D, rot", [(4, 2, 64, 32), (6, 3, 20, 8), (16, 4, 128, 64), (9, 3, 11, 6), (2, 1, 200, 0), (12, 12, 56, 24), (32, 4, 128, 128), (3, 3, 300, 24)])
def test_prep_folds_the_mixing_into_the_queries(H, G, D, rot):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  B, S, max_len, eps = 3, 9, 30, 1e-3
  begin, new = [0, 4, 25], [9, 3, 5]
  pos = torch.tensor(begin)[:, None] + torch.arange(S)[None]
  base = 300.0
  inv = (1.0 / base ** (2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float()
  for dtype in DTYPES:
    p = torch.randn(B * S, (H + G) * D + 8, generator=g).to(dtype)
    talk = torch.randn(H, H, generator=g).to(dtype)
    pc = p.cuda()
    q, k = pc[:, :H * D], pc[:, H * D:(H + G) * D]
    qp, kp = torch.full((B * S, H, G * D), 9.0, dtype=dtype, device="cuda"), torch.full((B * S, G, D), 9.0, dtype=dtype, device="cuda")
    kc, vc = (torch.full((B + 1, max_len, G, D), 5.0, dtype=dtype, device="cuda") for _ in range(2))
    E.qkv_prep(q, k, k, D, D, pos.reshape(-1).cuda(), inv.cuda() if rot else None, rot, eps, qp, kp, None, kc, vc, torch.arange(B, device="cuda") + 1,
               torch.tensor(begin, device="cuda"), torch.tensor(new, device="cuda"), talk=talk.cuda())

    def turned(x, heads):
      x = x.double().cpu().view(B, S, heads, D)
      out = torch.zeros_like(x)
      for b in range(B):                             # positions begin at begin[b]: rotate a longer sequence and keep its end
        longer = torch.cat([torch.zeros(begin[b], heads, D, dtype=torch.float64), x[b]])
        out[b] = O.rotate_halves(longer, base, rot)[begin[b]:]
      return O.rms(out, eps)
    nq, nk = turned(q, H), turned(k, G)
    want = torch.einsum("hcj,bscjd->bshcd", talk.double().view(H, G, H // G), nq.view(B, S, G, H // G, D))
    assert _rows(qp.view(B, S, H, G * D), want.flatten(3)) < TOL[dtype]
    assert _rows(kp.view(B, S, G, D), nk) < TOL[dtype]
    raw = k.cpu().view(B, S, G, D)
    for b in range(B):
      lo, hi = begin[b], begin[b] + new[b]
      assert _rows(kc[b + 1, lo:hi], nk[b, :new[b]]) < TOL[dtype] and torch.equal(vc[b + 1, lo:hi].cpu(), raw[b, :new[b]])
      for c in (kc, vc):                             # nothing else was written
        assert float((c[b + 1, :lo] - 5).abs().sum() + (c[b + 1, hi:] - 5).abs().sum()) == 0
    assert float((kc[0] - 5).abs().max()) == 0


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T, E_n, k, D, Fd, shared", [(1, 8, 2, 64, 48, True), (5, 4, 4, 40, 24, False), (130, 3, 1, 72, 40, True), (40, 16, 3, 33, 21, True), (200, 2, 2, 128, 128, False),
                                                      (513, 4, 2, 256, 128, True), (128, 16, 2, 1024, 2048, False), (3, 1, 1, 24, 16, True), (2, 128, 8, 256, 64, False)])
def test_experts(T, E_n, k, D, Fd, shared):
  from maxtext_b200.ops import moe_ops
  g = torch.Generator().manual_seed(T)
  for dtype in DTYPES:
    P = lambda *s: type("P", (), {"data": (torch.randn(*s, generator=g) * s[-1] ** -0.5 * 1.5).to(dtype).cuda()})()  # noqa: E731
    layer = type("L", (), dict(style="prob_weighted", k=k, E=E_n, limit=0.0, gate=P(E_n, D), wi_0=P(E_n, Fd, D), wi_1=None, wo=P(E_n, D, Fd)))()
    x = torch.randn(T, D, generator=g).to(dtype)
    more = torch.randn(T, D, generator=g).to(dtype) if shared else None
    with torch.no_grad():
      rows = moe_ops.serve_scored(x.cuda(), layer)
      rows.extra = more.cuda() if shared else None
      got = rows.combine(torch.empty(T, D, device="cuda"))
    s = torch.softmax(x.double() @ layer.gate.data.double().cpu().t(), -1)
    top = torch.topk(s, min(k + 1, E_n), dim=-1).values
    clear = torch.ones(T, dtype=torch.bool) if k == E_n else (top[:, k - 1] - top[:, k]) > 1e-5
    assert int(clear.sum()) > 0.8 * T
    w0, wo = (p.data.double().cpu() for p in (layer.wi_0, layer.wo))
    want = more.double() if shared else torch.zeros(T, D, dtype=torch.float64)
    for t in range(T):
      for e in torch.topk(s[t], k).indices.tolist():
        want[t] += s[t, e] * O.expert(x[t].double(), w0[e], wo[e])
    assert _rows(got[clear.cuda()], want[clear]) < 2 * TOL[dtype], dtype


# ------------------------------------------------------------------------------------------ training
def test_training_on_a_gpu_follows_the_cpu(tmp_path):
  """The layers train through their differentiable forms; a layer's input survives the forward pass although the stream's kernels work in place."""
  from test_gukirax_cpu import train_losses, train_spec
  path = M.write_folder(tmp_path / "m", train_spec(), M.weights(train_spec()))
  cpu, _ = train_losses(path, "cpu")
  gpu, _ = train_losses(path, "cuda")
  assert max(abs(a - b) / a for a, b in zip(cpu, gpu)) < 1e-3, (cpu, gpu)
  bf, _ = train_losses(path, "cuda", 6, dtype="bfloat16")
  assert bf[-1] < bf[0] and all(x == x for x in bf)
