"""Tipidra on the CUDA kernels: the shared suite in fp32 and bf16, the decode graph, and the kernels on shapes of their own."""
import pytest
import torch

import tipidra_models as M
import tipidra_oracle as O
from tipidra_suite import Suite

pytestmark = pytest.mark.gpu


class TestTipidraGpu(Suite):
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
  """The captured decode step must leave recurrent states as if its warm-up had not happened."""
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


# ------------------------------------------------------------------------------------------ residual streams
@pytest.mark.parametrize("k, D, per, padded", [(1, 64, 1, False), (2, 388, 2, True), (3, 2048, 1, False), (4, 516, 3, False), (5, 96, 2, True), (2, 33, 1, False),
                                               (7, 21, 2, False)])
def test_stream_mix(k, D, per, padded):
  E = _ext()
  g = torch.Generator().manual_seed(k)
  N = 37
  for dtype in DTYPES:
    x = torch.randn(N, k, D, generator=g)
    rows = torch.randn(N * per + 20, D, generator=g).to(dtype)
    dest = torch.randperm(N * per + 20, generator=g)[:N * per].int()
    if not padded:
      rows, dest = rows[:N * per], torch.arange(N * per).int()
    mix, write, read = torch.randn(k, k, generator=g).to(dtype), torch.randn(k, generator=g).to(dtype), torch.randn(k, generator=g).to(dtype)
    w, b = torch.randn(D, generator=g).to(dtype), torch.randn(D, generator=g).to(dtype)
    y = rows.double()[dest.long()].view(N, per, D).sum(1)
    want = torch.einsum("st,nsd->ntd", mix.double(), x.double()) + write.double()[None, :, None] * y[:, None]
    for rd in (read, None):
      u = want.sum(1) if rd is None else torch.einsum("s,nsd->nd", rd.double(), want)
      gx, gy = x.cuda(), torch.empty(N, D, dtype=dtype, device="cuda")
      E.stream_mix(gx, rows.cuda(), dest.cuda() if padded else None, per, mix.cuda(), write.cuda(), rd.cuda() if rd is not None else None, w.cuda(), b.cuda(),
                   gy, 0.05)
      assert _rel(gx, want) < 1e-6
      assert _rows(gy, O.layer_norm(u, w.double(), b.double(), 0.05)) < TOL[dtype]
      only = torch.empty_like(gy)
      E.stream_mix(gx, None, None, 1, None, None, rd.cuda() if rd is not None else None, w.cuda(), b.cuda(), only, 0.05)      # reads what is there
      assert torch.equal(only, gy) and _rel(gx, want) < 1e-6


# ------------------------------------------------------------------------------------------ selective scan
def _scan_case(B, S, C, N, taps, rank, dtype, seed, slow=False):
  g = torch.Generator().manual_seed(seed)
  p = torch.randn(B * S, 2 * C, generator=g).to(dtype)
  w, bias = (torch.randn(taps, C, generator=g) * 0.6).to(dtype), torch.randn(C, generator=g).to(dtype)
  off = -(-rank // 8) * 8
  q = torch.randn(B * S, -(-(off + 2 * N) // 8) * 8, generator=g).to(dtype)
  dt = torch.randn(B * S, C, generator=g)
  dtb = (torch.randn(C, generator=g) - (6.0 if slow else 1.0)).to(dtype)
  A = torch.log(torch.rand(C, N, generator=g) * 4 + 0.01).to(dtype)
  D = torch.randn(C, generator=g).to(dtype)
  return p, w, bias, off, q, dt, dtb, A, D


def _scan_want(case, x, B, S, C, N, b, n):
  p, w, bias, off, q, dt, dtb, A, D = (t.double() if isinstance(t, torch.Tensor) else t for t in case)
  z = p.view(B, S, -1)[b, :n, C:]
  qb = q.view(B, S, -1)[b, :n]
  y = O.selective_scan(x, O.softplus(dt.view(B, S, C)[b, :n] + dtb), -torch.exp(A), qb[:, off:off + N], qb[:, off + N:off + 2 * N], D)
  return y * O.silu(z)


@pytest.mark.parametrize("B, S, C, N, taps, rank, lens, slow", [
    (2, 150, 64, 16, 4, 8, None, False), (1, 300, 160, 16, 3, 12, None, True), (3, 70, 40, 12, 2, 5, [70, 1, 65], False), (2, 90, 24, 1, 1, 1, None, False),
    (2, 130, 33, 6, 3, 2, [64, 130], False), (1, 67, 96, 32, 4, 16, None, False), (1, 80, 20, 64, 5, 4, None, False), (2, 40, 12, 100, 2, 3, [40, 33], False),
    (1, 45, 16, 250, 17, 2, None, True), (2, 64, 136, 8, 4, 3, None, False)])
def test_selective_scan(B, S, C, N, taps, rank, lens, slow):
  E = _ext()
  for dtype in DTYPES:
    case = _scan_case(B, S, C, N, taps, rank, dtype, 7, slow)
    p, w, bias, off, q, dt, dtb, A, D = (t.cuda() if isinstance(t, torch.Tensor) else t for t in case)
    slots = torch.arange(B, device="cuda") + 1
    length = torch.zeros(B, dtype=torch.long, device="cuda")
    new = torch.tensor(lens, device="cuda") if lens else None
    conv = torch.full((B + 1, taps - 1, C), 5.0, device="cuda")                # dirty slots
    rec = torch.full((B + 1, 1, C, N), 7.0, device="cuda")
    x = torch.empty(B * S, C, dtype=dtype, device="cuda")
    y = torch.empty(B * S, C, dtype=dtype, device="cuda")
    E.ssm_conv(p, w, bias, S, conv, slots, length, new, x)
    E.ssm_scan(x, p, q, dt, dtb, A, D, off, N, S, rec, slots, length, new, y)
    assert torch.isfinite(y).all()                                             # padding too
    for b in range(B):
      n = lens[b] if lens else S
      xin = case[0].double().view(B, S, -1)[b, :n, :C]
      want_x = O.silu(O.causal_conv(xin, case[1].double().t(), case[2].double()))
      assert _rows(x.view(B, S, C)[b, :n], want_x) < TOL[dtype]
      want = _scan_want(case, x.double().cpu().view(B, S, C)[b, :n], B, S, C, N, b, n)
      assert _rows(y.view(B, S, C)[b, :n], want) < 2 * TOL[dtype], (dtype, b)
      hist = torch.cat([torch.zeros(taps - 1, C).double(), xin])[n:n + taps - 1]
      assert torch.equal(conv[b + 1].double().cpu(), hist)
    assert float((rec[0] - 7.0).abs().max()) == 0.0 and (taps == 1 or float((conv[0] - 5.0).abs().max()) == 0.0)
    if lens:
      continue
    # the same in pieces, the last ones a token at a time
    cuts = [0, 1, S // 2, S // 2 + 2, S - 2, S - 1, S]
    conv2, rec2, outs = torch.full_like(conv, 9.0), torch.full_like(rec, 9.0), []
    for lo, hi in zip(cuts, cuts[1:]):
      def cut(t):
        return t.view(B, S, -1)[:, lo:hi].reshape(B * (hi - lo), -1).contiguous()
      m = hi - lo
      xx, yy = torch.empty(B * m, C, dtype=dtype, device="cuda"), torch.empty(B * m, C, dtype=dtype, device="cuda")
      at = torch.full_like(length, lo)
      E.ssm_conv(cut(p), w, bias, m, conv2, slots, at, None, xx)
      E.ssm_scan(xx, cut(p), cut(q), cut(dt), dtb, A, D, off, N, m, rec2, slots, at, None, yy)
      outs.append(yy.view(B, m, C))
    assert _rows(torch.cat(outs, 1).view(B * S, C), y) < TOL[dtype]
    assert _rel(rec2[1:], rec[1:]) < 1e-4 and torch.equal(conv2[1:], conv[1:])


# ------------------------------------------------------------------------------------------ attention over the cache
def _attend(q, k, v, n, s, scale, cap, window, sink):
  """The s last of n cached tokens of one sequence: q [s, H, D], k [n, G, D], v [n, G, Dv] -> [s, H, Dv] in fp64."""
  H, G = q.shape[1], k.shape[1]
  out = torch.zeros(s, H, v.shape[-1], dtype=torch.float64)
  for i in range(s):
    p = n - s + i
    lo = max(0, p - window + 1) if window else 0
    for h in range(H):
      g = h // (H // G)
      x = (k[lo:p + 1, g] @ q[i, h]) * scale
      x = O.soft_cap(x, cap) if cap else x
      e = torch.exp(x)
      out[i, h] = (e @ v[lo:p + 1, g]) / (e.sum() + (torch.exp(sink[h]) if sink is not None else 0.0))
  return out


@pytest.mark.parametrize("H, G, D, Dv, cap, window, sinks, gated", [
    (4, 2, 64, 64, 0.0, 0, False, False), (6, 2, 96, 40, 5.0, 0, True, True), (20, 1, 128, 128, 3.0, 33, True, False), (3, 3, 16, 24, 0.0, 1, False, True),
    (36, 2, 40, 72, 8.0, 64, True, True), (2, 1, 200, 136, 4.0, 0, True, True), (2, 2, 256, 256, 0.0, 100, False, False), (4, 1, 8, 8, 2.0, 16, True, True)])
def test_cached_decode(H, G, D, Dv, cap, window, sinks, gated):
  E = _ext()
  g = torch.Generator().manual_seed(H)
  max_len, lens = 220, [1, 2, 16, 17, 33, 34, 64, 65, 100, 101, 210, 220]
  B, slots_n = len(lens), len(lens) + 2
  bf = torch.bfloat16
  q, gate = torch.randn(B, H, D, generator=g).to(bf), torch.randn(B, H * Dv + 8, generator=g).to(bf)
  k, v = torch.randn(slots_n, max_len, G, D, generator=g).to(bf), torch.randn(slots_n, max_len, G, Dv, generator=g).to(bf)
  sink = torch.randn(H, generator=g).to(bf) if sinks else None
  slots = torch.randperm(slots_n, generator=g)[:B]
  scale = 3.0 / D ** 0.5
  for i, n in enumerate(lens):                       # what is beyond a sequence's end must not be read as a value
    k[slots[i], n:], v[slots[i], n:] = float("nan"), float("nan")
    if window and n > window:                        # a key just outside the window would win if it were seen; one just inside wins
      k[slots[i], n - window - 1] = (q[i, ::H // G].double() * 9).to(bf)
      k[slots[i], n - window] = (q[i, ::H // G].double() * 4 / D ** 0.5).to(bf)
  want = torch.stack([_attend(q[i:i + 1].double(), k[s, :n].double(), v[s, :n].double(), n, 1, scale, cap, window, sink.double() if sinks else None)[0]
                      for i, (n, s) in enumerate(zip(lens, slots.tolist()))])
  if gated:
    want = want * O.sigmoid(gate[:, :H * Dv].double()).view(B, H, Dv)
  length = torch.tensor(lens, device="cuda") - 1
  for splits in (1, 3, E.cached_decode_splits(B, H, G, max_len), 16):
    part, ml = torch.empty(B, H, splits, Dv, device="cuda"), torch.empty(B, H, splits, 2, device="cuda")
    out = torch.empty(B, H * Dv, dtype=bf, device="cuda")
    E.cached_decode(q.cuda(), k.cuda(), v.cuda(), slots.cuda(), length, scale, cap, window, sink.cuda() if sinks else None, gate.cuda() if gated else None, splits,
                    part, ml, out)
    assert _rows(out.view(B, H, Dv), want) < 1.5e-2, splits


@pytest.mark.parametrize("H, G, D, Dv, cap, window, sinks", [(4, 2, 20, 12, 5.0, 0, True), (3, 1, 33, 17, 0.0, 7, False), (2, 2, 64, 128, 2.0, 32, True),
                                                             (2, 1, 300, 290, 4.0, 0, True), (1, 1, 4, 512, 0.0, 50, True)])
def test_cached_attention(H, G, D, Dv, cap, window, sinks):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  max_len, S = 90, 37
  begin = [0, 5, 53, 40]
  B = len(begin)
  for dtype in DTYPES:
    q = torch.randn(B * S, H, D, generator=g).to(dtype)
    k, v = torch.randn(B + 1, max_len, G, D, generator=g).to(dtype), torch.randn(B + 1, max_len, G, Dv, generator=g).to(dtype)
    for b, n in enumerate(begin):
      k[b + 1, n + S:], v[b + 1, n + S:] = float("nan"), float("nan")
    sink = torch.randn(H, generator=g).to(dtype) if sinks else None
    out = torch.empty(B * S, H, Dv, dtype=dtype, device="cuda")
    E.cached_attention(q.cuda(), k.cuda(), v.cuda(), torch.arange(B, device="cuda") + 1, torch.tensor(begin, device="cuda"), S, 2.0 / D ** 0.5, cap, window,
                       sink.cuda() if sinks else None, out)
    for b, n in enumerate(begin):
      want = _attend(q.view(B, S, H, D)[b].double(), k[b + 1, :n + S].double(), v[b + 1, :n + S].double(), n + S, S, 2.0 / D ** 0.5, cap, window,
                     sink.double() if sinks else None)
      assert _rows(out.view(B, S, H, Dv)[b], want) < TOL[dtype], (dtype, b)


@pytest.mark.parametrize("D, Dv, rot, eps", [(20, 12, 8, 1e-5), (96, 40, 96, 0.3), (128, 128, 64, 1e-6), (11, 7, 6, 1e-5), (200, 136, 0, 1e-5), (300, 290, 24, 0.1),
                                             (64, 64, 32, -1.0)])
def test_qkv_prep(D, Dv, rot, eps):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  B, S, H, G, max_len = 3, 9, 4, 2, 30
  begin, new = [0, 4, 25], [9, 3, 5]
  pos = torch.tensor(begin)[:, None] + torch.arange(S)[None]
  base = 300.0
  inv = (1.0 / base ** (2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float()
  dq, dvp = (256 if D <= 256 else 512), -(-Dv // 64) * 64
  for dtype in DTYPES:
    p = torch.randn(B * S, H * D + G * D + G * Dv + 8, generator=g).to(dtype)
    q, k, v = p[:, :H * D], p[:, H * D:(H + G) * D], p[:, (H + G) * D:(H + G) * D + G * Dv]
    pc = p.cuda()
    qp, kp = torch.full((B * S, H, dq), 9.0, dtype=dtype, device="cuda"), torch.full((B * S, G, dq), 9.0, dtype=dtype, device="cuda")
    vp = torch.full((B * S, G, dvp), 9.0, dtype=dtype, device="cuda")
    kc, vc = torch.full((B + 1, max_len, G, D), 5.0, dtype=dtype, device="cuda"), torch.full((B + 1, max_len, G, Dv), 5.0, dtype=dtype, device="cuda")
    E.qkv_prep(pc[:, :H * D], pc[:, H * D:(H + G) * D], pc[:, (H + G) * D:(H + G) * D + G * Dv], D, Dv, pos.reshape(-1).cuda(), inv.cuda() if rot else None, rot, eps,
               qp, kp, vp, kc, vc, torch.arange(B, device="cuda") + 1, torch.tensor(begin, device="cuda"), torch.tensor(new, device="cuda"))

    def want(x, heads):
      x = x.double().view(B, S, heads, D)
      turned = torch.zeros_like(x)
      for b in range(B):                             # positions begin at begin[b]: rotate a longer sequence and keep its end
        longer = torch.cat([torch.zeros(begin[b], heads, D, dtype=torch.float64), x[b]])
        turned[b] = O.rotate_halves(longer, base, rot)[begin[b]:]
      return O.rms(turned, eps) if eps >= 0 else turned
    wq, wk, wv = want(q, H), want(k, G), v.double().view(B, S, G, Dv)
    assert _rows(qp.view(B, S, H, dq)[..., :D], wq) < TOL[dtype] and float(qp[..., D:].abs().max() if dq > D else 0) == 0
    assert _rows(kp.view(B, S, G, dq)[..., :D], wk) < TOL[dtype] and float(kp[..., D:].abs().max() if dq > D else 0) == 0
    assert torch.equal(vp.view(B, S, G, dvp)[..., :Dv].double().cpu(), wv) and (dvp == Dv or float(vp[..., Dv:].abs().max()) == 0)
    for b in range(B):
      lo, hi = begin[b], begin[b] + new[b]
      assert _rows(kc[b + 1, lo:hi], wk[b, :new[b]]) < TOL[dtype] and torch.equal(vc[b + 1, lo:hi].double().cpu(), wv[b, :new[b]])
      for c in (kc, vc):                             # nothing else was written
        assert float((c[b + 1, :lo] - 5).abs().sum() + (c[b + 1, hi:] - 5).abs().sum()) == 0
    assert float((kc[0] - 5).abs().max()) == 0


@pytest.mark.parametrize("mode, reach", [("CAP_EXACT", 4.0), ("CAP_SMALL", 0.3)])
def test_flash_soft_cap_is_exact(mode, reach):
  """Scores up to `reach` caps, with one key that stands out per query: the tanh instruction would be off by a part in a thousand of the cap."""
  from maxtext_b200.ops import functional as F
  g = torch.Generator().manual_seed(2)
  B, S, H, D, cap = 1, 300, 2, 64, 50.0
  q, k, v = (torch.randn(B, S, H, D, generator=g).bfloat16() for _ in range(3))
  raw = torch.einsum("bqhd,bkhd->bhqk", q.double(), k.double())
  scale = float(reach * cap / raw.abs().max())
  sinks = torch.tensor([1.0, -2.0])
  mask = torch.tril(torch.ones(S, S, dtype=torch.bool))
  x = (O.soft_cap(raw * scale, cap)).masked_fill(~mask, -1e30)
  lse = torch.logsumexp(torch.cat([x, sinks.double().view(1, H, 1, 1).expand(B, H, S, 1)], -1), -1)
  want = torch.einsum("bhqk,bkhd->bqhd", torch.exp(x - lse[..., None]), v.double())
  with torch.no_grad():
    out, got_lse = F.attention_fwd(q.cuda(), k.cuda(), v.cuda(), None, None, scale, cap, 0, sinks=sinks.cuda(), cap_mode=getattr(F, mode))
  assert float((got_lse.double().cpu() - lse).abs().max()) < 2e-4
  assert _rows(out, want) < 2e-2


# ------------------------------------------------------------------------------------------ experts
def _layer(E_n, k, D, Fd, limit, dtype, g):
  P = lambda *s: type("P", (), {"data": (torch.randn(*s, generator=g) * s[-1] ** -0.5 * 1.5).to(dtype).cuda()})()  # noqa: E731
  return type("L", (), dict(style="scaled_input", k=k, E=E_n, limit=limit, gate=P(E_n, D), wi_0=P(E_n, Fd, D), wi_1=P(E_n, Fd, D), wo=P(E_n, D, Fd)))()


@pytest.mark.parametrize("T, E_n, k, D, Fd", [(1, 8, 2, 64, 48), (5, 4, 4, 40, 24), (130, 3, 1, 72, 40), (40, 16, 3, 33, 21), (200, 2, 2, 128, 128), (513, 4, 2, 256, 128),
                                              (64, 8, 2, 512, 1024), (128, 16, 2, 1024, 2048), (3, 1, 1, 24, 16), (2, 128, 8, 256, 64)])
def test_experts(T, E_n, k, D, Fd):
  from maxtext_b200.ops import moe_ops
  g = torch.Generator().manual_seed(T)
  limit = 0.8
  for dtype in DTYPES:
    layer = _layer(E_n, k, D, Fd, limit, dtype, g)
    x = torch.randn(T, D, generator=g).to(dtype)
    with torch.no_grad():
      rows = moe_ops.serve_scored(x.cuda(), layer)
      got = rows.combine(torch.empty(T, D, device="cuda"))
    s = torch.sigmoid(x.double() @ layer.gate.data.double().cpu().t())
    top = torch.topk(s, min(k + 1, E_n), dim=-1).values
    clear = torch.ones(T, dtype=torch.bool) if k == E_n else (top[:, k - 1] - top[:, k]) > 1e-5
    assert int(clear.sum()) > 0.8 * T
    w0, w1, wo = (p.data.double().cpu() for p in (layer.wi_0, layer.wi_1, layer.wo))
    want = torch.zeros(T, D, dtype=torch.float64)
    for t in range(T):
      for e in torch.topk(s[t], k).indices.tolist():
        want[t] += O.clamped_expert(s[t, e] * x[t].double(), w0[e], w1[e], wo[e], limit)
    assert _rows(got[clear.cuda()], want[clear]) < 2 * TOL[dtype], dtype


def test_every_row_of_an_expert_is_computed():
  """All tokens choose the same two experts, so that one expert owns many 32-row passes and others none."""
  from maxtext_b200.ops import moe_ops
  g = torch.Generator().manual_seed(4)
  for T, D, Fd in ((97, 48, 32), (150, 128, 128)):
    layer = _layer(6, 2, D, Fd, 1.0, torch.bfloat16, g)
    x = torch.randn(T, D, generator=g).bfloat16()
    x[:, 0] = 4.0
    layer.gate.data.zero_()
    layer.gate.data[3, 0], layer.gate.data[5, 0] = 0.5, 0.25
    with torch.no_grad():
      got = moe_ops.serve_scored(x.cuda(), layer).combine(torch.empty(T, D, device="cuda"))
    w0, w1, wo = (p.data.double().cpu() for p in (layer.wi_0, layer.wi_1, layer.wo))
    want = sum(O.clamped_expert(float(torch.sigmoid(torch.tensor(v, dtype=torch.float64))) * x.double(), w0[e], w1[e], wo[e], 1.0) for e, v in ((3, 2.0), (5, 1.0)))
    assert _rows(got, want) < 2.5e-2


# ------------------------------------------------------------------------------------------ the same kernels behind the other families' caches
@pytest.mark.parametrize("D, Dv, H, G, window, cap, sinks", [(64, 64, 4, 2, 0, 0.0, False), (128, 128, 8, 1, 9, 4.0, True), (32, 32, 4, 4, 0, 0.0, True),
                                                             (48, 80, 6, 2, 5, 3.0, False), (208, 144, 2, 1, 0, 2.0, True)])
def test_layer_cache_attends_on_the_kernels(D, Dv, H, G, window, cap, sinks):
  """Prompts, portions, single tokens and packed prompts through LayerKVCache.attend against the definition on fp32 copies."""
  from maxtext_b200.inference.kvcache import LayerKVCache
  from maxtext_b200.ops import cached_attention as CA, reference as ref
  g = torch.Generator().manual_seed(D)
  B, total, bf = 2, 40, torch.bfloat16
  q, k, v = (torch.randn(B, total, n, w, generator=g).to(bf).cuda() for n, w in ((H, D), (G, D), (G, Dv)))
  q = (q * (2.0 / D ** 0.5)).to(bf)
  sk = torch.randn(H, generator=g).to(bf).cuda() if sinks else None
  param = type("P", (), {"data": sk})() if sinks else None
  pos = torch.arange(total, device="cuda")[None].expand(B, -1)
  want = ref.attention(q.float(), k.float(), v.float(), ref.attention_mask(pos, pos, None, None, True, window), 1.0, cap, sinks=sk)
  slots = torch.tensor([2, 0], device="cuda")

  def ctx(mode, lo, hi, seg=None):
    return type("C", (), {"mode": mode, "positions": pos[:, lo:hi].contiguous(), "segment_ids": seg, "bidir": None})()
  with torch.no_grad():
    for cuts in ([0, total], [0, 17, 19, 39, 40], [0, 1, 2, 3, total]):
      cache = LayerKVCache(3, 64, G, D, Dv, bf, "cuda")
      outs = []
      for lo, hi in zip(cuts, cuts[1:]):
        cache.bind(slots, torch.full((B,), lo, dtype=torch.long, device="cuda"))
        c = ctx("prefill" if lo == 0 else "decode", lo, hi)
        assert CA.attends(q[:, lo:hi], cache, c)
        outs.append(cache.attend(q[:, lo:hi], k[:, lo:hi], v[:, lo:hi], c, window, cap, param))
      assert _rows(torch.cat(outs, 1), want) < 2e-2, cuts
    if CA.flash_widths(D, Dv) is not None:
      seg = torch.cat([torch.full((B, 15), 1), torch.full((B, 25), 2)], 1).int().cuda()
      want2 = ref.attention(q.float(), k.float(), v.float(), ref.attention_mask(pos, pos, seg, seg, True, window), 1.0, cap, sinks=sk)
      cache = LayerKVCache(3, 64, G, D, Dv, bf, "cuda")
      cache.bind(slots, torch.zeros(B, dtype=torch.long, device="cuda"))
      assert _rows(cache.attend(q, k, v, ctx("prefill", 0, total, seg), window, cap, param), want2) < 2e-2


def test_training_step_in_bf16(tmp_path):
  """The layers train through their differentiable forms, with the fp32 streams crossing units."""
  from helpers import BASE_YML
  from maxtext_b200.config import pyconfig
  from maxtext_b200.input_pipeline.synthetic import SyntheticDataIterator
  from maxtext_b200.train.engine import TrainEngine
  sp = M.spec([(M.scan(128, 8, 16, 3), M.dense(128)), (M.attention(4, 2, 64, 64, 32, 0.1, 9.0), M.moe(4, 2, 64, 2.0))], 128, streams=3, vocab=512)
  path = M.write_folder(tmp_path / "m", sp, M.weights(sp))
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype="bfloat16", max_target_length=64, per_device_batch_size=2,
                            dataset_type="synthetic", hardware="gpu", enable_checkpointing=False, log_config=False, steps=5, learning_rate=2e-3,
                            warmup_steps_fraction=0.0)
  eng = TrainEngine(cfg, None, torch.device("cuda", 0))
  batch = next(SyntheticDataIterator(cfg))
  losses = [float(eng.train_step(batch)["learning/loss"]) for _ in range(5)]
  assert losses[-1] < losses[0] and all(x == x for x in losses), losses
