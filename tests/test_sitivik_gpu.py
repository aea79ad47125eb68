"""Sitivik on the CUDA kernels: the shared suite in fp32 and bf16, the decode graph, and the kernels on shapes of their own."""
import pytest
import torch

import sitivik_models as M
import sitivik_oracle as O
from sitivik_suite import Suite

pytestmark = pytest.mark.gpu


class TestSitivikGpu(Suite):
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
      path = M.folder(tmp_path / (dtype + name), sp, M.weights(sp))
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


def test_forward_without_a_cache(tmp_path):
  """A plain forward pass (evaluation) runs the same layers on the differentiable forms and the flash kernel."""
  for name in ("mixed", "mixed_even"):
    sp = M.SPECS[name]
    W = M.weights(sp)
    toks = M.prompt(70, sp)
    want = M.oracle_logits(sp, W, toks)
    for dtype, worst in (("float32", 5e-5), ("bfloat16", 0.3)):
      eng = M.engine(M.folder(tmp_path / (name + dtype), sp, W), dtype, "cuda")
      e = M.rel_rows(eng.model.forward(torch.tensor(toks, device="cuda")[None])[0], want)
      assert float(e.max()) < worst and float(e.median()) < (1e-5 if dtype == "float32" else 0.04), (name, dtype, e.max())


# ------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("D, two, norms, bias, lanes, nxt", [
    (64, True, True, True, True, "norm"), (2048, True, True, False, True, "norm"), (388, True, False, True, True, "as_is"), (33, True, True, True, False, "norm"),
    (1028, False, True, True, True, "as_is"), (4096, False, False, False, True, "norm"), (5000, True, True, False, False, None), (8192, True, False, False, True, "norm"),
    (1030, True, True, True, True, "norm"), (7, False, False, False, False, "as_is")])
def test_residual_join(D, two, norms, bias, lanes, nxt):
  E = _ext()
  g = torch.Generator().manual_seed(D)
  N, eps = 19, 0.02
  for dtype in DTYPES:
    x = torch.randn(N, D, generator=g) * 3
    a, b = (torch.randn(N, D, generator=g).to(dtype) for _ in range(2))
    v = [torch.randn(D, generator=g).to(dtype) for _ in range(5)]
    bias_a, wa, wb, ln, wn = (t.double() for t in v)
    ta, tb = a.double() + (bias_a if bias else 0.0), b.double()
    if norms:
      ta, tb = O.rms(ta, eps) * wa, O.rms(tb, eps) * wb
    total = 0.7 * ta + (-1.3 * tb if two else 0.0)
    want = x.double() + (ln * total if lanes else total)
    c = [t.cuda() for t in v]
    gx, gy = x.cuda(), torch.empty(N, D, dtype=dtype, device="cuda") if nxt else None
    E.residual_join(gx, a.cuda(), c[0] if bias else None, c[1] if norms else None, 0.7, b.cuda() if two else None, None, c[2] if norms and two else None, -1.3,
                    c[3] if lanes else None, c[4] if nxt == "norm" else None, gy, eps)
    assert _rel(gx, want) < 1e-6
    if nxt:
      assert _rows(gy, O.rms(want, eps) * wn if nxt == "norm" else want) < TOL[dtype]


@pytest.mark.parametrize("dim, N", [(24, 5), (64, 300), (7, 33), (256, 1)])
def test_token_gate(dim, N):
  E = _ext()
  g = torch.Generator().manual_seed(dim)
  for dtype in DTYPES:
    x, table = (torch.randn(N, dim, generator=g) * 2).to(dtype), torch.randn(50, dim, generator=g).to(dtype)
    tok = torch.randint(0, 50, (N,), generator=g)
    out = torch.empty(N, dim, dtype=dtype, device="cuda")
    E.token_gate(x.cuda(), table.cuda(), tok.cuda(), out)
    assert _rows(out, O.gelu_tanh(x.double()) * table.double()[tok]) < TOL[dtype]


# ------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("H, G, D, Dv, rot, paired, maps, norm, temp, bias", [
    (4, 2, 20, 12, 8, True, 1, "all", 0, True), (6, 1, 128, 96, 64, True, 1, "all", 0, True), (4, 4, 64, 64, 64, True, 1, "head", 0, True),
    (5, 1, 11, 7, 6, True, 1, "head", 3, False), (3, 1, 200, 136, 100, False, 1, "head", 0, False), (4, 2, 48, 96, 0, False, 2, None, 5, True),
    (2, 1, 104, 72, 24, True, 2, "head", 7, True), (6, 3, 9, 5, 4, False, 2, None, 1, False), (1, 1, 300, 290, 24, True, 1, "all", 0, True)])
def test_prep(H, G, D, Dv, rot, paired, maps, norm, temp, bias):
  """Bias, norm, rotation, temperature, cache rows and padded operands of the attention kernels."""
  E = _ext()
  g = torch.Generator().manual_seed(D)
  B, S, max_len, eps, base = 3, 9, 30, 0.05, 300.0
  begin, new = [0, 4, 25], [9, 3, 5]
  pos = torch.tensor(begin)[:, None] + torch.arange(S)[None]
  inv = (1.0 / base ** (2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float()
  HM, GM, kw = H * maps, G * maps, D * maps
  dq, dvp = -(-kw // 64) * 64 + 64, -(-Dv // 64) * 64
  for dtype in DTYPES:
    p = torch.randn(B * S, HM * D + GM * D + G * Dv + 8, generator=g).to(dtype)
    cut = torch.split(p, [HM * D, GM * D, G * Dv, 8], 1)
    bq, bk, bv = (torch.randn(t.shape[1], generator=g).to(dtype) if bias else None for t in cut[:3])
    wn = {"all": (HM * D, GM * D), "head": (D, D)}.get(norm)
    wq, wk = (torch.randn(n, generator=g).to(dtype) for n in wn) if wn else (None, None)
    pc = torch.split(p.cuda(), [HM * D, GM * D, G * Dv, 8], 1)
    qp, kp = torch.full((B * S, HM, dq), 9.0, dtype=dtype, device="cuda"), torch.full((B * S, G, dq), 9.0, dtype=dtype, device="cuda")
    vp = torch.full((B * S, G, dvp), 9.0, dtype=dtype, device="cuda")
    kc, vc = torch.full((B + 1, max_len, G, kw), 5.0, dtype=dtype, device="cuda"), torch.full((B + 1, max_len, G, Dv), 5.0, dtype=dtype, device="cuda")
    dev = lambda t: t.cuda() if t is not None else None  # noqa: E731
    E.qkv_prep(*pc[:3], D, Dv, pos.reshape(-1).cuda(), inv.cuda() if rot else None, rot, eps if norm else -1.0, qp, kp, vp, kc, vc,
               torch.arange(B, device="cuda") + 1, torch.tensor(begin, device="cuda"), torch.tensor(new, device="cuda"), dev(bq), dev(bk), dev(bv), dev(wq), dev(wk),
               paired, maps, 0.4, float(temp))

    def want(x, b, w, heads, warm):
      x = x.double() + (b.double() if bias else 0.0)
      if norm == "all":
        x = O.rms(x, eps) * w.double()
      x = x.view(B, S, heads, D)
      if norm == "head":
        x = O.rms(x, eps) * w.double()
      x = torch.stack([O.rotate(x[b_], {"base": base, "dims": rot}, paired, begin[b_]) for b_ in range(B)])
      if warm and temp:
        x = x * (1 + 0.4 * torch.log(torch.floor((pos.double() + 1) / temp) + 1))[..., None, None]
      return x
    gq, gk, gv = want(cut[0], bq, wq, HM, True), want(cut[1], bk, wk, GM, False), (cut[2].double() + (bv.double() if bias else 0.0)).view(B, S, G, Dv)
    qv = qp.view(B, S, H, maps, dq)
    for m in range(maps):
      assert _rows(qv[:, :, :, m, m * D:(m + 1) * D], gq.view(B, S, H, maps, D)[:, :, :, m]) < TOL[dtype]
      rest = torch.cat([qv[:, :, :, m, :m * D], qv[:, :, :, m, (m + 1) * D:]], -1)
      assert float(rest.abs().max()) == 0
    gk = gk.reshape(B, S, G, kw)
    assert _rows(kp.view(B, S, G, dq)[..., :kw], gk) < TOL[dtype] and float(kp[..., kw:].abs().max()) == 0
    assert _rows(vp.view(B, S, G, dvp)[..., :Dv], gv) < TOL[dtype] and (dvp == Dv or float(vp[..., Dv:].abs().max()) == 0)
    for b in range(B):
      lo, hi = begin[b], begin[b] + new[b]
      assert _rows(kc[b + 1, lo:hi], gk[b, :new[b]]) < TOL[dtype] and _rows(vc[b + 1, lo:hi], gv[b, :new[b]]) < TOL[dtype]
      for c in (kc, vc):                             # nothing else was written
        assert float((c[b + 1, :lo] - 5).abs().sum() + (c[b + 1, hi:] - 5).abs().sum()) == 0
    assert float((kc[0] - 5).abs().max()) == 0


def _attend(q, k, v, n, scale, first, one):
  """The last of n cached tokens: q [H, D], k [n, G, D], v [n, G, Dv] -> [H, Dv]; keys from `first` on, `one` added to the denominator."""
  H, G = q.shape[0], k.shape[1]
  out = torch.zeros(H, v.shape[-1], dtype=torch.float64)
  for h in range(H):
    g = h // (H // G)
    e = torch.exp((k[first:n, g] @ q[h]) * scale)
    out[h] = (e @ v[first:n, g]) / (e.sum() + (1.0 if one else 0.0))
  return out


@pytest.mark.parametrize("H, G, D, Dv, chunk, one, per_head", [(4, 2, 64, 64, 33, True, False), (20, 1, 96, 40, 16, False, True), (3, 3, 24, 16, 1, True, False),
                                                                (8, 2, 128, 128, 100, True, True), (2, 1, 200, 136, 64, False, False)])
def test_chunked_decode(H, G, D, Dv, chunk, one, per_head):
  """Both kernels over the cache; a key just outside the chunk would win if it were seen, one just inside wins."""
  E = _ext()
  g = torch.Generator().manual_seed(H)
  max_len, lens = 220, [1, 2, 16, 17, 32, 33, 34, 64, 65, 99, 100, 101, 132, 133, 201, 220]
  B, scale, bf = len(lens), 2.0 / D ** 0.5, torch.bfloat16
  q, gate = torch.randn(B, H, D, generator=g).to(bf), torch.randn(B, H * Dv + 8, generator=g).to(bf)
  k, v = torch.randn(B + 2, max_len, G, D, generator=g).to(bf), torch.randn(B + 2, max_len, G, Dv, generator=g).to(bf)
  slots = torch.randperm(B + 2, generator=g)[:B]
  for i, n in enumerate(lens):
    first = (n - 1) // chunk * chunk
    k[slots[i], n:], v[slots[i], n:] = float("nan"), float("nan")
    k[slots[i], first] = (q[i, ::H // G].double() * 4 / D ** 0.5).to(bf)
    if first:
      k[slots[i], first - 1] = (q[i, ::H // G].double() * 9).to(bf)
  sink = torch.zeros(H, dtype=bf, device="cuda") if one else None
  for dtype in DTYPES:
    qd, kd, vd, gd = (t.to(dtype) for t in (q, k, v, gate))
    want = torch.stack([_attend(qd[i].double(), kd[s].double(), vd[s].double(), n, scale, (n - 1) // chunk * chunk, one)
                        for i, (n, s) in enumerate(zip(lens, slots.tolist()))])
    length = torch.tensor(lens, device="cuda") - 1
    out = torch.empty(B, H, Dv, dtype=dtype, device="cuda")
    E.cached_attention(qd.cuda(), kd.cuda(), vd.cuda(), slots.cuda(), length, 1, scale, 0.0, 0, sink.to(dtype) if one else None, out, chunk)
    assert _rows(out, want) < 2 * TOL[dtype]
    if dtype == bf:
      wanted = want * (O.sigmoid(gate.double()[:, :H])[..., None] if per_head else O.sigmoid(gate[:, :H * Dv].double()).view(B, H, Dv))
      for splits in (1, 3, 16):
        part, ml = torch.empty(B, H, splits, Dv, device="cuda"), torch.empty(B, H, splits, 2, device="cuda")
        got = torch.empty(B, H * Dv, dtype=bf, device="cuda")
        E.cached_decode(qd.cuda(), kd.cuda(), vd.cuda(), slots.cuda(), length, scale, 0.0, 0, sink, gate.cuda(), splits, part, ml, got, chunk=chunk,
                        per_head=per_head)
        assert _rows(got.view(B, H, Dv), wanted) < 1.5e-2, splits


@pytest.mark.parametrize("H, G, D, Dv, per_head", [(4, 2, 32, 64, True), (12, 1, 64, 128, True), (2, 2, 24, 40, False), (3, 1, 128, 200, True), (1, 1, 8, 8, False)])
def test_differential_decode(H, G, D, Dv, per_head):
  E = _ext()
  g = torch.Generator().manual_seed(H + D)
  max_len, lens, bf = 150, [1, 2, 16, 17, 65, 149, 150], torch.bfloat16
  B, scale, diff, eps = len(lens), 3.0 / D ** 0.5, 0.3, 0.02
  q, gate = torch.randn(B, H, 2, D, generator=g).to(bf), torch.randn(B, H * Dv, generator=g).to(bf)
  k, v = torch.randn(B, max_len, G, 2 * D, generator=g).to(bf), torch.randn(B, max_len, G, Dv, generator=g).to(bf)
  lam = [(torch.randn(D, generator=g) * 0.5 * D ** -0.25).to(bf) for _ in range(4)]
  l = [t.double() for t in lam]
  lv = torch.exp((l[0] * l[1]).sum()) - torch.exp((l[2] * l[3]).sum()) + diff
  for i, n in enumerate(lens):
    k[i, n:], v[i, n:] = float("nan"), float("nan")
  kd = k.double().view(B, max_len, G, 2, D)
  a = [torch.stack([_attend(q[i, :, m].double(), kd[i, :, :, m], v[i].double(), n, scale, 0, False) for i, n in enumerate(lens)]) for m in (0, 1)]
  want = O.difference(a[0], a[1], lv, diff, eps)
  want = want * (O.sigmoid(gate.double()[:, :H])[..., None] if per_head else O.sigmoid(gate.double()).view(B, H, Dv))
  qp = torch.zeros(B, H, 2, 2 * D, dtype=bf)
  qp[:, :, 0, :D], qp[:, :, 1, D:] = q[:, :, 0], q[:, :, 1]
  qp = qp.view(B, 2 * H, 2 * D).cuda()
  slots, length = torch.arange(B, device="cuda"), torch.tensor(lens, device="cuda") - 1
  lc = [t.cuda() for t in lam]
  o = torch.empty(B, 2 * H, Dv, dtype=bf, device="cuda")
  E.cached_attention(qp, k.cuda(), v.cuda(), slots, length, 1, scale, 0.0, 0, None, o, 0)
  out = torch.empty(B, H * Dv, dtype=bf, device="cuda")
  E.diff_combine(o, lc, diff, eps, gate.cuda(), Dv, out, per_head)
  assert _rows(out.view(B, H, Dv), want) < 3e-2
  o32 = torch.stack(a, 2).view(B, 2 * H, Dv).float().cuda()
  pad = torch.nn.functional.pad(o32, (0, 5)).contiguous()
  out32 = torch.empty(B, H * Dv, device="cuda")
  E.diff_combine(pad, [t.float() for t in lc], diff, eps, gate.float().cuda(), Dv, out32, per_head)
  assert _rows(out32.view(B, H, Dv), want) < 1e-5
  for splits in (1, 3, 16):
    part, ml = torch.empty(B, 2 * H, splits, Dv, device="cuda"), torch.empty(B, 2 * H, splits, 2, device="cuda")
    got = torch.empty(B, H * Dv, dtype=bf, device="cuda")
    E.cached_decode(qp, k.cuda(), v.cuda(), slots, length, scale, 0.0, 0, None, gate.cuda(), splits, part, ml, got, per_head=per_head, lam=lc, diff=diff, eps=eps)
    assert _rows(got.view(B, H, Dv), want) < 2e-2, splits


# ------------------------------------------------------------------------------------------ recurrences
def _pieces(S):
  cuts = [0, 1, S // 3, S // 2 + 2, S - 2, S - 1, S]
  return [(a, b) for a, b in zip(cuts, cuts[1:]) if b > a]


@pytest.mark.parametrize("B, S, H, dk, dv, rot, lens", [
    (2, 150, 3, 64, 48, 64, None), (1, 300, 2, 128, 64, 32, None), (3, 70, 2, 16, 16, 6, [70, 1, 65]), (2, 130, 2, 112, 32, 0, [64, 130]), (1, 90, 2, 20, 12, 10, None),
    (2, 40, 1, 200, 250, 44, [40, 33]), (1, 67, 4, 7, 5, 2, None)])
def test_retention(B, S, H, dk, dv, rot, lens):
  E = _ext()
  g = torch.Generator().manual_seed(S)
  eps, base = 0.01, 50.0
  decay = (torch.rand(H, generator=g, dtype=torch.float64) * 0.5 + 0.5) ** 0.2
  decay[0] = 0.9999
  inv = (1.0 / base ** (2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float().cuda() if rot else None
  ld = torch.log(decay).float().cuda()
  for dtype in DTYPES:
    p = torch.randn(B * S, 2 * H * (dk + dv) + 16, generator=g).to(dtype)
    pd = p.double().view(B, S, -1)
    qkvz = torch.split(pd, [H * dk, H * dk, H * dv, H * dv, 16], -1)
    slots, length = torch.arange(B, device="cuda") + 1, torch.zeros(B, dtype=torch.long, device="cuda")
    new = torch.tensor(lens, device="cuda") if lens else None
    pc = p.cuda()

    def wanted(b, n):
      q, k, v = qkvz[0][b, :n].reshape(n, H, dk), qkvz[1][b, :n].reshape(n, H, dk), qkvz[2][b, :n].reshape(n, H, dv)
      turn = {"base": base, "dims": rot}
      return O.retention_scan(O.rotate(q, turn, False) * dk ** -0.5, O.rotate(k, turn, False), v, decay)
    forms = [E.retention_scan] + ([E.retention_chunks] if dtype == torch.bfloat16 and E.chunk_supported(dk, dv) else [])
    for form in forms:
      rec = torch.full((B + 1, H, dk, dv), 7.0, device="cuda")                 # dirty slots
      o = torch.empty(B * S, H * dv, dtype=dtype, device="cuda")
      form(pc, ld, inv, rot, H, dk, dv, S, rec, slots, length, new, o)
      assert torch.isfinite(o).all() and float((rec[0] - 7).abs().max()) == 0
      for b in range(B):
        n = lens[b] if lens else S
        assert _rows(o.view(B, S, H, dv)[b, :n], wanted(b, n)) < (2e-5 if dtype == torch.float32 else 1e-2), (dtype, form, b)
      if lens:
        continue
      rec2 = torch.full_like(rec, 9.0)
      for lo, hi in _pieces(S):
        m = hi - lo
        cut = pc.view(B, S, -1)[:, lo:hi].reshape(B * m, -1).contiguous()
        oo, at = torch.empty(B * m, H * dv, dtype=dtype, device="cuda"), torch.full_like(length, lo)
        if m > 1:
          form(cut, ld, inv, rot, H, dk, dv, m, rec2, slots, at, None, oo)
          assert _rows(oo.view(B, m, H * dv), o.view(B, S, -1)[:, lo:hi]) < TOL[dtype]
        else:
          E.retention_decode(cut, ld, inv, rot, eps, H, dk, dv, rec2, slots, at, oo)
          want = torch.stack([O.rms(wanted(b, hi)[-1], eps).reshape(-1) * O.silu(qkvz[3][b, lo]) for b in range(B)])
          assert _rows(oo, want) < TOL[dtype]
      assert _rel(rec2[1:], rec[1:]) < 1e-4


@pytest.mark.parametrize("B, S, hk, hv, dk, dv, taps, lens, rate", [
    (2, 150, 2, 4, 64, 48, 4, None, 0.0), (1, 200, 2, 2, 128, 64, 2, None, -4.0), (3, 70, 1, 2, 16, 16, 3, [70, 1, 65], 0.0), (2, 130, 1, 3, 32, 32, 1, [64, 130], 2.0),
    (1, 90, 2, 2, 112, 16, 4, None, 3.5), (1, 90, 3, 3, 20, 12, 6, None, 0.0), (2, 40, 1, 1, 200, 250, 4, [40, 33], 0.0), (1, 67, 1, 2, 7, 5, 3, None, 1.0),
    (1, 128, 1, 1, 48, 32, 4, None, -8.0)])
def test_channel_delta(B, S, hk, hv, dk, dv, taps, lens, rate):
  """Decays from nearly one (rate -8) to nearly nothing (3.5: the exponents of a block of tokens no longer fit one split)."""
  E = _ext()
  g = torch.Generator().manual_seed(S)
  eps, C = 0.01, 2 * hk * dk + hv * dv
  for dtype in DTYPES:
    x = torch.randn(B * S, C + 8, generator=g).to(dtype)[:, :C] if C % 8 == 0 else torch.randn(B * S, C, generator=g).to(dtype)
    w, beta = (torch.randn(taps, C, generator=g) * 0.6).to(dtype), torch.randn(B * S, -(-hv // 8) * 8, generator=g).to(dtype)
    da, A = torch.randn(B * S, hv * dk, generator=g), (torch.randn(hv, generator=g) * 0.5 + rate).to(dtype)
    dtb, z, nw = torch.randn(hv * dk, generator=g).to(dtype), torch.randn(B * S, hv * dv, generator=g).to(dtype), torch.randn(dv, generator=g).to(dtype)
    slots, length = torch.arange(B, device="cuda") + 1, torch.zeros(B, dtype=torch.long, device="cuda")
    new = torch.tensor(lens, device="cuda") if lens else None
    dev = [t.cuda() for t in (x, w, beta, da, A, dtb, z, nw)]
    xc, wc, bc, dac, Ac, dtc, zc, nwc = dev

    def wanted(b, n, mixed):
      q, k, v = torch.split(mixed, [hk * dk, hk * dk, hv * dv], -1)
      q, k = (O.unit(t.view(n, hk, dk)).repeat_interleave(hv // hk, 1) for t in (q, k))
      step = O.softplus(da.double().view(B, S, hv, dk)[b, :n] + dtb.double().view(hv, dk))
      gg = torch.exp(-torch.exp(A.double())[None, :, None] * step)
      return O.delta_scan(q * dk ** -0.5, k, v.view(n, hv, dv), gg, O.sigmoid(beta.double().view(B, S, -1)[b, :n, :hv]))
    conv0, rec0 = torch.full((B + 1, taps - 1, C), 5.0, device="cuda"), torch.full((B + 1, hv, dk, dv), 7.0, device="cuda")    # dirty slots
    mixed = torch.empty(B * S, C, dtype=dtype, device="cuda")
    E.ssm_conv(xc, wc, None, S, conv0, slots, length, new, mixed)
    for b in range(B):
      n = lens[b] if lens else S
      assert _rows(mixed.view(B, S, C)[b, :n], O.silu(O.causal_conv(x.double().view(B, S, C)[b, :n], w.double().t()))) < TOL[dtype]
    for chunked in (False,) + ((True,) if dtype == torch.bfloat16 and E.chunk_supported(dk, dv) and C % 8 == 0 else ()):
      rec = rec0.clone()
      o = torch.empty(B * S, hv * dv, dtype=dtype, device="cuda")
      E.channel_delta_scan(mixed, bc, dac, Ac, dtc, hk, hv, dk, dv, S, rec, slots, length, new, o, chunked)
      assert torch.isfinite(o).all() and float((rec[0] - 7).abs().max()) == 0
      for b in range(B):
        n = lens[b] if lens else S
        want = wanted(b, n, mixed.double().cpu().view(B, S, C)[b, :n])
        assert _rows(o.view(B, S, hv, dv)[b, :n], want) < (3e-5 if dtype == torch.float32 else 1e-2), (dtype, chunked, b)
      if lens:
        continue
      conv2, rec2 = torch.full_like(conv0, 9.0), torch.full_like(rec, 9.0)
      for lo, hi in _pieces(S):
        def cut(t):
          return t.view(B, S, -1)[:, lo:hi].reshape(B * m, -1).contiguous()
        m, at = hi - lo, torch.full_like(length, lo)
        oo = torch.empty(B * m, hv * dv, dtype=dtype, device="cuda")
        xx = x.view(B, S, -1)[:, lo:hi].reshape(B * m, -1).contiguous().cuda()
        if m > 1:
          mm = torch.empty(B * m, C, dtype=dtype, device="cuda")
          E.ssm_conv(xx, wc, None, m, conv2, slots, at, None, mm)
          E.channel_delta_scan(mm, cut(bc), cut(dac), Ac, dtc, hk, hv, dk, dv, m, rec2, slots, at, None, oo, chunked)
          assert _rows(oo.view(B, m, -1), o.view(B, S, -1)[:, lo:hi]) < TOL[dtype]
        else:
          E.channel_delta_decode(xx, cut(bc), wc, cut(dac), Ac, dtc, cut(zc), nwc, eps, hk, hv, dk, dv, conv2, rec2, slots, at, oo)
          want = torch.stack([(O.rms(wanted(b, hi, mixed.double().cpu().view(B, S, C)[b, :hi])[-1], eps) * nw.double()
                               * O.sigmoid(z.double().view(B, S, hv, dv)[b, lo])).reshape(-1) for b in range(B)])
          assert _rows(oo, want) < 1.5 * TOL[dtype]
      assert _rel(rec2[1:], rec[1:]) < 1e-4 and torch.equal(conv2[1:], conv0[1:])


@pytest.mark.parametrize("H, dv, sig, weight", [(3, 64, True, True), (2, 20, False, False), (5, 7, True, False), (1, 256, False, True)])
def test_gated_head_norm(H, dv, sig, weight):
  E = _ext()
  g = torch.Generator().manual_seed(dv)
  N, eps = 21, 0.03
  for dtype in DTYPES:
    o, z, w = torch.randn(N, H * dv, generator=g).to(dtype), torch.randn(N, H * dv, generator=g).to(dtype), torch.randn(dv, generator=g).to(dtype)
    out = torch.empty(N, H * dv, dtype=dtype, device="cuda")
    E.gated_head_norm(o.cuda(), z.cuda(), H, dv, 1, 0, dv, w.cuda() if weight else None, eps, out, sig)
    zz = z.double().view(N, H, dv)
    want = O.rms(o.double().view(N, H, dv), eps) * (w.double() if weight else 1.0) * (O.sigmoid(zz) if sig else O.silu(zz))
    assert _rows(out.view(N, H, dv), want) < TOL[dtype]


def test_training_step_in_bf16(tmp_path):
  """The layers train through their differentiable forms, with the fp32 stream crossing units."""
  from helpers import BASE_YML
  from maxtext_b200.config import pyconfig
  from maxtext_b200.input_pipeline.synthetic import SyntheticDataIterator
  from maxtext_b200.train.engine import TrainEngine
  sp = M.spec([(M.parallel(M.window(4, 2, 64, 64, 32, 24, 0.12), M.retention(32, 64, 32, (0.9, 0.99))), 128), (M.differential(4, 2, 32, 64, 0.2), 128),
               (M.parallel_2(M.window(4, 4, 64, 64, 64, 40, 0.12), M.delta(4, 2, 32, 32, 4, 16, 8)), 128)], 128, vocab=512, side=16)
  path = M.folder(tmp_path / "m", sp, M.weights(sp))
  cfg = pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype="bfloat16", max_target_length=64, per_device_batch_size=2,
                            dataset_type="synthetic", hardware="gpu", enable_checkpointing=False, log_config=False, steps=5, learning_rate=2e-3,
                            warmup_steps_fraction=0.0)
  eng = TrainEngine(cfg, None, torch.device("cuda", 0))
  batch = next(SyntheticDataIterator(cfg))
  losses = [float(eng.train_step(batch)["learning/loss"]) for _ in range(5)]
  assert losses[-1] < losses[0] and all(x == x for x in losses), losses
