"""Mechanism-level checks shared by the CPU and the GPU tests: ops of the package against tests/oracle_layered.py, with
inputs made so that one key out of place, a sink left out or a wrong denominator dominates the result."""
import torch

import oracle_layered as O
from xfastertransformer_b200 import ops


def paged(x, block=64, spare=3, seed=0):
    """[T, G, d] -> (pool [nb, G, block, d], block table [1, W]): pages in scrambled order, unused rows hold large values."""
    T, G, d = x.shape
    n = (T + block - 1) // block
    g = torch.Generator().manual_seed(seed)
    perm = torch.randperm(n + spare, generator=g)[:n]
    pool = torch.full((n + spare, G, block, d), 25.0, dtype=x.dtype)
    for t in range(T):
        pool[perm[t // block], :, t % block] = x[t]
    return pool, perm.int().view(1, n)


def attend(dev, dtype, q, k, v, decode, start=0, pad=0, **kw):
    """ops.paged_attention of queries start .. T - 1 over all keys of one sequence: as a prompt portion, or each as a
    decode step of its own sequence sharing the pages (one batch)."""
    T, H, _ = q.shape
    if pad:                                          # heads padded with zeros, as the decoder pads them at load
        z = lambda t: torch.cat([t, torch.zeros(*t.shape[:2], pad - t.shape[2], dtype=t.dtype)], -1)
        q, k, vd, v = z(q), z(k), v.shape[2], z(v)
    kp, bt = paged(k.to(dtype))
    vp, _ = paged(v.to(dtype))
    n = T - start
    qd = q[start:].to(dtype).to(dev).contiguous()
    if decode:
        cu, lens, table = list(range(n + 1)), [i + 1 for i in range(start, T)], bt.repeat(n, 1)
    else:
        cu, lens, table = [0, n], [T], bt
    out = ops.paged_attention(qd, kp.to(dev), vp.to(dev), table.to(dev), cu, lens, kw.pop("scale"), **kw)
    if dev.type == "cuda":
        from xfastertransformer_b200.ops import native
        native.Workspace.get(dev).check_status()
    out = out.float().cpu()
    return out[..., :vd] if pad else out


def _close(got, want, tol, what):
    e = (got - want).abs().amax(dim=(-1, -2)) / want.abs().max()
    assert bool((e <= tol).all()), f"{what}: query {int(e.argmax())} is off by {float(e.max()):.3g}"


def _inputs(T, H, G, d, dv, dtype, seed):
    """Keys and queries so quiet that every visible key weighs the same, values so distinct that each one shows."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    return r(T, H, d) / 16, r(T, G, d), r(T, G, dv)


def window_edges(dev, dtype, d, dv, window, keep, decode, tol, T=200, H=4, G=2, **kw):
    """For every distance that is special — just inside and just outside the window, the last kept token and the first that
    is not, a page's first and last token — one key is made to stand out (score about +20 for every query).  Queries that
    see it return its value almost alone; queries that do not must not feel it."""
    q, k, v = _inputs(T, H, G, d, dv, dtype, window * 31 + keep)
    q[..., 0] = 2.0
    k[..., 0] = 0.0
    mask = {"size": window, "keep_first": keep}
    sink = torch.linspace(-1.0, 1.5, H)
    i = T - 30
    for j in sorted({i - window, i - window + 1, i - window - 1, keep - 1, keep, 63, 64, 127, 128, 0, i}):
        if not 0 <= j < T:
            continue
        kk = k.clone()
        kk[j, :, 0] = 10.0
        want = O.attention(q.double(), kk.double(), v.double(), 1.0, 40.0, mask, sink.double())[100:].float()
        got = attend(dev, dtype, q, kk, v, decode, 100, scale=1.0, softcap=40.0, window=window, keep_first=keep,
                     sinks=sink.to(dev), **kw)
        _close(got, want, tol, f"window {window}, kept {keep}, key {j}")


def sink_counts_once(dev, dtype, d, tol, T=150, H=3, G=1, **kw):
    """Sinks from negligible to dominant: a sink that is scaled, capped, left out or counted per split or per tile changes
    the output's size."""
    q, k, v = _inputs(T, H, G, d, d, dtype, 5)
    v = v + 2.0                                       # means do not cancel: the output's size is the visible weight
    for sink in (torch.tensor([-30.0, 0.0, 3.0]), torch.tensor([5.0, 8.0, 60.0])):
        want = O.attention(q.double(), k.double(), v.double(), 0.7, 6.0, None, sink.double())
        for decode in (False, True):
            got = attend(dev, dtype, q, k, v, decode, 0, scale=0.7, softcap=6.0, sinks=sink.to(dev), **kw)
            for h in range(H):
                w = want[:, h:h + 1].float()
                if float(w.abs().max()) > 1e-9:
                    _close(got[:, h:h + 1], w, tol, f"sink {float(sink[h])}, decode {decode}")
                else:
                    assert float(got[:, h].abs().max()) < 1e-6


def softcap(dev, dtype, d, tol, T=140, H=2, G=2, **kw):
    """Scores far above and far below the cap."""
    g = torch.Generator().manual_seed(9)
    r = lambda a, *s: (a * torch.randn(*s, generator=g)).to(dtype).float()
    q, k, v = r(3, T, H, d), r(3, T, G, d), r(1, T, G, d)
    for cap in (1.5, 30.0):
        want = O.attention(q.double(), k.double(), v.double(), 0.4, cap, {"size": 77, "keep_first": 3}, None).float()
        for decode in (False, True):
            got = attend(dev, dtype, q, k, v, decode, 0, scale=0.4, softcap=cap, window=77, keep_first=3, **kw)
            _close(got, want, tol, f"cap {cap}, decode {decode}")


def residual_norm(dev, H, kind, y_dtype, h_dtype, tol, T=9):
    """Every form of the op: embedding, sum, norm before the sum, norm after it, selected rows; means far from zero."""
    g = torch.Generator().manual_seed(H)
    HP = (H + 7) // 8 * 8 if dev.type == "cuda" else H
    wide = lambda t: torch.cat([t, torch.zeros(*t.shape[:-1], HP - H, dtype=t.dtype)], -1).to(dev).contiguous()
    x = torch.randn(T, H, generator=g) * 3 + 5
    y = (torch.randn(T, H, generator=g) * 0.1 + 2).to(y_dtype)
    w1, w2 = torch.randn(H, generator=g), torch.randn(H, generator=g)
    b1, b2 = torch.randn(H, generator=g), torch.randn(H, generator=g)
    table = torch.randn(20, H, generator=g).bfloat16()
    ids = torch.tensor([3, 19, 0, 7, 3], dtype=torch.int32)
    rows = torch.tensor([8, 0, 3], dtype=torch.int32)
    eps = 1e-3

    def norm(t, w, b=None):
        if kind == "layer":
            n = O.layer_norm(t.double(), w.double(), eps)
        else:
            n = t.double() / torch.sqrt((t.double() ** 2).mean(-1, keepdim=True) + eps) * w.double()
        return n if b is None else n + b.double()

    def run(x_, y_, post, nxt, **kw):
        dv = lambda p: None if p is None else tuple(None if t is None else t.to(dev) for t in p)
        a, h = ops.residual_norm(None if x_ is None else wide(x_), None if y_ is None else wide(y_), dv(post), dv(nxt), eps, kind,
                                 h_dtype=h_dtype, **kw)
        for t in (a, h):
            if t is not None and HP > H:
                assert bool((t[:, H:] == 0).all()), "padding columns must be zero"
        return (None if a is None else a[:, :H].float().cpu()), (None if h is None else h[:, :H].float().cpu())

    def close(got, want, t, what):
        e = float((got.double() - want).abs().max() / want.abs().max())
        assert e <= t, f"{what} ({H}, {kind}): {e:.3g}"

    ht = tol if h_dtype == torch.float32 else 6e-3
    a, h = run(x, y, (w1, None), (w2, None))
    xs = x.double() + norm(y, w1)
    close(a, xs, tol, "sum of a normed sublayer")
    close(h, norm(xs, w2), ht, "next norm")
    a, h = run(x, y, (w1, b1), (w2, b2))
    close(h, norm(x.double() + norm(y, w1, b1), w2, b2), ht, "biases")
    a, h = run(x, y, None, (w2, None))
    close(a, x.double() + y.double(), tol, "plain sum")
    a, h = run(x, y, (w1, None), None)
    assert h is None
    close(a, xs, tol, "sum alone")
    a, h = run(x, None, None, (w2, None))
    close(h, norm(x, w2), ht, "norm alone")
    a, h = run(x, y, (w1, None), (w2, None), rows=rows.to(dev), keep_x=False)
    assert a is None
    close(h, norm(xs, w2)[rows.long()], ht, "selected rows")
    a, h = run(None, None, None, (w2, None), ids=ids.to(dev), table=wide(table))
    close(a, table[ids.long()].double(), 0.0, "embedding")
    close(h, norm(table[ids.long()], w2), ht, "embedding's norm")


def rotation(dev, dtype, rot, d, dv, tol, hq=3, hkv=2, T=90):
    """Split, rotation and append of one packed projection, with positions that start late and slots out of order."""
    from xfastertransformer_b200.ops import reference as R
    g = torch.Generator().manual_seed(d)
    qkv = torch.randn(T, hq * d + hkv * (d + dv), generator=g).to(dtype)
    pos = list(range(37, 37 + T))
    sc = rot.get("scaling")
    if sc:
        tab = R.rope_table(256, rot["dims"], rot["base"], "yarn", sc["factor"], sc["original"], sc["fast"], sc["slow"],
                           table_scale=O.rotary_frequencies(rot)[1])
    else:
        tab = R.rope_table(256, rot["dims"], rot["base"])
    nb = 4
    kc, vc = torch.zeros(nb, hkv, 64, d, dtype=dtype), torch.zeros(nb, hkv, 64, dv, dtype=dtype)
    slots = torch.randperm(nb * 64, generator=g)[:T].int()
    kc, vc = kc.to(dev), vc.to(dev)
    q = ops.qkv_rope_cache(qkv.to(dev), hq, hkv, d, torch.tensor(pos, dtype=torch.int32).to(dev), tab.to(dev), rot["dims"], "half",
                           kc, vc, None, None, slots.to(dev), dv=dv)
    x = qkv.double()
    wq = O.rotate(x[:, :hq * d].reshape(T, hq, d), pos, rot)
    wk = O.rotate(x[:, hq * d:(hq + hkv) * d].reshape(T, hkv, d), pos, rot)
    wv = x[:, (hq + hkv) * d:].reshape(T, hkv, dv)
    b, o = (slots // 64).long(), (slots % 64).long()
    for got, want, what in ((q, wq, "queries"), (kc.cpu()[b, :, o], wk, "keys"), (vc.cpu()[b, :, o], wv, "values")):
        e = float((got.double().cpu() - want).abs().max())
        assert e <= tol * float(want.abs().max()), f"{what}: {e:.3g}"
    q2 = ops.qkv_rope_cache(qkv[:, :hq * d].contiguous().to(dev), hq, 0, d, torch.tensor(pos, dtype=torch.int32).to(dev),
                            tab.to(dev), rot["dims"], "half", kc, vc, None, None, slots.to(dev), dv=dv)
    assert torch.equal(q2, q), "a layer with queries only rotates them like any other"
