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


def _latent_layer(H, d, rd, R, dv, T, seed, quiet=1 / 16):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    q = r(T, H, d + rd) * quiet
    return q, r(T, R), r(T, rd), r(H, d, R) / R ** 0.5, r(H, dv, R) / R ** 0.5, r(T, H * dv)


def latent_run(dev, dtype, q, c, kr, uk, uv, gate, scale, window, decode, start, extra=0, sinks=None):
    """ops.latent_attention of queries start .. T - 1, as one portion or as decode steps that share the pages; with `extra`,
    the portion's batch also holds `extra` short portions of two tokens (the last ones, over the same pages)."""
    T, H, _ = q.shape
    d, R, dv = uk.shape[1], uk.shape[2], uv.shape[1]
    rd = kr.shape[1]
    up = (lambda n: (n + 63) // 64 * 64) if dev.type == "cuda" and dtype == torch.bfloat16 else (lambda n: n)
    rank = next((x for x in (64, 128, 256, 512) if R <= x), up(R)) if up(1) > 1 else R
    per_head = gate.shape[1] == H and dv > 1               # one gate value per head
    dims = ops.LatentDims(H, up(d), up(rd), rank, up(dv), False, True, R, per_head, 8 if up(1) > 1 else 1)

    def pad(t, *shape):
        out = torch.zeros(*shape, dtype=t.dtype)
        out[tuple(slice(n) for n in t.shape)] = t
        return out
    qp = torch.cat([pad(q[..., :d], T, H, dims.dim), pad(q[..., d:], T, H, dims.rot)], -1).reshape(T, -1)
    x = torch.cat([qp, gate if per_head else pad(gate.view(T, H, dv), T, H, dims.vdim).reshape(T, -1)], -1)
    x = pad(x, T, dims.row)
    rows = torch.cat([pad(c, T, dims.rank), pad(kr, T, dims.rot)], -1)
    pool, bt = paged(rows[:, None].to(dtype))
    w = ops.LatentWeights(pad(uk, H, dims.dim, dims.rank).to(dtype).to(dev), pad(uv, H, dims.vdim, dims.rank).to(dtype).to(dev))
    n = T - start
    xs, cu, lens = x[start:], [0, n], [T]
    if decode:
        cu, lens = list(range(n + 1)), [i + 1 for i in range(start, T)]
    for i in range(extra):
        xs, cu, lens = torch.cat([xs, x[T - 2 - i:T - i]]), cu + [cu[-1] + 2], lens + [T - i]
    xs = xs.to(dtype).to(dev).contiguous()
    out = ops.latent_attention(xs, dims, pool.to(dev), bt.repeat(len(lens), 1).to(dev), cu, lens, w, scale, window, sinks=sinks)
    if dev.type == "cuda":
        from xfastertransformer_b200.ops import native
        native.Workspace.get(dev).check_status()
    return out.float().cpu().view(-1, H, dims.vdim)[..., :dv]


def latent_want(q, c, kr, uk, uv, gate, scale, window):
    a = O.latent_attention(q.double(), c.double(), kr.double(), uk.double(), uv.double(), scale, {"size": window} if window else None)
    return (a * torch.sigmoid(gate.double()).view(a.shape)).float()


def latent_window_edges(dev, dtype, window, decode, tol, T=200, H=3, d=24, rd=12, R=40, dv=20, extra=0):
    """One key stands out at every distance that is special, once through the shared rotated part and once through the
    latent: a query that sees it returns its value almost alone."""
    q, c, kr, uk, uv, gate = _latent_layer(H, d, rd, R, dv, T, window)
    q[..., d], kr[:, 0] = 2.0, 0.0
    start, i = 100, T - 30
    for j in sorted({i - window - 1, i - window, i - window + 1, 63, 64, 127, 128, 0, i}):
        if not 0 <= j < T:
            continue
        k2 = kr.clone()
        k2[j, 0] = 10.0
        want = latent_want(q, c, k2, uk, uv, gate, 1.0, window)
        got = latent_run(dev, dtype, q, c, k2, uk, uv, gate, 1.0, window, decode, start, extra)
        rows = list(range(start, T)) + [t for e in range(extra) for t in (T - 2 - e, T - 1 - e)]
        _close(got, want[rows], tol, f"window {window}, key {j}")


def latent_heads_differ(dev, dtype, tol, decode, T=150, H=20, d=32, rd=16, R=64, dv=48, window=60, extra=0):
    """Scores spread over several units, every head with matrices of its own: a head that uses another's is far off."""
    q, c, kr, uk, uv, gate = _latent_layer(H, d, rd, R, dv, T, 3, quiet=0.7)
    want = latent_want(q, c, kr, uk, uv, gate, 0.5, window)
    got = latent_run(dev, dtype, q, c, kr, uk, uv, gate, 0.5, window, decode, 40, extra)
    rows = list(range(40, T)) + [t for e in range(extra) for t in (T - 2 - e, T - 1 - e)]
    e = (got - want[rows]).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()
    assert float(e) <= tol, f"off by {float(e):.3g}"


def latent_prep(dev, dtype, tol, T=70, H=5, d=24, rd=12, R=40, spare=4):
    """Rotation of the queries' rotated part in place (columns past the rotated ones pass), norm over the real latent only,
    append in scrambled slots; a layer that reads another's rows only rotates."""
    from xfastertransformer_b200.ops import reference as Rf
    g = torch.Generator().manual_seed(8)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype)
    rot = {"dims": rd, "base": 700.0, "scaling": {"factor": 3.0, "original": 50, "fast": 5.0, "slow": 0.5}}
    tab = Rf.rope_table(256, rd, 700.0, "yarn", 3.0, 50, 5.0, 0.5, table_scale=O.rotary_frequencies(rot)[1], angle_dtype=torch.float64)
    rp, rk = rd + spare, R + spare
    dims = ops.LatentDims(H, d, rp, rk, 8, True, True, R)
    x = r(T, dims.row)
    x[:, dims.q_width + R:dims.q_width + rk] = 0
    w = torch.cat([torch.rand(R, generator=g) + 0.5, torch.zeros(spare)])
    pos = list(range(31, 31 + T))
    pool = torch.zeros(3, 1, 64, rk + rp, dtype=dtype).to(dev)
    slots = torch.randperm(3 * 64, generator=g)[:T].int()
    y = x.clone().to(dev)
    p = torch.tensor(pos, dtype=torch.int32).to(dev)
    ops.latent_prep(y, dims, p, tab.to(dev), rd, w.to(dev), 1e-3, pool, slots.to(dev))
    xd = x.double()
    q = xd[:, :dims.q_width].view(T, H, d + rp).clone()
    q[..., d:] = O.rotate(q[..., d:], pos, rot, True)
    c = torch.cat([O.rms_norm(xd[:, dims.q_width:dims.q_width + R], w[:R].double(), 1e-3), torch.zeros(T, spare)], -1)
    k = O.rotate(xd[:, None, dims.q_width + rk:dims.gate_at], pos, rot, True)[:, 0]
    got = pool.cpu()[(slots // 64).long(), 0, (slots % 64).long()]
    for a, b, what in ((y[:, :dims.q_width].view(T, H, -1), q, "queries"), (got[:, :rk], c, "latents"), (got[:, rk:], k, "shared keys"),
                       (y[:, dims.gate_at:], xd[:, dims.gate_at:], "gate")):
        e = float((a.double().cpu() - b).abs().max() / b.abs().max())
        assert e <= tol, f"{what}: {e:.3g}"
    reader = ops.LatentDims(H, d, rp, rk, 8, False, True, R)
    z = torch.cat([x[:, :dims.q_width], x[:, dims.gate_at:]], -1).contiguous().to(dev)
    before = pool.clone()
    ops.latent_prep(z, reader, p, tab.to(dev), rd, None, 1e-3, pool, slots.to(dev))
    assert torch.equal(z[:, :dims.q_width], y[:, :dims.q_width]) and torch.equal(pool, before)


def experts(dev, dtype, tol, T, E, top, ff, shared, width=72, spread=2.0):
    """Router and gate-free experts against the plain form; unused experts and experts that get every token included."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T * 31 + E)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    h = r(T, width)
    W = {"embed": torch.zeros(1, width), "l0.mlp.router": r(E, width) * (spread / width ** 0.5)}
    W["l0.mlp.router"] = W["l0.mlp.router"].bfloat16().float()
    sizes = [(f"e{e}", ff) for e in range(E)] + ([("shared", shared)] if shared else [])
    for n, f in sizes:
        W[f"l0.mlp.{n}.up"], W[f"l0.mlp.{n}.down"] = (r(f, width) / width ** 0.5).bfloat16().float(), (r(width, f) / f ** 0.5).bfloat16().float()
    W = {k: v.double() for k, v in W.items()}
    want = O.experts(h.double(), {"router": {"top": top}, "shared": bool(shared)}, W, "l0")
    kind = "bf16" if dtype == torch.bfloat16 else "fp32"
    lin = lambda n: make_linear(W["l0.mlp." + n].float().to(dev), kind)
    x = h.to(dtype).to(dev)
    idx, w = ops.route(ops.linear(x, lin("router"), out_dtype=torch.float32), "deepseek", top, norm_topk=True, scoring="softmax")
    pair = lambda n: (lin(n + ".up"), lin(n + ".down"))
    add = None
    if shared:
        up, down = pair("shared")
        add = ops.linear(ops.linear(x, up, act="relu2"), down, out_dtype=torch.float32)
    got = ops.moe_experts(x, idx, w, [pair(f"e{e}") for e in range(E)], "relu2", 0, gated=False, add=add)
    assert got.dtype == torch.float32
    wi, ww = O.router(h.double() @ W["l0.mlp.router"].T, top)
    assert torch.equal(torch.sort(idx.cpu().long(), -1).values, torch.sort(wi, -1).values), "other experts"
    assert float((w.cpu().double().sum(-1) - 1).abs().max()) < 1e-5
    e = float((got.double().cpu() - want).abs().max() / want.abs().max())
    assert e <= tol, f"{T} tokens, {top} of {E}: {e:.3g}"


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
    a, h = run(None, None, None, (w2, None), ids=ids.to(dev), table=wide(table), embed_scale=2.75)
    close(a, table[ids.long()].double() * 2.75, 0.0, "scaled embedding")
    close(h, norm(table[ids.long()].double() * 2.75, w2), ht, "scaled embedding's norm")
    a, h = run(None, None, None, (w2, None), ids=ids.to(dev), table=wide(table))
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


# ------------------------------------------------------------------------------------------ recurrent mechanisms
class Portions:
    """Sequences cut into portions that run in batches: steps() yields (cu_q, kv_lens, which sequence and tokens)."""

    def __init__(self, lengths, sizes, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.at, self.n, self.sizes, self.g = [0] * len(lengths), list(lengths), sizes, g

    def steps(self):
        k = 0
        while any(a < n for a, n in zip(self.at, self.n)):
            live = [i for i in range(len(self.n)) if self.at[i] < self.n[i]]
            if len(live) > 1 and k % 3 == 2:
                live = live[1:]                           # some sit a step out
            cu, lens, parts = [0], [], []
            for i in live:
                m = min(self.sizes[(k + i) % len(self.sizes)], self.n[i] - self.at[i])
                parts.append((i, self.at[i], self.at[i] + m))
                self.at[i] += m
                cu.append(cu[-1] + m)
                lens.append(self.at[i])
            k += 1
            yield cu, lens, parts


def gated_linear(dev, dtype, tol, H, d, dv, rank, tau, lengths, sizes, z_around=1.5, spread=2.0):
    """Batches of unequal portions over states that start out as garbage, against the recurrence token by token.  In every
    head one key channel hardly decays and one token's key, 5 places in, owns it: its value must still be there at the end."""
    g = torch.Generator().manual_seed(d * 7 + dv)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    gpu = dev.type == "cuda"
    D = ops.LinearDims(H, d, dv, rank, 8 if gpu else 1)
    a2 = (r(H * d, rank) * spread / rank ** 0.5).to(dtype).float()
    bias, gain = z_around + r(H * d), 1 + 0.2 * r(dv)
    bias[::d] = 14.0                                      # the first channel of every head
    a2[::d] = 0
    a2p = torch.zeros(H * d, D.up(rank))
    a2p[:, :rank] = a2
    W = ops.LinearWeights(a2p.to(dtype).to(dev).contiguous(), bias.to(dev), tau, gain.to(dev))
    n = len(lengths)
    state = torch.full((n + 2, H, d, dv), 50.0, device=dev)
    slots = torch.randperm(n + 2, generator=g)[:n].int()
    seqs, want = [], []
    for T in lengths:
        q, k, v, gate, a1 = r(T, H, d), r(T, H, d), r(T, H, dv), r(T, H * dv), r(T, rank)
        k = ((k + q) / d ** 0.25).to(dtype).float()
        q[:, :, 0], k[:, :, 0] = 4.0, 0.0
        if T > 5:
            k[5, :, 0] = 4.0
        seqs.append((q, k, v, gate, a1))
        z = a1.double() @ a2.double().T + bias.double()
        o = O.gated_linear(q.double() * d ** -0.5, k.double(), v.double(), torch.exp(O.log_decay(z, tau)).view(T, H, d))
        o = O.rms_norm(o, gain.double(), 1e-5).reshape(T, -1)
        want.append(o * gate.double() * O.output_gate(gate.double(), torch.eye(H * dv, dtype=torch.float64)))
    got = [torch.zeros(T, H * dv) for T in lengths]
    for cu, lens, parts in Portions(lengths, sizes).steps():
        x = torch.full((cu[-1], D.up(D.a_at + rank)), 9.0)
        x[:, D.a_at:] = 0
        for (i, a, b), c in zip(parts, cu):
            q, k, v, gate, a1 = seqs[i]
            s = slice(c, c + b - a)
            x[s, :H * d], x[s, D.k_at:D.k_at + H * d] = q[a:b].reshape(b - a, -1), k[a:b].reshape(b - a, -1)
            x[s, D.v_at:D.v_at + H * dv], x[s, D.g_at:D.g_at + H * dv] = v[a:b].reshape(b - a, -1), gate[a:b]
            x[s, D.a_at:D.a_at + rank] = a1[a:b]
        out = ops.gated_linear(x.to(dtype).to(dev), D, W, 1e-5, state, slots[[p[0] for p in parts]].to(dev), cu, lens)
        out = out.float().cpu()
        assert bool((out[:, H * dv:] == 0).all())
        for (i, a, b), c in zip(parts, cu):
            got[i][a:b] = out[c:c + b - a, :H * dv]
    if gpu:
        from xfastertransformer_b200.ops import native
        native.Workspace.get(dev).check_status()
    for i, (x, w) in enumerate(zip(got, want)):
        e = (x.double() - w).abs().amax(-1) / w.abs().max()
        assert bool((e <= tol).all()), f"sequence {i}: token {int(e.argmax())} of {len(e)} is off by {float(e.max()):.3g}"
    untouched = [s for s in range(n + 2) if s not in slots.tolist()]
    assert bool((state[untouched] == 50.0).all())


def head_prep(dev, dtype, tol, hq, hkv, d, padded, taps, lengths, sizes, rot=None, norm=True):
    """Convolution, norm, rotation and append over unequal portions; every tap weighs about as much, so a state that is one
    token off, or not zero before the first token, shows."""
    from xfastertransformer_b200.ops import reference as R
    g = torch.Generator().manual_seed(d * 11 + taps)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    C = (hq + hkv) * d
    conv = 0.6 + 0.5 * r(C, taps) if taps else None
    qn, kn = 1 + 0.3 * r(d), 1 + 0.3 * r(d)
    prep = ops.HeadPrep(hq, hkv, d, padded, conv.t().contiguous().to(dev) if taps else None, qn.to(dev) if norm else None,
                        kn.to(dev) if norm else None)
    tab = None
    if rot:
        sc = rot.get("scaling")
        tab = R.rope_table(2000, rot["dims"], rot["base"], "banded", sc["factor"], sc["original"], sc["high"], sc["low"],
                           angle_dtype=torch.float64) if sc else R.rope_table(2000, rot["dims"], rot["base"], angle_dtype=torch.float64)
        tab = tab.to(dev)
    n = len(lengths)
    state = torch.full((n + 1, max(taps - 1, 0), C), 50.0, dtype=dtype, device=dev) if taps > 1 else None
    slot_of = torch.randperm(n + 1, generator=g)[:n].int()
    us = [r(T, C) for T in lengths]
    nb = sum((T + 63) // 64 for T in lengths) + 1
    place = torch.randperm(nb * 64, generator=g)
    where = [place[sum(lengths[:i]):sum(lengths[:i + 1])] for i in range(n)]
    kc, vc = (torch.full((nb, hkv, 64, padded), 7.0, dtype=dtype, device=dev) for _ in range(2))
    qs = [torch.zeros(T, hq, padded) for T in lengths]
    for cu, lens, parts in Portions(lengths, sizes).steps():
        x = torch.cat([us[i][a:b] for i, a, b in parts])
        wide = C + (-C % 8) + 8
        x = torch.cat([x, torch.full((x.shape[0], wide - C), 99.0)], 1).to(dtype).to(dev)
        pos = torch.cat([torch.arange(a, b) for _, a, b in parts]).int().to(dev)
        slots = torch.cat([where[i][a:b] for i, a, b in parts]).int().to(dev)
        q = ops.head_prep(x, prep, 1e-4, pos, tab, rot["dims"] if rot else 0, kc, vc, slots, state,
                          slot_of[[p[0] for p in parts]].to(dev), cu, lens).float().cpu()
        for (i, a, b), c in zip(parts, cu):
            qs[i][a:b] = q[c:c + b - a]
    if dev.type == "cuda":
        from xfastertransformer_b200.ops import native
        native.Workspace.get(dev).check_status()
    for i, T in enumerate(lengths):
        y = O.short_conv(us[i].double(), conv.double()) if taps else us[i].double()
        wq, wv = y[:, :hq * d].view(T, hq, d), y[:, hq * d:].view(T, hkv, d)
        wk = wv
        if norm:
            wq, wk = O.rms_norm(wq, qn.double(), 1e-4), O.rms_norm(wv, kn.double(), 1e-4)
        wq, wk = O.rotate(wq, list(range(T)), rot), O.rotate(wk, list(range(T)), rot)
        b, o = where[i] // 64, where[i] % 64
        for got, want, what in ((qs[i], wq, "queries"), (kc.float().cpu()[b, :, o], wk, "keys"), (vc.float().cpu()[b, :, o], wv, "values")):
            e = (got[..., :d].double() - want).abs().amax(dim=(-1, -2)) / want.abs().max()
            assert bool((e <= tol).all()), f"{what} of sequence {i}: token {int(e.argmax())} of {T} is off by {float(e.max()):.3g}"
            assert bool((got[..., d:] == 0).all()), f"{what}: padding"
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, C), us[i]])[-(taps - 1):]
            m = min(taps - 1, T)                          # rows before the first token are never read
            assert torch.equal(state[int(slot_of[i])].float().cpu()[-m:], tail[-m:]), f"state of sequence {i}"


def residual_extras(dev, H, dtype, tol):
    """The factor on what joins the residual stream, the vector added to every row, and the stream itself as the output."""
    g = torch.Generator().manual_seed(H)
    HP = (H + 7) // 8 * 8 if dev.type == "cuda" else H
    wide = lambda t: torch.cat([t, torch.zeros(*t.shape[:-1], HP - H, dtype=t.dtype)], -1).to(dev).contiguous()
    x, y, w, v = torch.randn(7, H, generator=g), torch.randn(7, H, generator=g).to(dtype), torch.randn(H, generator=g), torch.randn(H, generator=g)
    table, ids = torch.randn(11, H, generator=g).bfloat16(), torch.tensor([2, 10, 0], dtype=torch.int32)
    d = lambda t: t.double()
    gain = (w.to(dev), None)
    ht = tol if dtype == torch.float32 else 6e-3

    def close(got, want, t):
        assert float((got[:, :H].double().cpu() - want).abs().max() / want.abs().max()) <= t
        assert bool((got[:, H:] == 0).all())
    a, h = ops.residual_norm(wide(x), wide(y), gain, gain, 1e-3, "rms", h_dtype=dtype, mult=0.3, add=v.to(dev))
    want = d(x) + 0.3 * O.rms_norm(d(y), d(w), 1e-3) + d(v)
    close(a, want, tol)
    close(h, O.rms_norm(want, d(w), 1e-3), ht)
    a, h = ops.residual_norm(wide(x), wide(y), None, None, 1e-3, "rms", h_dtype=dtype, mult=-1.7, raw=True)
    close(a, d(x) - 1.7 * d(y), tol)
    assert torch.equal(h, a.to(dtype))
    a, h = ops.residual_norm(None, None, None, gain, 1e-3, "rms", h_dtype=dtype, ids=ids.to(dev), table=wide(table), embed_scale=3.0, add=v.to(dev))
    close(a, d(table)[ids.long()] * 3 + d(v), tol)
    a, h = ops.residual_norm(wide(x), None, None, gain, 1e-3, "rms", h_dtype=dtype, add=v.to(dev))
    close(h, O.rms_norm(d(x) + d(v), d(w), 1e-3), ht)


def linear_times(dev, dtype, tol, T, K, N):
    """gelu(x W^T) times rows that are a column range of a wider table."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T + N)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    x, w, e = r(T, K), (r(N, K) * 2 / K ** 0.5).bfloat16().float(), r(T, 3 * N)
    W = make_linear(w.to(dev), "bf16" if dtype == torch.bfloat16 else "fp32")
    got = ops.linear(x.to(dtype).to(dev), W, act="gelu_tanh", times=e.to(dtype).to(dev)[:, N:2 * N])
    want = O.gelu_tanh(x.double() @ w.double().T) * e[:, N:2 * N].double()
    err = float((got.double().cpu() - want).abs().max() / want.abs().max())
    assert err <= tol, f"{T} x {K} x {N}: {err:.3g}"


def grouped_route(dev, E, top, groups, T=60):
    """Choice with corrections (also such that choice scores are negative), weights without them and not renormalised; among
    groups, and among all."""
    g = torch.Generator().manual_seed(E + top)
    z = torch.randn(T, E, generator=g) * 3
    for shift in (0.0, -4.0):
        c = torch.randn(E, generator=g) * 0.7 + shift
        wi, ww = O.grouped_router(z.double(), c.double(), top, 1.9, dict(zip(("count", "keep"), groups)) if groups else None)
        count, keep = groups or (1, 1)
        idx, w = ops.route(z.to(dev), "deepseek", top, c.to(dev), count, keep, 1.9, False, "sigmoid")
        order, worder = idx.cpu().long().sort(-1), wi.sort(-1)
        assert torch.equal(order.values, worder.values), f"{top} of {E} in {groups}, corrections around {shift}"
        e = (w.cpu().double().gather(1, order.indices) - ww.gather(1, worder.indices)).abs().max()
        assert float(e) < 1e-5


def gated_experts(dev, dtype, tol, T, E, top, ff, width=72, groups=None):
    """Sigmoid-scored experts with a gate product: router, plan, products and weighted sum."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T * 13 + E)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    h = r(T, width)
    W = {"embed": torch.zeros(1, width), "l0.mlp.router": (r(E, width) * 2 / width ** 0.5).bfloat16().float(), "l0.mlp.correction": r(E)}
    for e in range(E):
        for n, (o, i) in dict(gate=(ff, width), up=(ff, width), down=(width, ff)).items():
            W[f"l0.mlp.e{e}.{n}"] = (r(o, i) * 1.5 / i ** 0.5).bfloat16().float()
    f = {"router": {"experts": E, "top": top, "scale": 0.8}}
    if groups:
        f["router"]["groups"] = dict(zip(("count", "keep"), groups))
    want = O.grouped_experts(h.double(), f, {k: v.double() for k, v in W.items()}, "l0")
    kind = "bf16" if dtype == torch.bfloat16 else "fp32"
    lin = lambda *n: make_linear(torch.cat([W["l0.mlp." + x] for x in n]).to(dev), kind)
    x = h.to(dtype).to(dev)
    idx, w = ops.route(ops.linear(x, lin("router"), out_dtype=torch.float32), "deepseek", top, W["l0.mlp.correction"].to(dev),
                       *(groups or (1, 1)), 0.8, False, "sigmoid")
    got = ops.moe_experts(x, idx, w, [(lin(f"e{e}.gate", f"e{e}.up"), lin(f"e{e}.down")) for e in range(E)], "silu", 0, gated=True)
    e = float((got.double().cpu() - want).abs().max() / want.abs().max())
    assert e <= tol, f"{T} tokens, {top} of {E}: {e:.3g}"


# ------------------------------------------------------------------------------------------ Dagezen's mechanisms
def time_mix(dev, dtype, tol, H, d, rank, lengths, sizes, around=-1.5, spread=1.5, one_gain=False):
    """As `gated_linear`, with decays exp(-exp(z)) and a bonus for the current token.  The first channel of every head hardly decays,
    and one token's key owns it; the bonus differs from one by much, so a token that reads itself through the state shows."""
    g = torch.Generator().manual_seed(d * 5 + rank)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    gpu = dev.type == "cuda"
    D = ops.LinearDims(H, d, d, rank, 8 if gpu else 1)
    a2 = (r(H * d, rank) * spread / rank ** 0.5).to(dtype).float()
    bias, gain, u = around + r(H * d), 1 + 0.2 * r(H * d), (2 + 0.5 * r(H, d)).abs()
    bias[::d] = -12.0
    a2[::d] = 0
    a2p = torch.zeros(H * d, D.up(rank))
    a2p[:, :rank] = a2
    W = ops.LinearWeights(a2p.to(dtype).to(dev).contiguous(), bias.to(dev), 1.0, gain.to(dev), 1.0, u.to(dev), 0.6)
    n = len(lengths)
    state = torch.full((n + 2, H, d, d), 50.0, device=dev)
    slots = torch.randperm(n + 2, generator=g)[:n].int()
    seqs, want = [], []
    for T in lengths:
        q, k, v, gate, a1 = r(T, H, d), r(T, H, d), r(T, H, d), r(T, H * d), r(T, rank)
        k = ((k + q) / d ** 0.25).to(dtype).float()
        q[:, :, 0], k[:, :, 0] = 4.0, 0.0
        if T > 5:
            k[5, :, 0] = 4.0
        seqs.append((q, k, v, gate, a1))
        w = torch.exp(-torch.exp(a1.double() @ a2.double().T + bias.double()))
        o = O.time_mix(q.double(), k.double(), v.double(), w.view(T, H, d), u.double())
        o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-5)
        want.append(0.6 * o.reshape(T, -1) * gain.double() * O.silu(gate.double()))
    got = [torch.zeros(T, H * d) for T in lengths]
    for cu, lens, parts in Portions(lengths, sizes).steps():
        x = torch.full((cu[-1], D.up(D.a_at + rank)), 9.0)
        x[:, D.a_at:] = 0
        for (i, a, b), c in zip(parts, cu):
            s = slice(c, c + b - a)
            for at, t in zip((0, D.k_at, D.v_at, D.g_at), seqs[i]):
                x[s, at:at + H * d] = t[a:b].reshape(b - a, -1)
            x[s, D.a_at:D.a_at + rank] = seqs[i][4][a:b]
        wide = torch.full((cu[-1], 16 + D.up(H * d)), 7.0, dtype=dtype, device=dev)        # the result is a part of wider rows
        ops.gated_linear(x.to(dtype).to(dev), D, W, 1e-5, state, slots[[p[0] for p in parts]].to(dev), cu, lens, out=wide[:, 16:])
        assert bool((wide[:, :16] == 7).all()) and bool((wide[:, 16 + H * d:] == 0).all())
        out = wide[:, 16:].float().cpu()
        for (i, a, b), c in zip(parts, cu):
            got[i][a:b] = out[c:c + b - a, :H * d]
    _status(dev)
    for i, (x, w) in enumerate(zip(got, want)):
        e = (x.double() - w).abs().amax(-1) / w.abs().max()
        assert bool((e <= tol).all()), f"sequence {i}: token {int(e.argmax())} of {len(e)} is off by {float(e.max()):.3g}"
    untouched = [s for s in range(n + 2) if s not in slots.tolist()]
    assert bool((state[untouched] == 50.0).all())


def _status(dev):
    if dev.type == "cuda":
        from xfastertransformer_b200.ops import native
        native.Workspace.get(dev).check_status()


def token_shift(dev, dtype, lengths, sizes, width=72, n_mix=5):
    """Mixes with the token before, across portions and at a sequence's start, over states that hold garbage."""
    g = torch.Generator().manual_seed(width + n_mix)
    mu = torch.randn(n_mix, width, generator=g)
    n = len(lengths)
    state = torch.full((n + 1, width), 50.0, device=dev)
    slots = torch.randperm(n + 1, generator=g)[:n].int()
    xs = [torch.randn(T, width, generator=g) for T in lengths]
    for cu, lens, parts in Portions(lengths, sizes).steps():
        x = torch.cat([xs[i][a:b] for i, a, b in parts]).to(dev)
        got = ops.token_shift(x, mu.to(dev), state, slots[[p[0] for p in parts]].to(dev), cu, lens, dtype).float().cpu()
        want = torch.cat([(xs[i][:, None] + (O.shifted(xs[i]) - xs[i])[:, None] * mu).reshape(-1, n_mix * width)[a:b] for i, a, b in parts])
        assert float((got - want).abs().max()) <= (1e-5 if dtype == torch.float32 else 0.08)
    _status(dev)
    for i, x in enumerate(xs):
        assert torch.equal(state[int(slots[i])].cpu(), x[-1])


def state_space(dev, dtype, tol, H, P, N, G, parts_n, taps, lengths, sizes, dt_around=-1.0, rate_around=0.0):
    """Batches of unequal portions over garbage states.  Head 0 hardly decays, and one token, 5 places in, drives it far harder than
    the others: it must still be there at the end."""
    g = torch.Generator().manual_seed(P * 3 + N)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    gpu = dev.type == "cuda"
    D = ops.StateDims(H, N, P, G, parts_n, taps, 8 if gpu else 1)
    C_, inner = D.channels, D.inner
    conv, cb = (0.5 + 0.4 * r(C_, taps)), 0.3 * r(C_)
    dtb, rate, skip, gain = dt_around + r(H), torch.exp(rate_around + r(H)), 1 + 0.5 * r(H), 1 + 0.2 * r(inner)
    dtb[0], rate[0] = -2.0, 1e-4
    f = lambda t: t.float().contiguous().to(dev)
    W = ops.StateWeights(f(conv.t()), f(cb), f(dtb), f(rate), f(skip), f(gain))
    n = len(lengths)
    state = torch.full((n + 2, H, N, P), 50.0, device=dev)
    cstate = torch.full((n + 2, taps - 1, C_), 50.0, dtype=dtype, device=dev) if taps > 1 else None
    slots = torch.randperm(n + 2, generator=g)[:n].int()
    seqs, want = [], []
    for T in lengths:
        z, u, dt = r(T, inner), r(T, C_), r(T, H)
        if T > 5:
            dt[5, 0] = 6.0
        seqs.append((z, u, dt))
        c = O.silu(O.short_conv(u.double(), conv.double()) + cb.double()).to(dtype).double()         # rows of the activations' type
        y = O.state_space(c[:, :inner].reshape(T, H, P), c[:, inner:inner + G * N].reshape(T, G, N), c[:, inner + G * N:].reshape(T, G, N),
                          O.softplus(dt.double() + dtb.double()), torch.log(rate.double()), skip.double()).reshape(T, -1)
        want.append(O.grouped_rms(y * O.silu(z.double()), gain.double(), parts_n, 1e-5))
    got = [torch.zeros(T, inner) for T in lengths]
    for cu, lens, parts in Portions(lengths, sizes).steps():
        x = torch.full((cu[-1], D.row + 8), 9.0)
        for (i, a, b), c in zip(parts, cu):
            z, u, dt = seqs[i]
            s = slice(c, c + b - a)
            x[s, :inner], x[s, D.x_at:D.x_at + C_], x[s, D.dt_at:D.dt_at + H] = z[a:b], u[a:b], dt[a:b]
        out = ops.state_space(x.to(dtype).to(dev), D, W, 1e-5, state, cstate, slots[[p[0] for p in parts]].to(dev), cu, lens).float().cpu()
        assert bool((out[:, inner:] == 0).all())
        for (i, a, b), c in zip(parts, cu):
            got[i][a:b] = out[c:c + b - a, :inner]
    _status(dev)
    for i, (x, w) in enumerate(zip(got, want)):
        e = (x.double() - w).abs().amax(-1) / w.abs().max()
        assert bool((e <= tol).all()), f"sequence {i}: token {int(e.argmax())} of {len(e)} is off by {float(e.max()):.3g}"
        if taps > 1:
            u = seqs[i][1]
            tail, m = torch.cat([torch.zeros(taps - 1, C_), u])[-(taps - 1):], min(taps - 1, len(u))
            assert torch.equal(cstate[int(slots[i])].float().cpu()[-m:], tail[-m:]), f"state of sequence {i}"
    untouched = [s for s in range(n + 2) if s not in slots.tolist()]
    assert bool((state[untouched] == 50.0).all())


def _talking(dev, dtype, H, G, d, padded, talk, r1, r2, mult=1.0):
    one = lambda n: torch.ones(n, device=dev)
    return ops.TalkingHeads(H, G, d, padded, one(H * d), one(G * d), r1.float().to(dev), r2.float().to(dev), talk.float().contiguous().to(dev), mult,
                            8 if dev.type == "cuda" else 1)


def talking_run(dev, dtype, q, k, v, gate, D, scale, window, decode, start, extra=()):
    """ops.talking_attention of queries start .. T - 1, as one portion or as decode steps that share the pages; `extra` are the lengths
    of more portions, over the same pages, in the same batch."""
    T, H, d = q.shape
    pad = lambda t: torch.cat([t, torch.zeros(*t.shape[:2], D.padded - d)], -1)
    kp, bt = paged(pad(k).to(dtype))
    vp, _ = paged(pad(v).to(dtype))
    n = T - start
    rows, cu, lens = list(range(start, T)), [0, n], [T]
    if decode:
        cu, lens = list(range(n + 1)), [i + 1 for i in range(start, T)]
    for i, m in enumerate(extra):
        rows += range(T - i - m, T - i)
        cu, lens = cu + [cu[-1] + m], lens + [T - i]
    x = torch.full((len(rows), D.row), 3.0)
    x[:, D.gate_at:D.gate_at + H * D.padded] = pad(gate.view(T, H, d))[rows].reshape(len(rows), -1)
    wide = torch.full((len(rows), H * D.padded + 8), 7.0, dtype=dtype, device=dev)
    ops.talking_attention(pad(q)[rows].to(dtype).to(dev).contiguous(), x.to(dtype).to(dev), D, kp.to(dev), vp.to(dev),
                          bt.repeat(len(lens), 1).to(dev), cu, lens, scale, window, out=wide[:, :H * D.padded])
    _status(dev)
    assert bool((wide[:, H * D.padded:] == 7).all())
    return wide[:, :H * D.padded].float().cpu().view(-1, H, D.padded)[..., :d], rows


def talking_want(q, k, v, gate, talk, r1, r2, scale, window, mult):
    T, H, d = q.shape
    own = [h // (H // k.shape[1]) for h in range(H)]
    mask = {"size": window} if window else None
    w = torch.stack([O.masked_softmax(O.distance_scores(q[:, h].double(), k[:, own[h]].double(), scale, r1[h].double(), r2[h].double()), mask)
                     for h in range(H)])
    w = O.talking_heads(w, talk.double())
    a = torch.stack([w[h] @ v[:, own[h]].double() for h in range(H)], 1)
    return (a * torch.sigmoid(gate.double()).view(a.shape) * mult).float()


def talking_edges(dev, dtype, tol, H, G, d, padded, window, decode, T=200, start=100, extra=()):
    """One key stands out, for one head alone, at every distance that is special; that head's weight is mixed into the others with
    factors far from each other, so a head that is left out, mixed by the transpose, or applied to another head's values shows."""
    g = torch.Generator().manual_seed(window * 7 + H)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    q, k, v, gate = r(T, H, d) / 16, r(T, G, d), r(T, G, d), r(T, H * d)
    talk = (torch.eye(H) * 0.5 + torch.randn(H, H, generator=g)).bfloat16().float()
    r1, r2 = (0.6 + 0.3 * torch.rand(H, generator=g)).bfloat16().float(), torch.rand(H, generator=g).bfloat16().float()
    D = _talking(dev, dtype, H, G, d, padded, talk, r1, r2, 0.7)
    special = H // 2
    q[:, special, 0] = 4.0
    k[:, :, 0] = 0.0
    i = T - 30
    for j in sorted({i - window - 1, i - window, i - window + 1, 63, 64, 127, 128, 0, i}):
        if not 0 <= j < T:
            continue
        k2 = k.clone()
        k2[j, :, 0] = 6.0
        want = talking_want(q, k2, v, gate, talk, r1, r2, 1.0, window, 0.7)
        got, rows = talking_run(dev, dtype, q, k2, v, gate, D, 1.0, window, decode, start, extra)
        _close(got, want[rows], tol, f"window {window}, key {j}, {'decode' if decode else 'portion'}")


def talking_scores(dev, dtype, tol, H, G, d, padded, window, decode, T=150, start=0, scale=0.3, extra=()):
    """Unequal heads, a strong distance bias (also none at all, in every third head), scores that spread over many units."""
    g = torch.Generator().manual_seed(d + H)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    q, k, v, gate = 3 * r(T, H, d) / d ** 0.25, 3 * r(T, G, d) / d ** 0.25, r(T, G, d), 2 * r(T, H * d)
    talk = torch.randn(H, H, generator=g).bfloat16().float() / H ** 0.5
    talk = talk.bfloat16().float()
    r1, r2 = 2 * torch.rand(H, generator=g), 3 * torch.rand(H, generator=g)
    r1[::3] = 0.0
    D = _talking(dev, dtype, H, G, d, padded, talk, r1, r2)
    want = talking_want(q, k, v, gate, talk, r1, r2, scale, window, 1.0)
    got, rows = talking_run(dev, dtype, q, k, v, gate, D, scale, window, decode, start, extra)
    _close(got, want[rows], tol, f"{H} heads of {d}, window {window}")


def talking_prep(dev, dtype, tol, hq, hkv, d, padded, T=37):
    """Norms over whole projections; the heads' sizes differ by much, so a norm per head shows.  Values are the keys before it."""
    g = torch.Generator().manual_seed(d + hq)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    D = _talking(dev, dtype, hq, hkv, d, padded, torch.eye(hq), torch.ones(hq), torch.ones(hq))
    qn, kn = 1 + 0.3 * r(hq * d), 1 + 0.3 * r(hkv * d)
    D.q_norm, D.k_norm = qn.to(dev), kn.to(dev)
    q = (r(T, hq, d) * (1 + torch.arange(hq))[:, None]).reshape(T, -1).to(dtype).float()
    k = (r(T, hkv, d) * (1 + 2 * torch.arange(hkv))[:, None]).reshape(T, -1).to(dtype).float()
    x = torch.full((T, D.row), 99.0)
    x[:, :hq * d], x[:, D.k_at:D.k_at + hkv * d] = q, k
    kc, vc = (torch.full((3, hkv, 64, padded), 7.0, dtype=dtype, device=dev) for _ in range(2))
    slots = torch.randperm(3 * 64, generator=g)[:T].int()
    got = ops.talking_prep(x.to(dtype).to(dev), D, 1e-3, kc, vc, slots.to(dev)).float().cpu()
    _status(dev)
    b, o = slots.long() // 64, slots.long() % 64
    wq, wk = O.rms_norm(q.double(), qn.double(), 1e-3).view(T, hq, d), O.rms_norm(k.double(), kn.double(), 1e-3).view(T, hkv, d)
    for a, w, t in ((got, wq, tol), (kc.float().cpu()[b, :, o], wk, tol), (vc.float().cpu()[b, :, o], k.double().view(T, hkv, d), 0.0)):
        assert float((a[..., :d].double() - w).abs().max() / w.abs().max()) <= t and bool((a[..., d:] == 0).all())
    free = torch.ones(3, 64, dtype=torch.bool)
    free[b, o] = False
    assert bool((kc.float().cpu().permute(0, 2, 1, 3)[free] == 7).all())


def latent_sinks(dev, dtype, tol, decode, T=150, H=20, d=32, rd=16, R=64, dv=48, start=40, extra=0):
    """Sinks from dominant to negligible and one gate value per head; a sink that is left out, counted per part or scaled shows."""
    q, c, kr, uk, uv, _ = _latent_layer(H, d, rd, R, dv, T, d + H, 0.5)
    g = torch.Generator().manual_seed(H)
    gate = (2 * torch.randn(T, H, generator=g)).to(dtype).float()
    sinks = torch.linspace(8.0, -6.0, H)
    s, v = O.latent_scores_and_values(q.double(), c.double(), kr.double(), uk.double(), uv.double(), 0.4, rd)
    want = torch.stack([O.sink_softmax(s[h], sinks[h].double()) @ v[:, h] for h in range(H)], 1) * torch.sigmoid(gate.double())[:, :, None]
    got = latent_run(dev, dtype, q, c, kr, uk, uv, gate, 0.4, 0, decode, start, extra, sinks=sinks.to(dev))
    rows = list(range(start, T)) + [t for e in range(extra) for t in (T - 2 - e, T - 1 - e)]
    for h in range(H):                                    # every head on its own scale
        _close(got[:, h:h + 1], want[rows][:, h:h + 1].float(), tol, f"head {h}, sink {float(sinks[h]):.1f}")


def sum_norm(dev, H, dtype, tol, T=9):
    """x = norm(alpha x + y) with a bias; the stream and the next input are the same, or one more norm follows on some rows."""
    g = torch.Generator().manual_seed(H)
    HP = (H + 7) // 8 * 8 if dev.type == "cuda" else H
    wide = lambda t: torch.cat([t, torch.zeros(*t.shape[:-1], HP - H, dtype=t.dtype)], -1).to(dev).contiguous()
    x, y = torch.randn(T, H, generator=g) + 2, torch.randn(T, H, generator=g).to(dtype)
    w, b, w2, b2 = (torch.randn(H, generator=g) for _ in range(4))
    post, nxt = (w.to(dev), b.to(dev)), (w2.to(dev), b2.to(dev))
    d = lambda t: t.double()
    want = O.layer_norm_bias(2.5 * d(x) + d(y), d(w), d(b), 1e-2)
    a, h = ops.residual_norm(wide(x), wide(y), post, None, 1e-2, "layer", h_dtype=dtype, carry=2.5, post_sum=True, raw=True)
    assert float((a[:, :H].double().cpu() - want).abs().max()) <= tol * float(want.abs().max()) and bool((a[:, H:] == 0).all())
    assert torch.equal(h, a.to(dtype))
    rows = torch.tensor([3, 0, T - 1], dtype=torch.int32, device=dev)
    a, h = ops.residual_norm(wide(x), wide(y), post, nxt, 1e-2, "layer", rows=rows, h_dtype=dtype, keep_x=False, carry=2.5, post_sum=True)
    want = O.layer_norm_bias(want, d(w2), d(b2), 1e-2)[rows.long().cpu()]
    assert a is None
    assert float((h[:, :H].double().cpu() - want).abs().max()) <= (tol if dtype == torch.float32 else 6e-3) * float(want.abs().max())


def clamped_gate(dev, dtype, tol, T, K, N, limit):
    """Values on both sides of every limit; the up value's lower limit and the gate's missing one show."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T + N)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    x, w, b = r(T, K), (r(2 * N, K) * 2 / K ** 0.5).bfloat16().float(), torch.randn(2 * N, generator=g)
    W = make_linear(w.to(dev), "bf16" if dtype == torch.bfloat16 else "fp32")
    got = ops.linear_gated(x.to(dtype).to(dev), W, "clamped", b.to(dev), limit)
    y = x.double() @ w.double().T + b.double()
    gt, up = y[:, :N].clamp(max=limit), y[:, N:].clamp(-limit, limit)
    want = gt / (1 + torch.exp(-1.702 * gt)) * (up + 1)
    assert float((got.double().cpu() - want).abs().max() / want.abs().max()) <= tol


def activations(dev, dtype, tol, T, K, N):
    """gelu with the error function, tanh, and the tanh cap of logits (fp32 rows)."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T + K)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    x, w = r(T, K), (r(N, K) * 2 / K ** 0.5).bfloat16().float()
    W = make_linear(w.to(dev), "bf16" if dtype == torch.bfloat16 else "fp32")
    y, xd = x.double() @ w.double().T, x.to(dtype).to(dev)
    for act, want in (("gelu_erf", O.gelu(y)), ("tanh", torch.tanh(y))):
        got = ops.linear(xd, W, act=act)
        assert float((got.double().cpu() - want).abs().max() / want.abs().max()) <= tol, act
    got = ops.linear(xd, W, act="softcap", res_scale=1.7, out_dtype=torch.float32)
    assert got.dtype == torch.float32 and float((got.double().cpu() - 1.7 * torch.tanh(y / 1.7)).abs().max()) <= (1e-5 if dtype == torch.float32 else 1e-4)
    rows = torch.full((T, N + 24), 7.0, dtype=dtype, device=dev)
    ops.linear(xd, W, act="tanh", out=rows[:, 16:])
    assert bool((rows[:, :16] == 7).all()) and bool((rows[:, 16 + N:] == 7).all())
    assert float((rows[:, 16:16 + N].double().cpu() - torch.tanh(y)).abs().max()) <= tol


def linear_parts(dev, dtype, tol, T, K, N, n=4):
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T + N)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    x, w = r(T, (n + 1) * K), (r(n * N, K) * 2 / K ** 0.5).bfloat16().float()
    W = make_linear(w.to(dev), "bf16" if dtype == torch.bfloat16 else "fp32")
    rows = torch.full((T, n * N + 16), 7.0, dtype=dtype, device=dev)
    ops.linear_parts(x.to(dtype).to(dev)[:, :n * K], W, n, rows)
    want = torch.cat([x[:, i * K:(i + 1) * K].double() @ w[i * N:(i + 1) * N].double().T for i in range(n)], 1)
    assert float((rows[:, :n * N].double().cpu() - want).abs().max() / want.abs().max()) <= tol and bool((rows[:, n * N:] == 7).all())


def chosen_experts(dev, dtype, tol, T, E, top, ff, width=72):
    """Experts weighted by the softmax over the chosen logits, a bias in the router, gelu with the error function, no gate."""
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(T * 13 + E)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    h = r(T, width)
    W = {"embed": torch.zeros(1, width), "l0.mlp.router": (r(E, width) * 2 / width ** 0.5).bfloat16().float(), "l0.mlp.router.b": 2 * r(E)}
    for e in range(E):
        for n, (o, i) in dict(up=(ff, width), down=(width, ff)).items():
            W[f"l0.mlp.e{e}.{n}"] = (r(o, i) * 1.5 / i ** 0.5).bfloat16().float()
    want = O.gelu_experts(h.double(), {"router": {"experts": E, "top": top}}, {k: v.double() for k, v in W.items()}, "l0")
    kind = "bf16" if dtype == torch.bfloat16 else "fp32"
    lin = lambda n: make_linear(W["l0.mlp." + n].to(dev), kind)
    x = h.to(dtype).to(dev)
    idx, w = ops.route(ops.linear(x, lin("router"), W["l0.mlp.router.b"].to(dev), out_dtype=torch.float32), "mixtral", top)
    got = ops.moe_experts(x, idx, w, [(lin(f"e{e}.up"), lin(f"e{e}.down")) for e in range(E)], "gelu_erf", 0, gated=False)
    e = float((got.double().cpu() - want).abs().max() / want.abs().max())
    assert e <= tol, f"{T} tokens, {top} of {E}: {e:.3g}"
