"""A plain, slow implementation of the layered designs (Kafipel, Vepivik, Botusun, Dagezen), one function per mechanism, for the tests to
compare against.

It works on one whole sequence at a time, without a cache, in the precision of the tensors it is given (tests use fp64
or fp32), straight from the equations; nothing here is shared with the package.

`cfg` is the dictionary of a ``config.json``; `W` maps tensor names to tensors.
"""
import json
import math
import os
import struct

import torch


def layer_norm(x, w, eps):
    mu = x.sum(-1, keepdim=True) / x.shape[-1]
    d = x - mu
    var = (d * d).sum(-1, keepdim=True) / x.shape[-1]
    return d / torch.sqrt(var + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps) * w


def banded(f, sc):
    """A frequency scaled by wavelength: short waves keep it, long waves are slowed by the factor, with a ramp between."""
    wave = 2 * math.pi / f
    if wave < sc["original"] / sc["high"]:
        return f
    if wave > sc["original"] / sc["low"]:
        return f / sc["factor"]
    s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
    return (1 - s) * f / sc["factor"] + s * f


def rotary_frequencies(rot):
    """(frequency of each pair, factor on cosine and sine)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    if "low" in sc:
        return [banded(fi, sc) for fi in f], 1.0

    def dim_of(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = (i - lo) / max(hi - lo, 0.001)
        ramp = min(max(ramp, 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, interleaved=False):
    """x [T, heads, dim]: dimension i < dims/2 turns together with dimension i + dims/2, or, interleaved, dimension 2i with
    dimension 2i + 1."""
    if not rot:
        return x
    f, m = rotary_frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for i in range(half):
        a = [p * f[i] for p in positions]
        c = torch.tensor([math.cos(t) * m for t in a], dtype=x.dtype)[:, None]
        s = torch.tensor([math.sin(t) * m for t in a], dtype=x.dtype)[:, None]
        iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        u, v = x[:, :, iu], x[:, :, iv]
        y[:, :, iu] = u * c - v * s
        y[:, :, iv] = v * c + u * s
    return y


def sees(i, j, mask):
    """Whether position i attends to position j."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


_VISIBLE = {}


def visible(T, mask):
    """The table of `sees` for one sequence."""
    key = (T, tuple(sorted(mask.items())) if mask else None)
    if key not in _VISIBLE:
        _VISIBLE[key] = torch.tensor([[sees(i, j, mask) for j in range(T)] for i in range(T)])
    return _VISIBLE[key]


def attention(q, k, v, scale, softcap, mask, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv] (already rotated) -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    vis = visible(T, mask)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = torch.where(vis, s, torch.full_like(s, -math.inf))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (e / den) @ v[:, g]
    return out


def mixer(h, m, W, prefix, positions, kept):
    """Attention sublayer.  `kept` maps a layer index to its (keys after rotation, values)."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rotate((h @ W[prefix + ".mix.q"].T).view(T, H, d), positions, m.get("rot"))
    src = m.get("kv_from")
    if src is None:
        k = rotate((h @ W[prefix + ".mix.k"].T).view(T, G, d), positions, m.get("rot"))
        v = (h @ W[prefix + ".mix.v"].T).view(T, G, m["vdim"])
    else:
        k, v = kept[src]
    kept[int(prefix[1:])] = (k, v)
    sink = W.get(prefix + ".mix.sink")
    a = attention(q, k, v, m["scale"], m.get("softcap"), m.get("mask"), sink)
    return a.reshape(T, -1) @ W[prefix + ".mix.o"].T


def latent_scores_and_values(q, c, kr, uk, uv, scale, rot_dim):
    """Scores [H, T, T] (no mask) and values [T, H, vdim] from latents c [T, rank], shared rotated keys kr [T, rot_dim],
    queries q [T, H, dim + rot_dim] and the per-head matrices uk [H, dim, rank], uv [H, vdim, rank]."""
    H, d = uk.shape[:2]
    s = torch.stack([(q[:, h, :d] @ (c @ uk[h].T).T + q[:, h, d:] @ kr.T) * scale for h in range(H)])
    v = torch.stack([c @ uv[h].T for h in range(H)], 1)
    return s, v


def masked_softmax(s, mask):
    """Weights of the visible keys; s [..., T, T]."""
    vis = visible(s.shape[-1], mask)
    e = torch.where(vis, torch.exp(s - torch.where(vis, s, torch.full_like(s, -math.inf)).max(-1, keepdim=True).values), 0.0)
    return e / e.sum(-1, keepdim=True)


def latent_attention(q, c, kr, uk, uv, scale, mask):
    """-> [T, H, vdim]"""
    s, v = latent_scores_and_values(q, c, kr, uk, uv, scale, kr.shape[1])
    return torch.stack([masked_softmax(s[h], mask) @ v[:, h] for h in range(s.shape[0])], 1)


def latent_mixer(h, m, W, prefix, positions, kept, eps):
    """Latent attention sublayer.  `kept` maps a layer index to its (latents after the norm, shared key part after rotation)."""
    T, H, d, rd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    P = prefix + ".mix."
    q = (h @ W[P + "q"].T).view(T, H, d + rd).clone()
    q[:, :, d:] = rotate(q[:, :, d:], positions, m["rot"], interleaved=True)
    if m.get("kv_from") is None:
        kv = h @ W[P + "dkv"].T
        c = rms_norm(kv[:, :R], W[P + "dkv.norm"], eps)
        kr = rotate(kv[:, None, R:], positions, m["rot"], interleaved=True)[:, 0]
    else:
        c, kr = kept[m["kv_from"]]
    kept[int(prefix[1:])] = (c, kr)
    a = latent_attention(q, c, kr, W[P + "uk"].view(H, d, R), W[P + "uv"].view(H, m["vdim"], R), m["scale"], m.get("mask"))
    a = a.reshape(T, -1) * output_gate(h, W[P + "g"])
    return a @ W[P + "o"].T


def output_gate(h, wg):
    return 1 / (1 + torch.exp(-(h @ wg.T)))


def router(z, top):
    """Chosen experts [T, top] (best first) and their weights."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    idx = torch.argsort(s, -1, descending=True)[:, :top]
    w = torch.gather(s, 1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


def expert(h, up, down):
    u = h @ up.T
    u = torch.where(u > 0, u, torch.zeros_like(u))
    return (u * u) @ down.T


def experts(h, f, W, prefix):
    """Mixture of experts: the chosen experts' weighted outputs plus the shared expert's."""
    P = prefix + ".mlp."
    idx, w = router(h @ W[P + "router"].T, f["router"]["top"])
    out = torch.zeros(h.shape[0], W["embed"].shape[1], dtype=h.dtype)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            out[t] += we * expert(h[t:t + 1], W[P + f"e{e}.up"], W[P + f"e{e}.down"])[0]
    if f.get("shared"):
        out = out + expert(h, W[P + "shared.up"], W[P + "shared.down"])
    return out


def grouped_router(z, correction, top, scale, groups=None):
    """Chosen experts [T, top] (best first) and their weights: sigmoid scores choose with a correction added and weigh
    without it; with `groups` {count, keep} only experts of the groups with the best sum of two choice scores."""
    s = 1 / (1 + torch.exp(-z))
    choice = s + correction
    T, E = z.shape
    if groups:
        n = E // groups["count"]
        for t in range(T):
            score = [sum(sorted(choice[t, g * n:(g + 1) * n].tolist())[-2:]) for g in range(groups["count"])]
            best = sorted(range(groups["count"]), key=lambda g: -score[g])[:groups["keep"]]
            for e in range(E):
                if e // n not in best:
                    choice[t, e] = -math.inf
    idx = torch.argsort(choice, -1, descending=True)[:, :top]
    return idx, torch.gather(s, 1, idx) * scale


def gated_expert(h, gate, up, down):
    g = h @ gate.T
    return (g / (1 + torch.exp(-g)) * (h @ up.T)) @ down.T


def grouped_experts(h, f, W, prefix):
    P, r = prefix + ".mlp.", f["router"]
    idx, w = grouped_router(h @ W[P + "router"].T, W[P + "correction"], r["top"], r["scale"], r.get("groups"))
    out = torch.zeros(h.shape[0], W["embed"].shape[1], dtype=h.dtype)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            out[t] += we * gated_expert(h[t:t + 1], *(W[P + f"e{e}.{n}"] for n in ("gate", "up", "down")))[0]
    return out


def short_conv(u, w):
    """u [T, C], w [C, taps]: every channel's weighted sum of its last `taps` values, the newest one last."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def shared_kv_mixer(h, m, W, prefix, positions, eps):
    """Attention whose values are its keys: projections with biases, short convolutions, then a norm per head and rotation
    on queries and keys; the values are the convolved keys.  A sink of score 0 joins the softmax."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    P = prefix + ".mix."
    q, k = h @ W[P + "q"].T + W[P + "q.b"], h @ W[P + "k"].T + W[P + "k.b"]
    if m.get("conv"):
        q, k = short_conv(q, W[P + "q.conv"]), short_conv(k, W[P + "k.conv"])
    q, k = q.view(T, H, d), k.view(T, G, d)
    v = k
    q = rotate(rms_norm(q, W[P + "q.norm"], eps), positions, m.get("rot"))
    k = rotate(rms_norm(k, W[P + "k.norm"], eps), positions, m.get("rot"))
    a = attention(q, k, v, m["scale"], None, m.get("mask"), torch.zeros(H, dtype=h.dtype))
    return a.reshape(T, -1) @ W[P + "o"].T


def log_decay(z, tau):
    """log(sigmoid(z)^(1/tau))"""
    return torch.nn.functional.logsigmoid(z) / tau


def gated_linear(q, k, v, decay):
    """q, k, decay [T, H, d], v [T, H, dv] -> [T, H, dv]: per head S <- diag(decay) S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def linear_mixer(h, m, W, prefix, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    P = prefix + ".mix."
    q = (h @ W[P + "q"].T * d ** -0.5).view(T, H, d)
    k, v = (h @ W[P + "k"].T).view(T, H, d), (h @ W[P + "v"].T).view(T, H, dv)
    z = (h @ W[P + "a1"].T) @ W[P + "a2"].T + W[P + "a2.b"]
    o = gated_linear(q, k, v, torch.exp(log_decay(z, m["tau"])).view(T, H, d))
    o = rms_norm(o, W[P + "norm"], eps).reshape(T, -1)
    g = h @ W[P + "g"].T
    return (o * (g / (1 + torch.exp(-g)))) @ W[P + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def token_side(x, tokens, W, i, dim, eps):
    """What the token's own side embedding adds after layer i."""
    e = W["side.embed"][torch.tensor(tokens), i * dim:(i + 1) * dim]
    g = gelu_tanh(x @ W[f"l{i}.side.gate"].T) * e
    return rms_norm(g @ W[f"l{i}.side.proj"].T, W[f"l{i}.side.norm"], eps)


def layer_runs(cfg):
    """(layer, pass, first layer of a pass) in the order they run: the looped layers several times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, 0, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, 0, False) for i in range(a)] + [(i, t, i == a) for t in range(loop["times"]) for i in range(a, b)] + \
        [(i, 0, False) for i in range(b, n)]


def feed_forward(h, W, prefix):
    g, u = h @ W[prefix + ".mlp.gate"].T, h @ W[prefix + ".mlp.up"].T
    return (g / (1 + torch.exp(-g)) * u) @ W[prefix + ".mlp.down"].T


def forward(cfg, W, tokens, layers_out=None, dtype=torch.float64):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) collects the residual stream after every layer."""
    W = {n: (t.to(dtype) if t.is_floating_point() else t) for n, t in W.items()}
    run = {"Kafipel": _kafipel, "Vepivik": _vepivik, "Botusun": _botusun, "Dagezen": _dagezen}[cfg["architecture"]]
    return run(cfg, W, tokens, [] if layers_out is None else layers_out)


def _kafipel(cfg, W, tokens, layers_out):
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = W["embed"][torch.tensor(tokens)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        y = mixer(layer_norm(x, W[p + ".norm1"], eps), layer["mixer"], W, p, positions, kept)
        x = x + layer_norm(y, W[p + ".norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(layer_norm(x, W[p + ".norm2"], eps), W, p)
            x = x + layer_norm(y, W[p + ".norm2b"], eps)
        layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T


def _vepivik(cfg, W, tokens, layers_out):
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        h = rms_norm(x, W[p + ".norm1"], eps)
        if layer["type"] == "latent_attention":
            x = x + latent_mixer(h, layer["mixer"], W, p, positions, kept, eps)
        else:
            x = x + mixer(h, layer["mixer"], W, p, positions, kept)
        if layer.get("mlp"):
            x = x + experts(rms_norm(x, W[p + ".norm2"], eps), layer["mlp"], W, p)
        layers_out.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T


def _botusun(cfg, W, tokens, layers_out):
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    positions = list(range(len(tokens)))
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, t, begins in layer_runs(cfg):
        p, layer = f"l{i}", cfg["layers"][i]
        if begins:
            x = x + W["loop.step"][t]
        h = rms_norm(x, W[p + ".norm1"], eps)
        if layer["type"] == "gla":
            x = x + m * linear_mixer(h, layer["mixer"], W, p, eps)
        else:
            x = x + m * shared_kv_mixer(h, layer["mixer"], W, p, positions, eps)
        f = layer.get("mlp")
        if f:
            h = rms_norm(x, W[p + ".norm2"], eps)
            x = x + m * (feed_forward(h, W, p) if f["kind"] == "dense" else grouped_experts(h, f, W, p))
        if cfg.get("token_side"):
            x = x + m * token_side(x, tokens, W, i, cfg["token_side"]["dim"], eps)
        layers_out.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T


# ------------------------------------------------------------------------------------------ Dagezen
def layer_norm_bias(x, w, b, eps):
    return layer_norm(x, w, eps) + b


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0)


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (after the softplus) -> [T, H, P]: per head
    S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype)
    group = [h // (H // G) for h in range(H)]
    out = []
    for t in range(T):
        keep = torch.exp(-torch.exp(A_log) * dt[t])
        S = keep[:, None, None] * S + (dt[t][:, None] * B[t][group])[:, :, None] * x[t][:, None, :]
        out.append((S * C[t][group][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(out)


def grouped_rms(y, w, n, eps):
    """RMS norm of every row in `n` equal parts."""
    T = y.shape[0]
    parts = y.view(T, n, -1)
    return (parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)).reshape(T, -1) * w


def mamba_mixer(h, m, W, prefix, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    Q, inner = prefix + ".mix.", m["heads"] * m["vdim"]
    z, u, dt = torch.split(h @ W[Q + "in"].T, [inner, inner + 2 * G * N, H], 1)
    u = silu(short_conv(u, W[Q + "conv"]) + W[Q + "conv.b"])
    x, B, C = torch.split(u, [inner, G * N, G * N], 1)
    dt = softplus(dt + W[Q + "dt_bias"])
    y = state_space(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, W[Q + "A_log"], W[Q + "D"]).reshape(T, -1)
    return grouped_rms(y * silu(z), W[Q + "norm"], m["norm_groups"], eps) @ W[Q + "o"].T


def sink_softmax(s, sink):
    """Weights of the visible keys of one head with a score that has no key; s [T, T]."""
    vis = visible(s.shape[-1], None)
    s = torch.where(vis, s, torch.full_like(s, -math.inf))
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_sink_mixer(h, m, W, prefix, positions, eps):
    """Latent attention with a sink per head and one gate value per head."""
    T, H, d, rd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    P = prefix + ".mix."
    q = (h @ W[P + "q"].T).view(T, H, d + rd).clone()
    q[:, :, d:] = rotate(q[:, :, d:], positions, m["rot"], interleaved=True)
    kv = h @ W[P + "dkv"].T
    c = rms_norm(kv[:, :R], W[P + "dkv.norm"], eps)
    kr = rotate(kv[:, None, R:], positions, m["rot"], interleaved=True)[:, 0]
    s, v = latent_scores_and_values(q, c, kr, W[P + "uk"].view(H, d, R), W[P + "uv"].view(H, m["vdim"], R), m["scale"], rd)
    a = torch.stack([sink_softmax(s[n], W[P + "sink"][n]) @ v[:, n] for n in range(H)], 1)
    a = a * output_gate(h, W[P + "g"])[:, :, None]
    return a.reshape(T, -1) @ W[P + "o"].T


def distance_scores(q, k, scale, r1, r2):
    """Scores of one head with the bias r1 ln(1 + r2 distance) taken off (keys behind the query: no meaning)."""
    T = q.shape[0]
    i = torch.arange(T, dtype=q.dtype)
    return (q @ k.T) * scale - r1 * torch.log(1 + r2 * torch.clamp(i[:, None] - i[None, :], min=0))


def talking_heads(w, T_):
    """w [H, T, T] weights: head h gets sum_g T_[h, g] w[g]."""
    return torch.einsum("hg,gij->hij", T_, w)


def talking_mixer(h, m, W, P, eps):
    """Attention whose values are its keys (before the norm), normalised over the whole projection, with a distance bias and
    weights mixed between the heads.  -> before the output projection: [T, H * dim], gated."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ W[P + "q"].T, h @ W[P + "k"].T
    v = k.view(T, G, d)
    q, k = rms_norm(q, W[P + "q.norm"], eps).view(T, H, d), rms_norm(k, W[P + "k.norm"], eps).view(T, G, d)
    own = [n // (H // G) for n in range(H)]
    w = torch.stack([masked_softmax(distance_scores(q[:, n], k[:, own[n]], m["scale"], W[P + "r1"][n], W[P + "r2"][n]), m.get("mask"))
                     for n in range(H)])
    w = talking_heads(w, W[P + "talk"])
    a = torch.stack([w[n] @ v[:, own[n]] for n in range(H)], 1).reshape(T, -1)
    return (a * output_gate(h, W[P + "g"])) @ W[P + "o"].T


def shifted(h):
    """The previous token's row (zeros for the first)."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def time_mix(r, k, v, w, u):
    """r, k, w [T, H, d], v [T, H, d], u [H, d]: o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype)
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out)


def time_mixer(h, m, W, P, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    mix = {n: h + (shifted(h) - h) * W[P + "mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ W[P + n].T).view(T, H, d) for n in "rkv")
    gate = silu(mix["g"] @ W[P + "g"].T)
    w = torch.exp(-torch.exp(torch.tanh(mix["w"] @ W[P + "w1"].T) @ W[P + "w2"].T + W[P + "w0"]))
    o = time_mix(r, k, v, w.view(T, H, d), W[P + "u"])
    o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)).reshape(T, -1)
    return (o * W[P + "norm"] * gate) @ W[P + "o"].T


def parallel_mixer(h, m, W, prefix, eps):
    P = prefix + ".mix."
    return m["left_scale"] * talking_mixer(h, m["left"], W, P + "left.", eps) + \
        m["right_scale"] * time_mixer(h, m["right"], W, P + "right.", eps)


def clamped_feed_forward(h, f, W, prefix):
    P, lim = prefix + ".mlp.", f["limit"]
    g = torch.clamp(h @ W[P + "gate"].T + W[P + "gate.b"], max=lim)
    u = torch.clamp(h @ W[P + "up"].T + W[P + "up.b"], min=-lim, max=lim)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ W[P + "down"].T + W[P + "down.b"]


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def chosen_softmax(z, top):
    """Chosen experts [T, top] (best first) and the softmax over their logits alone."""
    idx = torch.argsort(z, -1, descending=True)[:, :top]
    e = torch.exp(torch.gather(z, 1, idx) - z.max(-1, keepdim=True).values)
    return idx, e / e.sum(-1, keepdim=True)


def gelu_experts(h, f, W, prefix):
    P = prefix + ".mlp."
    idx, w = chosen_softmax(h @ W[P + "router"].T + W[P + "router.b"], f["router"]["top"])
    out = torch.zeros(h.shape[0], W["embed"].shape[1], dtype=h.dtype)
    for e in range(f["router"]["experts"]):
        y = gelu(h @ W[P + f"e{e}.up"].T) @ W[P + f"e{e}.down"].T
        out = out + y * torch.where(idx == e, w, torch.zeros_like(w)).sum(-1, keepdim=True)
    return out


def _dagezen(cfg, W, tokens, layers_out):
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    positions = list(range(len(tokens)))
    x = W["embed"][torch.tensor(tokens)]
    norm = lambda v, n: layer_norm_bias(v, W[n], W[n + ".b"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer.get("mlp")
        if layer["type"] == "mamba2":
            y = mamba_mixer(x, m, W, p, eps)
        elif layer["type"] == "latent_attention":
            y = latent_sink_mixer(x, m, W, p, positions, eps)
        else:
            y = parallel_mixer(x, m, W, p, eps)
        x = norm(alpha * x + y, p + ".norm1")
        if f:
            y = clamped_feed_forward(x, f, W, p) if f["kind"] == "dense" else gelu_experts(x, f, W, p)
            x = norm(alpha * x + y, p + ".norm2")
        layers_out.append(x.clone())
    z = norm(x, "final.norm") @ W["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


# ------------------------------------------------------------------------------------------ small checkpoints
def attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, size=24, keep=3, rot_dims=16, base=10000.0, scaling=None,
                    scale=None, softcap=30.0, kv_from=None, ff=96, mask=True, rot=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale else dim ** -0.5}
    if softcap:
        m["softcap"] = softcap
    if mask:
        m["mask"] = {"size": size, "keep_first": keep}
    if rot:
        m["rot"] = {"dims": rot_dims, "base": base}
        if scaling:
            m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=96, vocab=210, eps=1e-5):
    return {"architecture": "Kafipel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def moe(ff=40, experts=6, top=2, shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared} if shared else None}


def window_layer(heads=4, kv_heads=2, dim=32, vdim=24, size=24, scale=None, mlp=None, mask=True):
    """Attention without rotation."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale else dim ** -0.5}
    if mask:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent_layer(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=40, size=24, base=10000.0, scaling=None, scale=None, kv_from=None,
                 mlp=None, mask=True):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": scale if scale else (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": base}}
    if scaling:
        m["rot"]["scaling"] = scaling
    if mask:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def vepivik(layers, width=96, vocab=210, eps=1e-5, scale=2.0):
    return {"architecture": "Vepivik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale}}


def botusun(layers, width=96, vocab=210, eps=1e-5, scale=2.0, mult=0.4, loop=None, side=None):
    """`loop`: (start, stop, times)."""
    cfg = {"architecture": "Botusun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "embedding": {"scale": scale}, "residual_mult": mult}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


def shared_kv_layer(heads=4, kv_heads=2, dim=32, size=24, rot_dims=16, base=10000.0, scaling=None, scale=None, conv=4, mlp=None,
                    mask=True, rot=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale else dim ** -0.5}
    if conv:
        m["conv"] = conv
    if mask:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot_dims, "base": base}
        if scaling:
            m["rot"]["scaling"] = scaling
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gla_layer(heads=2, dim=16, vdim=24, tau=8.0, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def grouped_moe(ff=40, experts=6, top=2, scale=1.3, groups=None):
    """`groups`: (count, keep)."""
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def mamba_layer(heads=4, vdim=16, state=24, groups=2, norm_groups=2, conv=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                                    "conv": conv}}


def sink_latent_layer(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=40, base=10000.0, scale=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": scale if scale else (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": base}}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel_layer(heads=4, kv_heads=2, dim=32, size=24, scale=None, right_heads=3, right_dim=16, scales=(0.7, 1.3), mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale else dim ** -0.5, "mask": {"size": size}}
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": {"heads": right_heads, "dim": right_dim},
                                                      "left_scale": scales[0], "right_scale": scales[1]}}


def clamped(ff=48, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def chosen_moe(ff=40, experts=6, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def dagezen(layers, width=96, vocab=210, eps=1e-5, alpha=2.0, cap=20.0):
    cfg = {"architecture": "Dagezen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "postln_alpha": alpha}
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


def random_weights(cfg, seed=0, gain=1.0):
    if cfg["architecture"] == "Botusun":
        return _botusun_weights(cfg, seed)
    if cfg["architecture"] == "Dagezen":
        return _dagezen_weights(cfg, seed)
    return _weights(cfg, seed, gain)


def _botusun_weights(cfg, seed):
    """As `_weights`.  The code that decides about experts is one per kind of router: a group's levels lie next to each other,
    so that the groups' order is as clear as the experts'; corrections move single experts to the front or to the back of
    their group, far enough that it shows."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / math.sqrt(i))).bfloat16()

    def vec(n, around=1.0, s=0.2):
        return (around + s * torch.randn(n, generator=g)).bfloat16()
    perm = lambda n: torch.randperm(n, generator=g)
    W = {"embed": (torch.randn(V, D, generator=g) / math.sqrt(D)).bfloat16(), "final.norm": vec(D)}
    code, used = {}, 0
    for layer in cfg["layers"]:
        if (layer.get("mlp") or {}).get("kind") == "moe":
            r = layer["mlp"]["router"]
            E, n = r["experts"], (r.get("groups") or {"count": 1})["count"]
            if (E, n) not in code:
                levels = ((torch.arange(E) - (E - 1) / 2) * 3.0 / math.sqrt(D)).view(n, E // n)
                rows = [torch.cat([levels[k][perm(E // n)] for k in perm(n)]) for _ in range(V)]
                W["embed"][:, used:used + E] = torch.stack(rows).bfloat16()
                code[E, n] = used
                used += E
    if cfg.get("loop"):
        W["loop.step"] = (torch.randn(cfg["loop"]["times"], D, generator=g) * 0.7 / math.sqrt(D) * cfg["embedding"]["scale"]).bfloat16()
        W["loop.step"][:, :used] = 0
    side = (cfg.get("token_side") or {}).get("dim")
    if side:
        W["side.embed"] = torch.randn(V, side * len(cfg["layers"]), generator=g).bfloat16()
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer.get("mlp")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        P = p + ".mix."
        W[p + ".norm1"] = vec(D)
        if layer["type"] == "gla":
            rank = (5, 16, 24, 33)[i % 4] if d <= 128 else 9
            W[P + "q"], W[P + "v"], W[P + "g"] = mat(H * d, D), mat(H * dv, D), mat(H * dv, D, 2.0)
            # keys akin to their queries: a first token whose key misses its query has an output of nothing but rounding,
            # which the norm behind it would blow up
            W[P + "k"] = (W[P + "q"].float() + 0.7 * mat(H * d, D).float()).bfloat16()
            W[P + "a1"], W[P + "a2"], W[P + "a2.b"] = mat(rank, D), mat(H * d, rank, 2.0), vec(H * d, 1.0, 2.0)
            W[P + "norm"] = vec(dv)
        else:
            for x, n in (("q", H), ("k", m["kv_heads"])):
                W[P + x], W[P + x + ".b"], W[P + x + ".norm"] = mat(n * d, D), vec(n * d, 0.0, 0.3), vec(d, 1.3)
                if m.get("conv"):
                    W[P + x + ".conv"] = vec(n * d * m["conv"], 0.4, 0.6).view(n * d, m["conv"])
        W[P + "o"] = mat(D, H * dv, 2.0)
        if f:
            W[p + ".norm2"] = vec(D)
            if f["kind"] == "moe":
                r = f["router"]
                E, n = r["experts"], (r.get("groups") or {"count": 1})["count"]
                at, per = code[E, n], E // n
                W[p + ".norm2"][at:at + E] = 1.0
                columns = torch.cat([k * per + perm(per) for k in perm(n)])     # experts of a group read a group of the code
                w = 0.001 * torch.randn(E, D, generator=g)
                w[:, at:at + E] = torch.eye(E)[columns]
                W[p + ".mlp.router"] = w.bfloat16()
                c = torch.zeros(E)
                for k in range(n):
                    c[k * per + int(perm(per)[0])] += 2.0
                    c[k * per + int(perm(per)[0])] -= 1.0 if per > 2 else 0.0
                W[p + ".mlp.correction"] = c.bfloat16()
            for x, ff in [(f".e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] if f["kind"] == "moe" else [("", f["ff"])]:
                W[p + f".mlp{x}.gate"], W[p + f".mlp{x}.up"], W[p + f".mlp{x}.down"] = mat(ff, D, 2.0), mat(ff, D, 2.0), mat(D, ff, 2.0)
        if side:
            W[p + ".side.gate"], W[p + ".side.proj"], W[p + ".side.norm"] = mat(side, D), mat(D, side), vec(D, 0.5)
    for n, t in W.items():
        if n.endswith((".mix.o", ".down", ".side.proj")):
            t[:used] = 0
    return W


def _dagezen_weights(cfg, seed):
    """As `_weights`.  The norms keep the code's order (one gain, no bias there, and about what
    the norm of the sum takes from it is given back); router biases are a part of its steps, so that
    they change the weights and no choice."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / math.sqrt(i))).bfloat16()

    def vec(n, around=0.0, s=0.2):
        return (around + s * torch.randn(n, generator=g)).bfloat16()
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if (l.get("mlp") or {}).get("kind") == "moe"], default=0)
    W = {"embed": torch.randn(V, D, generator=g).bfloat16()}
    if E:
        levels = (torch.arange(E) - (E - 1) / 2) * (4.0 / E)
        W["embed"][:, :E] = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(V)]).bfloat16()

    def norm(name):
        W[name], W[name + ".b"] = vec(D, 1.0), vec(D, 0.0, 0.3)
        if not name.startswith("final"):
            W[name][:E], W[name + ".b"][:E] = 1.6, 0.0
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer.get("mlp")
        P = p + ".mix."
        norm(p + ".norm1")
        if layer["type"] == "mamba2":
            H, n = m["heads"], m["heads"] * m["vdim"]
            c = n + 2 * m["groups"] * m["state"]
            W[P + "in"] = mat(n + c + H, D, 1.3)
            W[P + "conv"], W[P + "conv.b"] = vec(c * m["conv"], 0.4, 0.5).view(c, m["conv"]), vec(c, 0.2, 0.3)
            W[P + "dt_bias"], W[P + "A_log"], W[P + "D"], W[P + "norm"] = vec(H, -1.5, 1.5), vec(H, 0.0, 1.2), vec(H, 1.0, 0.5), vec(n, 1.0)
            W[P + "o"] = mat(D, n, 1.5)
        elif layer["type"] == "latent_attention":
            H = m["heads"]
            W[P + "q"] = mat(H * (m["dim"] + m["rot_dim"]), D, 1.6)
            W[P + "dkv"], W[P + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], D, 1.3), vec(m["kv_rank"], 1.0)
            W[P + "uk"], W[P + "uv"] = mat(H * m["dim"], m["kv_rank"], 1.6), mat(H * m["vdim"], m["kv_rank"])
            W[P + "sink"], W[P + "g"], W[P + "o"] = vec(H, 1.0, 1.0), mat(H, D, 2.0), mat(D, H * m["vdim"], 2.0)
        else:
            l, r = m["left"], m["right"]
            H, d = l["heads"], l["dim"]
            L = P + "left."
            W[L + "q"], W[L + "k"], W[L + "g"] = mat(H * d, D), mat(l["kv_heads"] * d, D), mat(H * d, D, 2.0)
            W[L + "q.norm"], W[L + "k.norm"] = vec(H * d, 1.5), vec(l["kv_heads"] * d, 1.5)
            W[L + "r1"], W[L + "r2"] = vec(H, 1.0, 0.5).abs(), vec(H, 0.3, 0.2).abs()
            W[L + "talk"] = (0.8 * torch.eye(H) + 0.4 * torch.randn(H, H, generator=g) / math.sqrt(H)).bfloat16()
            W[L + "o"] = mat(D, H * d, 2.0)
            R, H, d, rank = P + "right.", r["heads"], r["dim"], (5, 16, 24, 33)[i % 4] if r["dim"] <= 128 else 9
            for x in "rkvgw":
                W[R + "mu." + x] = vec(D, 0.5, 0.2) if x != "k" else (W[R + "mu.r"].float() + 0.05 * torch.randn(D, generator=g)).bfloat16()
            W[R + "r"], W[R + "v"], W[R + "g"] = mat(H * d, D, 1.5), mat(H * d, D), mat(H * d, D, 2.0)
            # keys akin to their queries: an output of nothing but rounding would be blown up by the norm behind it
            W[R + "k"] = (W[R + "r"].float() + 0.7 * mat(H * d, D).float()).bfloat16()
            W[R + "w1"], W[R + "w2"], W[R + "w0"] = mat(rank, D), mat(H * d, rank, 1.5), vec(H * d, -1.5, 1.5)
            W[R + "u"], W[R + "norm"], W[R + "o"] = vec(H * d, 1.0, 0.3).abs().view(H, d), vec(H * d, 1.0), mat(D, H * d, 1.5)
        if not f:
            continue
        norm(p + ".norm2")
        if f["kind"] == "moe":
            n = f["router"]["experts"]
            r = 0.001 * torch.randn(n, D, generator=g)
            r[:, :E] = 2.0 * torch.eye(E)[torch.randperm(E, generator=g)[:n]]
            W[p + ".mlp.router"] = r.bfloat16()
            W[p + ".mlp.router.b"] = (0.15 * (4.0 / E) * torch.randn(n, generator=g).clamp(-1.5, 1.5)).bfloat16()
            for e in range(n):
                W[p + f".mlp.e{e}.up"], W[p + f".mlp.e{e}.down"] = mat(f["expert"]["ff"], D, 1.5), mat(D, f["expert"]["ff"], 1.5)
        else:
            for x, (o, k) in dict(gate=(f["ff"], D), up=(f["ff"], D), down=(D, f["ff"])).items():
                W[p + f".mlp.{x}"], W[p + f".mlp.{x}.b"] = mat(o, k, 1.5), vec(o, 0.0, 0.3)
    for n, t in W.items():
        if n.endswith((".o", ".down", ".down.b")):
            t[:E] = 0
    return W


def _weights(cfg, seed, gain):
    """bf16-representable weights, scaled so that scores spread over several units and every mechanism matters.

    Experts: the first columns of the residual stream hold a code that the embedding alone writes, a permutation of equally
    spaced levels per token, and each router reads little else.  So every token has experts of its own, other ones in every
    layer, and no choice is close enough for rounding to turn it."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s * gain / math.sqrt(i))).bfloat16()

    def vec(n, around=1.0, s=0.2):
        return (around + s * torch.randn(n, generator=g)).bfloat16()

    D = cfg["width"]
    kafipel = cfg["architecture"] == "Kafipel"
    W = {"embed": torch.randn(cfg["vocab"], D, generator=g).bfloat16(), "final.norm": vec(D)}
    if kafipel:
        W["head"] = mat(cfg["vocab"], D)
    else:
        W["embed"] = (W["embed"].float() / math.sqrt(D)).bfloat16()
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if (l.get("mlp") or {}).get("kind") == "moe"], default=0)
    if E:
        levels = (torch.arange(E) - (E - 1) / 2) * 3.0 / math.sqrt(D)
        W["embed"][:, :E] = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(cfg["vocab"])]).bfloat16()
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        W[p + ".norm1"] = vec(D)
        if kafipel:
            W[p + ".norm1b"] = vec(D, 0.7)
        if layer["type"] == "latent_attention":
            W[p + ".mix.q"] = mat(m["heads"] * (m["dim"] + m["rot_dim"]), D, 1.6)
            if m.get("kv_from") is None:
                W[p + ".mix.dkv"] = mat(m["kv_rank"] + m["rot_dim"], D, 1.3)
                W[p + ".mix.dkv.norm"] = vec(m["kv_rank"])
            W[p + ".mix.uk"] = mat(m["heads"] * m["dim"], m["kv_rank"], 1.6)
            W[p + ".mix.uv"] = mat(m["heads"] * m["vdim"], m["kv_rank"])
            W[p + ".mix.g"] = mat(m["heads"] * m["vdim"], D, 2.0)
        else:
            W[p + ".mix.q"] = mat(m["heads"] * m["dim"], D, 1.6)
            if m.get("kv_from") is None:
                W[p + ".mix.k"] = mat(m["kv_heads"] * m["dim"], D, 1.6)
                W[p + ".mix.v"] = mat(m["kv_heads"] * m["vdim"], D)
            if kafipel:
                W[p + ".mix.sink"] = vec(m["heads"], 1.0, 1.0)
        W[p + ".mix.o"] = mat(D, m["heads"] * m["vdim"])
        f = layer.get("mlp")
        if not f:
            continue
        W[p + ".norm2"] = vec(D)
        if f["kind"] == "moe":
            n = f["router"]["experts"]
            r = 0.001 * torch.randn(n, D, generator=g)
            r[:, :E] = torch.eye(E)[torch.randperm(E, generator=g)[:n]]
            W[p + ".mlp.router"] = r.bfloat16()
            W[p + ".norm2"][:E] = 1.0
            for n, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + \
                    ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
                W[p + f".mlp.{n}.up"], W[p + f".mlp.{n}.down"] = mat(ff, D), mat(D, ff, 0.8)
        else:
            W[p + ".norm2b"] = vec(D, 0.7)
            W[p + ".mlp.gate"], W[p + ".mlp.up"], W[p + ".mlp.down"] = mat(f["ff"], D), mat(f["ff"], D), mat(D, f["ff"])
    for n, t in W.items():
        if E and (n.endswith(".mix.o") or n.endswith(".down")):
            t[:E] = 0
    return W


def write_checkpoint(path, cfg, W):
    """config.json and model.safetensors, written byte by byte (bf16)."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for n, t in W.items():
        b = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[n] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return path
