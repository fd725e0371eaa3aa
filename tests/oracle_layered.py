"""A plain, slow implementation of the Kafipel design, one function per mechanism, for the tests to compare against.

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


def rotary_frequencies(rot):
    """(frequency of each pair, factor on cosine and sine)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

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


def rotate(x, positions, rot):
    """x [T, heads, dim]: dimension i < dims/2 turns together with dimension i + dims/2."""
    if not rot:
        return x
    f, m = rotary_frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for i in range(half):
        a = [p * f[i] for p in positions]
        c = torch.tensor([math.cos(t) * m for t in a], dtype=x.dtype)[:, None]
        s = torch.tensor([math.sin(t) * m for t in a], dtype=x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * c - v * s
        y[:, :, i + half] = v * c + u * s
    return y


def sees(i, j, mask):
    """Whether position i attends to position j."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask["keep_first"]


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


def feed_forward(h, W, prefix):
    g, u = h @ W[prefix + ".mlp.gate"].T, h @ W[prefix + ".mlp.up"].T
    return (g / (1 + torch.exp(-g)) * u) @ W[prefix + ".mlp.down"].T


def forward(cfg, W, tokens, layers_out=None, dtype=torch.float64):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) collects the residual stream after every layer."""
    W = {n: (t.to(dtype) if t.is_floating_point() else t) for n, t in W.items()}
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
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T


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


def random_weights(cfg, seed=0, gain=1.0):
    """bf16-representable weights, scaled so that scores spread over several units and every mechanism matters."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s * gain / math.sqrt(i))).bfloat16()

    def vec(n, around=1.0, s=0.2):
        return (around + s * torch.randn(n, generator=g)).bfloat16()

    D = cfg["width"]
    W = {"embed": torch.randn(cfg["vocab"], D, generator=g).bfloat16(), "final.norm": vec(D),
         "head": mat(cfg["vocab"], D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        W[p + ".norm1"], W[p + ".norm1b"] = vec(D), vec(D, 0.7)
        W[p + ".mix.q"] = mat(m["heads"] * m["dim"], D, 1.6)
        if m.get("kv_from") is None:
            W[p + ".mix.k"] = mat(m["kv_heads"] * m["dim"], D, 1.6)
            W[p + ".mix.v"] = mat(m["kv_heads"] * m["vdim"], D)
        W[p + ".mix.sink"] = vec(m["heads"], 1.0, 1.0)
        W[p + ".mix.o"] = mat(D, m["heads"] * m["vdim"])
        if layer.get("mlp"):
            f = layer["mlp"]["ff"]
            W[p + ".norm2"], W[p + ".norm2b"] = vec(D), vec(D, 0.7)
            W[p + ".mlp.gate"], W[p + ".mlp.up"], W[p + ".mlp.down"] = mat(f, D), mat(f, D), mat(D, f)
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
