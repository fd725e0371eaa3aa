"""Scenarios of the layered decoder, run on CPU by test_layered_cpu.py and on a GPU by test_layered_gpu.py: the engine
against tests/oracle_layered.py.  Every function takes the dtype it runs the engine in; `tolerance` says how far logits
may be from the fp64 result (root mean square over the vocabulary, mean taken off, relative to the logits' spread)."""
import random

import torch

import oracle_layered as O
import xfastertransformer_b200 as xft
from xfastertransformer_b200.tools.trace_run import TraceRunner

YARN = {"factor": 3.0, "original": 96, "fast": 12.0, "slow": 1.0}

# name -> config; none of the sizes repeat within a config unless that is the point
CONFIGS = {
    # unequal layers: heads, sizes, windows, rotation, a layer without feed-forward, one that reads another's keys
    "unequal": O.config([
        O.attention_layer(heads=6, kv_heads=3, dim=20, vdim=36, size=17, keep=3, rot_dims=12, scaling=YARN, softcap=9.0,
                          ff=70),
        O.attention_layer(heads=4, kv_heads=4, dim=48, vdim=24, size=70, keep=1, rot_dims=48, base=500.0, softcap=25.0,
                          ff=None),
        O.attention_layer(heads=6, kv_heads=3, dim=20, vdim=36, size=33, keep=6, rot_dims=12, scaling=YARN, softcap=4.0,
                          scale=0.31, kv_from=0, ff=104)], width=90, vocab=131, eps=3e-4),
    # head size 128: the tensor-core prompt kernel and the fused QKV epilogue; windows off the 64-token pages
    "heads128": O.config([
        O.attention_layer(heads=6, kv_heads=2, dim=128, vdim=128, size=100, keep=5, rot_dims=64, scaling=YARN,
                          softcap=20.0, ff=200),
        O.attention_layer(heads=6, kv_heads=2, dim=128, vdim=128, size=65, keep=2, rot_dims=64, scaling=YARN,
                          softcap=20.0, kv_from=0, ff=136)], width=160, vocab=300),
    # sizes between the kernels' head sizes, keys longer than values
    "padded": O.config([
        O.attention_layer(heads=5, kv_heads=1, dim=112, vdim=80, size=64, keep=64, rot_dims=16, softcap=15.0, ff=88),
        O.attention_layer(heads=2, kv_heads=2, dim=160, vdim=200, size=1, keep=4, rot_dims=160, base=77.0, softcap=8.0,
                          ff=64)], width=104, vocab=97),
    # larger than any tensor-core attention kernel takes
    "large_heads": O.config([
        O.attention_layer(heads=2, kv_heads=1, dim=264, vdim=304, size=30, keep=2, rot_dims=32, softcap=12.0, ff=72)],
        width=64, vocab=83),
    # mechanisms left out one by one: no cap, no window, no rotation, no scaling, nothing kept, a window past the end
    "bare": O.config([
        O.attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, softcap=None, mask=False, rot=False, ff=48),
        O.attention_layer(heads=3, kv_heads=1, dim=64, vdim=64, softcap=None, size=21, keep=0, rot_dims=64, ff=40),
        O.attention_layer(heads=3, kv_heads=3, dim=16, vdim=8, size=5000, keep=2, rot_dims=2, softcap=2.0, ff=24),
        O.attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, softcap=6.0, mask=False, rot=False, kv_from=0, ff=56)],
        width=72, vocab=150),
    # two layers that read the same keys, each with a window of its own, wider and narrower than the owner's
    "shared": O.config([
        O.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, size=24, keep=4, rot_dims=20, softcap=11.0, ff=96),
        O.attention_layer(heads=8, kv_heads=1, dim=64, vdim=64, size=40, keep=0, rot_dims=64, softcap=13.0, ff=96),
        O.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, size=90, keep=9, rot_dims=20, softcap=11.0, kv_from=0,
                          ff=None),
        O.attention_layer(heads=8, kv_heads=1, dim=64, vdim=64, size=7, keep=1, rot_dims=64, softcap=13.0, kv_from=1,
                          ff=32)], width=128, vocab=220),
    # Vepivik: both mixers, unequal sizes, a reader with other heads and another window than the layer whose latents it
    # reads, a layer without feed-forward, one expert per token
    "latent": O.vepivik([
        O.window_layer(heads=6, kv_heads=3, dim=20, vdim=36, size=17, mlp=O.moe(ff=36, experts=5, top=3, shared=20)),
        O.latent_layer(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=28, size=33, scaling=YARN, mlp=O.moe(ff=44, experts=7, top=1,
                                                                                                        shared=12)),
        O.latent_layer(heads=5, dim=40, rot_dim=12, vdim=12, kv_rank=28, size=70, scaling=YARN, scale=0.2, kv_from=1),
        O.window_layer(heads=4, kv_heads=1, dim=56, vdim=16, size=70, mlp=O.moe(ff=24, experts=3, top=2, shared=60))],
        width=90, vocab=131, eps=3e-4, scale=1.7),
    # sizes of the kernels without padding; the expanded form's two head chunks, a window off the 64-token pages
    "latent128": O.vepivik([
        O.latent_layer(heads=18, dim=128, rot_dim=64, vdim=128, kv_rank=128, size=100, scaling=YARN,
                       mlp=O.moe(ff=64, experts=6, top=2, shared=128)),
        O.window_layer(heads=6, kv_heads=2, dim=128, vdim=128, size=65, mlp=O.moe(ff=64, experts=4, top=4, shared=64)),
        O.latent_layer(heads=2, dim=64, rot_dim=64, vdim=64, kv_rank=256, size=64, base=500.0,
                       mlp=O.moe(ff=128, experts=2, top=1, shared=32))], width=160, vocab=300),
    # mechanisms left out one by one: no window, no scaling, no shared expert, every expert chosen, one head, no feed-forward
    "latent_bare": O.vepivik([
        O.latent_layer(heads=1, dim=16, rot_dim=2, vdim=8, kv_rank=12, mask=False, scale=0.11, mlp=O.moe(ff=16, experts=3, top=3, shared=None)),
        O.window_layer(heads=2, kv_heads=2, dim=32, vdim=32, mask=False, mlp=None),
        O.latent_layer(heads=2, dim=8, rot_dim=2, vdim=64, kv_rank=12, size=1, kv_from=0, mlp=O.moe(ff=8, experts=1, top=1, shared=8)),
        O.latent_layer(heads=2, dim=72, rot_dim=70, vdim=24, kv_rank=20, size=5000, scale=0.04, mlp=None)], width=72, vocab=150, scale=0.5),
    # larger than any tensor-core latent kernel takes; three key chunks of the expanded form
    "latent_large": O.vepivik([
        O.latent_layer(heads=2, dim=208, rot_dim=80, vdim=144, kv_rank=520, size=30, scaling=YARN, mlp=O.moe()),
        O.latent_layer(heads=3, dim=136, rot_dim=24, vdim=72, kv_rank=300, size=41, mlp=O.moe(top=3))], width=64, vocab=83),
}
BANDS = {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 80}
CONFIGS.update({
    # Botusun: both mixers, unequal sizes, looped layers inside others, a side embedding off the 16-byte rows, experts in groups
    "recurrent": O.botusun([
        O.shared_kv_layer(heads=6, kv_heads=3, dim=20, size=17, rot_dims=12, scaling=BANDS, conv=3, mlp=O.dense(70)),
        O.gla_layer(heads=3, dim=12, vdim=20, tau=4.0, mlp=O.grouped_moe(ff=36, experts=9, top=3, scale=1.7, groups=(3, 2))),
        O.shared_kv_layer(heads=4, kv_heads=4, dim=48, size=70, rot_dims=48, base=500.0, scale=0.21, conv=1),
        O.gla_layer(heads=2, dim=40, vdim=24, tau=1.0, mlp=O.dense(44))],
        width=90, vocab=131, eps=3e-4, scale=1.7, mult=0.35, loop=(1, 3, 3), side=6),
    # sizes of the kernels without padding; several chunks, a window off the 64-token pages
    "recurrent128": O.botusun([
        O.shared_kv_layer(heads=6, kv_heads=2, dim=128, size=100, rot_dims=64, scaling=BANDS, conv=4,
                          mlp=O.grouped_moe(ff=64, experts=8, top=3, groups=(4, 2))),
        O.gla_layer(heads=2, dim=128, vdim=128, tau=16.0, mlp=O.grouped_moe(ff=64, experts=5, top=1, scale=2.5)),
        O.gla_layer(heads=3, dim=64, vdim=64, tau=12.0)], width=160, vocab=300, loop=(0, 2, 2), side=16),
    # mechanisms left out one by one: no loop, no side embedding, no convolution, window, rotation or scaling, no groups, every
    # expert chosen, factors of one
    "recurrent_bare": O.botusun([
        O.shared_kv_layer(heads=2, kv_heads=1, dim=32, conv=None, mask=False, rot=False, mlp=O.grouped_moe(ff=24, experts=3, top=3, scale=1.0)),
        O.gla_layer(heads=1, dim=24, vdim=16, tau=1.0),
        O.shared_kv_layer(heads=3, kv_heads=3, dim=16, size=1, rot_dims=2, conv=2, mlp=O.grouped_moe(ff=16, experts=4, top=1, groups=(4, 1))),
        O.shared_kv_layer(heads=3, kv_heads=1, dim=64, size=5000, rot_dims=64, conv=4, mlp=O.dense(40))],
        width=72, vocab=150, scale=1.0, mult=1.0),
    # larger than the tensor-core kernels take, many taps, output columns over several CTAs; a loop of one pass
    "recurrent_large": O.botusun([
        O.shared_kv_layer(heads=2, kv_heads=1, dim=264, size=30, rot_dims=32, conv=7, mlp=O.dense(72)),
        O.gla_layer(heads=2, dim=200, vdim=144, tau=10.0),
        O.gla_layer(heads=1, dim=300, vdim=72, tau=6.0, mlp=O.grouped_moe(ff=24, experts=4, top=2, groups=(2, 1)))],
        width=104, vocab=83, loop=(1, 2, 1), side=24),
    # decays from none to e^-40 per token: chunks that go in pieces, pieces that go by differences
    "recurrent_fast": O.botusun([
        O.gla_layer(heads=2, dim=24, vdim=40, tau=0.2), O.gla_layer(heads=2, dim=72, vdim=80, tau=1.5, mlp=O.dense(40)),
        O.shared_kv_layer(heads=2, kv_heads=1, dim=36, size=9, rot_dims=20, conv=5)], width=88, vocab=120, mult=0.5, loop=(0, 1, 2)),
})
CONFIGS.update({
    # Dagezen: all mixers, unequal sizes, a layer without feed-forward, widths off the 16-byte rows
    "mixed_heads": O.dagezen([
        O.mamba_layer(heads=6, vdim=12, state=20, groups=3, norm_groups=2, conv=3, mlp=O.chosen_moe(ff=36, experts=7, top=3)),
        O.sink_latent_layer(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=28, base=900.0, mlp=O.clamped(70, 0.8)),
        O.parallel_layer(heads=6, kv_heads=3, dim=20, size=17, right_heads=2, right_dim=24, scales=(0.5, 1.7)),
        O.parallel_layer(heads=4, kv_heads=1, dim=36, size=70, right_heads=3, right_dim=12, mlp=O.chosen_moe(ff=20, experts=5, top=1))],
        width=90, vocab=131, eps=3e-4, alpha=1.6, cap=11.0),
    # sizes of the kernels without padding; several chunks, a window off the 64-token pages, 16 heads
    "mixed_heads128": O.dagezen([
        O.parallel_layer(heads=16, kv_heads=4, dim=128, size=100, right_heads=2, right_dim=128, mlp=O.clamped(64, 2.0)),
        O.mamba_layer(heads=4, vdim=64, state=128, groups=1, norm_groups=1, conv=4, mlp=O.clamped(128, 1.2)),
        O.sink_latent_layer(heads=18, dim=128, rot_dim=64, vdim=128, kv_rank=128, mlp=O.chosen_moe(ff=64, experts=6, top=2)),
        O.parallel_layer(heads=8, kv_heads=8, dim=64, size=65, right_heads=3, right_dim=64)], width=160, vocab=300),
    # mechanisms at their least: one head, one group, one tap, one expert, no cap, factors of one, a window of one, one past the end
    "mixed_heads_bare": O.dagezen([
        O.parallel_layer(heads=1, kv_heads=1, dim=16, size=1, right_heads=1, right_dim=8, scales=(1.0, 1.0), mlp=O.chosen_moe(ff=8, experts=1, top=1)),
        O.mamba_layer(heads=2, vdim=8, state=8, groups=1, norm_groups=1, conv=1),
        O.sink_latent_layer(heads=1, dim=16, rot_dim=2, vdim=8, kv_rank=12, scale=0.11, mlp=O.chosen_moe(ff=16, experts=4, top=4)),
        O.parallel_layer(heads=3, kv_heads=3, dim=64, size=5000, right_heads=1, right_dim=64, mlp=O.clamped(40, 100.0))],
        width=72, vocab=150, alpha=1.5, cap=None),
    # larger than the tensor-core kernels take, many heads, many taps, norm parts that cut through heads
    "mixed_heads_large": O.dagezen([
        O.parallel_layer(heads=2, kv_heads=1, dim=264, size=30, right_heads=1, right_dim=200, mlp=O.clamped(72)),
        O.mamba_layer(heads=5, vdim=136, state=264, groups=5, norm_groups=4, conv=7),
        O.sink_latent_layer(heads=2, dim=208, rot_dim=80, vdim=144, kv_rank=520, mlp=O.clamped(24)),
        O.parallel_layer(heads=24, kv_heads=2, dim=24, size=66, right_heads=2, right_dim=300),
        O.mamba_layer(heads=3, vdim=72, state=130, groups=1, norm_groups=3, conv=2)], width=104, vocab=83, alpha=1.0),
})
MIXED_HEADS = ["mixed_heads", "mixed_heads128", "mixed_heads_bare", "mixed_heads_large"]
RECURRENT = [n for n in sorted(CONFIGS) if n.startswith("recurrent")]
LATENT = ["latent", "latent128", "latent_bare", "latent_large"]

TOLERANCE = {"fp32": 3e-5, "bf16": 0.05}


def tolerance(dtype, what=""):
    """(A stream that is normalised after every sublayer carries the rounding of all of them at full weight.)"""
    return TOLERANCE[dtype] * (1.6 if dtype == "bf16" and what.startswith("mixed_heads") else 1.0)


class Case:
    """A checkpoint on disk, its weights, and the oracle's logits of prompts (computed once)."""

    def __init__(self, root, name):
        self.name, self.cfg = name, CONFIGS[name]
        self.W = O.random_weights(self.cfg, seed=sum(map(ord, name)))
        self.path = O.write_checkpoint(str(root / name), self.cfg, self.W)
        self._want = {}

    def tokens(self, n, seed=0):
        r = random.Random(seed * 1000 + n)
        return [r.randrange(self.cfg["vocab"]) for _ in range(n)]

    def want(self, tokens):
        key = tuple(tokens)
        if key not in self._want:
            self._want[key] = O.forward(self.cfg, self.W, list(tokens))
        return self._want[key]


def error(got, want):
    """Per row: rms difference over the vocabulary (means taken off) over the spread of the wanted logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / float((want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())


def check(got, want, dtype, what=""):
    assert got.shape == want.shape, (got.shape, want.shape)
    e = error(got, want)
    bad = int(e.argmax())
    assert bool((e <= tolerance(dtype, what)).all()), f"{what}: row {bad} of {len(e)} is off by {float(e[bad]):.3g}"


def cuts(n, sizes):
    """Portions of a prompt of n tokens, cycling through `sizes`."""
    out, at, i = [], 0, 0
    while at < n:
        s = min(sizes[i % len(sizes)], n - at)
        out.append((at, at + s))
        at += s
        i += 1
    return out


def run_portions(runner, rid, tokens, portions):
    """All positions' logits of one request fed in portions."""
    rows = []
    for k, (a, b) in enumerate(portions):
        last = k + 1 == len(portions)
        rows.append(runner.step([{"id": rid, "tokens": tokens[a:b], "want": list(range(b - a))}], [rid] if last else []))
    return torch.cat(rows)


# ------------------------------------------------------------------------------------------ scenarios
def whole_prompt(case, dtype, n):
    toks = case.tokens(n)
    m = xft.AutoModel.from_pretrained(case.path, dtype=dtype)
    check(m([toks])[0], case.want(toks), dtype, f"{case.name}: whole prompt of {n}")


def first_tokens(case, dtype):
    """Prompts of 1, 2, 3 ... tokens in one ragged batch."""
    prompts = [case.tokens(n, 5) for n in (1, 2, 3, 5, 9)]
    m = xft.AutoModel.from_pretrained(case.path, dtype=dtype)
    got = m(prompts)
    check(got, torch.cat([case.want(p) for p in prompts]), dtype, f"{case.name}: first tokens")


def token_by_token(case, dtype, n, start=1):
    """A prompt, then single tokens through the cache, against the prompt in one piece."""
    toks = case.tokens(n, 1)
    r = TraceRunner(case.path, dtype, n)
    got = run_portions(r, "a", toks, [(0, start)] + [(i, i + 1) for i in range(start, n)])
    check(got, case.want(toks), dtype, f"{case.name}: token by token")


def portions(case, dtype, n, sizes):
    toks = case.tokens(n, 2)
    r = TraceRunner(case.path, dtype, n)
    check(run_portions(r, "a", toks, cuts(n, sizes)), case.want(toks), dtype, f"{case.name}: portions {sizes}")


def mixed_batches(case, dtype, seed=0, lengths=(150, 97, 64, 30, 1, 129), live=3):
    """Requests of unequal lengths in random portions — prompts' portions beside single tokens, some left out of a step —
    over pools just large enough for those alive, so that freed blocks are used again (and are filled with large values
    in between: a masked key must not leak)."""
    r = random.Random(seed)
    toks = {str(i): case.tokens(n, 10 + i) for i, n in enumerate(lengths)}
    pages = lambda n: (n + 63) // 64 * 64
    run = TraceRunner(case.path, dtype, sum(sorted((pages(n) for n in lengths), reverse=True)[:live]))
    cache = run.model.model.cache
    if cache.has_state:                                  # no more slots than live requests need
        assert cache.max_states - 4 in (0, 1)
    size, states = cache.alloc.num_blocks, cache.state_alloc.num_blocks
    at, got = {k: 0 for k in toks}, {k: [] for k in toks}
    waiting, alive = list(toks), []
    steps = 0
    while waiting or alive:
        while waiting and len(alive) < live:
            alive.append(waiting.pop(0))
        entries, end = [], []
        for k in r.sample(alive, r.randint(1, len(alive))):
            left = len(toks[k]) - at[k]
            n = min(left, r.choice([1, 1, 2, 3, 7, 29, 64, 90]))
            entries.append({"id": k, "tokens": toks[k][at[k]:at[k] + n], "want": list(range(n))})
            at[k] += n
            if n == left:
                end.append(k)
        rows = run.step(entries, end)
        for e in entries:
            n = len(e["tokens"])
            got[e["id"]].append(rows[:n])
            rows = rows[n:]
        for k in end:
            alive.remove(k)
        for b in cache.alloc.free:                       # what freed pages hold must not matter
            for pool in (cache.k, cache.v):
                for t in pool:
                    if t is not None:
                        t[b].fill_(30.0)
        for s in cache.state_alloc.free:                 # nor what freed states hold
            for t in cache.state:
                t[s].fill_(30.0)
        steps += 1
    assert (cache.alloc.num_blocks, cache.state_alloc.num_blocks) == (size, states) and not cache.state_slot
    assert not cache.tables, "requests were left behind"
    for k, rows in got.items():
        check(torch.cat(rows), case.want(toks[k]), dtype, f"{case.name}: request {k} of {len(toks[k])} tokens")
    return steps


def greedy(case, dtype, n_prompt, n_new):
    """generate() on a batch of unequal prompts (through the engine's batching, decode runner and sampler): each emitted
    token is the best one, up to rounding, given everything before it."""
    prompts = [case.tokens(n_prompt, 30), case.tokens(n_prompt, 31)]
    m = xft.AutoModel.from_pretrained(case.path, dtype=dtype)
    out = m.generate(torch.tensor(prompts), max_length=n_prompt + n_new).tolist()
    for p, row in zip(prompts, out):
        assert row[:n_prompt] == p and len(row) == n_prompt + n_new
        w = case.want(row[:-1])[n_prompt - 1:]
        spread = float((w - w.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        picked = w.gather(1, torch.tensor(row[n_prompt:])[:, None])[:, 0]
        short = (w.max(-1).values - picked) / spread
        assert float(short.max()) <= (1e-4 if dtype == "fp32" else 6 * tolerance(dtype)), f"a worse token by {float(short.max())}"
    return out


def rows_and_order(case, dtype):
    """`want` may be empty, partial or out of order; a step in which nothing is wanted still fills the cache."""
    a, b = case.tokens(40, 3), case.tokens(25, 4)
    r = TraceRunner(case.path, dtype, 192)
    assert r.step([{"id": "a", "tokens": a[:17], "want": []}]).shape == (0, case.cfg["vocab"])
    got = r.step([{"id": "b", "tokens": b, "want": [24, 0, 7]}, {"id": "a", "tokens": a[17:30], "want": [12]}], ["b"])
    wa, wb = case.want(a), case.want(b)
    check(got, torch.stack([wb[24], wb[0], wb[7], wa[29]]), dtype, "rows")
    got = r.step([{"id": "a", "tokens": a[30:], "want": [3, 9]}], ["a"])
    check(got, torch.stack([wa[33], wa[39]]), dtype, "rows of a later portion")
    assert not r.model.model.cache.tables
