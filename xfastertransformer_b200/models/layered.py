"""Decoder for designs described layer by layer (``ModelConfig.layers``): Kafipel, Vepivik, Botusun, Dagezen.

It is the generic decoder with sizes, rotation, mask and cache pool taken from each layer's own entry, served by the same
engine, paged cache, decode runner, sampler and kernels.  What these designs add to it, each as an op with its constants
as arguments:

* a 32-bit residual stream with a norm before and (per design) after every sublayer, one launch between two products
  (`ops.residual_norm`): x += norm_b(y) and h = norm(x) for the product that follows;
* attention with a sliding window that keeps the first tokens, a tanh cap on the scores and a sink per head
  (`ops.paged_attention(window=, keep_first=, softcap=, sinks=)`);
* layers without keys and values of their own, which read the pool of an earlier layer (`kv_from`);
* query/key and value heads of different sizes;
* latent attention with a window, an output gate and layers that read another layer's latents
  (`ops.latent_prep`, `ops.latent_attention`); its pools have one row per token and no values;
* attention whose values are its keys, with short convolutions, a norm per head and rotation between the projection and the
  cache (`ops.head_prep`), the convolutions' last inputs kept as a state;
* gated linear attention, a recurrent layer with a state instead of a cache (`ops.gated_linear`);
* mixtures of experts with or without a gate product, chosen by group or among all (`ops.route`, `ops.moe_experts`), next to
  a shared expert;
* a residual stream that is the norm of alpha * x + sublayer(x), the sublayers reading the stream itself
  (`FamilySpec.sum_norm`);
* state-space layers (`ops.state_space`): convolution, recurrence and grouped norm between their two projections;
* mixers side by side on the same input (`MixerConfig.parts`), with one output projection over all of their heads: attention
  with mixed heads (`ops.talking_prep`, `ops.talking_attention`) and time mixing (`ops.token_shift`, `ops.gated_linear` with a
  bonus);
* dense feed-forwards with a clamped gate and biases, experts weighted by the softmax over the chosen ones, a tanh cap on the
  logits;
* layers that run several times in a row (`ModelConfig.runs`), each pass with a cache and states of its own;
* a part of the token's own side embedding after every layer, gated by the residual stream;
* a scaled embedding, a factor on everything that joins the residual stream, and logits from the embedding table.

Widths that the 16-byte rows of the tensor-core kernels do not allow are padded with zeros at load: the hidden and the
feed-forward width to a multiple of 8, heads to the next size the attention kernels have, each part of a latent head to a
multiple of 64.  A zero dimension adds nothing
to a score or a sum.  The 32-bit path (dtype "fp32") and CPU tensors keep the heads as they are.
"""
from __future__ import annotations

import copy
import math
from typing import Dict, List, Optional

import torch

from .. import ops
from ..config import PARALLEL_PARTS, LayerConfig, MixerConfig, ModelConfig, MoeConfig, RotaryConfig
from ..ops import reference as R
from ..parallel import partition as P
from ..parallel.dist import DistContext
from ..runtime.kv_cache import PagedKVCache
from ..runtime.loader import SafetensorsSource, make_linear
from ..utils import debugger
from ..utils.progress import ProgressBar
from ..utils.trace import TimeLine
from .decoder import Batch, Decoder, Layer

ATTENTION_HEADS = (64, 128, 256)          # head sizes of the tensor-core attention kernels
LATENTS = (64, 128, 256, 512)             # latent sizes of the tensor-core latent attention


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def _pad(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """`t` in the corner of a zero tensor of `shape`."""
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(n) for n in t.shape)] = t
    return out


class LayeredDecoder(Decoder):
    def __init__(self, cfg: ModelConfig, ctx: DistContext, path: str, weight_dtype: str,
                 act_dtype: Optional[torch.dtype] = None, embed_from: Optional["LayeredDecoder"] = None):
        self._setup(cfg, ctx, weight_dtype, act_dtype)
        self.hidden_dtype = torch.float32
        self.exact = self.kind == "fp32"
        self.eps = cfg.layernorm_eps
        self.W = cfg.hidden_size
        gpu = self.device.type == "cuda"
        self.hidden_width = self.WP = _up(self.W, 8) if gpu else self.W
        self.pad_heads = gpu and not self.exact
        self.src = SafetensorsSource(path, self.device)
        self._ropes: Dict[RotaryConfig, torch.Tensor] = {}
        self._old_ropes: List[torch.Tensor] = []
        self.slopes = None
        self.has_moe = False
        with TimeLine("Decoder.loadWeights"):
            self._load_ends(embed_from)
            # pipeline stages are ranges of runs; a looped layer's weights are loaded once
            runs = cfg.runs()
            self.l0, self.l1 = P.pp_layer_range(len(runs), ctx.pp_size, ctx.pp_rank)
            runs = runs[self.l0:self.l1]
            loaded = {i: self._load_layer(i) for i in ProgressBar.wrap(sorted({i for i, _ in runs}), "Loading layers")}
        self.layers: List[Layer] = list(loaded.values())
        self.runs: List[Layer] = []
        for i, t in runs:
            L = copy.copy(loaded[i])
            L.parts = [copy.copy(q) for q in L.parts]
            L.step = self._step_vector(t) if cfg.loop is not None and i == cfg.loop.start and t >= 0 else None
            self.runs.append(L)
        # cache pools: one per run with keys and values of its own; state pools: the ones each run asks for
        self.pools: Dict[int, int] = {}
        self.pool_shapes, self.state_shapes = [], []
        for L in self.runs:
            for q in L.parts or [L]:
                if q.own_kv:
                    self.pools[L.idx] = len(self.pool_shapes)
                    self.pool_shapes.append((1, q.kd, 0) if q.mix.kind == "latent" else (q.hkv, q.kd, q.vd))
                q.pool = self.pools.get(q.kv_layer, -1)
                if q.pool < 0 and q.mix.has_kv:
                    raise ValueError(f"layer {L.idx} reads the keys of layer {q.kv_layer}, which is on another pipeline stage")
                q.state = list(range(len(self.state_shapes), len(self.state_shapes) + len(q.state_shapes)))
                self.state_shapes.extend(q.state_shapes)
        L = (self.layers[0].parts or self.layers)[0]
        self.D, self.hq, self.hkv, self.group, self.scale = L.kd, L.hq, L.hkv, L.group, L.mix.scale
        for L in self.layers:
            self._rope(L.mix.rot, 2048)

    # ------------------------------------------------------------------------------------
    # rotary tables: one per distinct rotation, grown when a longer context comes up
    # ------------------------------------------------------------------------------------
    def _rope(self, rot: Optional[RotaryConfig], positions: int) -> Optional[torch.Tensor]:
        if rot is None or rot.dims == 0:
            return None
        tab = self._ropes.get(rot)
        if tab is None or tab.shape[0] < positions:
            n = max(_up(positions, 2048), 2 * tab.shape[0] if tab is not None else 0)
            if rot.factor > 0 and rot.scaling == "banded":
                new = R.rope_table(n, rot.dims, rot.base, "banded", rot.factor, rot.original, rot.high, rot.low,
                                   angle_dtype=torch.float64)
            elif rot.factor > 0:
                new = R.rope_table(n, rot.dims, rot.base, "yarn", rot.factor, rot.original, rot.fast, rot.slow,
                                   table_scale=0.1 * math.log(rot.factor) + 1.0, angle_dtype=torch.float64)
            else:
                new = R.rope_table(n, rot.dims, rot.base, angle_dtype=torch.float64)
            if tab is not None:
                self._old_ropes.append(tab)       # captured decode graphs keep reading it (their positions fit it)
            tab = self._ropes[rot] = new.to(self.device)
        return tab

    def _ensure_positions(self, b: Batch, cache: PagedKVCache) -> None:
        need = max(b.max_kv, b.block_table.shape[1] * cache.block)     # a captured step may run to the table's width
        for rot in list(self._ropes):
            self._rope(rot, need)

    # ------------------------------------------------------------------------------------
    # weights
    # ------------------------------------------------------------------------------------
    def _gain(self, name: str):
        bias = self.src.vector(name + ".b", self.W) if self.spec.norm_bias else None
        return self.src.vector(name, self.W, fake_ones=True), bias

    def _step_vector(self, t: int) -> torch.Tensor:
        """What joins the residual stream in front of pass `t` of the looped layers."""
        return self.src.matrix("loop.step", (self.cfg.loop.times, self.W), rows=(t, t + 1))[0].float().contiguous()

    def _load_ends(self, share: Optional["LayeredDecoder"]) -> None:
        c = self.cfg
        self.v0, self.v1 = P.vocab_range(c.vocab_size, self.tp, self.tpr)
        if share is not None:
            self.wte, self.final, self.lm_head, self.side_embed = share.wte, share.final, share.lm_head, share.side_embed
            return
        self.wte = self.final = self.lm_head = self.side_embed = None
        if c.side_dim:
            # the part of each layer padded to the products' 16-byte rows
            n, d = len(c.layers), c.side_dim
            w = self.src.matrix("side.embed", (c.vocab_size, n * d)).view(c.vocab_size, n, d)
            w = _pad(w, c.vocab_size, n, self._ff_size(d)).reshape(c.vocab_size, -1)
            self.side_embed = w.to(torch.bfloat16 if self.device.type == "cuda" else w.dtype)
        if self.first_stage:
            self.wte = _pad(self.src.matrix("embed", (c.vocab_size, self.W)).to(torch.bfloat16), c.vocab_size, self.WP)
        if self.last_stage:
            self.final = self._gain("final.norm")
            w = self.src.matrix("embed" if self.spec.tied_head else "head", (c.vocab_size, self.W), rows=(self.v0, self.v1))
            kind = "fp32" if self.exact or self.device.type == "cpu" else "bf16"
            if self.spec.tied_head and self.wte is not None and kind == "bf16":
                w = self.wte[self.v0:self.v1]                  # one copy serves both ends
            self.lm_head = make_linear(_pad(w, w.shape[0], self.WP), kind)

    def _head_size(self, n: int) -> int:
        if not self.pad_heads:
            return n
        return next((d for d in ATTENTION_HEADS if n <= d), _up(n, 8))

    def _rows(self, name: str, heads: int, rng, *parts) -> torch.Tensor:
        """Rows of heads rng[0] .. rng[1] of a [heads * size, width] projection.  `parts` lists (rows, padded rows) of a
        head, in order."""
        dim, padded = sum(a for a, _ in parts), sum(b for _, b in parts)
        w = self.src.matrix(name, (heads * dim, self.W), rows=(rng[0] * dim, rng[1] * dim))
        n = rng[1] - rng[0]
        w, out, at = w.view(n, dim, self.W), [], 0
        for a, b in parts:
            out.append(_pad(w[:, at:at + a], n, b, self.WP))
            at += a
        return torch.cat(out, 1).reshape(n * padded, self.WP)

    def _out_rows(self, L: Layer, p: str, heads: int, rng, vdim: int, width: int = 0) -> None:
        """The output projection: its columns are heads of `vdim`, padded to L.vd, and all of them to `width`."""
        w = self.src.matrix(p + "o", (self.W, heads * vdim), cols=(rng[0] * vdim, rng[1] * vdim))
        w = _pad(w.reshape(self.W, L.hq, vdim), self.WP, L.hq, L.vd).reshape(self.WP, L.hq * L.vd)
        L.o_rows = _pad(w, self.WP, max(width, L.hq * L.vd))

    def _load_layer(self, i: int) -> Layer:
        lc: LayerConfig = self.cfg.layers[i]
        m = lc.mixer
        p = f"l{i}."
        L = Layer()
        L.idx, L.ff = i, lc.ff
        second = self._gain if self.spec.post_norm else lambda name: None
        L.norm1, L.norm1b = self._gain(p + "norm1"), second(p + "norm1b")
        L.parts = []
        if m.parts:
            L.mix, L.own_kv, L.state_shapes = m, False, []
            for (name, _), q, mult in zip(PARALLEL_PARTS, m.parts, m.part_scales):
                Q = Layer()
                Q.idx, Q.mult = i, mult
                self._load_mixer(Q, f"{p}mix.{name}.", q)
                Q.width = Q.o_rows.shape[1]
                L.parts.append(Q)
            # one output projection over all parts' heads
            L.o = make_linear(torch.cat([q.o_rows for q in L.parts], 1), self.kind)
            for q in L.parts:
                del q.o_rows
            L.hq, L.hkv = L.parts[0].hq, L.parts[0].hkv
        else:
            L.mult = 1.0
            self._load_mixer(L, p + "mix.", m)
            L.o = make_linear(L.o_rows, self.kind)
            del L.o_rows
        L.mlp_kind = "none"
        if lc.ff_kind == "moe" or lc.ff:
            L.norm2, L.norm2b = self._gain(p + "norm2"), second(p + "norm2b")
        if lc.ff_kind == "moe":
            self._load_experts(L, p, lc.moe)
        elif lc.ff:
            L.mlp_kind, gpu = "llama", self.device.type == "cuda"
            r = self._ffn_range(lc.ff)
            n = r[1] - r[0]
            np_ = self._ff_size(n)
            gate, up = (_pad(self.src.matrix(p + "mlp." + x, (lc.ff, self.W), rows=r), np_, self.WP) for x in ("gate", "up"))
            kind = "bf16" if gpu and lc.act == "clamped" and not self.exact else self.kind       # not in the quantised products
            L.gate_up = make_linear(torch.cat([gate, up]), kind)
            L.down = make_linear(_pad(self.src.matrix(p + "mlp.down", (self.W, lc.ff), cols=r), self.WP, np_), self.kind)
            L.act, L.limit, L.gate_up_b, L.down_b = lc.act, lc.limit, None, None
            if lc.ff_bias:
                L.gate_up_b = torch.cat([_pad(self.src.vector(f"{p}mlp.{x}.b", lc.ff, rng=r), np_) for x in ("gate", "up")]).contiguous()
                L.down_b = _pad(self.src.vector(p + "mlp.down.b", self.W), self.WP).contiguous()
        L.side_gate = None
        if self.cfg.side_dim:
            d, kind = self.cfg.side_dim, "fp32" if self.exact or self.device.type == "cpu" else "bf16"
            n = self._ff_size(d)
            L.side_gate = make_linear(_pad(self.src.matrix(p + "side.gate", (d, self.W)), n, self.WP), kind)
            L.side_proj = make_linear(_pad(self.src.matrix(p + "side.proj", (self.W, d)), self.WP, n), kind)
            L.side_norm = self._gain(p + "side.norm")
            L.side_at = i * n
        return L

    def _load_mixer(self, L: Layer, p: str, m: MixerConfig) -> None:
        """Weights of one mixer, the tensors `p`*; leaves its output projection in L.o_rows."""
        L.mix = m
        L.replicated = m.kind in ("ssd", "talking", "time_mix")      # norms, groups and mixes go across heads: on every rank
        tp, tpr = (1, 0) if L.replicated else (self.tp, self.tpr)
        # this rank's heads; query head h reads key/value head h // (heads / kv_heads)
        (qs, qe), (ks, ke) = P.head_range(m.heads, m.kv_heads, tp, tpr)
        L.hq, L.hkv, L.group = qe - qs, ke - ks, m.heads // m.kv_heads
        L.q_off = qs - ks * L.group
        if L.hq <= 0:
            raise ValueError(f"layer {L.idx}: {m.heads} heads cannot be split over {tp} ranks")
        L.own_kv = m.has_kv and m.kv_from < 0
        L.state_shapes = []
        L.kv_layer = L.idx if L.own_kv else m.kv_from
        if m.kind == "latent":
            self._load_latent(L, p, (qs, qe))
        elif m.kind == "gla":
            self._load_linear(L, p, (qs, qe))
        elif m.kind == "ssd":
            self._load_state_space(L, p)
        elif m.kind == "talking":
            self._load_talking(L, p)
        elif m.kind == "time_mix":
            self._load_time_mix(L, p)
        elif m.values_from_keys:
            self._load_shared_kv(L, p, (qs, qe), (ks, ke))
        else:
            self._load_attention(L, p, (qs, qe), (ks, ke))

    def _ff_size(self, n: int) -> int:
        return _up(n, 8) if self.device.type == "cuda" else n

    def _load_attention(self, L: Layer, p: str, q, kv) -> None:
        m = L.mix
        L.kd, L.vd = self._head_size(m.dim), self._head_size(m.vdim)
        if self.pad_heads:
            L.kd = L.vd = max(L.kd, L.vd)         # the tensor-core kernels have one size for keys and values
        parts = [self._rows(p + "q", m.heads, q, (m.dim, L.kd))]
        if L.own_kv:
            parts.append(self._rows(p + "k", m.kv_heads, kv, (m.dim, L.kd)))
            parts.append(self._rows(p + "v", m.kv_heads, kv, (m.vdim, L.vd)))
        L.qkv = make_linear(torch.cat(parts), self.kind)
        L.sinks = None
        if self.spec.sinks and (self.src.exists(p + "sink") or self.src.fake):
            L.sinks = self.src.vector(p + "sink", m.heads, rng=q).contiguous()
        self._out_rows(L, p, m.heads, q, m.vdim)

    def _load_shared_kv(self, L: Layer, p: str, q, kv) -> None:
        """Attention whose values are its keys.  Rows leave the projection with the heads' real size; `head_prep` pads them."""
        m, n = L.mix, (L.hq + L.hkv) * L.mix.dim
        L.kd = L.vd = self._head_size(m.dim)
        parts = [(p + "q", m.heads, q), (p + "k", m.kv_heads, kv)]
        w = torch.cat([self._rows(name, heads, rng, (m.dim, m.dim)) for name, heads, rng in parts])
        L.qkv = make_linear(_pad(w, self._ff_size(n), self.WP), self.kind)
        cut = lambda rng: (rng[0] * m.dim, rng[1] * m.dim)
        L.qkv_b = None
        if m.qk_bias:
            b = [self.src.vector(name + ".b", heads * m.dim, rng=cut(rng)) for name, heads, rng in parts]
            L.qkv_b = _pad(torch.cat(b), L.qkv.out_features).contiguous()
        conv = None
        if m.conv:
            conv = [self.src.matrix(name + ".conv", (heads * m.dim, m.conv), rows=cut(rng)) for name, heads, rng in parts]
            conv = torch.cat(conv).float().t().contiguous()                # [taps, channels]
            if m.conv > 1:
                L.state_shapes.append(((m.conv - 1, n), self.act_dtype))
        norms = [self.src.vector(p + f"{x}.norm", m.dim, fake_ones=True).contiguous() if m.qk_norm else None for x in "qk"]
        L.prep = ops.HeadPrep(L.hq, L.hkv, m.dim, L.kd, conv, *norms)
        L.sinks = None if m.sink is None else torch.full((L.hq,), m.sink, dtype=torch.float32, device=self.device)
        self._out_rows(L, p, m.heads, q, m.vdim)

    def _load_linear(self, L: Layer, p: str, rng) -> None:
        """Gated linear attention: queries, keys, values, output gate and the decay's first product are one projection."""
        m, gpu = L.mix, self.device.type == "cuda"
        rank = self.src.shape(p + "a1", (16, self.W))[0]
        d = L.dims = ops.LinearDims(L.hq, m.dim, m.vdim, rank, 8 if gpu else 1)
        L.kd, L.vd = m.dim, m.vdim
        rows = [self._rows(p + "" + x, m.heads, rng, (n, n)) for x, n in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim))]
        rows.append(_pad(self.src.matrix(p + "a1", (rank, self.W)), rank, self.WP))
        L.qkv = make_linear(torch.cat([_pad(r, d.up(r.shape[0]), self.WP) for r in rows]), self.kind)
        a2 = self.src.matrix(p + "a2", (m.heads * m.dim, rank), rows=(rng[0] * m.dim, rng[1] * m.dim)).to(self.act_dtype)
        bias = self.src.vector(p + "a2.b", m.heads * m.dim, rng=(rng[0] * m.dim, rng[1] * m.dim))
        gain = self.src.vector(p + "norm", m.vdim, fake_ones=True)
        L.decay = ops.LinearWeights(_pad(a2, a2.shape[0], d.up(rank)).contiguous(), bias.contiguous(), m.tau, gain.contiguous())
        L.state_shapes.append(((L.hq, m.dim, m.vdim), torch.float32))
        self._out_rows(L, p, m.heads, rng, m.vdim, d.up(L.hq * m.vdim))

    def _load_state_space(self, L: Layer, p: str) -> None:
        """Mamba-2: gate, convolved channels and step sizes are one projection."""
        m, gpu = L.mix, self.device.type == "cuda"
        H, n = m.heads, m.heads * m.vdim
        d = L.dims = ops.StateDims(H, m.dim, m.vdim, m.groups, m.norm_groups, max(m.conv, 1), 8 if gpu else 1)
        L.kd, L.vd = m.dim, m.vdim
        w = self.src.matrix(p + "in", (n + d.channels + H, self.W))
        rows = [w[:n], w[n:n + d.channels], w[n + d.channels:]]
        L.qkv = make_linear(torch.cat([_pad(r, d.up(r.shape[0]), self.WP) for r in rows]), self.kind)
        f32 = lambda name, k: self.src.vector(p + name, k).contiguous()
        conv = self.src.matrix(p + "conv", (d.channels, d.taps)).float().t().contiguous()              # [taps, channels]
        L.ssm = ops.StateWeights(conv, f32("conv.b", d.channels), f32("dt_bias", H), torch.exp(f32("A_log", H)), f32("D", H),
                                 self.src.vector(p + "norm", n, fake_ones=True).contiguous())
        L.state_shapes.append(((H, m.dim, m.vdim), torch.float32))
        if d.taps > 1:
            L.state_shapes.append(((d.taps - 1, d.channels), self.act_dtype))
        self._out_rows(L, p, H, (0, H), m.vdim, d.up(n))

    def _load_talking(self, L: Layer, p: str) -> None:
        """Attention with mixed heads: queries, keys and gate are one projection; heads are padded behind the norms."""
        m, gpu = L.mix, self.device.type == "cuda"
        L.kd = L.vd = self._head_size(m.dim)
        f32 = lambda name, k, ones=False: self.src.vector(p + name, k, fake_ones=ones).contiguous()
        talk = self.src.matrix(p + "talk", (m.heads, m.heads)).float().contiguous()
        d = L.talk = ops.TalkingHeads(m.heads, m.kv_heads, m.dim, L.kd, f32("q.norm", m.heads * m.dim, True),
                                      f32("k.norm", m.kv_heads * m.dim, True), f32("r1", m.heads), f32("r2", m.heads), talk,
                                      L.mult, 8 if gpu else 1)
        rows = [self._rows(p + "q", m.heads, (0, m.heads), (m.dim, m.dim)),
                self._rows(p + "k", m.kv_heads, (0, m.kv_heads), (m.dim, m.dim)),
                self._rows(p + "g", m.heads, (0, m.heads), (m.vdim, L.vd))]
        L.qkv = make_linear(torch.cat([_pad(r, d.up(r.shape[0]), self.WP) for r in rows]), self.kind)
        self._out_rows(L, p, m.heads, (0, m.heads), m.vdim)

    def _load_time_mix(self, L: Layer, p: str) -> None:
        """Time mixing: four products of one size on four mixes of the input, and the decay's two."""
        m, gpu = L.mix, self.device.type == "cuda"
        n, rank = m.heads * m.dim, self.src.shape(p + "w1", (32, self.W))[0]
        d = L.dims = ops.LinearDims(m.heads, m.dim, m.vdim, rank, 8 if gpu else 1)
        L.kd, L.vd = m.dim, m.vdim
        L.mu = torch.stack([_pad(self.src.vector(p + "mu." + x, self.W), self.WP) for x in "rkvgw"]).contiguous()
        rows = [self._rows(p + x, m.heads, (0, m.heads), (m.dim, m.dim)) for x in "rkvg"]
        kind = "fp32" if self.exact or self.device.type == "cpu" else "bf16"
        L.rkvg = make_linear(torch.cat([_pad(r, d.up(n), self.WP) for r in rows]), kind)
        L.w1 = make_linear(_pad(self.src.matrix(p + "w1", (rank, self.W)), d.up(rank), self.WP), kind)
        a2 = self.src.matrix(p + "w2", (n, rank)).to(self.act_dtype)
        L.decay = ops.LinearWeights(_pad(a2, n, d.up(rank)).contiguous(), self.src.vector(p + "w0", n).contiguous(), 1.0,
                                    self.src.vector(p + "norm", n, fake_ones=True).contiguous(), 1.0,
                                    self.src.matrix(p + "u", (m.heads, m.dim)).float().contiguous(), L.mult)
        L.state_shapes.append(((m.heads, m.dim, m.vdim), torch.float32))
        L.state_shapes.append(((self.WP,), torch.float32))
        self._out_rows(L, p, m.heads, (0, m.heads), m.vdim, d.up(n))

    def _load_latent(self, L: Layer, p: str, q) -> None:
        """Latent attention: heads are split over ranks, the latents (one row per token) are on every rank."""
        m = L.mix
        size = (lambda n: _up(n, 64)) if self.pad_heads else (lambda n: n)
        rank = next((r for r in LATENTS if m.kv_rank <= r), size(m.kv_rank)) if self.pad_heads else m.kv_rank
        d = L.dims = ops.LatentDims(L.hq, size(m.dim), size(m.rot_dim), rank, size(m.vdim), L.own_kv, m.gate, m.kv_rank,
                                  m.head_gate, 8 if self.device.type == "cuda" else 1)
        L.kd, L.vd = d.rank + d.rot, d.vdim
        parts = [self._rows(p + "q", m.heads, q, (m.dim, d.dim), (m.rot_dim, d.rot))]
        L.latent_norm = None
        if L.own_kv:
            parts.append(self._rows(p + "dkv", 1, (0, 1), (m.kv_rank, d.rank), (m.rot_dim, d.rot)))
            L.latent_norm = _pad(self.src.vector(p + "dkv.norm", m.kv_rank, fake_ones=True), d.rank)
        if d.gate:
            parts.append(self._rows(p + "g", m.heads, q, (1, 1) if d.head_gate else (m.vdim, d.vdim)))
        w = torch.cat(parts)
        L.qkv = make_linear(_pad(w, d.row, self.WP), self.kind)
        L.sinks = self.src.vector(p + "sink", m.heads, rng=q).contiguous() if m.sinks else None

        def per_head(name, n, padded):
            w = self.src.matrix(p + name, (m.heads * n, m.kv_rank), rows=(q[0] * n, q[1] * n))
            return _pad(w.view(L.hq, n, m.kv_rank), L.hq, padded, d.rank).to(self.act_dtype)
        L.up = ops.LatentWeights(per_head("uk", m.dim, d.dim), per_head("uv", m.vdim, d.vdim))
        self._out_rows(L, p, m.heads, q, m.vdim)

    def _load_experts(self, L: Layer, p: str, f: MoeConfig) -> None:
        """Router and experts; an expert's width is split over tensor-parallel ranks (whole experts with XFT_EXPERT_PARALLEL)."""
        L.mlp_kind, L.moe, L.act = "moe", f, f.act
        kind = "fp32" if self.exact or self.device.type == "cpu" else "bf16"
        L.router = make_linear(_pad(self.src.matrix(p + "mlp.router", (f.experts, self.W)), f.experts, self.WP), kind)

        L.router_b = self.src.vector(p + "mlp.router.b", f.experts).contiguous() if f.router_bias else None
        L.correction = self.src.vector(p + "mlp.correction", f.experts).contiguous() if f.correction else None
        first = ("gate", "up") if f.gated else ("up",)

        def pair(name, ff, r):
            n = self._ff_size(r[1] - r[0])
            w = [_pad(self.src.matrix(f"{p}{name}.{x}", (ff, self.W), rows=r), n, self.WP) for x in first]
            return (make_linear(torch.cat(w), self.kind),
                    make_linear(_pad(self.src.matrix(p + name + ".down", (self.W, ff), cols=r), self.WP, n), self.kind))
        L.e0, L.e1 = self._local_experts(f.experts)
        r = (0, f.ff) if self.ctx.ep_size > 1 else self._ffn_range(f.ff)
        L.experts = [pair(f"mlp.e{e}", f.ff, r) for e in range(L.e0, L.e1)]
        L.shared = pair("mlp.shared", f.shared, self._ffn_range(f.shared)) if f.shared else None

    # ------------------------------------------------------------------------------------
    # forward
    # ------------------------------------------------------------------------------------
    def _mixer(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache, x: torch.Tensor) -> torch.Tensor:
        """Token-mixing sublayer: its input `h` (the stream itself is `x`) -> output projection (summed over tensor-parallel ranks)."""
        if L.parts:
            a = torch.empty(h.shape[0], L.o.in_features, dtype=h.dtype, device=h.device)
            at = 0
            for q in L.parts:
                n = q.width
                self._heads(q, h, b, cache, x, a[:, at:at + n])
                at += n
        else:
            a = self._heads(L, h, b, cache, x)
        with TimeLine("Output"):
            if (L.parts or [L])[0].replicated:
                return ops.linear(a, L.o)
            return self._row_parallel(a, L.o, None, None)

    def _heads(self, L: Layer, h, b: Batch, cache: PagedKVCache, x, out=None) -> torch.Tensor:
        """A mixer without its output projection."""
        kind = L.mix.kind
        if kind == "talking":
            return self._talking(L, h, b, cache, out)
        if kind == "time_mix":
            return self._time_mix(L, x, b, cache, out)
        if kind == "attention" and L.mix.values_from_keys:
            return self._shared_kv(L, h, b, cache)
        return {"latent": self._latent, "gla": self._linear, "ssd": self._state_space}.get(kind, self._attend)(L, h, b, cache)

    def _state_space(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache) -> torch.Tensor:
        with TimeLine("QKV.linear"):
            x = ops.linear(h, L.qkv)
        with TimeLine("SSD"):
            states = [cache.state[i] for i in L.state]
            return ops.state_space(x, L.dims, L.ssm, self.eps, states[0], states[1] if len(states) > 1 else None, b.state_slots, b.cu_q,
                                   b.kv_lens, meta=b)

    def _talking(self, L: Layer, h, b: Batch, cache: PagedKVCache, out) -> torch.Tensor:
        kc, vc = cache.k[L.pool], cache.v[L.pool]
        with TimeLine("QKV.linear"):
            x = ops.linear(h, L.qkv)
        with TimeLine("QKPO"):
            q = ops.talking_prep(x, L.talk, self.eps, kc, vc, b.slots)
        with TimeLine("MHA"):
            return ops.talking_attention(q, x, L.talk, kc, vc, b.block_table, b.cu_q, b.kv_lens, L.mix.scale, L.mix.window, meta=b, out=out)

    def _time_mix(self, L: Layer, x, b: Batch, cache: PagedKVCache, out) -> torch.Tensor:
        d, W = L.dims, L.mu.shape[1]
        with TimeLine("Shift"):
            mix = ops.token_shift(x, L.mu, cache.state[L.state[1]], b.state_slots, b.cu_q, b.kv_lens, self.act_dtype, meta=b)
        with TimeLine("QKV.linear"):
            rows = torch.empty(x.shape[0], d.a_at + d.up(d.rank), dtype=self.act_dtype, device=x.device)
            ops.linear_parts(mix[:, :4 * W], L.rkvg, 4, rows)
            ops.linear(mix[:, 4 * W:], L.w1, act="tanh", out=rows[:, d.a_at:])
        with TimeLine("GLA"):
            return ops.gated_linear(rows, d, L.decay, self.eps, cache.state[L.state[0]], b.state_slots, b.cu_q, b.kv_lens, meta=b, out=out)

    def _latent(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache) -> torch.Tensor:
        m, pool = L.mix, cache.k[L.pool]
        with TimeLine("QKV.linear"):
            x = ops.linear(h, L.qkv)
        with TimeLine("QKPO"):
            ops.latent_prep(x, L.dims, b.positions, self._rope(m.rot, 0), m.rot.dims if m.rot is not None else 0, L.latent_norm,
                            self.eps, pool, b.slots)
        with TimeLine("MHA"):
            return ops.latent_attention(x, L.dims, pool, b.block_table, b.cu_q, b.kv_lens, L.up, m.scale, m.window, meta=b, sinks=L.sinks)

    def _linear(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache) -> torch.Tensor:
        with TimeLine("QKV.linear"):
            x = ops.linear(h, L.qkv)
        with TimeLine("GLA"):
            return ops.gated_linear(x, L.dims, L.decay, self.eps, cache.state[L.state[0]], b.state_slots, b.cu_q, b.kv_lens, meta=b)

    def _shared_kv(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache) -> torch.Tensor:
        m, kc, vc = L.mix, cache.k[L.pool], cache.v[L.pool]
        with TimeLine("QKV.linear"):
            x = ops.linear(h, L.qkv, L.qkv_b)
        with TimeLine("QKPO"):
            q = ops.head_prep(x, L.prep, self.eps, b.positions, self._rope(m.rot, 0), m.rot.dims if m.rot is not None else 0, kc, vc,
                              b.slots, cache.state[L.state[0]] if m.conv > 1 else None, b.state_slots, b.cu_q, b.kv_lens, meta=b)
        with TimeLine("MHA"):
            a = ops.paged_attention(q, kc, vc, b.block_table, b.cu_q, b.kv_lens, m.scale, group=L.group, q_off=L.q_off, meta=b,
                                    softcap=m.softcap, window=m.window, keep_first=m.keep_first, sinks=L.sinks)
        return a.reshape(a.shape[0], -1)

    def _attend(self, L: Layer, h: torch.Tensor, b: Batch, cache: PagedKVCache) -> torch.Tensor:
        m, li = L.mix, L.pool
        kc, vc, ks, vs = cache.k[li], cache.v[li], cache.ks[li], cache.vs[li]
        table, rot = self._rope(m.rot, 0), m.rot.dims if m.rot is not None else 0
        style = m.rot.style if m.rot is not None else "half"
        new_kv = L.hkv if L.own_kv else 0
        if h.is_cuda and not self.exact and ops.can_fuse_qkv_rope(L.qkv, h.shape[0], L.kd, kc, ks, None, None, style):
            with TimeLine("QKV.linear+QKPO"):
                q = ops.qkv_linear_rope_cache(h, L.qkv, None, None, L.hq, new_kv, b.positions, table, rot, style, kc, vc,
                                              b.slots)
        else:
            with TimeLine("QKV.linear"):
                qkv = ops.linear(h, L.qkv)
            with TimeLine("QKPO"):
                q = ops.qkv_rope_cache(qkv, L.hq, new_kv, L.kd, b.positions, table, rot, style, kc, vc, ks, vs, b.slots,
                                       dv=L.vd)
        with TimeLine("MHA"):
            a = ops.paged_attention(q, kc, vc, b.block_table, b.cu_q, b.kv_lens, m.scale, ks, vs, group=L.group,
                                    q_off=L.q_off, meta=b, softcap=m.softcap, window=m.window, keep_first=m.keep_first,
                                    sinks=L.sinks)
        return a.reshape(a.shape[0], -1)

    def _ff(self, L: Layer, h: torch.Tensor) -> torch.Tensor:
        if L.mlp_kind == "moe":
            with TimeLine("MoE"):
                return self._experts(L, h)
        with TimeLine("LlamaMLP"):
            return self._row_parallel(ops.linear_gated(h, L.gate_up, L.act, L.gate_up_b, L.limit), L.down, L.down_b, None)

    def _experts(self, L: Layer, h: torch.Tensor) -> torch.Tensor:
        """Mixture of experts -> fp32 rows (summed over tensor-parallel ranks)."""
        f = L.moe
        logits = ops.linear(h, L.router, L.router_b, out_dtype=torch.float32)
        if f.scoring == "chosen":
            idx, w = ops.route(logits, "mixtral", f.top)
        else:
            idx, w = ops.route(logits, "deepseek", f.top, L.correction, f.groups, f.keep_groups, f.scale, f.renorm, f.scoring)
        shared = None
        if L.shared is not None:
            # few rows: the product leaves in fp32; prompts: in the activation type, like the experts' own rows
            u = ops.linear_gated(h, L.shared[0], L.act) if f.gated else ops.linear(h, L.shared[0], act=L.act)
            shared = ops.linear(u, L.shared[1], out_dtype=torch.float32 if h.shape[0] <= 128 else None)
        out = ops.moe_experts(h, idx, w, L.experts, L.act, L.e0, gated=f.gated, add=shared)
        if self.tp > 1:
            peer = getattr(self.ctx, "peer", None)
            if peer is not None and out.is_cuda and out.numel() <= peer.slot:
                return peer.all_reduce(out.contiguous())
            return self.ctx.all_reduce(out)
        return out

    def _side(self, L: Layer, x: torch.Tensor, e: torch.Tensor) -> torch.Tensor:
        """The token's own side embedding, gated by the residual stream `x` (in the activation type), as wide as it."""
        with TimeLine("Side"):
            n = L.side_gate.out_features
            g = ops.linear(x, L.side_gate, act="gelu_tanh", times=e[:, L.side_at:L.side_at + n])
            return ops.linear(g, L.side_proj)

    def _add_norm(self, x, y, post, nxt, **kw):
        return ops.residual_norm(x, y, post, nxt, self.eps, self.spec.norm, h_dtype=self.act_dtype, mult=self.cfg.residual_mult, **kw)

    def _sum_norm(self, x, y, post, nxt=None, **kw):
        """x = norm(alpha * x + y), and the same in the activation type or, with `nxt`, one more norm of it."""
        return self._add_norm(x, y, post, nxt, raw=nxt is None, carry=self.cfg.residual_carry, post_sum=True, **kw)

    def _logits(self, h):
        with TimeLine("DistLinear.forward"):
            cap = self.cfg.logit_softcap
            if cap > 0:
                return ops.linear(h, self.lm_head, act="softcap", res_scale=cap, out_dtype=torch.float32)
            return ops.linear(h, self.lm_head, out_dtype=torch.float32)

    def _forward_sum_norm(self, b: Batch, cache: PagedKVCache, hidden, step) -> torch.Tensor:
        """The stream is the norm of the residual sum: one launch behind each sublayer makes the sum, its norm, the stream and the
        next product's input; the last one makes the final norm too, on the rows whose logits are wanted."""
        dump = (lambda name, x: debugger.dump(name, x[:, :self.W], self.ctx.rank, step)) if debugger.enabled() else lambda name, x: None
        kw = dict(ids=b.ids, table=self.wte, embed_scale=self.cfg.embed_scale) if self.first_stage else {}
        x, h = self._add_norm(None if self.first_stage else hidden, None, None, None, raw=True, **kw)
        dump("embedding", x)
        for n, L in enumerate(self.runs):
            last = n + 1 == len(self.runs) and self.last_stage
            y, post = self._mixer(L, h, b, cache, x), L.norm1
            if L.mlp_kind != "none":
                x, h = self._sum_norm(x, y, post)
                dump(f"layer{L.idx}_attn_out", x)
                y, post = self._ff(L, h), L.norm2
            if last and not debugger.enabled():
                break
            x, h = self._sum_norm(x, y, post)
            dump(f"layer{L.idx}_ffn_out", x)
        if not self.last_stage:
            return x
        if b.logit_rows is not None and b.logit_rows.numel() == 0:
            return torch.empty(0, self.v1 - self.v0, dtype=torch.float32, device=x.device)
        if debugger.enabled():
            _, h = self._add_norm(x, None, None, self.final, rows=b.logit_rows, keep_x=False)
        else:
            _, h = self._sum_norm(x, y, post, self.final, rows=b.logit_rows, keep_x=False)
        return self._logits(h)

    def forward(self, b: Batch, cache: PagedKVCache, hidden: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Local logits on the last stage, the residual stream otherwise.  The norm of each sublayer's output, the
        residual sum, the vector in front of a pass of looped layers and the norm in front of the next sublayer are one
        launch; so are the embedding and the first norm, and on the last stage the last sum and the final norm, on the
        rows whose logits are wanted."""
        self._ensure_positions(b, cache)
        dbg = debugger.enabled()
        step = debugger.next_step() if dbg else 0
        with TimeLine("Decoder.forward"):
            if self.spec.sum_norm:
                return self._forward_sum_norm(b, cache, hidden, step)
            first = self.runs[0]
            if self.first_stage:
                x, h = self._add_norm(None, None, None, first.norm1, ids=b.ids, table=self.wte, embed_scale=self.cfg.embed_scale,
                                      add=first.step)
            else:
                x, h = self._add_norm(hidden, None, None, first.norm1, add=first.step)
            if dbg:
                debugger.dump("embedding", x[:, :self.W], self.ctx.rank, step)
            side = ops.embedding(b.ids, self.side_embed, 1.0, self.act_dtype) if self.side_embed is not None else None
            for n, L in enumerate(self.runs):
                nxt = self.runs[n + 1] if n + 1 < len(self.runs) else None
                y, post = self._mixer(L, h, b, cache, x), L.norm1b
                if L.mlp_kind != "none":
                    x, h = self._add_norm(x, y, post, L.norm2)
                    if dbg:
                        debugger.dump(f"layer{L.idx}_attn_out", x[:, :self.W], self.ctx.rank, step)
                    y, post = self._ff(L, h), L.norm2b
                if L.side_gate is not None:
                    x, h = self._add_norm(x, y, post, None, raw=True)
                    y, post = self._side(L, h, side), L.side_norm
                if dbg or nxt is None and not self.last_stage:
                    x, _ = self._add_norm(x, y, post, None)
                    y = post = None
                if dbg:
                    debugger.dump(f"layer{L.idx}_ffn_out", x[:, :self.W], self.ctx.rank, step)
                if nxt is not None:
                    x, h = self._add_norm(x, y, post, nxt.norm1, add=nxt.step)
            if not self.last_stage:
                return x
            if b.logit_rows is not None and b.logit_rows.numel() == 0:
                return torch.empty(0, self.v1 - self.v0, dtype=torch.float32, device=x.device)
            _, h = self._add_norm(x, y, post, self.final, rows=b.logit_rows, keep_x=False)
            return self._logits(h)

    # -- sizes ------------------------------------------------------------------------------
    def plan_splits(self, B: int, max_kv: int, int8: bool) -> Optional[int]:
        return None                               # windows differ from layer to layer: each launch plans its own split

    def kv_geometry(self):
        first = self.pool_shapes[0] if self.pool_shapes else (0, 0, 0)
        return dict(kv_heads=first[0], k_dim=first[1], v_dim=first[2], latent=False, layers=self.pool_shapes,
                    states=self.state_shapes)
