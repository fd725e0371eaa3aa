"""Synthetic checkpoints in the converted-model layout (config.ini + .bin), for tests and
benchmarks: random N(0, std) weights of a named architecture, written exactly where the
converters of the reference put them (``src/xfastertransformer/tools/llama_convert.py:177-233``,
``mixtral_convert.py:196-215``, ``qwen3_convert.py:120-160``, ``deepseek_moe_convert.py:182-375``,
``opt_convert.py``, ``chatglm2_convert.py``).

`config_only(path, cfg)` writes just config.ini: together with ``XFT_FAKE_MODEL=2`` the engine
draws the weights on the device, which is how the large benchmark configs are built.
"""
from __future__ import annotations

import os
from typing import Dict, Optional

import torch

from ..config import PARALLEL_PARTS, ModelConfig, RopeConfig
from ..ops import reference as R
from ..runtime.loader import write_bin, write_safetensors

PRESETS: Dict[str, dict] = {
    # BASELINE configs
    "tiny-llama": dict(model_type="llama", num_layer=2, hidden_size=256, head_num=4, kv_head_num=4, size_per_head=64,
                       inter_size=688, vocab_size=32000, max_pos_seq_len=2048, layernorm_eps=1e-6),
    "llama-2-7b": dict(model_type="llama", num_layer=32, hidden_size=4096, head_num=32, kv_head_num=32,
                       size_per_head=128, inter_size=11008, vocab_size=32000, max_pos_seq_len=4096),
    "llama-2-70b": dict(model_type="llama", num_layer=80, hidden_size=8192, head_num=64, kv_head_num=8,
                        size_per_head=128, inter_size=28672, vocab_size=32000, max_pos_seq_len=4096),
    # one tensor-parallel rank's share of Llama-2-70B at TP=8 (8 q heads + 1 kv head, FFN slice 3584, vocab slice
    # 4000) as a stand-alone model: isolates per-GPU kernel time from communication when profiling on one GPU
    "llama-2-70b-tp8-slice": dict(model_type="llama", num_layer=80, hidden_size=8192, head_num=8, kv_head_num=1,
                                  size_per_head=128, inter_size=3584, vocab_size=4000, max_pos_seq_len=4096),
    "mixtral-8x7b": dict(model_type="mixtral", num_layer=32, hidden_size=4096, head_num=32, kv_head_num=8,
                         size_per_head=128, inter_size=14336, vocab_size=32000, max_pos_seq_len=32768,
                         sparse_experts=8, num_experts_per_tok=2, rope=RopeConfig(theta=1e6)),
    "deepseek-v3": dict(model_type="deepseek_moe", num_layer=61, hidden_size=7168, head_num=128, kv_head_num=128,
                        size_per_head=128, inter_size=18432, vocab_size=129280, max_pos_seq_len=163840,
                        q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                        moe_intermediate_size=2048, first_k_dense_replace=3, dense_experts=1, sparse_experts=256,
                        routed_scaling_factor=2.5, topk_method="noaux_tc", n_group=8, topk_group=4,
                        num_experts_per_tok=8, norm_topk_prob=True, scoring_func="sigmoid",
                        weight_data_type="fp8_e4m3",
                        rope=RopeConfig(theta=10000, scaling_type="yarn", scaling_factor=40, original_max_pos=4096,
                                        beta_fast=32, beta_slow=1, mscale=1.0, mscale_all_dim=1.0)),
}


def kafipel_config(width: int, heads: int, kv_heads: int, ff: int, layers: int, vocab: int = 32000, dim: int = 128,
                   window: int = 1024, keep_first: int = 4, share: bool = True, eps: float = 1e-5) -> dict:
    """config.json of a Kafipel model with equal layers; with `share`, the second half of them reads the keys and values of
    the last layer of the first half."""
    out = []
    for i in range(layers):
        m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": 50.0,
             "rot": {"dims": dim // 2, "base": 500000.0,
                     "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}},
             "mask": {"size": window, "keep_first": keep_first}}
        if share and i >= max(layers // 2, 1):
            m["kv_from"] = max(layers // 2, 1) - 1
        out.append({"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Kafipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}


def vepivik_config(width: int, heads: int, kv_heads: int, layers: int, experts: int, top: int, ff: int, shared: int,
                   vocab: int = 32000, dim: int = 128, rot_dim: int = 64, vdim: int = 128, kv_rank: int = 512, window: int = 1024,
                   latent_window: int = 4096, latent_only: bool = False, share: bool = True, eps: float = 1e-5,
                   scale: float = 4.0) -> dict:
    """config.json of a Vepivik model: attention and latent-attention layers in turn (`latent_only`: the latter alone); with
    `share`, every second latent layer reads the latents of the one before it."""
    out, owner, n = [], None, 0
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    for i in range(layers):
        if i % 2 == 0 and not latent_only:
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "mask": {"size": window}}
            out.append({"type": "attention", "mixer": m, "mlp": mlp})
            continue
        m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": (dim + rot_dim) ** -0.5,
             "mask": {"size": latent_window},
             "rot": {"dims": rot_dim, "base": 10000.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        if share and n % 2 == 1:
            m["kv_from"] = owner
        else:
            owner = i
        n += 1
        out.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return {"architecture": "Vepivik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": out}


def botusun_config(width: int, heads: int, kv_heads: int, layers: int, ff: int, experts: int, top: int, groups: int, keep: int,
                   vocab: int = 32000, dim: int = 128, window: int = 1024, gla_heads: int = 16, gla_dim: int = 128,
                   gla_vdim: int = 128, tau: float = 16.0, conv: int = 4, times: int = 1, side: int = 128, gla_every: int = 2,
                   eps: float = 1e-5, scale: float = 4.0, mult: float = 0.5) -> dict:
    """config.json of a Botusun model: every `gla_every`-th layer is gated linear attention, the others windowed attention
    whose values are its keys; the middle half of the layers runs `times` times."""
    out = []
    for i in range(layers):
        mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": 1.0,
                                                               "groups": {"count": groups, "keep": keep}}}
        if gla_every and i % gla_every == gla_every - 1:
            m = {"heads": gla_heads, "dim": gla_dim, "vdim": gla_vdim, "tau": tau}
            out.append({"type": "gla", "mixer": m, "mlp": mlp})
        else:
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "conv": conv, "mask": {"size": window},
                 "rot": {"dims": dim // 2, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
            out.append({"type": "attention", "mixer": m, "mlp": mlp})
    return {"architecture": "Botusun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": out,
            "residual_mult": mult, "loop": {"start": layers // 4, "stop": layers - layers // 4, "times": times}, "token_side": {"dim": side}}


def dagezen_config(width: int, layers: int, heads: int, kv_heads: int, ff: int, experts: int, top: int, expert_ff: int, vocab: int = 32000,
                   dim: int = 128, window: int = 1024, right_heads: int = 0, latent_dim: int = 128, rot_dim: int = 64, vdim: int = 128,
                   kv_rank: int = 512, ssm_heads: int = 0, ssm_vdim: int = 64, state: int = 128, groups: int = 1, conv: int = 4,
                   norm_groups: int = 1, kinds: str = "mlp", eps: float = 1e-5, alpha: float = 2.5, cap: float = 30.0) -> dict:
    """config.json of a Dagezen model: the mixers take turns as `kinds` says (m: state space, l: latent attention, p: attention with
    mixed heads beside time mixing), dense feed-forwards and experts take turns by layer."""
    out = []
    for i in range(layers):
        k = kinds[i % len(kinds)]
        if k == "m":
            e = {"type": "mamba2", "mixer": {"heads": ssm_heads or 2 * width // ssm_vdim, "vdim": ssm_vdim, "state": state, "groups": groups,
                                             "norm_groups": norm_groups, "conv": conv}}
        elif k == "l":
            e = {"type": "latent_attention", "mixer": {"heads": heads, "dim": latent_dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                       "scale": (latent_dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": 50000.0}}}
        else:
            e = {"type": "parallel", "mixer": {
                "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window}},
                "right": {"heads": right_heads or heads, "dim": dim}, "left_scale": 0.7, "right_scale": 1.0}}
        dense = {"kind": "dense", "ff": ff, "limit": 7.0}
        e["mlp"] = dense if i % 2 == 0 or not experts else {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}}
        out.append(e)
    return {"architecture": "Dagezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out, "postln_alpha": alpha,
            "logit_softcap": cap}


LAYERED_PRESETS: Dict[str, tuple] = {
    "tiny-kafipel": (kafipel_config, dict(width=192, heads=6, kv_heads=2, ff=512, layers=3, vocab=1000, dim=64, window=48)),
    "kafipel-1b": (kafipel_config, dict(width=2048, heads=16, kv_heads=4, ff=5632, layers=16)),
    "kafipel-8b": (kafipel_config, dict(width=4096, heads=32, kv_heads=8, ff=14336, layers=32)),
    "tiny-vepivik": (vepivik_config, dict(width=192, heads=5, kv_heads=1, layers=4, experts=6, top=2, ff=56, shared=72, vocab=1000, dim=40,
                                          rot_dim=24, vdim=32, kv_rank=72, window=48, latent_window=90)),
    "tiny-botusun": (botusun_config, dict(width=192, heads=6, kv_heads=3, layers=4, ff=40, experts=6, top=2, groups=3, keep=2, vocab=1000,
                                          dim=40, window=48, gla_heads=3, gla_dim=24, gla_vdim=40, conv=3, times=2, side=20)),
    "tiny-dagezen": (dagezen_config, dict(width=192, layers=4, heads=6, kv_heads=3, ff=88, experts=6, top=2, expert_ff=40, vocab=1000, dim=40,
                                          window=48, right_heads=2, latent_dim=24, rot_dim=16, vdim=40, kv_rank=72, ssm_heads=6, ssm_vdim=24,
                                          state=40, groups=2, conv=3, norm_groups=3)),
    "dagezen-lite": (dagezen_config, dict(width=2048, layers=18, heads=16, kv_heads=4, ff=5632, experts=64, top=6, expert_ff=1408)),
    "botusun-lite": (botusun_config, dict(width=2048, heads=16, kv_heads=4, layers=16, ff=1408, experts=64, top=6, groups=8, keep=4)),
    "vepivik-lite": (vepivik_config, dict(width=2048, heads=16, kv_heads=4, layers=26, experts=64, top=6, ff=1408, shared=2816)),
}


def _write_layered(path: str, cfg: ModelConfig, seed: int, std: float) -> str:
    """config.json and model.safetensors of a layered design, every tensor N(0, std) (norm gains around one)."""
    from ..models.registry import family_for
    cfg.to_ini(path)
    spec = family_for(cfg)
    g = torch.Generator().manual_seed(seed)
    W, t = cfg.hidden_size, {}

    def put(name, *shape, around=0.0, s=std):
        t[name] = (around + torch.randn(*shape, generator=g) * s).bfloat16()

    def gain(name, n=W, bias=False):
        put(name, n, around=1.0, s=0.05)
        if bias:
            put(name + ".b", n)

    def sum_norm_mixer(p, m):
        """Tensors of the mixers that only designs with a normalised residual sum have."""
        if m.kind == "ssd":
            n = m.heads * m.vdim
            c = n + 2 * m.groups * m.dim
            put(p + "in", n + c + m.heads, W)
            put(p + "conv", c, m.conv, around=1.0 / m.conv, s=0.1)
            put(p + "conv.b", c)
            put(p + "dt_bias", m.heads, around=-2.0, s=1.0)
            put(p + "A_log", m.heads, around=0.5, s=0.7)
            put(p + "D", m.heads, around=1.0)
            gain(p + "norm", n)
            put(p + "o", W, n)
        elif m.kind == "talking":
            n, k = m.heads * m.dim, m.kv_heads * m.dim
            put(p + "q", n, W)
            put(p + "k", k, W)
            put(p + "g", n, W)
            gain(p + "q.norm", n)
            gain(p + "k.norm", k)
            put(p + "r1", m.heads, around=0.5, s=0.1)
            put(p + "r2", m.heads, around=0.1, s=0.02)
            t[p + "talk"] = (torch.eye(m.heads) + torch.randn(m.heads, m.heads, generator=g) * 0.1).bfloat16()
            put(p + "o", W, n)
        elif m.kind == "time_mix":
            n, rank = m.heads * m.dim, 16
            for x in "rkvgw":
                put(p + "mu." + x, W, around=0.5, s=0.1)
            for x in "rkvg":
                put(p + x, n, W)
            put(p + "w1", rank, W)
            put(p + "w2", n, rank)
            put(p + "w0", n, around=-2.0, s=1.0)
            put(p + "u", m.heads, m.dim, around=1.0)
            gain(p + "norm", n)
            put(p + "o", W, n)

    put("embed", cfg.vocab_size, W)
    gain("final.norm", bias=spec.norm_bias)
    if not spec.tied_head:
        put("head", cfg.vocab_size, W)
    for i, lc in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lc.mixer, lc.moe
        for n in ("norm1",) + (("norm2",) if lc.ff or f else ()):
            gain(p + n, bias=spec.norm_bias)
            if spec.post_norm:
                gain(p + n + "b")
        if spec.sum_norm and m.kind != "latent":
            for pre, q in zip([f"mix.{n}." for n, _ in PARALLEL_PARTS], m.parts) if m.parts else [("mix.", m)]:
                sum_norm_mixer(p + pre, q)
            m = None
        if m is not None:
            put(p + "mix.q", m.heads * (m.dim + m.rot_dim), W)
            if m.kind == "gla":
                rank = 16
                put(p + "mix.k", m.heads * m.dim, W)
                put(p + "mix.v", m.heads * m.vdim, W)
                put(p + "mix.g", m.heads * m.vdim, W)
                put(p + "mix.a1", rank, W)
                put(p + "mix.a2", m.heads * m.dim, rank)
                put(p + "mix.a2.b", m.heads * m.dim, around=2.0)
                gain(p + "mix.norm", m.vdim)
            if m.kind == "latent":
                if m.kv_from < 0:
                    put(p + "mix.dkv", m.kv_rank + m.rot_dim, W)
                    gain(p + "mix.dkv.norm", m.kv_rank)
                put(p + "mix.uk", m.heads * m.dim, m.kv_rank)
                put(p + "mix.uv", m.heads * m.vdim, m.kv_rank)
                if m.gate:
                    put(p + "mix.g", m.heads * (1 if m.head_gate else m.vdim), W)
            elif m.values_from_keys:
                put(p + "mix.k", m.kv_heads * m.dim, W)
                for x, n in (("q", m.heads), ("k", m.kv_heads)):
                    if m.qk_bias:
                        put(p + f"mix.{x}.b", n * m.dim)
                    if m.qk_norm:
                        gain(p + f"mix.{x}.norm", m.dim)
                    if m.conv:
                        put(p + f"mix.{x}.conv", n * m.dim, m.conv, around=1.0 / m.conv, s=0.1)
            elif m.kind != "gla" and m.kv_from < 0:
                put(p + "mix.k", m.kv_heads * m.dim, W)
                put(p + "mix.v", m.kv_heads * m.vdim, W)
            if spec.sinks or m.sinks:
                put(p + "mix.sink", m.heads, s=1.0)
            put(p + "mix.o", W, m.heads * m.vdim)
        if lc.ff:
            put(p + "mlp.gate", lc.ff, W)
            put(p + "mlp.up", lc.ff, W)
            put(p + "mlp.down", W, lc.ff)
            if lc.ff_bias:
                for x, n in (("gate", lc.ff), ("up", lc.ff), ("down", W)):
                    put(p + f"mlp.{x}.b", n)
        if f:
            put(p + "mlp.router", f.experts, W)
            if f.router_bias:
                put(p + "mlp.router.b", f.experts)
            if f.correction:
                put(p + "mlp.correction", f.experts)
            for n, ff in [(f"e{e}", f.ff) for e in range(f.experts)] + ([("shared", f.shared)] if f.shared else []):
                for x in ("gate", "up") if f.gated else ("up",):
                    put(p + f"mlp.{n}.{x}", ff, W)
                put(p + f"mlp.{n}.down", W, ff)
        if cfg.side_dim:
            put(p + "side.gate", cfg.side_dim, W)
            put(p + "side.proj", W, cfg.side_dim)
            gain(p + "side.norm")
    if cfg.side_dim:
        put("side.embed", cfg.vocab_size, cfg.side_dim * len(cfg.layers), s=1.0)
    if cfg.loop:
        put("loop.step", cfg.loop.times, W)
    write_safetensors(os.path.join(path, "model.safetensors"), t)
    return path


def preset(name: str, **over) -> ModelConfig:
    if name in LAYERED_PRESETS:
        make, sizes = LAYERED_PRESETS[name]
        return ModelConfig.from_dict(make(**dict(sizes, **over)))
    if name not in PRESETS:
        from .model_zoo import ZOO          # public model architectures (examples/model_config)
        if name not in ZOO:
            raise KeyError(f"unknown model preset '{name}'; known: {sorted(set(PRESETS) | set(LAYERED_PRESETS) | set(ZOO))}")
        d = dict(ZOO[name])
    else:
        d = dict(PRESETS[name])
    d.update(over)
    d.setdefault("activation_type", "silu")
    d.setdefault("weight_data_type", "bf16")
    d.setdefault("start_id", 1)
    d.setdefault("end_id", 2)
    return ModelConfig(**d)


def config_only(path: str, cfg: ModelConfig) -> str:
    cfg.to_ini(path)
    return path


def write_synthetic_checkpoint(path: str, cfg: ModelConfig, seed: int = 0, std: float = 0.02,
                               dtype: Optional[str] = None) -> str:
    """Write config.ini and every tensor.  Linear weights are drawn in HF orientation [out,in]
    in fp32, rounded to `dtype`, and stored transposed ([in,out]) like the converters do."""
    if cfg.layers:
        return _write_layered(path, cfg, seed, std)
    dtype = dtype or cfg.weight_data_type
    os.makedirs(path, exist_ok=True)
    cfg.weight_data_type = dtype
    cfg.to_ini(path)
    g = torch.Generator().manual_seed(seed)
    H, D = cfg.hidden_size, cfg.size_per_head
    mt = cfg.model_type

    def rnd(*shape, s=std):
        return torch.randn(*shape, generator=g) * s

    def put(name, t, dt=None):
        write_bin(os.path.join(path, name), t, dt or dtype)

    def put_lin(name, out_f, in_f, dt=None):
        """HF weight [out,in] -> file [in,out]."""
        put(name, rnd(out_f, in_f).t().contiguous(), dt)

    def put_fp8_lin(base, out_f, in_f):
        w = rnd(out_f, in_f)
        if dtype == "fp8_e4m3":
            q, s = R.quantize_fp8_block(w)              # [out,in], [out/128,in/128]
            put(base + ".weight.bin", q.view(torch.uint8).t().contiguous().view(torch.float8_e4m3fn), "fp8_e4m3")
            put(base + ".weight_scale_inv.bin", s.t().contiguous(), "fp32")
        else:
            put(base + ".weight.bin", w.t().contiguous(), dtype)

    norm_dt = "bf16" if mt == "deepseek_moe" else dtype
    emb_dt = "bf16" if mt == "deepseek_moe" else dtype
    put("model.wte.bin", rnd(cfg.vocab_size, H), emb_dt)
    put("model.final_layernorm.weight.bin", 1.0 + rnd(H, s=0.05), norm_dt)
    put("model.lm_head.weight.bin", rnd(cfg.vocab_size, H), emb_dt)
    layer_norm = mt in ("gpt", "chatglm")
    if layer_norm:
        put("model.final_layernorm.bias.bin", rnd(H, s=0.05))
    if mt == "gpt":
        put("model.wpe.bin", rnd(cfg.max_pos_seq_len + 2, H))
    for i in range(cfg.num_layer):
        p = f"model.layers.{i}."
        put(p + "input_layernorm.weight.bin", 1.0 + rnd(H, s=0.05), norm_dt)
        put(p + "post_attention_layernorm.weight.bin", 1.0 + rnd(H, s=0.05), norm_dt)
        if layer_norm:
            put(p + "input_layernorm.bias.bin", rnd(H, s=0.05))
            put(p + "post_attention_layernorm.bias.bin", rnd(H, s=0.05))
        if mt == "deepseek_moe":
            nope, rope, vd = cfg.qk_nope_head_dim, cfg.qk_rope_head_dim, cfg.v_head_dim
            kvl, ql, nh = cfg.kv_lora_rank, cfg.q_lora_rank, cfg.head_num
            if ql > 0:
                put_fp8_lin(p + "self_attn.q_a_proj", ql, H)
                put(p + "self_attn.q_a_layernorm.weight.bin", 1.0 + rnd(ql, s=0.05), "bf16")
                put_fp8_lin(p + "self_attn.q_b_proj", nh * (nope + rope), ql)
            else:
                put_fp8_lin(p + "self_attn.q_a_proj", nh * (nope + rope), H)
            put_fp8_lin(p + "self_attn.kv_a_proj_with_mqa", kvl + rope, H)
            put(p + "self_attn.kv_a_layernorm.weight.bin", 1.0 + rnd(kvl, s=0.05), "bf16")
            put_fp8_lin(p + "self_attn.kv_b_proj", nh * (nope + vd), kvl)
            put_fp8_lin(p + "attention.dense", H, nh * vd)
            if i < cfg.first_k_dense_replace:
                for n, (o, k) in dict(gate=(cfg.inter_size, H), up=(cfg.inter_size, H), down=(H, cfg.inter_size)).items():
                    put_fp8_lin(p + f"mlp.{n}_proj", o, k)
            else:
                E, I = cfg.sparse_experts, cfg.moe_intermediate_size
                put(p + "mlp.gate.weight.bin", rnd(E, H, s=0.5).t().contiguous(), "bf16")
                if cfg.topk_method == "noaux_tc":
                    put(p + "mlp.gate.e_score_correction_bias.bin", rnd(E, s=0.1), "bf16")
                SI = cfg.dense_experts * I
                if SI:
                    for n, (o, k) in dict(gate=(SI, H), up=(SI, H), down=(H, SI)).items():
                        put_fp8_lin(p + f"mlp.shared_experts.{n}_proj", o, k)
                for e in range(E):
                    for n, (o, k) in dict(gate=(I, H), up=(I, H), down=(H, I)).items():
                        put_fp8_lin(p + f"mlp.experts.{e}.{n}_proj", o, k)
            continue
        qsz, kvsz = cfg.head_num * D, cfg.kv_head_num * D
        put_lin(p + "attention.query_key_value.weight.0.bin", qsz + 2 * kvsz, H)
        put_lin(p + "attention.dense.weight.0.bin", H, qsz)
        if mt in ("qwen", "qwen2", "chatglm", "chatglm2", "chatglm3", "chatglm4", "gpt"):
            put(p + "attention.query_key_value.bias.0.bin", rnd(qsz + 2 * kvsz, s=0.05))
        if mt in ("gpt", "chatglm", "telechat"):
            put(p + "attention.dense.bias.bin", rnd(H, s=0.05))
        if cfg.do_qk_norm:
            put(p + "attention.q_norm.weight.bin", 1.0 + rnd(D, s=0.05))
            put(p + "attention.k_norm.weight.bin", 1.0 + rnd(D, s=0.05))
        I = cfg.inter_size
        if mt in ("gpt", "chatglm"):
            put_lin(p + "mlp.dense_h_to_4h.weight.0.bin", I, H)
            put(p + "mlp.dense_h_to_4h.bias.0.bin", rnd(I, s=0.05))
            put_lin(p + "mlp.dense_4h_to_h.weight.0.bin", H, I)
            put(p + "mlp.dense_4h_to_h.bias.bin", rnd(H, s=0.05))
        elif mt in ("chatglm2", "chatglm3", "chatglm4"):
            put_lin(p + "mlp.dense_h_to_4h.weight.0.bin", 2 * I, H)
            put_lin(p + "mlp.dense_4h_to_h.weight.0.bin", H, I)
        elif mt == "mixtral":
            E = cfg.sparse_experts
            put(p + "moe.gate.weight.bin", rnd(E, H, s=0.5).t().contiguous())
            for e in range(E):
                put_lin(p + f"moe.sparse_experts.{e}.w1.0.bin", I, H)     # gate
                put_lin(p + f"moe.sparse_experts.{e}.w2.0.bin", I, H)     # up
                put_lin(p + f"moe.sparse_experts.{e}.w3.0.bin", H, I)     # down
        elif mt == "qwen3_moe":
            E, MI = cfg.sparse_experts, cfg.moe_intermediate_size or I
            put(p + "mlp.gate.weight.0.bin", rnd(E, H, s=0.5).t().contiguous())
            for e in range(E):
                put_lin(p + f"mlp.experts.{e}.gate_proj.weight.0.bin", MI, H)
                put_lin(p + f"mlp.experts.{e}.up_proj.weight.0.bin", MI, H)
                put_lin(p + f"mlp.experts.{e}.down_proj.weight.0.bin", H, MI)
        else:
            put_lin(p + "mlp.gate_proj.weight.0.bin", I, H)
            put_lin(p + "mlp.up_proj.weight.0.bin", I, H)
            put_lin(p + "mlp.down_proj.weight.0.bin", H, I)
    return path
