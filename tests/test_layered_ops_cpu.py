"""Mechanisms of layered designs one by one, on the CPU path, with inputs in which a fault stands out; and the files such
a model is read from."""
import json
import math
import os
import struct
import subprocess
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "tests"))

import layered_ops_cases as M  # noqa: E402
import oracle_layered as O  # noqa: E402
import xfastertransformer_b200 as xft  # noqa: E402
from xfastertransformer_b200.config import ModelConfig  # noqa: E402
from xfastertransformer_b200.models.registry import decoder_class, family_for  # noqa: E402
from xfastertransformer_b200.ops import reference as R  # noqa: E402
from xfastertransformer_b200.runtime.loader import SafetensorsFile, SafetensorsSource  # noqa: E402

CPU = torch.device("cpu")


@pytest.fixture(autouse=True)
def _cpu(monkeypatch):
    monkeypatch.setenv("XFT_ENGINE", "CPU")


@pytest.mark.parametrize("window,keep", [(40, 5), (64, 64), (1, 0), (1, 3), (129, 2), (300, 1), (33, 70)])
@pytest.mark.parametrize("decode", [False, True])
def test_window_edges(window, keep, decode):
    M.window_edges(CPU, torch.float32, 32, 32, window, keep, decode, 1e-5)


def test_sink_counts_once():
    M.sink_counts_once(CPU, torch.float32, 32, 1e-5)


def test_softcap():
    M.softcap(CPU, torch.float32, 32, 1e-5)


@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_residual_norm(kind):
    M.residual_norm(CPU, 77, kind, torch.float32, torch.float32, 2e-6)


@pytest.mark.parametrize("rot", [{"dims": 24, "base": 1000.0},
                                 {"dims": 16, "base": 50.0, "scaling": {"factor": 5.0, "original": 64, "fast": 6.0, "slow": 0.5}},
                                 {"dims": 40, "base": 1e5, "scaling": {"factor": 2.5, "original": 4096, "fast": 40.0, "slow": 2.0}},
                                 # the two ends of the ramp fall on one pair
                                 {"dims": 8, "base": 1e6, "scaling": {"factor": 3.0, "original": 32, "fast": 4.0, "slow": 3.9}},
                                 {"dims": 2, "base": 10.0, "scaling": {"factor": 7.0, "original": 10, "fast": 1.0, "slow": 1.0}}])
def test_rotation(rot):
    M.rotation(CPU, torch.float32, rot, 40, 24, 2e-5)


def test_rotation_table_grows(tmp_path):
    """Positions past the first table: it is made anew, longer, and the early rows stay what they were."""
    cfg = O.config([O.attention_layer(size=9, rot_dims=8, base=31.0)], width=64, vocab=50)
    p = O.write_checkpoint(str(tmp_path / "m"), cfg, O.random_weights(cfg))
    d = xft.AutoModel.from_pretrained(p, dtype="fp32").model.decoder
    rot = d.cfg.layers[0].mixer.rot
    a = d._rope(rot, 0)
    b = d._rope(rot, a.shape[0] + 1)
    assert b.shape[0] >= 2 * a.shape[0] and torch.equal(b[:a.shape[0]], a)
    f, _ = O.rotary_frequencies({"dims": 8, "base": 31.0})
    assert abs(float(b[-1, 1]) - math.cos((b.shape[0] - 1) * f[1])) < 2e-4


@pytest.mark.parametrize("window", [40, 64, 1, 129, 0])
@pytest.mark.parametrize("decode", [False, True])
def test_latent_window_edges(window, decode):
    M.latent_window_edges(CPU, torch.float32, window, decode, 1e-5)


def test_latent_heads_and_prep():
    M.latent_heads_differ(CPU, torch.float32, 1e-5, False)
    M.latent_prep(CPU, torch.float32, 2e-5)


@pytest.mark.parametrize("T,E,top,ff,shared", [(9, 5, 2, 24, 40), (1, 7, 7, 8, 0), (30, 1, 1, 16, 16), (40, 33, 3, 20, 8)])
def test_experts(T, E, top, ff, shared):
    M.experts(CPU, torch.float32, 1e-5, T, E, top, ff, shared)


# ------------------------------------------------------------------------------------------ configuration
def _write(tmp_path, cfg, name="m"):
    return O.write_checkpoint(str(tmp_path / name), cfg, O.random_weights(cfg))


@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 40, 3, 17)])
@pytest.mark.parametrize("tau", [1.0, 9.0])
def test_gated_linear(sizes, tau):
    M.gated_linear(CPU, torch.float32, 2e-5, 2, 12, 20, 5, tau, (70, 33, 1, 6), sizes)


@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 40, 3, 17)])
@pytest.mark.parametrize("taps", [0, 1, 2, 4, 7])
def test_head_prep(sizes, taps):
    M.head_prep(CPU, torch.float32, 2e-5, 3, 1, 12, 16, taps, (40, 13, 1, 2), sizes, {"dims": 6, "base": 300.0})
    M.head_prep(CPU, torch.float32, 2e-5, 2, 2, 8, 8, taps, (5, 20), sizes, norm=False)


@pytest.mark.parametrize("sc", [dict(factor=8.0, low=1.0, high=4.0, original=100), dict(factor=0.5, low=2.0, high=2.5, original=40),
                                dict(factor=3.0, low=1.0, high=50.0, original=5000), dict(factor=1.0, low=1.0, high=4.0, original=64)])
def test_banded_frequencies(sc):
    """Wavelengths on both sides of the bands and inside the ramp."""
    M.head_prep(CPU, torch.float32, 3e-5, 2, 1, 40, 40, 3, (500,), (600,), {"dims": 36, "base": 20000.0, "scaling": sc})


def test_residual_extras():
    M.residual_extras(CPU, 77, torch.float32, 2e-6)


def test_linear_times():
    M.linear_times(CPU, torch.float32, 1e-5, 9, 30, 12)


@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (8, 4, (2, 1)), (6, 2, (6, 3)), (9, 9, None), (5, 1, None), (10, 2, (1, 1))])
def test_grouped_route(E, top, groups):
    M.grouped_route(CPU, E, top, groups)


@pytest.mark.parametrize("T,E,top,ff,groups", [(9, 6, 2, 24, (3, 2)), (1, 4, 4, 8, None), (30, 8, 1, 16, (2, 1))])
def test_gated_experts(T, E, top, ff, groups):
    M.gated_experts(CPU, torch.float32, 1e-5, T, E, top, ff, groups=groups)


def test_layer_runs():
    """The order of looped layers, and what each run owns: a pass has pools and states of its own over shared weights."""
    import layered_cases as C
    for name in C.RECURRENT:
        cfg = C.CONFIGS[name]
        mine = [(i, max(t, 0)) for i, t in ModelConfig.from_dict(cfg).runs()]
        assert mine == [(i, t) for i, t, _ in O.layer_runs(cfg)], name


def test_recurrent_config_and_pools(tmp_path):
    import layered_cases as C
    cfg = C.CONFIGS["recurrent"]
    p = _write(tmp_path, cfg)
    c = ModelConfig.load(p)
    assert c.model_type == "botusun" and c.residual_mult == 0.35 and c.embed_scale == 1.7 and c.side_dim == 6
    a, g = c.layers[0].mixer, c.layers[1]
    assert (a.conv, a.values_from_keys, a.qk_norm, a.qk_bias, a.sink, a.rot.scaling) == (3, True, True, True, 0.0, "banded")
    assert (g.mixer.kind, g.mixer.tau, g.mixer.has_kv) == ("gla", 4.0, False)
    f = g.moe
    assert (f.scoring, f.renorm, f.scale, f.groups, f.keep_groups, f.gated, f.correction) == ("sigmoid", False, 1.7, 3, 2, True, True)
    m = xft.AutoModel.from_pretrained(p, dtype="fp32", max_cache_tokens=130, max_sequences=2)
    cache = m.model.cache
    # runs: 0, three times (1, 2), 3: four of them keep keys, four a matrix, one a convolution's inputs (layer 2 has one tap)
    assert len(cache.k) == 4 and [tuple(t.shape[1:]) for t in cache.state] == [(2, 180)] + [(3, 12, 20)] * 3 + [(2, 40, 24)]
    assert len(m.model.decoder.layers) == 4 and len(m.model.decoder.runs) == 8
    for i in range(2):
        m.set_input_cb([[1, 2, 3]], max_length=10)
    with pytest.raises(MemoryError, match="state"):
        m.set_input_cb([[1, 2, 3]], max_length=10)
    with pytest.raises(ValueError, match="int8"):
        xft.AutoModel.from_pretrained(p, dtype="bf16", kv_cache_dtype="int8")


def test_state_slots():
    """Slots of the state pools: taken and given back, copied by a fork, permuted by a reorder, kept when the pools grow."""
    from xfastertransformer_b200.runtime.kv_cache import PagedKVCache
    c = PagedKVCache(1, 1, 4, 4, "fp32", CPU, block_size=4, states=[((2,), torch.float32), ((3, 1), torch.float32)])
    for s in (7, 8, 9):
        c.add_sequence(s)
        c.append_slots(s, 5)
        for t in c.state:
            t[c.state_slot[s]] = s
    val = lambda s: [float(t[c.state_slot[s]].flatten()[0]) for t in c.state]
    c.fork(8, 20)
    assert val(20) == [8, 8] and c.state_slot[20] != c.state_slot[8]
    c.reorder([7, 8, 9], [1, 0, 0])
    assert [val(s) for s in (7, 8, 9)] == [[8, 8], [7, 7], [7, 7]]
    old, version = c.state_alloc.num_blocks, c.version
    for s in range(100, 100 + old):
        c.add_sequence(s)
    assert c.state_alloc.num_blocks > old and c.version > version and val(7) == [8, 8]
    with pytest.raises(RuntimeError, match="cannot go back"):
        c.truncate(7, 3)
    for s in [7, 8, 9, 20] + list(range(100, 100 + old)):
        c.free_sequence(s)
    assert c.state_alloc.num_free == c.state_alloc.num_blocks and not c.state_slot


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0]["mixer"].update(vdim=24), "size"), (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups")])
def test_recurrent_config_faults(tmp_path, change, match):
    import copy

    import layered_cases as C
    cfg = copy.deepcopy(C.CONFIGS["recurrent"])
    change(cfg)
    with pytest.raises(ValueError, match=match):
        ModelConfig.from_dict(cfg)


def test_config_is_read_per_layer(tmp_path):
    sc = {"factor": 2.5, "original": 77, "fast": 9.0, "slow": 0.7}
    cfg = O.config([O.attention_layer(heads=6, kv_heads=3, dim=20, vdim=28, size=11, keep=2, rot_dims=10, scaling=sc, scale=0.3,
                                      softcap=7.0, ff=44),
                    O.attention_layer(heads=2, kv_heads=2, mask=False, rot=False, softcap=None, ff=None)], eps=2e-3)
    c = ModelConfig.load(_write(tmp_path, cfg))
    a, b = c.layers
    assert (c.model_type, c.num_layer, c.hidden_size, c.vocab_size, c.layernorm_eps) == ("kafipel", 2, 96, 210, 2e-3)
    assert (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim, a.ff) == (6, 3, 20, 28, 44)
    assert (a.mixer.window, a.mixer.keep_first, a.mixer.softcap, a.mixer.scale, a.mixer.kv_from) == (11, 2, 7.0, 0.3, -1)
    r = a.mixer.rot
    assert (r.dims, r.base, r.factor, r.original, r.fast, r.slow) == (10, 10000.0, 2.5, 77, 9.0, 0.7)
    assert (b.mixer.window, b.mixer.softcap, b.mixer.rot, b.ff) == (0, 0.0, None, 0)
    assert family_for(c).layered and decoder_class(c).__name__ == "LayeredDecoder"
    c.to_ini(str(tmp_path / "again"))
    assert ModelConfig.load(str(tmp_path / "again")).layers == c.layers


def test_latent_config_is_read_per_layer(tmp_path):
    sc = {"factor": 2.5, "original": 77, "fast": 9.0, "slow": 0.7}
    cfg = O.vepivik([O.window_layer(heads=6, kv_heads=2, dim=20, vdim=28, size=11, scale=0.3, mlp=O.moe(ff=44, experts=9, top=4, shared=52)),
                     O.latent_layer(heads=5, dim=14, rot_dim=6, vdim=18, kv_rank=22, size=31, base=77.0, scaling=sc, scale=0.4),
                     O.latent_layer(heads=2, dim=30, rot_dim=6, vdim=4, kv_rank=22, base=77.0, scaling=sc, kv_from=1, mask=False,
                                    mlp=O.moe(shared=None))], eps=2e-3, scale=4.5)
    c = ModelConfig.load(_write(tmp_path, cfg))
    a, b, r = c.layers
    assert (c.model_type, c.embed_scale, c.layernorm_eps, c.num_layer) == ("vepivik", 4.5, 2e-3, 3)
    assert (a.mixer.kind, a.mixer.window, a.mixer.keep_first, a.mixer.rot, a.mixer.gate, a.ff) == ("attention", 11, 0, None, False, 0)
    assert (a.moe.experts, a.moe.top, a.moe.ff, a.moe.shared, a.ff_kind) == (9, 4, 44, 52, "moe")
    m = b.mixer
    assert (m.kind, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale) == ("latent", 5, 14, 6, 18, 22, 31, 0.4)
    assert (m.rot.dims, m.rot.base, m.rot.factor, m.rot.style, m.gate, b.moe, b.ff) == (6, 77.0, 2.5, "interleaved", True, None, 0)
    assert (r.mixer.kv_from, r.mixer.window, r.moe.shared) == (1, 0, 0)
    f = family_for(c)
    assert f.layered and f.tied_head and not f.post_norm and not f.sinks and f.norm == "rms"
    c.to_ini(str(tmp_path / "again"))
    assert ModelConfig.load(str(tmp_path / "again")).layers == c.layers


@pytest.mark.parametrize("change,match", [
    (lambda d: d["layers"][1]["mixer"].update(kv_rank=24), "heads differ"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(base=5.0), "heads differ"),
    (lambda d: d["layers"][1]["mixer"].update(kv_from=2), "not an earlier layer"),
    (lambda d: d["layers"][2]["mixer"].update(kv_from=0), "heads differ"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "of 6 experts"),
    (lambda d: d["layers"][0]["mlp"].update(kind="mixture"), "unsupported feed-forward"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "do not fit")])
def test_latent_config_faults(tmp_path, change, match):
    cfg = O.vepivik([O.latent_layer(mlp=O.moe()), O.latent_layer(kv_from=0), O.window_layer()])
    change(cfg)
    os.makedirs(tmp_path / "m")
    (tmp_path / "m" / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(ValueError, match=match):
        ModelConfig.load(str(tmp_path / "m"))


@pytest.mark.parametrize("change,match", [
    (lambda d: d.update(architecture="Other"), "unsupported architecture"),
    (lambda d: d["layers"][1].update(type="convolution"), "unsupported mixer"),
    (lambda d: d["layers"][1]["mlp"].update(kind="experts"), "unsupported feed-forward"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "query heads over"),
    (lambda d: d["layers"][1]["mixer"].update(kv_from=1), "not an earlier layer"),
    (lambda d: d["layers"][1]["mixer"].update(kv_from=0, dim=16), "heads differ"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=34), "do not fit")])
def test_config_faults(tmp_path, change, match):
    cfg = O.config([O.attention_layer(), O.attention_layer()])
    change(cfg)
    os.makedirs(tmp_path / "m")
    (tmp_path / "m" / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(ValueError, match=match):
        ModelConfig.load(str(tmp_path / "m"))


# ------------------------------------------------------------------------------------------ weights
def test_safetensors_faults(tmp_path):
    cfg = O.config([O.attention_layer()])
    p = _write(tmp_path, cfg)
    f = os.path.join(p, "model.safetensors")
    st = SafetensorsFile(f)
    W = O.random_weights(cfg)
    assert torch.equal(st.read("l0.mix.q", (128, 96)), W["l0.mix.q"])
    assert torch.equal(st.read("l0.mix.q", (128, 96), rows=(32, 64), cols=(3, 7)), W["l0.mix.q"][32:64, 3:7])
    with pytest.raises(ValueError, match="expected"):
        st.read("l0.mix.q", (96, 128))
    with pytest.raises(KeyError):
        st.read("l0.mix.z", (1,))
    raw = open(f, "rb").read()
    open(f, "wb").write(raw[:-2])
    with pytest.raises(ValueError, match="extent"):
        SafetensorsFile(f)
    open(f, "wb").write(raw[:5])
    with pytest.raises(ValueError, match="truncated"):
        SafetensorsFile(f)
    with pytest.raises(FileNotFoundError):
        SafetensorsSource(str(tmp_path), CPU)


def test_safetensors_types_and_odd_offsets(tmp_path):
    """fp32, int32 and bf16 tensors, one of them at an odd offset."""
    a = torch.arange(6, dtype=torch.int32).view(2, 3)
    b = torch.randn(3)
    c = torch.randn(5).bfloat16()
    parts = [("u", "U8", [1], b"\x07"), ("a", "I32", [2, 3], a.numpy().tobytes()), ("b", "F32", [3], b.numpy().tobytes()),
             ("c", "BF16", [5], c.view(torch.int16).numpy().tobytes())]
    head, off = {"__metadata__": {"x": "y"}}, 0
    for n, dt, sh, raw in parts:
        head[n] = {"dtype": dt, "shape": sh, "data_offsets": [off, off + len(raw)]}
        off += len(raw)
    h = json.dumps(head).encode()
    f = tmp_path / "t.safetensors"
    f.write_bytes(struct.pack("<Q", len(h)) + h + b"".join(x[3] for x in parts))
    st = SafetensorsFile(str(f))
    assert torch.equal(st.read("a", (2, 3)), a) and torch.equal(st.read("b", (3,)), b) and torch.equal(st.read("c", (5,)), c)


# ------------------------------------------------------------------------------------------ Dagezen's mechanisms
@pytest.mark.parametrize("sizes", [(1000,), (1,), (1, 40, 3, 17)])
def test_time_mix(sizes):
    M.time_mix(CPU, torch.float32, 4e-5, 2, 12, 5, (70, 33, 1, 6), sizes)


@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 5, 3)])
def test_token_shift(sizes):
    M.token_shift(CPU, torch.float32, (30, 9, 1, 2), sizes)


@pytest.mark.parametrize("sizes", [(1000,), (1,), (1, 40, 3, 17)])
@pytest.mark.parametrize("H,P,N,G,parts,taps", [(4, 12, 20, 2, 3, 3), (2, 8, 5, 1, 1, 1), (3, 16, 24, 3, 4, 7)])
def test_state_space(H, P, N, G, parts, taps, sizes):
    M.state_space(CPU, torch.float32, 4e-5, H, P, N, G, parts, taps, (70, 33, 1, 6), sizes)


@pytest.mark.parametrize("window", [40, 64, 1, 129, 0])
@pytest.mark.parametrize("decode", [False, True])
def test_talking_edges(window, decode):
    M.talking_edges(CPU, torch.float32, 2e-5, 6, 3, 20, 20, window, decode)


def test_talking_scores_and_prep():
    M.talking_scores(CPU, torch.float32, 2e-5, 4, 1, 24, 24, 33, False)
    M.talking_prep(CPU, torch.float32, 1e-5, 5, 1, 20, 20)


@pytest.mark.parametrize("decode", [False, True])
def test_latent_sinks(decode):
    M.latent_sinks(CPU, torch.float32, 2e-5, decode)


def test_sum_norm_gates_and_experts():
    M.sum_norm(CPU, 90, torch.float32, 4e-6)
    M.clamped_gate(CPU, torch.float32, 1e-5, 9, 40, 24, 0.7)
    M.activations(CPU, torch.float32, 1e-5, 9, 40, 24)
    M.linear_parts(CPU, torch.float32, 1e-5, 9, 40, 24)
    M.chosen_experts(CPU, torch.float32, 1e-5, 30, 6, 3, 20)


def test_dagezen_config_is_read_per_layer(tmp_path):
    cfg = O.dagezen([O.mamba_layer(heads=6, vdim=10, state=14, groups=3, norm_groups=5, conv=2, mlp=O.clamped(30, 0.25)),
                     O.sink_latent_layer(heads=5, dim=14, rot_dim=6, vdim=18, kv_rank=22, base=77.0, scale=0.4, mlp=O.chosen_moe(12, 9, 4)),
                     O.parallel_layer(heads=6, kv_heads=2, dim=20, size=11, scale=0.3, right_heads=7, right_dim=9, scales=(0.2, 3.0))],
                    eps=2e-3, alpha=1.25, cap=9.5)
    c = ModelConfig.load(_write(tmp_path, cfg))
    a, b, p = c.layers
    assert (c.model_type, c.residual_carry, c.logit_softcap, c.layernorm_eps) == ("dagezen", 1.25, 9.5, 2e-3)
    m = a.mixer
    assert (m.kind, m.heads, m.vdim, m.dim, m.groups, m.norm_groups, m.conv, m.has_kv) == ("ssd", 6, 10, 14, 3, 5, 2, False)
    assert (a.ff, a.act, a.limit, a.ff_bias) == (30, "clamped", 0.25, True)
    m = b.mixer
    assert (m.kind, m.gate, m.head_gate, m.sinks, m.window, m.scale, m.rot.style, m.rot.base) == ("latent", True, True, True, 0, 0.4, "interleaved", 77.0)
    assert (b.moe.act, b.moe.scoring, b.moe.router_bias, b.moe.shared, b.moe.experts, b.moe.top) == ("gelu_erf", "chosen", True, 0, 9, 4)
    l, r = p.mixer.parts
    assert p.mixer.part_scales == (0.2, 3.0) and p.mixer.has_kv and (l.kind, l.heads, l.kv_heads, l.dim, l.window, l.scale) == ("talking", 6, 2, 20, 11, 0.3)
    assert (r.kind, r.heads, r.dim, r.has_kv) == ("time_mix", 7, 9, False) and p.ff == 0 and p.moe is None
    with pytest.raises(ValueError, match="groups"):
        ModelConfig.from_dict(O.dagezen([O.mamba_layer(heads=4, groups=3)]))
    with pytest.raises(ValueError, match="int8"):
        xft.AutoModel.from_pretrained(str(tmp_path / "m"), dtype="bf16", kv_cache_dtype="int8")


# ------------------------------------------------------------------------------------------ limits and refusals
def test_fixed_pools_refuse_what_does_not_fit(tmp_path):
    cfg = O.config([O.attention_layer(), O.attention_layer(kv_from=0, size=5)])
    m = xft.AutoModel.from_pretrained(_write(tmp_path, cfg), dtype="fp32", max_cache_tokens=130)
    cache = m.model.cache
    assert cache.alloc.num_blocks == 3 and len(cache.k) == 1              # two layers, one pool
    m.set_input_cb([[1] * 100], max_length=1 << 30, on_demand=True)
    m.forward_cb()
    m.set_input_cb([[1] * 100], max_length=1 << 30, on_demand=True)
    with pytest.raises(MemoryError, match="limited to 3"):
        m.forward_cb()
    with pytest.raises(MemoryError):
        m.set_input_cb([[1] * 10], max_length=500)


def test_latent_pools(tmp_path):
    """A latent layer's pool has one row per token and no values; its reader has none; an int8 cache is refused."""
    cfg = O.vepivik([O.window_layer(), O.latent_layer(), O.latent_layer(kv_from=1)])
    p = _write(tmp_path, cfg)
    m = xft.AutoModel.from_pretrained(p, dtype="fp32", max_cache_tokens=130)
    cache = m.model.cache
    assert [tuple(k.shape) for k in cache.k] == [(3, 2, 64, 32), (3, 1, 64, 56)]
    assert cache.v[0].shape[3] == 24 and cache.v[1] is None
    assert cache.bytes_per_block() == 64 * 4 * (2 * 56 + 56)
    with pytest.raises(ValueError, match="int8"):
        xft.AutoModel.from_pretrained(p, dtype="bf16", kv_cache_dtype="int8")


def test_refusals(tmp_path):
    cfg = O.config([O.attention_layer()])
    p = _write(tmp_path, cfg)
    with pytest.raises(ValueError, match="fp32"):
        xft.AutoModel.from_pretrained(p, dtype="fp32", kv_cache_dtype="int8")
    m = xft.AutoModel.from_pretrained(p, dtype="fp32")
    with pytest.raises(ValueError, match="outside"):
        m.set_input_cb([[1, 2, 3]], max_length=8, rows=[[3]])
    with pytest.raises(ValueError, match="one list of rows"):
        m.set_input_cb([[1, 2, 3]], max_length=8, rows=[[0], [1]])


@pytest.mark.parametrize("dtype,kv,tol", [("int8", "bf16", 0.1), ("bf16_int8", "fp16", 0.1), ("bf16", "int8", 0.1)])
def test_other_weight_and_cache_types(tmp_path, dtype, kv, tol):
    """Quantised weights, hybrid types and an int8 cache go the way they go for the other families."""
    cfg = O.config([O.attention_layer(), O.attention_layer(kv_from=0, size=7)])
    W = O.random_weights(cfg)
    p = O.write_checkpoint(str(tmp_path / "q"), cfg, W)
    toks = list(range(3, 43))
    m = xft.AutoModel.from_pretrained(p, dtype=dtype, kv_cache_dtype=kv)
    want = O.forward(cfg, W, toks)
    got = m([toks])[0].double()
    assert float((got - want).pow(2).mean().sqrt() / want.std()) < tol
    assert m.generate(torch.tensor([toks]), max_length=50).shape == (1, 50)


def test_partial_library_has_what_layered_models_call():
    """bin/trace_run may build a part of the kernels only: its sources define every entry point the ops look up by name."""
    import importlib.util
    import re
    spec = importlib.util.spec_from_file_location("xft_build", os.path.join(ROOT, "csrc", "build.py"))
    b = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(b)
    text = "".join(open(os.path.join(ROOT, "csrc", "kernels", f)).read() for f in b.LAYERED)
    defined = set(re.findall(r'extern "C" \w+ (xft_\w+)\(', text))
    ops_dir = os.path.join(ROOT, "xfastertransformer_b200", "ops")
    src = {f: open(os.path.join(ops_dir, f)).read() for f in ("native.py", "native_latent.py", "native_linear.py", "native_moe.py", "native_talking.py")}
    wanted = {n for t in src.values() for n in re.findall(r'(?:lib\(\)\.|L\.|lib\.|")(xft_\w+)', t)}
    assert len(wanted) > 30 and wanted - defined <= {"xft_qgemm_grouped"}, wanted - defined


def test_command_line(tmp_path):
    """bin/trace_run as a program: JSON lines in, files of fp32 logits and a line per step out."""
    cfg = O.config([O.attention_layer(), O.attention_layer(kv_from=0, size=7)], vocab=61)
    W = O.random_weights(cfg)
    p, out = O.write_checkpoint(str(tmp_path / "m"), cfg, W), tmp_path / "out"
    out.mkdir()
    a, b = list(range(40)), list(range(60, 40, -1))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b, "want": [19, 2]}, {"id": "x", "tokens": a[30:31], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": a[31:], "want": [8]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", p, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(map(json.dumps, steps)) + "\n", text=True, capture_output=True,
                       env=dict(os.environ, XFT_ENGINE="CPU"), timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(out)) == ["1.f32", "2.f32"]
    wa, wb = O.forward(cfg, W, a), O.forward(cfg, W, b)
    for name, want in (("1.f32", torch.stack([wb[19], wb[2], wa[30]])), ("2.f32", wa[39:40])):
        got = torch.frombuffer(bytearray((out / name).read_bytes()), dtype=torch.float32).view(-1, 61)
        assert torch.allclose(got.double(), want, atol=2e-4)


@pytest.mark.parametrize("name", ["tiny-kafipel", "tiny-vepivik", "tiny-botusun", "tiny-dagezen"])
def test_synthetic_checkpoint_and_benchmark_tool(tmp_path, monkeypatch, name):
    """The presets write checkpoints that load, and the benchmark tool runs one by name with fake weights."""
    from xfastertransformer_b200.tools.synthetic import preset, write_synthetic_checkpoint
    c = preset(name)
    p = write_synthetic_checkpoint(str(tmp_path / "k"), c, seed=3, std=0.05)
    W = {n: SafetensorsFile(os.path.join(p, "model.safetensors")).read(n, e["shape"])
         for n, e in SafetensorsFile(os.path.join(p, "model.safetensors")).entries.items()}
    toks = list(range(60))
    got = xft.AutoModel.from_pretrained(p, dtype="fp32")([toks])[0].double()
    assert torch.allclose(got, O.forward(c.raw, W, toks), atol=1e-4)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "benchmarks", "benchmark.py"), "--model_name", name, "-in", "20",
                        "-out", "4", "-i", "1"], env=dict(os.environ, XFT_ENGINE="CPU", PYTHONPATH=ROOT), capture_output=True,
                       text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
