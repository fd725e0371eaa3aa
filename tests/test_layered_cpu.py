"""Layered designs (Kafipel, Vepivik, Botusun, Dagezen) on the CPU path: the engine, cache, batching and command-line tool against a plain
implementation of the equations."""
import os
import subprocess
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "tests"))

import layered_cases as C  # noqa: E402
import oracle_layered as O  # noqa: E402
import xfastertransformer_b200 as xft  # noqa: E402
from xfastertransformer_b200.config import ModelConfig  # noqa: E402


@pytest.fixture(autouse=True)
def _cpu(monkeypatch):
    monkeypatch.setenv("XFT_ENGINE", "CPU")


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    root, made = tmp_path_factory.mktemp("layered"), {}

    def get(name):
        if name not in made:
            made[name] = C.Case(root, name)
        return made[name]
    return get


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_whole_prompt(cases, name):
    C.whole_prompt(cases(name), "fp32", 75)


@pytest.mark.parametrize("name", ["unequal", "bare", "latent", "latent_bare", "recurrent", "recurrent_bare", "mixed_heads", "mixed_heads_bare"])
def test_first_tokens(cases, name):
    C.first_tokens(cases(name), "fp32")


@pytest.mark.parametrize("name,n,start", [("unequal", 75, 1), ("shared", 75, 60), ("latent", 75, 1), ("recurrent", 75, 1), ("recurrent_bare", 75, 30), ("mixed_heads", 75, 1),
                                          ("mixed_heads_bare", 75, 30)])
def test_token_by_token(cases, name, n, start):
    C.token_by_token(cases(name), "fp32", n, start)


@pytest.mark.parametrize("sizes", [(2,), (3, 64, 1), (17, 29)])
@pytest.mark.parametrize("name", ["unequal", "latent", "recurrent", "mixed_heads"])
def test_portions(cases, name, sizes):
    C.portions(cases(name), "fp32", 75, sizes)


@pytest.mark.parametrize("name", ["unequal", "shared", "latent", "recurrent", "recurrent_large", "mixed_heads", "mixed_heads_large"])
def test_mixed_batches_reuse_pages(cases, name):
    assert C.mixed_batches(cases(name), "fp32", lengths=(75, 50, 20, 1, 66), live=2) > 5


@pytest.mark.parametrize("name", ["unequal", "latent", "recurrent", "mixed_heads"])
def test_greedy_generation(cases, name):
    C.greedy(cases(name), "fp32", 20, 40)


@pytest.mark.parametrize("name", ["unequal", "latent", "recurrent", "mixed_heads"])
def test_rows_and_order(cases, name):
    C.rows_and_order(cases(name), "fp32")


@pytest.mark.parametrize("name", ["large_heads", "recurrent", "recurrent_fast", "mixed_heads"])
def test_long_decoding(cases, name):
    """Generation across several pages, far past every window, over states that have long forgotten the prompt or never do."""
    C.greedy(cases(name), "fp32", 5, 140)


@pytest.mark.parametrize("name", ["shared", "latent", "recurrent", "mixed_heads"])
def test_scheduler_serves_it(cases, name):
    """The serving scheduler (chunked prefill, mixed steps) emits generate()'s tokens."""
    from serving import openai_server as oai
    c = cases(name)
    m = xft.AutoModel.from_pretrained(c.path, dtype="fp32")
    prompts = [c.tokens(n, 40 + n) for n in (33, 7, 70)]
    want = [m.generate(torch.tensor([p]), max_length=len(p) + 12)[0, len(p):].tolist() for p in prompts]
    s = oai.Scheduler(m, max_batch=4, prefill_per_step=2)
    s.mixed_steps, s.prefill_chunk = True, 16
    s.start()
    try:
        reqs = [s.submit(oai.Request(p, 12, 0.0, 1.0, 0, [], None)) for p in prompts]
        for r, w in zip(reqs, want):
            got = []
            while True:
                t = r.out.get(timeout=60)
                if t is None or isinstance(t, Exception):
                    assert t is None, t
                    break
                got.append(t)
            assert got == w
    finally:
        s.shutdown()
        s.join(timeout=30)


@pytest.mark.parametrize("name", ["unequal", "latent", "recurrent", "mixed_heads"])
def test_beams_sampling_and_prefix_reuse(cases, monkeypatch, name):
    """The parts of the engine above the step function work on a layered model as on any other."""
    c = cases(name)
    p = c.tokens(70, 51 if name == "mixed_heads" else 50)         # prompts where three beams find more than greedy decoding does
    m = xft.AutoModel.from_pretrained(c.path, dtype="fp32")
    g = m.generate(torch.tensor([p]), max_length=80)
    b = m.generate(torch.tensor([p]), max_length=80, num_beams=3)
    assert b.shape == g.shape and b[0, :70].tolist() == p

    def score(row):
        lp = torch.log_softmax(c.want(row[:-1])[69:], -1)
        return float(lp.gather(1, torch.tensor(row[70:])[:, None]).sum())
    assert score(b[0].tolist()) >= score(g[0].tolist()) - 1e-6
    s1 = m.generate(torch.tensor([p]), max_length=80, do_sample=True, top_k=20, seed=3)
    s2 = m.generate(torch.tensor([p]), max_length=80, do_sample=True, top_k=20, seed=3)
    assert torch.equal(s1, s2)
    m.prefix_sharing(torch.tensor([p[:66]]))
    assert torch.equal(m.generate(torch.tensor([p]), max_length=80), g)
    m.disable_prefix_sharing()
    monkeypatch.setenv("XFT_SPEC_NGRAM", "3")
    from xfastertransformer_b200.utils.flags import Env
    Env.get().reload()
    assert torch.equal(m.generate(torch.tensor([p]), max_length=80), g)


# ------------------------------------------------------------------------------------------ several ranks
def _ranks(case, tmp_path, port, n=2, **env):
    out = str(tmp_path / "out.pt")
    e = dict(os.environ, XFT_ENGINE="CPU", PYTHONPATH=ROOT + os.pathsep + os.environ.get("PYTHONPATH", ""), **env)
    cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={n}", "--master-addr", "127.0.0.1",
           "--master-port", str(port), os.path.join(ROOT, "tests", "layered_worker.py"), case.path, out]
    r = subprocess.run(cmd, env=e, capture_output=True, text=True, timeout=300)
    return r, out


@pytest.mark.parametrize("name,heads,env", [("shared", [2, 4], {}), ("latent", [3, 2], {}),
                                            ("latent", [3, 2], {"XFT_EXPERT_PARALLEL": "1"}),
                                            ("recurrent", [3, 2], {}), ("mixed_heads", [6, 2], {}),
                                            ("mixed_heads", [6, 2], {"XFT_EXPERT_PARALLEL": "1"})])
def test_tensor_parallel_two_ranks(cases, tmp_path, name, heads, env):
    """Heads (also a key/value head or latents that both ranks read), sinks, feed-forward rows or experts and the logits
    split over two ranks."""
    c = cases(name)
    r, out = _ranks(c, tmp_path, 29831, **env)
    assert r.returncode == 0, r.stdout[-2000:] + r.stderr[-2000:]
    got = torch.load(out)
    C.check(got["rows"], torch.cat([c.want(got["prompts"][0])[[3, 49]], c.want(got["prompts"][1])[-1:]]), "fp32", "two ranks")
    assert got["heads"][0] == heads
    m = xft.AutoModel.from_pretrained(c.path, dtype="fp32")
    assert torch.equal(got["tokens"], m.generate(torch.tensor([got["prompts"][0]]), max_length=60))


def test_pipeline_stages(cases, tmp_path):
    """The residual stream crosses stages in 32 bits; a layer whose keys live on another stage is refused."""
    cfg = O.config([O.attention_layer(size=9), O.attention_layer(kv_from=0, size=14), O.attention_layer(heads=2, size=5),
                    O.attention_layer(ff=None, size=30)], width=76, vocab=111)
    c = C.Case.__new__(C.Case)
    c.name, c.cfg, c.W, c._want = "stages", cfg, O.random_weights(cfg, 4), {}
    c.path = O.write_checkpoint(str(tmp_path / "stages"), cfg, c.W)
    r, out = _ranks(c, tmp_path, 29841, XFT_PIPELINE_STAGE="2")
    assert r.returncode == 0, r.stdout[-2000:] + r.stderr[-2000:]
    got = torch.load(out)
    C.check(got["rows"], torch.cat([c.want(got["prompts"][0])[[3, 49]], c.want(got["prompts"][1])[-1:]]), "fp32", "stages")
    # looped layers: stages are ranges of runs, a stage's weights those of the layers it runs; a stream that is a norm
    for k, name in enumerate(("recurrent", "mixed_heads")):
        c = C.Case(tmp_path, name)
        r, out = _ranks(c, tmp_path, 29851 + 10 * k, XFT_PIPELINE_STAGE="2")
        assert r.returncode == 0, r.stdout[-2000:] + r.stderr[-2000:]
        got = torch.load(out)
        C.check(got["rows"], torch.cat([c.want(got["prompts"][0])[[3, 49]], c.want(got["prompts"][1])[-1:]]), "fp32", "stages")
    c = C.Case.__new__(C.Case)
    c.path = O.write_checkpoint(str(tmp_path / "stages"), cfg, O.random_weights(cfg, 4))
    from xfastertransformer_b200.models.layered import LayeredDecoder
    from xfastertransformer_b200.parallel.dist import DistContext
    ctx = DistContext.get()
    ctx.pp_size, ctx.pp_rank = 4, 1                     # the layer that reads layer 0's keys alone on its stage
    with pytest.raises(ValueError, match="another pipeline stage"):
        LayeredDecoder(ModelConfig.load(c.path), ctx, c.path, "fp32")
