"""The Latodra decoder through the framework (state, step, engine, command line) against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

import latent_cases as H
from helpers import check_status

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = [torch.float32, torch.bfloat16]
_cache = {}


def case(name, n):
    """(config, weights, tokens, expected logits), computed once."""
    if (name, n) not in _cache:
        cfg = H.CONFIGS[name]
        W = H.weights(cfg, seed=len(name))
        t = H.tokens(cfg, n, seed=n)
        _cache[name, n] = (cfg, W, t, H.expected(cfg, W, t))
    return _cache[name, n]


def build(cfg, W, dt):
    import model_registry as R
    return R.model_class(cfg).from_config(cfg, W, dt)


def feed(m, st, toks, cuts):
    out, at = [], 0
    for c in cuts:
        c = min(c, len(toks) - at)
        if c:
            out.append(m.forward(torch.tensor([toks[at:at + c]]), st, range(c)))
        at += c
    assert at == len(toks)
    return torch.cat(out)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", list(H.CONFIGS))
@pytest.mark.parametrize("cuts", [(210,), (70, 64, 76), (1,) * 6 + (2, 3, 130, 2) + (1,) * 67, (33, 2, 2, 63, 65, 1, 1, 43)], ids=["whole", "thirds", "mixed", "portions"])
def test_logits(dt, name, cuts):
    cfg, W, toks, want = case(name, 210)
    m = build(cfg, W, dt)
    got = feed(m, m.new_cache(1, 210), toks, cuts)
    check_status()
    assert H.error(got, want) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", ["loop_inside", "odd_sizes", "large_heads"])
@pytest.mark.parametrize("absorb", [True, False])
def test_both_forms_of_the_attention(dt, name, absorb, monkeypatch):
    """The form is a matter of cost: portions of every size give the same with either."""
    import mixers
    cfg, W, toks, want = case(name, 210)
    m = build(cfg, W, dt)
    monkeypatch.setattr(mixers.LatentAttention, "_absorb", lambda self, ctx: absorb or ctx.n == 1)
    assert H.error(feed(m, m.new_cache(1, 230), toks, (2, 125, 2, 64, 1, 16)), want) < H.TOL[dt]
    check_status()


@pytest.mark.parametrize("name", ["loop_inside", "loop_first", "odd_sizes", "no_loop"])
def test_residual_stream_after_every_layer(name):
    cfg, W, toks, _ = case(name, 40)
    m, want, got = build(cfg, W, torch.float32), [], []
    H.expected(cfg, W, toks, want)
    m.hidden(torch.tensor([toks]).cuda(), m.new_cache(1, 40), 0, got)
    for a, b in zip(got, want, strict=True):
        assert (a.double().cpu() - b).abs().max() < 2e-5 * b.abs().max()


@pytest.mark.parametrize("dt", DT)
def test_long_decoding_token_by_token(dt):
    """Two tokens, then 318 single ones (captured step): every pass of the loop keeps its own cache, tile borders pass over decoded tokens,
    positions leave the length that the rotation was made for."""
    cfg, W, toks, want = case("loop_inside", 320)
    m = build(cfg, W, dt)
    assert H.error(feed(m, m.new_cache(1, 320), toks, (2,) + (1,) * 318), want) < H.TOL[dt]
    m.use_graph = False
    assert H.error(feed(m, m.new_cache(1, 320), toks, (2,) + (1,) * 318), want) < H.TOL[dt]
    check_status()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("key", [0, 1, 126, 127, 128, 129, 254])
def test_one_far_key_counts(dt, key):
    """A marked token whose latent one query direction singles out: the logits of far positions must carry it, from a portion and decoded."""
    cfg, W = H.one_key_counts(39)
    toks = [3 + (7 * i) % 30 for i in range(260)]
    toks[key] = 39
    want = H.expected(cfg, W, toks)
    other = H.expected(cfg, W, toks[:key] + [38] + toks[key + 1:])
    assert H.error(other[255:], want[255:]) > 3 * H.TOL[dt]            # it shows
    m = build(cfg, W, dt)
    assert H.error(feed(m, m.new_cache(1, 260), toks, (260,)), want) < H.TOL[dt]
    assert H.error(feed(m, m.new_cache(1, 260), toks, (200, 50) + (1,) * 10), want) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_the_sink_shows(dt):
    """Sinks above all scores: leaving them out, scaling them or counting them per key would change everything."""
    cfg, W, toks, want = case("no_loop", 60)
    W2 = dict(W)
    W2["l0.mix.sink"] = W["l0.mix.sink"] + 4
    want2 = H.expected(cfg, W2, toks)
    assert H.error(want2, want) > 3 * H.TOL[dt]
    m = build(cfg, W2, dt)
    for cuts in ((60,), (1,) * 60, (2, 50, 8)):
        assert H.error(feed(m, m.new_cache(1, 60), toks, cuts), want2) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_batch_in_lockstep(dt):
    cfg, W, _, _ = case("loop_inside", 40)
    m = build(cfg, W, dt)
    B = 3
    rows = [H.tokens(cfg, 90, seed=50 + b) for b in range(B)]
    st = m.new_cache(B, 96)
    got = [[] for _ in range(B)]
    at = 0
    for n in (70, 5) + (1,) * 15:
        lg = m.forward(torch.tensor([r[at:at + n] for r in rows]), st, range(B * n)).view(B, n, -1)
        for b in range(B):
            got[b].append(lg[b])
        at += n
    for b in range(B):
        assert H.error(torch.cat(got[b]), H.expected(cfg, W, rows[b])) < H.TOL[dt]
    B = 20
    st = m.new_cache(B, 8)
    ids = torch.tensor([H.tokens(cfg, 5, seed=b) for b in range(B)])
    m.forward(ids[:, :3], st)
    lg = [m.forward(ids[:, t:t + 1], st, range(B)) for t in (3, 4)]
    for b in (0, 7, 19):
        assert H.error(torch.stack([lg[0][b], lg[1][b]]), H.expected(cfg, W, ids[b].tolist())[3:]) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_interleaved_requests_and_reused_slots(dt):
    """Unequal requests alternate; a finished one's state serves the next request, with its latents still in it."""
    from engine import Engine
    cfg, W, _, _ = case("loop_inside", 40)
    eng = Engine(build(cfg, W, dt), max_tokens=160)
    reqs = {r: H.tokens(cfg, n, seed=n) for r, n in (("a", 150), ("b", 31), ("c", 2), ("d", 97), ("e", 1), ("f", 64))}
    got = {r: [] for r in reqs}

    def step(r, n):
        at = sum(len(g) for g in got[r])
        part = reqs[r][at:at + n]
        got[r].append(eng.step(r, part, range(len(part)), end=at + len(part) == len(reqs[r])))
    for r, n in (("a", 70), ("b", 30), ("a", 1), ("b", 1), ("c", 2), ("a", 1), ("d", 3), ("a", 66), ("d", 1), ("e", 1), ("d", 93), ("a", 12), ("f", 64)):
        step(r, n)
    assert not eng.pool.live and len(eng.pool.free) == 3          # three slots served six requests
    for r in reqs:
        assert H.error(torch.cat(got[r]), H.expected(cfg, W, reqs[r])) < H.TOL[dt], r


@pytest.mark.parametrize("name", ["loop_inside", "odd_sizes", "one_pass"])
def test_greedy_generation_through_the_scheduler(name):
    from engine import Engine, SamplingParams
    cfg, W, _, _ = case(name, 40)
    m = build(cfg, W, torch.float32)
    prompts = [H.tokens(cfg, n, seed=n) for n in (1, 13, 70)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(6):
            seq.append(int(H.expected(cfg, W, seq)[-1].argmax()))
        want.append(seq[len(p):])
    for portion, live in ((2048, 8), (7, 1), (32, 2)):
        assert Engine(m, 96, portion, live).generate(prompts, SamplingParams(max_new=6)) == want


def test_registry_folder_command_line_and_trace(tmp_path):
    import model_registry as R
    import numpy as np
    cfg, W, toks, want = case("loop_inside", 40)
    R.save_model(str(tmp_path), cfg, W)
    m = R.load_model(str(tmp_path), "float32")
    assert H.error(m.prefill(torch.tensor([toks]), m.new_cache(1, 40)), want[-1:]) < H.TOL[torch.float32]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "qwen-palettize_b200", "cli.py"), "generate", "--model", str(tmp_path), "--dtype", "float32", "--tokens",
                        ",".join(map(str, toks[:20])), "--max-new", "1"], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert int(r.stdout) == int(want[19].argmax())
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:25], "want": [3, 24]}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": toks[25:26], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[26:], "want": [0, 13]}], "end": ["x"]}, {"step": 3, "entries": [{"id": "y", "tokens": toks[:1], "want": [0]}], "end": ["y"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "48"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines()] == [f"done {i}" for i in range(4)] and sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
    for i, rows in ((0, [3, 24]), (2, [26, 39]), (3, [0])):
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        assert H.error(got, want[rows]) < H.TOL[torch.float32]
