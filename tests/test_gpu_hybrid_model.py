"""The Gopunex decoder through the framework (state, step, engine, command line) against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

import hybrid_cases as H
from helpers import check_status

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = [torch.float32, torch.bfloat16]
_cache = {}


def case(name, n):
    """(config, weights, tokens, expected logits), computed once."""
    if (name, n) not in _cache:
        cfg = H.CONFIGS[name]
        W = H.weights(cfg, seed=14 if name == "narrow_window" else len(name))
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


@pytest.mark.parametrize("name", ["all", "odd_sizes"])
def test_residual_stream_after_every_layer(name):
    cfg, W, toks, _ = case(name, 40)
    m, want, got = build(cfg, W, torch.float32), [], []
    H.expected(cfg, W, toks, want)
    m.hidden(torch.tensor([toks]).cuda(), m.new_cache(1, 40), 0, got)
    for a, b in zip(got, want, strict=True):
        assert (a.double().cpu() - b).abs().max() < 2e-5 * b.abs().max()


@pytest.mark.parametrize("dt", DT)
def test_long_decoding_token_by_token(dt):
    """Two tokens, then 318 single ones (captured step): states, convolution inputs, bias table and cache all pass over decoded tokens."""
    cfg, W, toks, want = case("all", 320)
    m = build(cfg, W, dt)
    assert H.error(feed(m, m.new_cache(1, 320), toks, (2,) + (1,) * 318), want) < H.TOL[dt]
    m.use_graph = False
    assert H.error(feed(m, m.new_cache(1, 320), toks, (2,) + (1,) * 318), want) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_batch_in_lockstep(dt):
    cfg, W, _, _ = case("all", 40)
    m = build(cfg, W, dt)
    B = 3
    rows = [H.tokens(cfg, 90, seed=50 + b) for b in range(B)]
    st = m.new_cache(B, 90)
    got = [[] for _ in range(B)]
    at = 0
    for n in (70, 5) + (1,) * 15:
        lg = m.forward(torch.tensor([r[at:at + n] for r in rows]), st, range(B * n)).view(B, n, -1)
        for b in range(B):
            got[b].append(lg[b])
        at += n
    for b in range(B):
        assert H.error(torch.cat(got[b]), H.expected(cfg, W, rows[b])) < H.TOL[dt]
    # many sequences: the wider Linear kernels of the one-token step
    B = 20
    st = m.new_cache(B, 8)
    ids = torch.tensor([H.tokens(cfg, 5, seed=b) for b in range(B)])
    m.forward(ids[:, :3], st)
    lg = [m.forward(ids[:, t:t + 1], st, range(B)) for t in (3, 4)]
    for b in (0, 7, 19):
        assert H.error(torch.stack([lg[0][b], lg[1][b]]), H.expected(cfg, W, ids[b].tolist())[3:]) < H.TOL[dt]


@pytest.mark.parametrize("dt", DT)
def test_interleaved_requests_and_reused_slots(dt):
    """Unequal requests alternate; a finished one's state serves the next request and must start clean."""
    from engine import Engine
    cfg, W, _, _ = case("all", 40)
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


@pytest.mark.parametrize("name", ["all", "odd_sizes", "attention_first"])
def test_greedy_generation_through_the_scheduler(name):
    from engine import Engine, SamplingParams
    cfg, W, _, _ = case(name, 40)
    m = build(cfg, W, torch.float32)
    prompts = [H.tokens(cfg, n, seed=n) for n in (1, 13, 70)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(8):
            seq.append(int(H.expected(cfg, W, seq)[-1].argmax()))
        want.append(seq[len(p):])
    for portion, live in ((2048, 8), (7, 1), (32, 2)):
        assert Engine(m, 96, portion, live).generate(prompts, SamplingParams(max_new=8)) == want


def test_registry_folder_command_line_and_trace(tmp_path):
    import model_registry as R
    cfg, W, toks, want = case("all", 40)
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
    import numpy as np
    for i, rows in ((0, [3, 24]), (2, [26, 39]), (3, [0])):
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        assert H.error(got, want[rows]) < H.TOL[torch.float32]


def test_refusals():
    cfg, W, toks, _ = case("all", 40)
    m = build(cfg, W, torch.float32)
    st = m.new_cache(1, 16)
    with pytest.raises(ValueError, match="capacity"):
        m.forward(torch.tensor([toks[:17]]), st)
    with pytest.raises(ValueError, match="sequences"):
        m.forward(torch.tensor([toks[:2], toks[:2]]), st)
    bad = dict(W)
    bad["l0.mix.q"] = bad["l0.mix.q"][:, :-1]
    with pytest.raises(ValueError, match="shape"):
        build(cfg, bad, torch.float32)
    with pytest.raises(ValueError):
        build(cfg, W, torch.float16)


def test_the_palettized_model_through_the_same_engine(tmp_path):
    """The framework's other decoder: saved, loaded by the registry and served by the engine, equal to its own prefill and decode."""
    import decode_model as DM
    import model_registry as R
    from engine import Engine, SamplingParams
    cfg = DM.ModelConfig(hidden=256, n_heads=2, n_kv_heads=1, head_dim=128, intermediate=512, n_layers=2, vocab=512)
    m = DM.PalettizedQwen.random(cfg, torch.device("cuda", 0), seed=5, max_positions=512)
    m.embed = (torch.randn(cfg.vocab, cfg.hidden, generator=torch.Generator().manual_seed(1)) * 0.5).to(torch.bfloat16).cuda()
    R.save_model(str(tmp_path), {"architecture": "PalettizedQwen", "max_positions": 512, **{k: getattr(cfg, k) for k in cfg.__dataclass_fields__}}, m.state_dict())
    m2 = R.load_model(str(tmp_path))
    ids = torch.randint(0, 512, (1, 140), generator=torch.Generator().manual_seed(2))
    eng = Engine(m2, 192)
    got = eng.step("r", ids[0].tolist(), [5, 127, 139])
    c = m.new_cache(1, 192)
    h, last = m.prefill(ids[:, :128].cuda(), c)
    want = [m.logits(h[5:6])[0], last[0]]
    for t in range(128, 140):
        want_last = m.decode_step(ids[:, t].cuda().contiguous(), c)[0]
    for a, b in zip(got, want + [want_last]):
        assert torch.nn.functional.cosine_similarity(a.float(), b.float(), dim=0) > 0.9999
    eng.end("r")
    assert len(eng.generate([ids[0, :20].tolist()], SamplingParams(max_new=3))[0]) == 3
