"""Host side of the hybrid decoders: tensor files, registry, configuration, distance buckets, state pool, scheduler, command line."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import hybrid_cases as H

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_safetensors_round_trip_and_bad_files(tmp_path):
    import safetensors_io as st
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "scalar": torch.tensor(2.5), "none": torch.empty(0, 4),
         "u8": torch.arange(9, dtype=torch.uint8).view(3, 3)}
    p = str(tmp_path / "x.safetensors")
    st.save(p, t)
    f = st.SafeTensors(p)
    assert set(f.keys()) == set(t) and "a" in f and "z" not in f
    for k, v in t.items():
        assert f[k].dtype == v.dtype and f.shape(k) == tuple(v.shape) and torch.equal(f[k], v)
    with pytest.raises(KeyError):
        f["z"]
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-1])
    with pytest.raises(ValueError):
        st.SafeTensors(p)
    open(p, "wb").write((1 << 40).to_bytes(8, "little") + raw[8:])
    with pytest.raises(ValueError):
        st.SafeTensors(p)


def test_registry_and_configuration():
    import model_registry as R
    from hybrid_model import HybridConfig, tensor_shapes
    assert {"Gopunex", "PalettizedQwen"} <= set(R.ARCHITECTURES)
    with pytest.raises(ValueError, match="unknown architecture"):
        R.model_class({"architecture": "Nope"})
    assert R.check_dtype({"architecture": "Gopunex"}, "float32") == torch.float32
    with pytest.raises(R.UnsupportedDtype):
        R.check_dtype({"architecture": "PalettizedQwen"}, "float32")
    cfg = H.CONFIGS["no_mlp"]
    c = HybridConfig.from_dict(cfg)
    assert c.width == 48 and c.layers[0].mlp is None and c.layers[1].mlp["kind"] == "dense" and c.eps == 3e-5
    assert "l0.norm2" not in tensor_shapes(cfg) and "l1.norm2" in tensor_shapes(cfg)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        HybridConfig.from_dict(bad)


@pytest.mark.parametrize("B,D", [(32, 240), (12, 70), (8, 9), (2, 5), (16, 8), (16, 128), (7, 50)])
def test_distance_buckets(B, D):
    """The product's table against the definition, including distances whose logarithm is a whole number of buckets."""
    import gopunex_oracle as O
    import mixers
    row = [mixers.distance_bucket(n, B, D) for n in range(3 * D)]
    assert row == sorted(row) and row[-1] == B - 1 and row[0] == 0
    half = B // 2
    assert row[:half] == list(range(half))
    for n in range(half, 3 * D):
        if D <= half:
            assert row[n] == B - 1
            continue
        at = math.log(n / half) / math.log(D / half) * (B - half)
        if abs(at - round(at)) > 1e-6:
            assert row[n] == O.distance_bucket(n, B, D)
        else:
            assert row[n] == min(B - 1, half + round(at))
    rel = torch.randn(B, 3)
    tab = mixers.distance_table(rel, D)
    for n in range(3 * D):
        assert torch.equal(tab[:, min(n, tab.shape[1] - 1)], rel[row[n]])
    assert tab.shape[1] <= max(D, half) + 1


class _Fake:
    """A model of the engine's protocol without kernels: logits say 'previous token + number of tokens so far'."""
    vocab = 50

    class State:
        def __init__(self, cap):
            self.capacity, self.length, self.sum, self.resets = cap, 0, 0, 0

        def reset(self):
            self.length = self.sum = 0
            self.resets += 1

    def __init__(self):
        self.made, self.log = 0, []

    def new_cache(self, B, T):
        self.made += 1
        return self.State(T)

    def forward(self, ids, st, want=None):
        assert st.length + ids.shape[1] <= st.capacity
        rows = []
        for t in ids[0].tolist():
            st.length += 1
            st.sum += t
            rows.append(torch.nn.functional.one_hot(torch.tensor((t + st.length) % self.vocab), self.vocab).float())
        self.log.append(ids.shape[1])
        return torch.stack([rows[w] for w in want]) if want else None


@pytest.fixture
def fake_engine(monkeypatch):
    import engine
    import seq_ops
    monkeypatch.setattr(seq_ops, "sample", lambda lg, pos, *a: lg.argmax(-1))
    return engine


def _fake_generate(prompt, n):
    out, length, last = [], len(prompt), prompt[-1]
    for _ in range(n):
        last = (last + length) % _Fake.vocab
        out.append(last)
        length += 1
    return out


def test_scheduler_portions_turns_and_slots(fake_engine):
    m = _Fake()
    eng = fake_engine.Engine(m, max_tokens=64, portion=5, max_live=2)
    prompts = [[3], [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12], [7, 7], [9] * 6]
    got = eng.generate(prompts, fake_engine.SamplingParams(max_new=6))
    assert got == [_fake_generate(p, 6) for p in prompts]
    assert m.made == 2 and len(eng.pool.free) == 2 and not eng.pool.live          # two slots served four requests
    assert max(m.log) == 5 and [5, 5, 2] == [n for n in m.log if n > 1][:3]
    # a stop token ends a request early and is kept
    stop = got[0][2]
    assert eng.generate([prompts[0]], fake_engine.SamplingParams(max_new=6, stop=(stop,))) == [got[0][:3]]


def test_engine_refuses_what_it_cannot_run(fake_engine):
    eng = fake_engine.Engine(_Fake(), max_tokens=8)
    with pytest.raises(ValueError):
        eng.submit([])
    with pytest.raises(ValueError):
        eng.submit([1] * 7, fake_engine.SamplingParams(max_new=2))
    with pytest.raises(ValueError):
        eng.step("a", [50])
    with pytest.raises(ValueError):
        eng.step("a", [1, 2], [2])
    with pytest.raises(ValueError):
        fake_engine.Engine(_Fake(), 8, portion=0)
    assert not eng.pool.live                       # nothing was taken by the refused calls
    eng.step("a", [1, 2, 3], end=True)
    assert "a" not in eng.pool
    eng.end("a")                                   # ending twice is harmless


def test_runner_refuses_an_unsupported_type(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "PalettizedQwen"}))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "8"], capture_output=True, text=True, stdin=subprocess.DEVNULL)
    assert r.returncode == 3 and "does not run in float32" in r.stderr
    r = subprocess.run([sys.executable, os.path.join(ROOT, "qwen-palettize_b200", "cli.py"), "models"], capture_output=True, text=True)
    assert r.returncode == 0 and "Gopunex bfloat16,float32" in r.stdout


def test_oracle_against_closed_forms():
    """The plain implementation on inputs whose answers are known."""
    import gopunex_oracle as O
    d = torch.float64
    torch.manual_seed(0)
    # decay 0: only the current token is left
    q, k, v = (torch.randn(5, 3, dtype=d) for _ in range(3))
    o = O.decayed_linear_attention(q, k, v, 0.0)
    assert torch.allclose(o, (q * k).sum(-1, keepdim=True) * v)
    # decay 1: linear attention with a causal mask
    o = O.decayed_linear_attention(q, k, v, 1.0)
    assert torch.allclose(o, torch.tril(q @ k.T) @ v)
    # delta rule with unit keys, beta 1 and no decay: reading with the key just written returns its value exactly
    k = O.unit(k)
    o = O.gated_delta(k, k, v, torch.ones(5, 3, dtype=d), torch.ones(5, dtype=d))
    assert torch.allclose(o, v, atol=1e-5)
    # the sink: scores far below zero leave nothing, one large score takes everything
    s = torch.full((1, 4), -40.0, dtype=d)
    m = torch.ones(1, 4, dtype=torch.bool)
    assert O.softmax_off_by_one(s, m).sum() < 1e-15
    s[0, 2] = 40.0
    assert abs(O.softmax_off_by_one(s, m)[0, 2] - 1) < 1e-12
    assert torch.allclose(O.softmax_off_by_one(torch.zeros(1, 4, dtype=d), m), torch.full((1, 4), 0.2, dtype=d))
    # convolution: a unit tap on the last column is the identity, on the first a delay
    x = torch.randn(6, 2, dtype=d)
    w = torch.zeros(2, 3, dtype=d)
    w[:, 2] = 1
    assert torch.equal(O.causal_conv(x, w), x)
    w = torch.zeros(2, 3, dtype=d)
    w[:, 0] = 1
    assert torch.equal(O.causal_conv(x, w)[2:], x[:4]) and O.causal_conv(x, w)[:2].abs().max() == 0
