"""CPU: the plain Nufalorn statement (oracle/nufalorn.py) agrees with itself where two formulations must agree, the test models show
every mechanism (a planted mistake in the plain statement moves the logits far beyond the GPU tests' tolerances), and the host-side
parts -- registry, JSON reader, command line -- behave without a GPU."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import nufalorn_cases as C
from oracle import nufalorn as N

ROOT = Path(__file__).resolve().parent.parent


def run(cfg, w, toks):
    return N.Nufalorn(cfg, w).run(toks)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def rms_diff(a, b):
    return np.sqrt(np.mean((a - b) ** 2, axis=-1)) / np.sqrt(np.mean(b ** 2))


def test_recurrence_carries_its_state():
    r = np.random.default_rng(1)
    q, k, a = r.standard_normal((3, 30, 2, 5))
    a = N.sigmoid(a)
    v = r.standard_normal((30, 2, 7))
    whole, S = N.decay_scan(q, k, v, a)
    o1, S1 = N.decay_scan(q[:11], k[:11], v[:11], a[:11])
    o2, S2 = N.decay_scan(q[11:], k[11:], v[11:], a[11:], S1)
    assert np.allclose(np.concatenate([o1, o2]), whole) and np.allclose(S, S2)
    # closed form of one read-out: sum_j (q_t . prod_{j<u<=t} a_u . k_j) v_j
    t = 17
    o = sum((q[t, 0] * np.prod(a[j + 1:t + 1, 0], axis=0) * k[j, 0]).sum() * v[j, 0] for j in range(t + 1))
    assert np.allclose(o, whole[t, 0])


def test_sink_and_block_mask():
    s = np.array([[2.0, -1.0, 0.5]])
    p = N.softmax_with_sink(s, np.array([[True, True, False]]))
    assert np.allclose(p, [[np.exp(2) / (1 + np.exp(2) + np.exp(-1)), np.exp(-1) / (1 + np.exp(2) + np.exp(-1)), 0]])
    assert np.allclose(N.softmax_with_sink(s + 800, np.ones((1, 3), bool)).sum(), 1) and np.allclose(N.softmax_with_sink(s - 800, np.ones((1, 3), bool)), 0)
    m = N.chunk_mask(9, 4)
    assert m[3].tolist() == [1, 1, 1, 1, 0, 0, 0, 0, 0] and m[4].tolist() == [0, 0, 0, 0, 1, 0, 0, 0, 0] and m[8, 8] and not m[8, 7]


def test_rotations_depend_on_distance_only():
    r = np.random.default_rng(2)
    q, k = r.standard_normal((2, 1, 1, 12))
    d = [(N.rotate_pairs(q, [i + s], 50.0, 8) * N.rotate_pairs(k, [i], 50.0, 8)).sum() for i, s in ((0, 3), (40, 3), (7, 3), (7, 4))]
    assert np.allclose(d[0], d[1]) and np.allclose(d[0], d[2]) and abs(d[0] - d[3]) > 1e-3
    x = r.standard_normal((5, 2, 12))
    assert np.allclose(N.rotate_pairs(N.rotate_pairs(x, np.arange(5), 9.0, 12), np.arange(5), 9.0, 12, sign=-1.0), x)


def shift_block(cfg, d):
    c = copy.deepcopy(cfg)
    for layer in c["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["mask"]["size"] += d
    return c


MISTAKES = {
    "no sink": lambda mp: mp.setattr(N, "softmax_with_sink", lambda s, m: np.exp(np.where(m, s, -np.inf) - np.max(np.where(m, s, -np.inf), -1, keepdims=True)) /
                                     np.exp(np.where(m, s, -np.inf) - np.max(np.where(m, s, -np.inf), -1, keepdims=True)).sum(-1, keepdims=True)),
    "blocks counted from 1": lambda mp: mp.setattr(N, "chunk_mask", lambda n, b: np.tril(np.ones((n, n), bool)) & (
        ((np.arange(n) + 1) // b)[None, :] == ((np.arange(n) + 1) // b)[:, None])),
    "values not turned back": lambda mp: mp.setattr(N, "rotate_pairs", (lambda f: lambda x, pos, base, dims, sign=1.0: x if sign < 0 else f(x, pos, base, dims))(N.rotate_pairs)),
    "forget gate not complementary": lambda mp: mp.setattr(N, "hgrn2_inputs", (lambda f: lambda *a: (lambda q, k, v, g: (q, np.ones_like(k), v, g))(*f(*a)))(N.hgrn2_inputs)),
    "state lost after 16 tokens": lambda mp: mp.setattr(N, "decay_scan", (lambda f: lambda q, k, v, a, state=None: (lambda s: f(q, k, v, np.where(np.arange(len(a)) == 16, 0.0, 1.0)[:, None, None] * a, s))(state))(N.decay_scan)),
    "gate temperature": lambda mp: mp.setattr(N, "gla_inputs", (lambda f: lambda h, p, c: f(h, p, dict(c, tau=c["tau"] * 1.1)))(N.gla_inputs)),
    "norm weight not around one": lambda mp: mp.setattr(N, "rms_norm_zero_centred", lambda x, w, eps: N.rms(x, eps) * np.where(w == 0, 1, 1 + w * 0.5)),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_test_model_shows_mistake(name, monkeypatch):
    cfg = C.CASES["mixed"]
    w, toks = C.tensors(cfg, 3), tokens(cfg, 60)
    good = run(cfg, w, toks)
    MISTAKES[name](monkeypatch)
    assert np.max(rms_diff(run(cfg, w, toks), good)) > 0.02, name


def test_block_edges_show():
    """one position more or less in a block changes the rows at the edge and leaves the rows before it alone"""
    cfg = C.config(48, 64, [C.att(4, 2, 16, 16, 21, scale=1.0)])
    w, toks = C.tensors(cfg, 8), tokens(cfg, 64)
    good = run(cfg, w, toks)
    for d in (-1, 1):
        diff = rms_diff(run(shift_block(cfg, d), w, toks), good)
        assert diff[:20].max() < 1e-12 and diff[20:23].max() > 0.05


# ---- host side -----------------------------------------------------------------------------------------------
def test_registry(lb):
    from lithos_b200 import model as M
    assert {"Nufalorn", "Qwen3.5-hybrid"} <= set(M.architectures())
    images = M.config_images(json.dumps(C.CASES["mixed"]))
    kdir = ROOT / "lithos_b200" / "kernels"
    assert images and all((kdir / f"{i}.cubin").exists() for i in images) and "chain" not in images
    for text in ('{"architecture": "none of these"}', "{}", "[1, 2", '{"architecture": 3}', '{"architecture": "Nufalorn"} x', ""):
        assert M.config_images(text) is None
    assert M.config_images('{"note": "a \\"quoted\\" \\u00e9 {", "x": [1, -2.5e3, true, null, {"y": []}], "architecture": "Nufalorn"}') == images


def test_command_line_lists_architectures(lb):
    r = subprocess.run([sys.executable, "-m", "lithos_b200", "architectures"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0 and "Nufalorn" in r.stdout.split()
