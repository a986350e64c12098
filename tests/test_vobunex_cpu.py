"""CPU: the plain Vobunex statement (oracle/vobunex.py) agrees with itself where two formulations must agree, the test models show every
mechanism (a planted mistake in the plain statement moves the logits far beyond the GPU tests' tolerances), and the registry knows the design."""
import json
from pathlib import Path

import numpy as np
import pytest

import vobunex_cases as C
from oracle import vobunex as V

ROOT = Path(__file__).resolve().parent.parent


def run(cfg, w, toks):
    return V.Vobunex(cfg, w).run(toks)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def rms_diff(a, b):
    return np.sqrt(np.mean((a - b) ** 2, axis=-1)) / np.sqrt(np.mean(b ** 2))


def test_recurrence_carries_its_state():
    r = np.random.default_rng(1)
    x, B, Cm = r.standard_normal((30, 4, 5)), r.standard_normal((30, 2, 7)), r.standard_normal((30, 2, 7))
    dt, A, D = r.uniform(0.01, 1, (30, 4)), r.standard_normal(4), r.standard_normal(4)
    whole, S = V.ssm_scan(x, B, Cm, dt, A, D)
    o1, S1 = V.ssm_scan(x[:11], B[:11], Cm[:11], dt[:11], A, D)
    o2, S2 = V.ssm_scan(x[11:], B[11:], Cm[11:], dt[11:], A, D, S1)
    assert np.allclose(np.concatenate([o1, o2]), whole) and np.allclose(S, S2)
    # closed form of one read-out: head 3 (group 1), token 17
    t, h = 17, 3
    o = D[h] * x[t, h] + sum(np.exp(-np.exp(A[h]) * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (Cm[t, 1] @ B[j, 1]) * x[j, h] for j in range(t + 1))
    assert np.allclose(o, whole[t, h])


def test_absorbed_latent_attention_is_the_same():
    """scores against the latent itself with W_uk^T q, and W_uv applied to the weighted latent"""
    cfg = C.config(40, 30, [C.latent(3, 10, 6, 8, 12, 20)])
    w = {k: np.asarray(t, np.float64) for k, t in C.tensors(cfg, 2).items()}
    p, c = {k[7:]: t for k, t in w.items() if k.startswith("l0.mix.")}, cfg["layers"][0]["mixer"]
    h = np.random.default_rng(3).standard_normal((25, 40))
    lat, kr = V.latent_cache(h, p, c, 1e-5)
    q = ((V.rms(h @ p["dq"].T, 1e-5) * p["dq.norm"]) @ p["uq"].T).reshape(25, 3, 16)
    freq, mul = V.yarn(6, c["rot"]["base"], c["rot"]["scaling"])
    qr = V.rotate_pairs(q[..., 10:], np.arange(25), freq, mul)
    out = []
    for a in range(3):
        ql = q[:, a, :10] @ p["uk"][10 * a:10 * a + 10]
        s = (ql @ lat.T + qr[:, a] @ kr.T) * c["scale"]
        out.append(V.softmax_with_sink(s, V.causal_mask(25), p["sink"][a]) @ lat @ p["uv"][8 * a:8 * a + 8].T)
    assert np.allclose(np.concatenate(out, -1) @ p["o"].T, V.latent_attention(h, p, c, 1e-5))


def test_rotation_frequencies():
    f, m = V.yarn(8, 100.0, None)
    assert np.allclose(f, 100.0 ** (-np.arange(4) / 4)) and m == 1.0
    g, m = V.yarn(8, 100.0, {"factor": 4.0, "original": 1e12, "fast": 2.0, "slow": 1.0})
    assert np.allclose(g, f) and np.isclose(m, 1 + 0.1 * np.log(4))
    g, _ = V.yarn(8, 100.0, {"factor": 4.0, "original": 1.0, "fast": 2.0, "slow": 1.0})
    assert np.allclose(g, [f[0], f[1] / 4, f[2] / 4, f[3] / 4])
    assert V.bigram_rows([5, 7, 5], 11, 3, 2).tolist() == [11, (15 + 14) % 11, (21 + 10) % 11]


def no_sink(s, m, sink):
    e = np.exp(np.where(m, s, -np.inf) - np.max(np.where(m, s, -np.inf), -1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def wrap(name, make):
    def plant(mp):
        mp.setattr(V, name, make(getattr(V, name)))
    return plant


MISTAKES = {
    "no sink": wrap("softmax_with_sink", lambda f: no_sink),
    "sink of one": wrap("softmax_with_sink", lambda f: lambda s, m, sink: f(s, m, 0.0)),
    "a key too few": wrap("causal_mask", lambda f: lambda n: np.tril(np.ones((n, n), bool), -1) | (np.arange(n)[:, None] + np.arange(n) == 0)),
    "cosines not scaled": wrap("yarn", lambda f: lambda *a: (f(*a)[0], 1.0)),
    "frequencies not scaled": wrap("yarn", lambda f: lambda d, b, s: (f(d, b, None)[0], f(d, b, s)[1])),
    "halves rotated instead of neighbours": wrap("rotate_pairs", lambda f: lambda x, *a: f(x.reshape(*x.shape[:-1], 2, -1).swapaxes(-1, -2).reshape(x.shape), *a)),
    "pairs not mixed in": wrap("bigram_rows", lambda f: lambda t, b, p, c: f(t, b, 0, c)),
    "first token as if token 0 came before": wrap("bigram_rows", lambda f: lambda t, b, p, c: f([0] + list(t), b, p, c)[1:]),
    "convolution reversed": wrap("causal_conv", lambda f: lambda u, w, b: f(u, w[:, ::-1], b)),
    "convolution without its bias": wrap("causal_conv", lambda f: lambda u, w, b: f(u, w, 0.0)),
    "decay without the step size": wrap("ssm_scan", lambda f: lambda x, B, Cm, dt, A, D, state=None: f(x * dt[..., None], B, Cm, np.ones_like(dt), A, D)),
    "no skip": wrap("ssm_scan", lambda f: lambda x, B, Cm, dt, A, D, state=None: f(x, B, Cm, dt, A, 0 * D)),
    "groups interleaved": wrap("ssm_scan", lambda f: lambda x, B, Cm, dt, A, D, state=None: f(x, B[:, ::-1], Cm[:, ::-1], dt, A, D)),
    "state lost after 16 tokens": wrap("ssm_scan", lambda f: lambda x, B, Cm, dt, A, D, state=None: (np.concatenate([f(x[:16], B[:16], Cm[:16], dt[:16], A, D)[0],
                                                                                                                       f(x[16:], B[16:], Cm[16:], dt[16:], A, D)[0]]), None)),
    "step size without softplus": wrap("softplus", lambda f: np.exp),
    "ReLU not squared": wrap("squared_relu", lambda f: lambda h, p: np.maximum(h @ p["up"].T, 0) @ p["down"].T),
    "gate not clamped": wrap("clamped_expert", lambda f: lambda h, g, u, d, limit: f(h, g, u, d, 1e9)),
    "weights not shared out": wrap("table_experts", lambda f: lambda h, t, p, c: f(h, t, p, c) * c["router"]["top"]),
    "experts of the next token": wrap("table_experts", lambda f: lambda h, t, p, c: f(h, t[1:] + t[:1], p, c)),
    "mean not taken off": wrap("layer_norm", lambda f: lambda x, w, b, eps: V.rms(x, eps) * w + b),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_test_model_shows_mistake(name, monkeypatch):
    cfg = C.CASES["mixed"]
    w, toks = C.tensors(cfg, 3), tokens(cfg, 60)
    good = run(cfg, w, toks)
    MISTAKES[name](monkeypatch)
    assert np.max(rms_diff(run(cfg, w, toks), good)) > 0.06, name


def test_registry(lb):
    from lithos_b200 import model as M
    assert "Vobunex" in M.architectures()
    images = M.config_images(json.dumps(C.CASES["mixed"]))
    kdir = ROOT / "lithos_b200" / "kernels"
    assert images and all((kdir / f"{i}.cubin").exists() for i in images) and "decay_attention" not in images
