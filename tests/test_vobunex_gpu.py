"""GPU: Vobunex models through the library against the plain statement in oracle/vobunex.py: every mechanism, prompts, portions,
decoding, what the caches and states hold, reuse, generation, the command line and the trace replay.

Tolerances: root mean square over the vocabulary of the logit difference, over the root mean square of all logits.  fp32 models:
3e-5 (rounding).  bf16 models: 6e-2 per position and 2e-2 on average (operands of the projections have 8 bits)."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import vobunex_cases as C
from oracle import vobunex as V

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": (3e-5, 3e-5), "bfloat16": (6e-2, 2e-2)}
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def errors(got, want):
    return np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want ** 2))


def check(got, want, dtype, what=""):
    e = errors(np.asarray(got, np.float64), want)
    assert np.isfinite(e).all() and e.max() <= TOL[dtype][0] and e.mean() <= TOL[dtype][1], (what, dtype, int(e.argmax()), e.max(), e.mean())


class Case:
    def __init__(self, path, ctx, cfg, seed, tweak=None):
        self.cfg, self.w = cfg, C.tensors(cfg, seed)
        if tweak:
            tweak(self.w)
        self.dir, self.ctx = C.write(path, cfg, self.w), ctx

    def open(self, dtype, max_ctx):
        from lithos_b200 import model as M
        return M.Model.open(self.ctx, self.dir, max_ctx, dtype)

    def want(self, toks):
        return V.Vobunex(self.cfg, self.w).run(toks)


def feed(m, toks, cuts):
    """logits of every token, the sequence cut at `cuts`"""
    out, pos = [], 0
    for n in cuts:
        out.append(m.forward(toks[pos:pos + n], pos, list(range(n))))
        pos += n
    assert pos == len(toks)
    return np.concatenate(out)


@BOTH
@pytest.mark.parametrize("name", list(C.CASES))
def test_prompt_decode_and_portions(ctx, lb, tmp_path, name, dtype):
    """whole prompt, token by token, and portions down to two tokens: the same logits"""
    c = Case(tmp_path, ctx, C.CASES[name], 11)
    n = 150
    toks = tokens(c.cfg, n)
    want = c.want(toks)
    m = c.open(dtype, n)
    check(m.forward(toks, 0, list(range(n))), want, dtype, "whole")
    m.reset_state()
    check(feed(m, toks, [1] * n), want, dtype, "decode")
    for cuts in ([64, 2, 2, 1, 30, 1, 1, 7, 42], [2] * 75, [17, 130, 3], [149, 1], [1, 149], [15, 16, 33, 65, 21]):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.close()


MECHANISMS = {
    "latent": [C.latent(4, 20, 8, 24, 36, 56)],
    "latent_no_scaling": [C.latent(4, 24, 24, 24, 36, 56, scaling=None)],
    "yarn_all_slow": [C.latent(3, 8, 16, 16, 20, 24, scaling={"factor": 3.0, "original": 8, "fast": 2.0, "slow": 1.0})],
    "yarn_all_fast": [C.latent(3, 8, 16, 16, 20, 24, scaling={"factor": 3.0, "original": 1e9, "fast": 2.0, "slow": 1.0})],
    "yarn_no_ramp": [C.latent(3, 8, 16, 16, 20, 24, base=100.0, scaling={"factor": 1.0, "original": 64, "fast": 4.0, "slow": 4.0})],
    "mamba2": [C.mamba2(6, 24, 40, groups=2, conv=4, norm_groups=3)],
    "mamba2_one_tap": [C.mamba2(2, 16, 16, conv=1)],
    "squared_relu": [C.mamba2(1, 4, 4, mlp=C.dense(150))],
    "experts": [C.mamba2(1, 4, 4, mlp=C.moe(50, 9, 4, limit=0.5))],
    "all_experts": [C.mamba2(1, 4, 4, mlp=C.moe(24, 3, 3))],
}


@pytest.mark.parametrize("name", list(MECHANISMS))
def test_one_mechanism(ctx, lb, tmp_path, name):
    c = Case(tmp_path, ctx, C.config(56, 75, MECHANISMS[name]), 21)
    toks = tokens(c.cfg, 90)
    want = c.want(toks)
    for dtype in ("float32", "bfloat16"):
        m = c.open(dtype, 90)
        check(m.forward(toks, 0, list(range(90))), want, dtype)
        m.reset_state()
        check(feed(m, toks, [40] + [1] * 50), want, dtype)
        m.close()


def test_caches_and_states_hold_what_they_should(ctx, lb, tmp_path):
    """normed latents and rotated key parts; states and the convolution's last inputs -- after a prompt, and after decoding"""
    cfg = C.config(60, 70, [C.latent(4, 20, 8, 12, 24, 40), C.mamba2(4, 18, 24, groups=2, conv=3)])
    c = Case(tmp_path, ctx, cfg, 5)
    toks = tokens(cfg, 40)
    om, eps = V.Vobunex(cfg, c.w), cfg["norm"]["eps"]
    keep = []
    om.run(toks, keep)
    h0, h1 = om._norm(om.embed(toks), "l0.norm1"), om._norm(keep[0], "l1.norm1")
    lat, rot = V.latent_cache(h0, om._sub("l0.mix."), cfg["layers"][0]["mixer"], eps)
    p1 = om._sub("l1.mix.")
    _, S = V.mamba2(h1, p1, cfg["layers"][1]["mixer"], eps)
    chan = 4 * 18 + 2 * 2 * 24
    pre = (h1 @ p1["in"].T)[:, 72:72 + chan]
    for cuts in ([40], [23] + [1] * 17, [2] * 20):
        m = c.open("float32", 48)
        feed(m, toks, cuts)
        row = m.get_state(0, 0, np.float32, 48 * (64 + 16)).reshape(48, 80)   # latent padded to 64, key part to 16
        assert np.allclose(row[:40, :40], lat, atol=2e-5) and np.allclose(row[:40, 64:72], rot, atol=2e-5)
        assert not row[:, 40:64].any() and not row[:, 72:].any() and not row[40:].any()
        assert np.allclose(m.get_state(1, 0, np.float32, S.size).reshape(S.shape), S, atol=2e-5 * np.abs(S).max())
        ring = m.get_state(1, 1, np.float32, 3 * chan).reshape(3, chan)
        for pos in (38, 39):
            assert np.allclose(ring[pos % 3], pre[pos], atol=2e-5)
        m.close()


def far_key(w):
    """tokens 0 and 1: the pair's own feature is all of their embedding, the first head's query of token 1 asks for the latent of token 0"""
    d = np.zeros(64, np.float32)
    d[7] = 24.0
    w["embed"][0] = C.bf16(d)
    w["embed"][1] = C.bf16(-d)
    w["l0.mix.dkv"][:, :] *= 0.25
    w["l0.mix.dkv"][3, :] = 0
    w["l0.mix.dkv"][3, 7] = 1.0        # latent feature 3: large for token 0
    w["l0.mix.dq"][:, :] *= 0.25
    w["l0.mix.dq"][5, :] = 0
    w["l0.mix.dq"][5, 7] = -1.0        # query latent 5: large for token 1
    w["l0.mix.uk"][:16] = 0
    w["l0.mix.uk"][2, 3] = 6.0
    w["l0.mix.uq"][:24] = 0
    w["l0.mix.uq"][2, 5] = 2.0


@BOTH
def test_far_key(ctx, lb, tmp_path, dtype):
    """one key among hundreds stands out: asked for from near and from far, in a prompt, in portions and in decoding"""
    cfg = C.config(64, 90, [C.latent(3, 16, 8, 16, 20, 32, scale=0.5, mlp=C.dense(32))], bigram=None)
    c = Case(tmp_path, ctx, cfg, 31, tweak=far_key)
    n = 700
    base = np.random.default_rng(4).integers(2, 90, n)
    base[0] = 0
    ask = [1, 31, 63, 64, 65, 127, 128, 300, 512, 640, 698, 699]
    base[ask] = 1
    toks = base.tolist()
    want = c.want(toks)
    other = list(toks)
    other[0] = 5
    moved = errors(c.want(other), want)
    assert moved[ask].min() > 0.1       # the key matters wherever it is asked for
    m = c.open(dtype, n)
    check(m.forward(toks, 0, list(range(n))), want, dtype, "prompt")
    for cuts in ([60] + [1] * 10 + [230] + [1] * 4 + [396], [64, 64, 2, 170, 213, 187], [299, 2, 5, 2, 390, 2], [690] + [1] * 10):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.close()


@BOTH
@pytest.mark.parametrize("sink", [-30.0, 0.0, 12.0])
def test_sinks(ctx, lb, tmp_path, sink, dtype):
    """sinks that take nothing and sinks that take nearly everything, at the first positions and later; scores far above and below zero"""
    for scale in (0.25, -1.5, 1.5):
        cfg = C.config(64, 50, [C.latent(3, 16, 8, 16, 20, 32, scale=scale)])

        def tweak(w):
            w["l0.mix.sink"][:2] = sink
        c = Case(tmp_path / str(scale), ctx, cfg, 7, tweak=tweak)
        toks = tokens(cfg, 45)
        want = c.want(toks)
        m = c.open(dtype, 64)
        check(m.forward(toks, 0, list(range(45))), want, dtype)
        m.reset_state()
        check(feed(m, toks, [1] * 20 + [3] * 5 + [1] * 10), want, dtype)
        m.close()


@BOTH
def test_pair_embedding_across_portions(ctx, lb, tmp_path, dtype):
    """the same token after different tokens, the pair cut by a portion's edge, and a first token that equals the last of the sequence before"""
    cfg = C.config(48, 40, [C.mamba2(2, 8, 8, conv=2)], bigram=(53, 19, 3))
    c = Case(tmp_path, ctx, cfg, 43)
    toks = [3, 9, 3, 9, 9, 3, 12, 3, 3, 9, 12, 9]
    want = c.want(toks)
    m = c.open(dtype, 32)
    for cuts in ([12], [1] * 12, [5, 7], [4, 2, 6], [1, 11], [6, 1, 2, 1, 2]):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.reset_state()
    check(feed(m, [9], [1]), c.want([9]), dtype)
    m.close()


@BOTH
def test_slow_decay_keeps_a_distant_token(ctx, lb, tmp_path, dtype):
    """heads that hardly forget: the first token shows in the state hundreds of tokens later, whatever the blocks and portions"""
    cfg = C.config(64, 60, [C.mamba2(4, 16, 24, groups=2, conv=3)], bigram=None)

    def tweak(w):
        w["l0.mix.A_log"][:] = -9.0
        w["l0.mix.dt_bias"][:] = C.bf16(np.float32([-4, -3, -2, -1]))
        w["embed"][0] *= 8
    c = Case(tmp_path, ctx, cfg, 47, tweak=tweak)
    n = 1000                                          # several segments side by side in a prompt's chunk
    toks = np.random.default_rng(9).integers(1, 60, n)
    toks[0] = 0
    toks = toks.tolist()
    want = c.want(toks)
    m = c.open(dtype, n)
    check(m.forward(toks, 0, list(range(n))), want, dtype, "prompt")
    for cuts in ([63, 2, 64, 1, 128, 65, 677], [2, 998], [513, 387] + [1] * 100):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.close()


@BOTH
def test_long_prompt_many_chunks(ctx, lb, tmp_path, dtype):
    """2700 tokens: several chunks of the prompt pass over four streams, then decoding"""
    cfg = C.config(64, 101, [C.latent(4, 16, 8, 32, 24, 48, mlp=C.dense(40)), C.mamba2(4, 16, 16, groups=2, norm_groups=2, mlp=C.moe(24, 6, 2)),
                             C.latent(2, 16, 16, 16, 16, 32, mlp=C.moe(32, 5, 3)), C.mamba2(2, 24, 16)])
    c = Case(tmp_path, ctx, cfg, 13)
    n, tail = 2700, 20
    toks = tokens(cfg, n + tail)
    want = c.want(toks)
    m = c.open(dtype, n + tail)
    places = sorted({p for e in range(0, n, 256) for p in (e, e + 1, e + 255) if p < n} | {n - 1})
    check(m.forward(toks[:n], 0, places), want[places], dtype, "prompt")
    check(feed_from(m, toks, n), want[n:], dtype, "decode")
    m.close()


def feed_from(m, toks, pos):
    return np.concatenate([m.forward([t], pos + i, [0]) for i, t in enumerate(toks[pos:])])


def test_long_decoding(ctx, lb, tmp_path):
    """500 tokens decoded one by one after a prompt: nothing drifts"""
    cfg = C.config(48, 60, [C.latent(2, 16, 8, 16, 16, 24, mlp=C.dense(32)), C.mamba2(2, 12, 12, mlp=C.moe(16, 4, 2))])
    c = Case(tmp_path, ctx, cfg, 17)
    toks = tokens(cfg, 520)
    want = c.want(toks)
    m = c.open("float32", 520)
    m.forward(toks[:20], 0)
    check(feed_from(m, toks, 20), want[20:], "float32")
    m.close()


@BOTH
def test_caches_used_again(ctx, lb, tmp_path, dtype):
    """a second sequence in the same caches and states gives bit for bit what it gives in a fresh model"""
    c = Case(tmp_path, ctx, C.CASES["mixed"], 19)
    a, b = tokens(c.cfg, 140, 1), tokens(c.cfg, 77, 2)
    fresh = c.open(dtype, 140)
    want = feed(fresh, b, [50] + [1] * 5 + [22])
    fresh.close()
    m = c.open(dtype, 140)
    feed(m, a, [100] + [1] * 40)
    m.reset_state()
    assert np.array_equal(feed(m, b, [50] + [1] * 5 + [22]), want)
    m.reset_state()
    m.forward(a[:3], 0)
    m.reset_state()
    assert np.array_equal(feed(m, b, [50] + [1] * 5 + [22]), want)
    m.close()


def test_checkpoint_and_rollback(ctx, lb, tmp_path):
    c = Case(tmp_path, ctx, C.CASES["large_state"], 23)
    toks = tokens(c.cfg, 60)
    m = c.open("float32", 80)
    m.forward(toks[:40], 0)
    m.checkpoint()
    first = feed_from(m, toks, 40)
    m.rollback()
    assert np.array_equal(feed_from(m, toks, 40), first)
    m.close()


def greedy(cfg, w, prompt, n):
    om, toks, margin = V.Vobunex(cfg, w), list(prompt), []
    for _ in range(n):
        z = om.run(toks)[-1]
        s = np.sort(z)
        margin.append(s[-1] - s[-2])
        toks.append(int(np.argmax(z)))
    return toks[len(prompt):], margin


def test_greedy_generation(ctx, lb, tmp_path):
    """prompt pass, captured decode step and arg-max through lb_model_generate, and the command line, give the plain statement's tokens"""
    c = Case(tmp_path, ctx, C.CASES["mixed"], 29)
    prompt = tokens(c.cfg, 30)
    want, margin = greedy(c.cfg, c.w, prompt, 24)
    assert min(margin) > 1e-3
    m = c.open("float32", 64)
    assert m.generate(prompt, 24) == want
    m.reset_state()
    nxt, got = m.prefill(prompt), []
    for i in range(24):                               # launch by launch
        got.append(nxt)
        nxt = m.decode(nxt, 30 + i)
    assert got == want
    m.reset_state()
    eos = want[5]
    assert m.generate(prompt, 24, eos=eos) == want[:want.index(eos) + 1]
    m.reset_state()
    m.set_sampling(1.5, 8, seed=3)
    s1 = m.generate(prompt, 24)
    m.reset_state()
    assert m.generate(prompt, 24) == s1 and all(0 <= t < c.cfg["vocab"] for t in s1)
    m.close()
    r = subprocess.run([sys.executable, "-m", "lithos_b200", "generate", "--model", str(c.dir), "--prompt-ids", ",".join(map(str, prompt)), "--max-new", "24",
                        "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.splitlines()[-1])["tokens"] == want


def test_trace_replay(ctx, lb, tmp_path):
    c = Case(tmp_path / "m", ctx, C.CASES["odd_width"], 37)
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(c.cfg, 33, 1), tokens(c.cfg, 10, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [3, 0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [9]}], "end": ["b"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(c.dir), "--dtype", "float32", "--out", str(out), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, cwd=tmp_path)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = c.want(a), c.want(b)
    for i, want in ((0, wa[[3, 0, 19]]), (2, wa[[32]]), (3, wb[[9]])):
        check(np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, c.cfg["vocab"]), want, "float32", i)
    assert not (out / "1.f32").exists()


def test_bad_models_are_refused(ctx, lb, tmp_path):
    from lithos_b200 import model as M
    cfg = C.config(64, 40, [C.latent(4, 16, 8, 16, 20, 32, mlp=C.moe(16, 4, 2)), C.mamba2(2, 8, 8, mlp=C.dense(16))])
    w = C.tensors(cfg, 1)

    def refused(change_cfg=None, change_w=None, status=None):
        c2, w2 = json.loads(json.dumps(cfg)), dict(w)
        if change_cfg:
            change_cfg(c2)
        if change_w:
            change_w(w2)
        with pytest.raises(lb.LithosError) as e:
            M.Model.open(ctx, C.write(tmp_path / "x", c2, w2), 32)
        assert status is None or e.value.status == status, e.value

    refused(change_w=lambda t: t.pop("l0.mix.uk"), status=lb.LB_ERR_IO)
    refused(change_w=lambda t: t.pop("bigram"), status=lb.LB_ERR_IO)
    refused(change_w=lambda t: t.update({"l0.mlp.table": t["l0.mlp.table"] + 3}), status=lb.LB_ERR_IO)
    refused(change_w=lambda t: t.update({"l1.mix.conv": t["l1.mix.conv"][:, :-1]}), status=lb.LB_ERR_IO)
    refused(lambda c: c["layers"][0]["mixer"].update(kv_rank=1000), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][1]["mixer"].update(groups=3), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=5), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0].update(type="something else"), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][1]["mlp"].update(kind="none"), status=lb.LB_ERR_INVALID)
    m = M.Model.open(ctx, C.write(tmp_path / "ok", cfg, w), 32)
    for toks, pos, want in (([1] * 40, 0, []), ([1], 32, [0]), ([40], 0, [0]), ([1, 2], 0, [2]), ([1, 2], 0, [1, 0])):
        with pytest.raises(lb.LithosError):
            m.forward(toks, pos, want)
    m.close()


def test_generated_weights(ctx, lb):
    from lithos_b200 import model as M
    for name in ("mixed", "wide_heads"):
        m = M.Model.open_synthetic(ctx, C.CASES[name], 64, "bfloat16", 9)
        a = m.generate(list(range(10)), 8)
        m.reset_state()
        assert m.generate(list(range(10)), 8) == a and m.architecture == "stack"
        m.close()
