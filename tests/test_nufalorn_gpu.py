"""GPU: Nufalorn models through the library against the plain statement in oracle/nufalorn.py: every mechanism, prompts, portions,
decoding, what the caches and states hold, reuse, generation, the command line and the trace replay.

Tolerances: root mean square over the vocabulary of the logit difference, over the root mean square of all logits.  fp32 models:
2e-5 (rounding).  bf16 models: 4e-2 per position and 1.5e-2 on average (operands of the projections have 8 bits)."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import nufalorn_cases as C
from oracle import nufalorn as N

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": (2e-5, 2e-5), "bfloat16": (4e-2, 1.5e-2)}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def errors(got, want):
    return np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want ** 2))


def check(got, want, dtype, what=""):
    e = errors(np.asarray(got, np.float64), want)
    assert np.isfinite(e).all() and e.max() <= TOL[dtype][0] and e.mean() <= TOL[dtype][1], (what, dtype, int(e.argmax()), e.max(), e.mean())


class Case:
    def __init__(self, path, ctx, cfg, seed, rank=5, tweak=None):
        self.cfg, self.w = cfg, C.tensors(cfg, seed, rank)
        if tweak:
            tweak(self.w)
        self.dir, self.ctx = C.write(path, cfg, self.w), ctx

    def open(self, dtype, max_ctx):
        from lithos_b200 import model as M
        return M.Model.open(self.ctx, self.dir, max_ctx, dtype)

    def want(self, toks):
        return N.Nufalorn(self.cfg, self.w).run(toks)


def feed(m, toks, cuts):
    """logits of every token, the sequence cut at `cuts`"""
    out, pos = [], 0
    for n in cuts:
        out.append(m.forward(toks[pos:pos + n], pos, list(range(n))))
        pos += n
    assert pos == len(toks)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    for cuts in ([64, 2, 2, 1, 30, 1, 1, 7, 42], [2] * 75, [17, 130, 3], [149, 1], [1, 149]):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.close()


@pytest.mark.parametrize("layer", ["att", "att_shared", "hgrn2", "gla", "ff"])
def test_one_mechanism(ctx, lb, tmp_path, layer):
    layers = {"att": [C.att(4, 2, 20, 24, 33, rot_dims=12)], "att_shared": [C.att(4, 4, 16, 8, 25), C.att(4, 4, 16, 8, 60, kv_from=0)],
              "hgrn2": [C.hgrn2(3, 24, 40)], "gla": [C.gla(3, 36, 20, tau=5.0)], "ff": [C.hgrn2(1, 4, 4, ff=150)]}[layer]
    c = Case(tmp_path, ctx, C.config(56, 75, layers), 21, rank=9)
    toks = tokens(c.cfg, 90)
    want = c.want(toks)
    for dtype in ("float32", "bfloat16"):
        m = c.open(dtype, 90)
        check(m.forward(toks, 0, list(range(90))), want, dtype)
        m.reset_state()
        check(feed(m, toks, [40] + [1] * 50), want, dtype)
        m.close()


def test_caches_and_states_hold_what_they_should(ctx, lb, tmp_path):
    """rotated keys; normed, rotated values; recurrent states -- after a prompt, and after decoding"""
    cfg = C.config(60, 70, [C.att(4, 2, 20, 12, 31, rot_dims=8), C.hgrn2(2, 24, 18), C.gla(3, 10, 22)])
    c = Case(tmp_path, ctx, cfg, 5)
    toks = tokens(cfg, 40)
    om, eps = N.Nufalorn(cfg, c.w), cfg["norm"]["eps"]
    keep = []
    om.run(toks, keep)
    x = [om.w["embed"][toks]] + keep
    h = [N.rms_norm_zero_centred(x[i], om.w[f"l{i}.norm1"], eps) for i in range(3)]
    k, v = N.keys_values(h[0], om._sub("l0.mix."), cfg["layers"][0]["mixer"], eps)
    _, S1 = N.hgrn2(h[1], om._sub("l1.mix."), cfg["layers"][1]["mixer"], eps)
    _, S2 = N.gla(h[2], om._sub("l2.mix."), cfg["layers"][2]["mixer"], eps)
    for cuts in ([40], [23] + [1] * 17):
        m = c.open("float32", 48)
        feed(m, toks, cuts)
        kg = m.get_state(0, 0, np.float32, 48 * 2 * 32).reshape(48, 2, 32)   # head sizes are padded to 16
        vg = m.get_state(0, 1, np.float32, 48 * 2 * 16).reshape(48, 2, 16)
        assert np.allclose(kg[:40, :, :20], k, atol=2e-5) and np.allclose(vg[:40, :, :12], v, atol=2e-5)
        assert not kg[:, :, 20:].any() and not vg[:, :, 12:].any() and not kg[40:].any()
        for i, S in ((1, S1), (2, S2)):
            assert np.allclose(m.get_state(i, 0, np.float32, S.size).reshape(S.shape), S, atol=2e-5 * np.abs(S).max())
        m.close()


def stand_out(w):
    """tokens 0 and 1 get embeddings along one direction that the first head's query and key pick out: a query token 1 asks for the
    key of token 0 whatever else is there"""
    d = np.zeros(64, np.float32)
    d[7] = 8.0
    w["embed"][0] = w["embed"][1] = C.bf16(d)
    for t in ("q", "k"):
        w[f"l0.mix.{t}"][:16] = 0
        w[f"l0.mix.{t}"][1, 7] = 1.0     # the second of a pair that hardly turns at this base


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_key_inside_and_outside_a_block(ctx, lb, tmp_path, dtype):
    """one key stands out among hundreds, from the first and from the last place of a block: seen up to the block's last position,
    not one position later; in a prompt, in portions and in decoding"""
    B = 300
    cfg = C.config(64, 90, [C.att(4, 1, 16, 16, B, rot_dims=2, base=1e9, scale=0.35, ff=32)])
    # rot_dims 2: the only rotated pair is (0, 1), one radian per position; move the match to an unrotated feature
    def tweak(w):
        stand_out(w)
        for t in ("q", "k"):
            w[f"l0.mix.{t}"][1, 7], w[f"l0.mix.{t}"][9, 7] = 0.0, 1.0
    c = Case(tmp_path, ctx, cfg, 31, tweak=tweak)
    n = 2 * B + 20
    base = np.random.default_rng(4).integers(2, 90, n)
    base[[0, B, 2 * B - 1]] = 0                        # keys: first place of blocks 0 and 1, last place of block 1
    ask = [B - 2, B - 1, B + 1, 2 * B - 2, 2 * B, 2 * B + 1]
    base[ask] = 1
    toks = base.tolist()
    want = c.want(toks)
    # the key matters where it is seen and nowhere else
    other = list(toks)
    other[0] = 5
    moved = errors(c.want(other), want)
    assert moved[B - 1] > 0.1 and moved[B + 1:].max() < 1e-12
    m = c.open(dtype, n)
    check(m.forward(toks, 0, list(range(n))), want, dtype, "prompt")
    for cuts in ([B - 3] + [1] * 8 + [B - 10] + [1] * 25, [B, B, 20], [B - 1, 2, B - 3, 5, 2, 15], [100, 150, 60, 289, 21]):
        m.reset_state()
        check(feed(m, toks, cuts), want, dtype, cuts)
    m.close()


def test_first_tokens_and_sink(ctx, lb, tmp_path):
    """scores far below zero (the sink takes all the weight), scores far above, and the first positions, where the sink is one of few"""
    for scale in (-4.0, 4.0, 0.01):
        cfg = C.config(64, 50, [C.att(2, 1, 16, 16, 40, scale=scale)])
        c = Case(tmp_path / str(scale), ctx, cfg, 7)
        toks = tokens(cfg, 45)
        want = c.want(toks)
        m = c.open("float32", 64)
        check(m.forward(toks, 0, list(range(45))), want, "float32")
        m.reset_state()
        check(feed(m, toks, [1] * 45), want, "float32")
        m.close()
        m = c.open("bfloat16", 64)
        m.forward(toks, 0, [0])
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompt_many_chunks(ctx, lb, tmp_path, dtype):
    """2700 tokens: six chunks of the prompt pass over four streams, then decoding; positions seen at every chunk's edge"""
    cfg = C.config(64, 101, [C.att(4, 2, 16, 32, 700, ff=40), C.hgrn2(2, 16, 16), C.gla(2, 16, 24, ff=24), C.att(4, 2, 16, 32, 700, kv_from=0)])
    c = Case(tmp_path, ctx, cfg, 13)
    n, tail = 2700, 20
    toks = tokens(cfg, n + tail)
    want = c.want(toks)
    m = c.open(dtype, n + tail)
    places = sorted({p for e in range(0, n, 512) for p in (e, e + 1, e + 511) if p < n} | {699, 700, 701, 1399, 1400, 2099, 2100, n - 1})
    check(m.forward(toks[:n], 0, places), want[places], dtype, "prompt")
    check(feed_from(m, toks, n), want[n:], dtype, "decode")
    m.close()


def feed_from(m, toks, pos):
    return np.concatenate([m.forward([t], pos + i, [0]) for i, t in enumerate(toks[pos:])])


def test_long_decoding(ctx, lb, tmp_path):
    """500 tokens decoded one by one after a prompt: nothing drifts"""
    cfg = C.config(48, 60, [C.att(2, 1, 16, 16, 90, ff=32), C.hgrn2(2, 12, 12), C.gla(2, 12, 12, tau=16.0)])
    c = Case(tmp_path, ctx, cfg, 17)
    toks = tokens(cfg, 520)
    want = c.want(toks)
    m = c.open("float32", 520)
    m.forward(toks[:20], 0)
    check(feed_from(m, toks, 20), want[20:], "float32")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    c = Case(tmp_path, ctx, C.CASES["many_groups"], 23)
    toks = tokens(c.cfg, 60)
    m = c.open("float32", 80)
    m.forward(toks[:40], 0)
    m.checkpoint()
    first = feed_from(m, toks, 40)
    m.rollback()
    assert np.array_equal(feed_from(m, toks, 40), first)
    m.close()


def greedy(cfg, w, prompt, n):
    om, toks, margin = N.Nufalorn(cfg, w), list(prompt), []
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
    c = Case(tmp_path / "m", ctx, C.CASES["many_groups"], 37)
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
    V = c.cfg["vocab"]
    for i, want in ((0, wa[[3, 0, 19]]), (2, wa[[32]]), (3, wb[[9]])):
        check(np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, V), want, "float32", i)
    assert not (out / "1.f32").exists()


def test_bad_models_are_refused(ctx, lb, tmp_path):
    from lithos_b200 import model as M
    cfg = C.config(64, 40, [C.att(4, 2, 16, 16, 20, ff=16), C.gla(2, 8, 8), C.att(4, 2, 16, 16, 20, kv_from=0)])
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

    refused(change_w=lambda t: t.pop("l0.mix.q"), status=lb.LB_ERR_IO)
    refused(change_w=lambda t: t.update({"head": t["head"][:, :-1]}), status=lb.LB_ERR_IO)
    refused(lambda c: c["layers"][0]["mixer"].update(kv_heads=3), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0]["mixer"].update(dim=1000), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][2]["mixer"].update(kv_from=1), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0].update(type="something else"), status=lb.LB_ERR_INVALID)
    refused(lambda c: c["layers"][0]["mlp"].update(kind="experts"), status=lb.LB_ERR_INVALID)
    refused(lambda c: c.update(architecture="unheard of"), status=lb.LB_ERR_INVALID)
    m = M.Model.open(ctx, C.write(tmp_path / "ok", cfg, w), 32)
    for toks, pos, want in (([1] * 40, 0, []), ([1], 32, [0]), ([40], 0, [0]), ([1, 2], 0, [2]), ([1, 2], 0, [1, 0])):
        with pytest.raises(lb.LithosError):
            m.forward(toks, pos, want)
    m.close()


def test_generated_weights_and_the_hybrid_through_the_registry(ctx, lb):
    """the registry also opens the int4 hybrid, and both classes fill themselves with seeded weights"""
    from lithos_b200 import model as M
    m = M.Model.open_synthetic(ctx, C.CASES["mixed"], 64, "bfloat16", 9)
    a = m.generate(list(range(10)), 8)
    m.reset_state()
    assert m.generate(list(range(10)), 8) == a and m.architecture == "stack"
    m.close()
    t = M.tiny(max_ctx=64)
    cfg = {"architecture": "Qwen3.5-hybrid", **{n: getattr(t, n) for n, _ in M.ModelCfg._fields_ if n not in ("max_ctx", "reserved")}}
    m, d = M.Model.open_synthetic(ctx, cfg, 64, "bfloat16", 7), M.Model(ctx, t)
    d.fill_synthetic(7)
    assert m.architecture == "hybrid"
    prompt = list(range(3, 40))
    got = m.forward(prompt, 0, [5, 36])
    d.prefill(prompt)
    assert np.array_equal(got[1], d.logits())
    d.reset_state()
    d.prefill(prompt[:6])
    assert errors(got[:1].astype(np.float64), d.logits()[None].astype(np.float64)).max() < 1e-2  # 6 and 37 tokens: different product kernels
    with pytest.raises(lb.LithosError):
        M.Model.open_synthetic(ctx, cfg, 64, "float32", 7)
    m.close()
    d.close()
