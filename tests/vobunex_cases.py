"""Small random Vobunex models for the tests: configurations, weights (bf16-exact), model directories."""
import json
import struct

import numpy as np

from nufalorn_cases import bf16

YARN = {"factor": 8.0, "original": 256, "fast": 16.0, "slow": 2.0}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, base=5000.0, scaling=YARN, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale or (dim + rot_dim) ** -0.5, "rot": rot}, "mlp": mlp}


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, bigram=(97, 13, 7), eps=1e-5):
    c = {"architecture": "Vobunex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}
    c["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))} if bigram else None
    return c


def tensors(cfg, seed):
    """random weights: step sizes and decays spread from fast to nearly no forgetting, sinks on both sides of the scores"""
    r = np.random.default_rng(seed)
    W, w = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = bf16(r.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean, std):
        w[name] = bf16(mean + std * r.standard_normal(n))

    def norm(name):
        vec(name, W, 1.0, 0.1)
        vec(name + ".b", W, 0.0, 0.1)

    w["embed"] = bf16(r.standard_normal((cfg["vocab"], W)))
    if cfg["embedding"]:
        w["bigram"] = bf16(r.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, W)) * 0.7)
    mat("head", cfg["vocab"], W)
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, V = m["heads"], m["vdim"]
        norm(f"l{i}.norm1")
        if layer["type"] == "latent_attention":
            mat(p + "dq", m["q_rank"], W)
            vec(p + "dq.norm", m["q_rank"], 1.0, 0.2)
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + "dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(p + "uk", H * m["dim"], m["kv_rank"], 1.5)
            mat(p + "uv", H * V, m["kv_rank"])
            vec(p + "sink", H, 0.5, 1.5)
        else:
            C = H * V + 2 * m["groups"] * m["state"]
            mat(p + "in", H * V + C + H, W)
            w[p + "conv"] = bf16(r.standard_normal((C, m["conv"])) * 0.6)
            vec(p + "conv.b", C, 0.0, 0.2)
            w[p + "dt_bias"] = bf16(r.uniform(-5, 0, H))
            w[p + "A_log"] = bf16(r.uniform(-1.5, 2.0, H))
            vec(p + "D", H, 1.0, 0.3)
            vec(p + "norm", H * V, 1.0, 0.2)
        mat(p + "o", W, H * V, 1.5)
        f, p = layer["mlp"], f"l{i}.mlp."
        if f is None:
            continue
        norm(f"l{i}.norm2")
        if f["kind"] == "dense":
            mat(p + "up", f["ff"], W)
            mat(p + "down", W, f["ff"])
        else:
            F, E, top = f["expert"]["ff"], f["router"]["experts"], f["router"]["top"]
            for e in range(E):
                mat(f"{p}e{e}.gate", F, W, 1.5)
                mat(f"{p}e{e}.up", F, W, 1.5)
                mat(f"{p}e{e}.down", W, F, 2.0)
            w[p + "table"] = np.stack([r.permutation(E)[:top] for _ in range(cfg["vocab"])]).astype(np.int32)
    return w


def write(path, cfg, w):
    """a model directory: config.json and model.safetensors"""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blob = {}, b""
    for name, a in w.items():
        if a.dtype == np.int32:
            kind, raw = "I32", a.astype("<i4").tobytes()
        else:
            kind, raw = "BF16", (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    js = json.dumps(head).encode()
    js += b" " * (-len(js) % 8)
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(js)) + js + blob)
    return path


# sizes on purpose unlike one another: odd vocabularies and widths, head sizes that are no multiple of anything, key and value sizes that differ,
# state sizes of every kernel, one and several groups, every expert and one expert per token, layers without feed-forward, no pair embedding
CASES = {
    "mixed": config(72, 131, [latent(5, 20, 12, 28, 40, 72, mlp=dense(90)), mamba2(6, 20, 36, groups=3, conv=3, norm_groups=2, mlp=moe(28, 7, 3)),
                              mamba2(4, 12, 70, groups=1, conv=2, norm_groups=4, mlp=None), latent(3, 14, 24, 10, 24, 40, scaling=None, mlp=moe(40, 3, 1)),
                              mamba2(3, 40, 12, groups=3, conv=5, norm_groups=1, mlp=dense(33))]),
    "wide_heads": config(192, 200, [latent(20, 128, 64, 96, 160, 320, mlp=moe(72, 10, 2, limit=0.7)), mamba2(8, 64, 128, groups=2, conv=4, norm_groups=8, mlp=dense(200)),
                                    latent(9, 200, 100, 130, 72, 500, mlp=None)], bigram=(1000, 31, 2), eps=1e-6),
    "large_state": config(100, 97, [mamba2(2, 33, 200, groups=2, conv=8, norm_groups=3, mlp=moe(16, 4, 4)), mamba2(5, 31, 250, groups=1, conv=1, norm_groups=5, mlp=moe(90, 2, 1))], bigram=None),
    "odd_width": config(75, 64, [latent(2, 7, 2, 5, 9, 11, mlp=moe(13, 5, 2)), mamba2(3, 5, 5, mlp=dense(7)), latent(17, 16, 16, 32, 64, 128, mlp=None)], bigram=(1, 0, 0)),
}
