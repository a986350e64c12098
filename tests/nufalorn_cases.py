"""Small random Nufalorn models for the tests: configurations, weights (bf16-exact), model directories."""
import json
import struct

import numpy as np


def bf16(a):
    """float32 values a bf16 holds"""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint32) << 16).view(np.float32)


def att(heads, kv_heads, dim, vdim, block, rot_dims=None, base=1000.0, scale=None, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": block}, "scale": scale or dim ** -0.5,
         "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def gla(heads, dim, vdim, tau=8.0, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(width, vocab, layers, residual_mult=0.7, cap=20.0, eps=1e-5):
    return {"architecture": "Nufalorn", "width": width, "vocab": vocab, "layers": layers, "residual_mult": residual_mult, "logit_softcap": cap,
            "norm": {"eps": eps}}


def tensors(cfg, seed, rank=5):
    """random weights: gates spread from fast to nearly no forgetting, lower bounds from 0 to 0.9"""
    r = np.random.default_rng(seed)
    W, w = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = bf16(r.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean, std):
        w[name] = bf16(mean + std * r.standard_normal(n))

    w["embed"] = bf16(r.standard_normal((cfg["vocab"], W)))
    mat("head", cfg["vocab"], W, 3.0)
    vec("final.norm", W, 0.0, 0.1)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        vec(f"l{i}.norm1", W, 0.0, 0.1)
        mat(p + "q", H * dk, W, 1.5)
        if layer["type"] == "attention":
            if "kv_from" not in m:
                mat(p + "k", m["kv_heads"] * dk, W, 1.5)
                mat(p + "v", m["kv_heads"] * dv, W)
        elif layer["type"] == "hgrn2":
            mat(p + "f", H * dk, W)
            w[p + "f.b"] = bf16(r.uniform(-1, 7, H * dk))
            w[p + "lower"] = bf16(r.uniform(0, 0.9, H * dk) * (r.random(H * dk) > 0.3))
            mat(p + "v", H * dv, W)
            vec(p + "norm", dv, 1.0, 0.2)
        else:
            mat(p + "k", H * dk, W)
            mat(p + "v", H * dv, W)
            mat(p + "g", H * dv, W)
            mat(p + "a1", rank, W)
            mat(p + "a2", H * dk, rank)
            w[p + "a2.b"] = bf16(r.uniform(-2, 4, H * dk))
            vec(p + "norm", dv, 1.0, 0.2)
        mat(p + "o", W, H * dv, 1.5)
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            vec(f"l{i}.norm2", W, 0.0, 0.1)
            mat(f"l{i}.mlp.gate", F, W)
            mat(f"l{i}.mlp.up", F, W)
            mat(f"l{i}.mlp.down", W, F)
    return w


def write(path, cfg, w):
    """a model directory: config.json and model.safetensors"""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blob = {}, b""
    for name, a in w.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    js = json.dumps(head).encode()
    js += b" " * (-len(js) % 8)
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(js)) + js + blob)
    return path


# sizes on purpose unlike one another: odd vocabularies and widths, head sizes that are no multiple of anything, every ratio of query to
# KV heads the kernels treat differently, rotated parts of a head, layers without feed-forward, shared caches with a block of their own
CASES = {
    "mixed": config(72, 131, [att(6, 2, 24, 20, 37, rot_dims=16, ff=90), hgrn2(3, 20, 36, ff=45), gla(5, 12, 28, ff=64),
                              att(6, 2, 24, 20, 19, rot_dims=16, kv_from=0), gla(2, 30, 16, tau=3.0), hgrn2(2, 44, 10, ff=33)]),
    "wide_heads": config(192, 200, [att(8, 1, 160, 192, 50, ff=100), hgrn2(2, 200, 72), gla(2, 128, 128, ff=128), att(8, 1, 160, 192, 50, kv_from=0, ff=20)],
                         residual_mult=1.0),
    "many_groups": config(80, 97, [att(12, 1, 32, 64, 64, ff=32), att(3, 3, 18, 14, 23, rot_dims=4, ff=32), gla(1, 65, 33), hgrn2(4, 16, 64, ff=70)], cap=8.0),
    "one_block": config(64, 64, [hgrn2(1, 8, 8, ff=16), att(2, 1, 16, 16, 100000, ff=16), gla(1, 8, 8, tau=1.0, ff=16)], residual_mult=0.25, eps=1e-6),
}
