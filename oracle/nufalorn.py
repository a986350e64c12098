"""Plain numpy statement of the Nufalorn decoder -- TEST INFRASTRUCTURE, slow on purpose, float64 throughout.

One function per mechanism, every one written from its equation and none of them sharing code with the library:
tests compare the kernels, the cache and the step function with these.  Sequences are [tokens, features] arrays.
"""
from __future__ import annotations

import numpy as np


# ---- element-wise pieces ---------------------------------------------------------------------------
def sigmoid(z):
    z = np.asarray(z, np.float64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def relu_glu(h, gate, up, down):
    return (np.maximum(h @ gate.T, 0.0) * (h @ up.T)) @ down.T


# ---- rotations ---------------------------------------------------------------------------------------
def rotate_pairs(x, pos, base, dims, sign=1.0):
    """neighbouring features (2i, 2i+1) of the first `dims` turn by sign * pos * base^(-2i/dims); x [T, heads, D]"""
    y = x.copy()
    i = np.arange(dims // 2)
    ang = sign * np.asarray(pos, np.float64)[:, None] * base ** (-2.0 * i / dims)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


# ---- attention -----------------------------------------------------------------------------------------
def chunk_mask(n, size):
    """[n, n]: row i sees column j <= i inside the same block of `size` positions (size 0: one block)"""
    i = np.arange(n)
    m = i[None, :] <= i[:, None]
    if size:
        m &= (i[None, :] // size) == (i[:, None] // size)
    return m


def softmax_with_sink(s, mask):
    """weights exp(s) / (1 + sum exp(s)) over the unmasked entries of the last axis"""
    s = np.where(mask, s, -np.inf)
    top = np.maximum(np.max(s, axis=-1, keepdims=True), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum(-1, keepdims=True))


def keys_values(h, p, c, eps):
    """what an attention layer caches: rotated keys [T, G, dim], normed and rotated values [T, G, vdim]"""
    n, G = len(h), c["kv_heads"]
    pos = np.arange(n)
    k = (h @ p["k"].T).reshape(n, G, c["dim"])
    v = (h @ p["v"].T).reshape(n, G, c["vdim"])
    k = rotate_pairs(k, pos, c["rot"]["base"], c["rot"]["dims"])
    v = rotate_pairs(rms(v, eps), pos, c["rot"]["base"], c["vdim"])
    return k, v


def attention(h, p, c, k, v):
    n, H, G = len(h), c["heads"], c["kv_heads"]
    pos = np.arange(n)
    q = rotate_pairs((h @ p["q"].T).reshape(n, H, c["dim"]), pos, c["rot"]["base"], c["rot"]["dims"])
    mask = chunk_mask(n, c["mask"]["size"])
    out = np.empty((n, H, c["vdim"]))
    for a in range(H):
        g = a // (H // G)
        w = softmax_with_sink((q[:, a] @ k[:, g].T) * c["scale"], mask)
        out[:, a] = w @ v[:, g]
    out = rotate_pairs(out, pos, c["rot"]["base"], c["vdim"], sign=-1.0)
    return out.reshape(n, -1) @ p["o"].T


# ---- linear attention with one decay per key channel ------------------------------------------------------
def decay_scan(q, k, v, a, state=None):
    """S <- diag(a) S + k v^T, o = S^T q per head; q, k, a [T, heads, dk], v [T, heads, dv]"""
    n, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[-1])) if state is None else state.astype(np.float64).copy()
    o = np.empty_like(v)
    for t in range(n):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hd,hdv->hv", q[t], S)
    return o, S


def hgrn2_inputs(h, p, c):
    n, H, dk = len(h), c["heads"], c["dim"]
    q = silu(h @ p["q"].T).reshape(n, H, dk)
    v = (h @ p["v"].T).reshape(n, H, c["vdim"])
    l = p["lower"]
    f = (l + (1.0 - l) * sigmoid(h @ p["f"].T + p["f.b"])).reshape(n, H, dk)
    return q, 1.0 - f, v, f


def gla_inputs(h, p, c):
    n, H, dk = len(h), c["heads"], c["dim"]
    q = (h @ p["q"].T).reshape(n, H, dk) / np.sqrt(dk)
    k = (h @ p["k"].T).reshape(n, H, dk)
    v = (h @ p["v"].T).reshape(n, H, c["vdim"])
    z = (h @ p["a1"].T) @ p["a2"].T + p["a2.b"]
    return q, k, v, (sigmoid(z) ** (1.0 / c["tau"])).reshape(n, H, dk)


def hgrn2(h, p, c, eps, state=None):
    o, S = decay_scan(*hgrn2_inputs(h, p, c), state)
    return (rms(o, eps) * p["norm"]).reshape(len(h), -1) @ p["o"].T, S


def gla(h, p, c, eps, state=None):
    o, S = decay_scan(*gla_inputs(h, p, c), state)
    y = (rms(o, eps) * p["norm"]).reshape(len(h), -1) * silu(h @ p["g"].T)
    return y @ p["o"].T, S


# ---- the model ---------------------------------------------------------------------------------------------
class Nufalorn:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.w = {k: np.asarray(t, np.float64) for k, t in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: t for k, t in self.w.items() if k.startswith(prefix)}

    def run(self, tokens, keep=None):
        """logits [T, vocab]; keep (a list) receives the residual stream after every layer"""
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = self.w["embed"][np.asarray(tokens)]
        kv = {}
        for i, layer in enumerate(cfg["layers"]):
            c, p = layer["mixer"], self._sub(f"l{i}.mix.")
            h = rms_norm_zero_centred(x, self.w[f"l{i}.norm1"], eps)
            if layer["type"] == "attention":
                j = c.get("kv_from", i)
                if j == i:
                    kv[i] = keys_values(h, p, c, eps)
                y = attention(h, p, c, *kv[j])
            elif layer["type"] == "hgrn2":
                y, _ = hgrn2(h, p, c, eps)
            else:
                y, _ = gla(h, p, c, eps)
            if layer["mlp"] is not None:
                f = self._sub(f"l{i}.mlp.")
                y = y + relu_glu(rms_norm_zero_centred(x, self.w[f"l{i}.norm2"], eps), f["gate"], f["up"], f["down"])
            x = x + cfg["residual_mult"] * y
            if keep is not None:
                keep.append(x.copy())
        z = rms_norm_zero_centred(x, self.w["final.norm"], eps) @ self.w["head"].T
        return soft_cap(z, cfg["logit_softcap"])
