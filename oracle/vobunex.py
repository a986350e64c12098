"""Plain numpy statement of the Vobunex decoder -- TEST INFRASTRUCTURE, slow on purpose, float64 throughout.

One function per mechanism, every one written from its equation and none of them sharing code with the library:
tests compare the kernels, the caches, the states and the step function with these.  Sequences are [tokens, features] arrays.
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


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


# ---- embedding -----------------------------------------------------------------------------------------
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """row of the bigram table for every token: a hash of (previous, current); a sequence's first token has a row of its own"""
    t = np.asarray(tokens, np.int64)
    rows = np.full(len(t), buckets, np.int64)
    rows[1:] = (t[:-1] * mul_prev + t[1:] * mul_cur) % buckets
    return rows


# ---- rotations ---------------------------------------------------------------------------------------
def yarn(dims, base, scaling):
    """(frequencies, factor of cos and sin): fast pairs keep their frequency, slow ones are slowed down by `factor`, a ramp between"""
    n = dims // 2
    f = np.array([base ** (-2.0 * i / dims) for i in range(n)])
    if not scaling:
        return f, 1.0
    s = scaling

    def turning(t):  # the (fractional) pair that makes t turns over the original length
        return dims * np.log(s["original"] / (2 * np.pi * t)) / (2 * np.log(base))

    lo = max(np.floor(turning(s["fast"])), 0)
    hi = min(np.ceil(turning(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(n) - lo) / max(hi - lo, 0.001), 0, 1)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(s["factor"]) + 1.0


def rotate_pairs(x, pos, freq, mul):
    """neighbouring features turn by pos * freq, scaled by mul; x [T, heads, 2 len(freq)]"""
    ang = np.asarray(pos, np.float64)[:, None] * freq[None, :]
    c, s = (np.cos(ang) * mul)[:, None, :], (np.sin(ang) * mul)[:, None, :]
    y = np.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    y[..., 0::2] = u * c - v * s
    y[..., 1::2] = v * c + u * s
    return y


# ---- latent attention --------------------------------------------------------------------------------------
def softmax_with_sink(s, mask, sink):
    """weights exp(s) / (exp(sink) + sum exp(s)) over the unmasked entries of the last axis"""
    s = np.where(mask, s, -np.inf)
    top = np.maximum(np.max(s, axis=-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (np.exp(sink - top) + e.sum(-1, keepdims=True))


def causal_mask(n):
    return np.tril(np.ones((n, n), bool))


def latent_cache(h, p, c, eps):
    """what a layer caches: the normed latent [T, kv_rank] and the rotated shared key part [T, rot_dim]"""
    z = h @ p["dkv"].T
    freq, mul = yarn(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
    lat = rms(z[:, :c["kv_rank"]], eps) * p["dkv.norm"]
    rot = rotate_pairs(z[:, None, c["kv_rank"]:], np.arange(len(h)), freq, mul)[:, 0]
    return lat, rot


def latent_attention(h, p, c, eps):
    n, H, D, R, V = len(h), c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    lat, kr = latent_cache(h, p, c, eps)
    q = ((rms(h @ p["dq"].T, eps) * p["dq.norm"]) @ p["uq"].T).reshape(n, H, D + R)
    freq, mul = yarn(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
    qr = rotate_pairs(q[..., D:], np.arange(n), freq, mul)
    k = (lat @ p["uk"].T).reshape(n, H, D)
    v = (lat @ p["uv"].T).reshape(n, H, V)
    mask = causal_mask(n)
    out = np.empty((n, H, V))
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + qr[:, a] @ kr.T) * c["scale"]
        out[:, a] = softmax_with_sink(s, mask, p["sink"][a]) @ v[:, a]
    return out.reshape(n, -1) @ p["o"].T


# ---- state-space mixer -------------------------------------------------------------------------------------
def causal_conv(u, w, b):
    """u [T, channels], w [channels, taps], last column = the current token"""
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(pad[j:j + len(u)] * w[:, j] for j in range(taps)) + b


def ssm_scan(x, B, C, dt, A_log, D, state=None):
    """S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x per head; x [T, H, V], B, C [T, G, N], dt [T, H]"""
    n, H, V = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, V)) if state is None else state.astype(np.float64).copy()
    y = np.empty_like(x)
    g = np.arange(H) // (H // G)
    for t in range(n):
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t, g][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, C[t, g]) + D[:, None] * x[t]
    return y, S


def mamba2(h, p, c, eps, state=None):
    n, H, V, N, G = len(h), c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * V
    u = h @ p["in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, p["conv"], p["conv.b"]))
    x = xbc[:, :inner].reshape(n, H, V)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    y, S = ssm_scan(x, B, C, softplus(dt + p["dt_bias"]), p["A_log"], p["D"], state)
    y = (y.reshape(n, inner) * silu(z)).reshape(n, c["norm_groups"], -1)
    return (rms(y, eps).reshape(n, inner) * p["norm"]) @ p["o"].T, S


# ---- feed-forward ----------------------------------------------------------------------------------------------
def squared_relu(h, p):
    return np.maximum(h @ p["up"].T, 0.0) ** 2 @ p["down"].T


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def table_experts(h, tokens, p, f):
    """experts by token id; equal weights"""
    table, top = p["table"].astype(np.int64), f["router"]["top"]
    y = np.zeros_like(h)
    picks = table[np.asarray(tokens)]
    for e in np.unique(picks):
        t = np.nonzero((picks == e).any(-1))[0]
        y[t] += clamped_expert(h[t], p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"], f["expert"]["limit"]) / top
    return y


# ---- the model ---------------------------------------------------------------------------------------------
class Vobunex:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.w = {k: np.asarray(t, np.float64) for k, t in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: t for k, t in self.w.items() if k.startswith(prefix)}

    def _norm(self, x, name):
        return layer_norm(x, self.w[name], self.w[name + ".b"], self.cfg["norm"]["eps"])

    def embed(self, tokens):
        x = self.w["embed"][np.asarray(tokens)]
        bg = (self.cfg.get("embedding") or {}).get("bigram")
        return x + self.w["bigram"][bigram_rows(tokens, bg["buckets"], bg["mul_prev"], bg["mul_cur"])] if bg else x

    def run(self, tokens, keep=None):
        """logits [T, vocab]; keep (a list) receives the residual stream after every layer"""
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = self.embed(tokens)
        for i, layer in enumerate(cfg["layers"]):
            c, p = layer["mixer"], self._sub(f"l{i}.mix.")
            h = self._norm(x, f"l{i}.norm1")
            x = x + (latent_attention(h, p, c, eps) if layer["type"] == "latent_attention" else mamba2(h, p, c, eps)[0])
            f = layer["mlp"]
            if f is not None:
                h, p = self._norm(x, f"l{i}.norm2"), self._sub(f"l{i}.mlp.")
                x = x + (squared_relu(h, p) if f["kind"] == "dense" else table_experts(h, tokens, p, f))
            if keep is not None:
                keep.append(x.copy())
        return self._norm(x, "final.norm") @ self.w["head"].T
