"""Nekotar, plainly: numpy in float64, one function per mechanism, a token at a time wherever the
design carries a state.  Shares no code with the package (own safetensors reader, own config walk).
Slow on purpose: keys and values are built from the latents for every head, attention is a loop over
queries, the recurrence a loop over tokens.

Notation: T tokens of ONE sequence from its first token, width W, H heads, key size D, value size V,
s residual streams.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np


# ---- files -------------------------------------------------------------------------------
def read_safetensors(path) -> dict:
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif info["dtype"] == "F32":
            arr = np.frombuffer(buf, dtype="<f4")
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        out[name] = arr.reshape(info["shape"]).astype(np.float64)
    return out


# ---- small functions -----------------------------------------------------------------------
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_divide(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_divide(x, eps) * w


# ---- rotations -----------------------------------------------------------------------------
def angles(n, dims, base, first=0):
    """[n, dims / 2]: position times base^(-2 i / dims)."""
    return (first + np.arange(n))[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)[None, :]


def turn(u, v, a):
    return u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)


def rotate_neighbours(x, base):
    """x [T, ..., dims]: entry 2i turns with entry 2i + 1."""
    a = angles(x.shape[0], x.shape[-1], base).reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (-1,))
    out = np.empty_like(x)
    out[..., 0::2], out[..., 1::2] = turn(x[..., 0::2], x[..., 1::2], a)
    return out


def rotate_halves(x, dims, base):
    """x [T, heads, D]: of the first ``dims`` entries, entry i turns with entry i + dims / 2."""
    a = angles(x.shape[0], dims, base)[:, None, :]
    out = x.copy()
    half = dims // 2
    out[..., :half], out[..., half:dims] = turn(x[..., :half], x[..., half:dims], a)
    return out


# ---- attention -------------------------------------------------------------------------------
def visible(i, j, window=0, keep=0):
    """May the query at position i see the key at position j?"""
    return j <= i and (window <= 0 or i - j < window or j < keep)


def attend(q, k, v, scale, window=0, keep=0):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: softmax over the visible keys."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        seen = [j for j in range(i + 1) if visible(i, j, window, keep)]
        for h in range(H):
            s = (k[seen, h // per] @ q[i, h]) * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[seen, h // per]
    return out


def windowed_attention(h, m, t, pre, eps=None):
    T, H, G, D, V = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ t[pre + "q"].T + t[pre + "q.b"]).reshape(T, H, D)
    k = (h @ t[pre + "k"].T + t[pre + "k.b"]).reshape(T, G, D)
    v = (h @ t[pre + "v"].T + t[pre + "v.b"]).reshape(T, G, V)
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q, k = rotate_halves(q, dims, base), rotate_halves(k, dims, base)
    mask = m.get("mask") or {}
    o = attend(q, k, v, float(m["scale"]), int(mask.get("size") or 0), int(mask.get("keep_first") or 0)).reshape(T, -1)
    return (o * sigmoid(h @ t[pre + "g"].T)) @ t[pre + "o"].T


# ---- latent attention ----------------------------------------------------------------------------
def latents(h, m, t, pre, eps):
    """What a token leaves behind: its normed latent and the one rotated key part all heads share."""
    d = h @ t[pre + "dkv"].T
    r = int(m["kv_rank"])
    return rms_norm(d[:, :r], t[pre + "dkv.norm"], eps), rotate_neighbours(d[:, r:], float(m["rot"]["base"]))


def latent_attention(h, m, t, pre, eps, kept=None):
    """``kept``: the latents and rotated keys of another layer (None: this layer makes its own)."""
    T, H, D, R, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    q = (h @ t[pre + "q"].T).reshape(T, H, D + R)
    qn, qr = q[:, :, :D], rotate_neighbours(q[:, :, D:], float(m["rot"]["base"]))
    c, kr = kept if kept is not None else latents(h, m, t, pre, eps)
    kn = (c @ t[pre + "uk"].T).reshape(T, H, D)
    v = (c @ t[pre + "uv"].T).reshape(T, H, V)
    k = np.concatenate([kn, np.broadcast_to(kr[:, None, :], (T, H, R))], axis=2)
    o = attend(np.concatenate([qn, qr], axis=2), k, v, float(m["scale"])).reshape(T, -1)
    return (o * sigmoid(h @ t[pre + "g"].T)) @ t[pre + "o"].T


# ---- time mixing with a decayed matrix state --------------------------------------------------------
def shifted(h, mu, before=None):
    """Every row mixed with the row in front of it (zeros in front of the first, or ``before``)."""
    prev = np.concatenate([np.zeros((1, h.shape[1])) if before is None else before[None], h[:-1]])
    return h + (prev - h) * mu


def key_decays(mixed, t, pre):
    """The factor in (0, 1) of every token and key channel (heads side by side)."""
    return np.exp(-np.exp(np.tanh(mixed @ t[pre + "w1"].T) @ t[pre + "w2"].T + t[pre + "w0"]))


def recurrence(r, k, v, w, u, S=None):
    """S [D, V] per head (from zero): o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(w_t) S + k_t v_t^T."""
    T, H, D = r.shape
    S = np.zeros((H, D, v.shape[2])) if S is None else S.copy()
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        kv = k[i][:, :, None] * v[i][:, None, :]
        out[i] = np.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[i])
        S = w[i][:, :, None] * S + kv
    return out


def wkv(h, m, t, pre, eps):
    T, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    mixed = {c: shifted(h, t[pre + "mu." + c]) for c in "rkvgw"}
    r, k, v = ((mixed[c] @ t[pre + c].T).reshape(T, H, D) for c in "rkv")
    w = key_decays(mixed["w"], t, pre).reshape(T, H, D)
    o = rms_divide(recurrence(r, k, v, w, t[pre + "u"]), eps).reshape(T, -1)
    return (o * t[pre + "norm"] * silu(mixed["g"] @ t[pre + "g"].T)) @ t[pre + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------
def gelu_mlp(h, t, pre):
    return gelu_tanh(h @ t[pre + "up"].T) @ t[pre + "down"].T


# ---- several residual streams ------------------------------------------------------------------------
def read_streams(X, a):
    """X [s, T, W] -> sum over streams of a[s] X[s]."""
    return np.einsum("s,stw->tw", a, X)


def write_streams(X, y, mix, out, m):
    """All streams at once: stream t becomes sum_s mix[s, t] X[s] + m out[t] y."""
    return np.einsum("st,sij->tij", mix, X) + m * out[:, None, None] * y[None]


# ---- the model -----------------------------------------------------------------------------------------
def forward(cfg, t, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence's tokens from its first.  ``layers_out``: a list that gets the
    sum of the streams after every layer."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = rms_norm(t["embed"][np.asarray(tokens)], t["embed.norm"], eps)
    X = np.repeat(x[None], int(cfg["streams"]), axis=0)
    kept = {}

    def sublayer(X, hc, norm, f):
        y = f(rms_norm(read_streams(X, t[hc + "in"]), t[norm], eps))
        return write_streams(X, y, t[hc + "mix"], t[hc + "out"], m)

    for i, layer in enumerate(cfg["layers"]):
        pre, mix, kind = f"l{i}.", layer["mixer"], layer["type"]

        def mixer(h):
            if kind == "wkv":
                return wkv(h, mix, t, pre + "mix.", eps)
            if kind == "attention":
                return windowed_attention(h, mix, t, pre + "mix.")
            if mix.get("kv_from") is None:
                kept[i] = latents(h, mix, t, pre + "mix.", eps)
            return latent_attention(h, mix, t, pre + "mix.", eps, kept[i if mix.get("kv_from") is None else mix["kv_from"]])
        X = sublayer(X, pre + "hc1.", pre + "norm1", mixer)
        if layer.get("mlp") is not None:
            X = sublayer(X, pre + "hc2.", pre + "norm2", lambda h: gelu_mlp(h, t, pre + "mlp."))
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return rms_norm(X.sum(0), t["final.norm"], eps) @ t["head"].T


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")
