"""Kubedra, plainly: numpy in float64, one function per mechanism, a token at a time wherever the
design carries a state.  Shares no code with the package (own safetensors reader, own config walk).
Slow on purpose: keys and values are built from the latents for every head, attention is a loop over
queries, the recurrence a loop over tokens.

Notation: T tokens of ONE sequence from its first token, width W, H heads, key size D, value size V.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np

SLOPE = 1.702             # slope of the sigmoid in the capped expert's gate


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


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms_divide(x, eps) * (1.0 + w)


# ---- embedding ---------------------------------------------------------------------------------
def embed(t, tokens, first=0):
    """The token's row plus the position's row."""
    tokens = np.asarray(tokens)
    return t["embed"][tokens] + t["pos"][first + np.arange(len(tokens))]


# ---- latent attention ----------------------------------------------------------------------------
def visible(i, j, window=0):
    """May the query at position i see the key at position j?"""
    return j <= i and (window <= 0 or i - j < window)


def attend(q, k, v, scale, window=0):
    """q [T, H, D], k [T, H, D], v [T, H, V] -> [T, H, V]: softmax over the visible keys."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = 0 if window <= 0 else max(0, i - window + 1)
        for h in range(H):
            s = (k[lo:i + 1, h] @ q[i, h]) * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, h]
    return out


def latents(h, t, pre, eps):
    """What a cache would hold: the normed down-projection, one row per token."""
    return rms_divide(h @ t[pre + "dkv"].T, eps) * t[pre + "dkv.norm"]


def latent_attention(h, m, t, pre, eps):
    T, H = h.shape[0], int(m["heads"])
    cq = rms_divide(h @ t[pre + "dq"].T, eps) * t[pre + "dq.norm"]
    q = (cq @ t[pre + "uq"].T).reshape(T, H, int(m["dim"]))
    c = latents(h, t, pre, eps)
    k = (c @ t[pre + "uk"].T).reshape(T, H, int(m["dim"]))
    v = (c @ t[pre + "uv"].T).reshape(T, H, int(m["vdim"]))
    window = int((m.get("mask") or {}).get("size") or 0)
    o = attend(q, k, v, float(m["scale"]), window)
    return o.reshape(T, -1) @ t[pre + "o"].T


# ---- gated linear attention ----------------------------------------------------------------------
def key_decays(h, m, t, pre):
    """The factor in (0, 1) of every token, head and key channel."""
    z = (h @ t[pre + "a1"].T) @ t[pre + "a2"].T + t[pre + "a2.b"]
    # sigmoid(z)^(1/tau) through its logarithm: log sigmoid(z) = -log(1 + exp(-z))
    return np.exp(-np.logaddexp(0.0, -z) / float(m["tau"])).reshape(h.shape[0], int(m["heads"]), int(m["dim"]))


def recurrence(q, k, v, alpha):
    """S [D, V] per head from zero: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, D = q.shape
    V = v.shape[2]
    S = np.zeros((H, D, V))
    out = np.zeros((T, H, V))
    for i in range(T):
        S = alpha[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = np.einsum("hdv,hd->hv", S, q[i])
    return out


def gla(h, m, t, pre, eps):
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ t[pre + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ t[pre + "k"].T).reshape(T, H, D)
    v = (h @ t[pre + "v"].T).reshape(T, H, V)
    o = recurrence(q, k, v, key_decays(h, m, t, pre))
    o = rms_divide(o, eps) * t[pre + "norm"]
    return (o.reshape(T, -1) * silu(h @ t[pre + "g"].T)) @ t[pre + "o"].T


# ---- feed-forwards ------------------------------------------------------------------------------
def gelu_ff(h, t, pre):
    return (gelu_tanh(h @ t[pre + "gate"].T) * (h @ t[pre + "up"].T)) @ t[pre + "down"].T


def capped_ff(h, t, pre, limit):
    g = np.minimum(h @ t[pre + "gate"].T, limit)
    u = np.clip(h @ t[pre + "up"].T, -limit, limit)
    return (g * sigmoid(SLOPE * g) * (u + 1.0)) @ t[pre + "down"].T


def route(z, top):
    """Router logits [E] of one token -> (the experts with the largest ones, softmax over just those)."""
    chosen = np.argsort(-z, kind="stable")[:top]
    e = np.exp(z[chosen] - z[chosen].max())
    return chosen, e / e.sum()


def router_logits(h, t, pre):
    return h @ t[pre + "router"].T + t[pre + "router.b"]


def routed_ff(h, mlp, t, pre):
    out = np.zeros_like(h)
    z = router_logits(h, t, pre)
    for i in range(h.shape[0]):
        for e, w in zip(*route(z[i], int(mlp["router"]["top"]))):
            out[i] += w * capped_ff(h[i:i + 1], t, f"{pre}e{e}.", float(mlp["expert"]["limit"]))[0]
    if mlp.get("shared") is not None:
        out += capped_ff(h, t, pre + "shared.", float(mlp["shared"]["limit"]))
    return out


def feed_forward(h, mlp, t, pre):
    if mlp["kind"] == "dense":
        return gelu_ff(h, t, pre)
    if mlp["kind"] == "moe":
        return routed_ff(h, mlp, t, pre)
    raise ValueError(mlp["kind"])


# ---- the model --------------------------------------------------------------------------------------
def layer_runs(cfg):
    """[(layer, whether the embedding output is added right before it)] in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    out = [(i, False) for i in range(start)]
    for turn in range(times):
        out += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return out + [(i, False) for i in range(stop, n)]


MIXERS = {"latent_attention": latent_attention, "gla": gla}


def forward(cfg, t, tokens, layers_out=None, watch=None):
    """Logits [T, vocab] of one sequence's tokens from its first.  ``layers_out``: a list that gets the
    stream after every layer run.  ``watch(i, h)``: called with the rows that layer i's feed-forward reads."""
    eps = float(cfg["norm"]["eps"])
    start = embed(t, tokens)
    x = start.copy()
    for i, again in layer_runs(cfg):
        layer, pre = cfg["layers"][i], f"l{i}."
        if again:
            x = x + start
        h = centred_norm(x, t[pre + "norm1"], eps)
        y = MIXERS[layer["type"]](h, layer["mixer"], t, pre + "mix.", eps)
        x = x + centred_norm(y, t[pre + "norm1b"], eps)
        if layer.get("mlp") is not None:
            h = centred_norm(x, t[pre + "norm2"], eps)
            if watch is not None:
                watch(i, h)
            x = x + centred_norm(feed_forward(h, layer["mlp"], t, pre + "mlp."), t[pre + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return centred_norm(x, t["final.norm"], eps) @ t["embed"].T


def routing_margin(z, top):
    """How far one token's last chosen logit stands above the best one left out (inf: nothing is left out)."""
    ranked = -np.sort(-z)
    return ranked[top - 1] - ranked[top] if top < len(ranked) else np.inf


class Stepper:
    """The same model a token at a time: what every layer run keeps of the tokens before is a list of latents or a
    state.  ``step(token)`` gives the token's logits; a snapshot can be returned to."""

    def __init__(self, cfg, t):
        self.cfg, self.t, self.n = cfg, t, 0
        self.runs = layer_runs(cfg)
        self.kept = [[] if cfg["layers"][i]["type"] == "latent_attention" else None for i, _ in self.runs]

    def snapshot(self):
        return self.n, [list(k) if isinstance(k, list) else k for k in self.kept]

    def restore(self, snap):
        self.n, self.kept = snap[0], [list(k) if isinstance(k, list) else k for k in snap[1]]

    def _latent(self, r, h, m, pre):
        t, eps, H = self.t, float(self.cfg["norm"]["eps"]), int(m["heads"])
        q = ((rms_divide(h @ t[pre + "dq"].T, eps) * t[pre + "dq.norm"]) @ t[pre + "uq"].T).reshape(H, -1)
        self.kept[r].append(latents(h, t, pre, eps)[0])
        window = int((m.get("mask") or {}).get("size") or 0)
        c = np.array(self.kept[r][-window:] if window else self.kept[r])
        k = (c @ t[pre + "uk"].T).reshape(len(c), H, -1)
        v = (c @ t[pre + "uv"].T).reshape(len(c), H, -1)
        s = np.einsum("nhd,hd->hn", k, q) * float(m["scale"])
        e = np.exp(s - s.max(axis=1, keepdims=True))
        o = np.einsum("hn,nhv->hv", e / e.sum(axis=1, keepdims=True), v)
        return o.reshape(1, -1) @ t[pre + "o"].T

    def _gla(self, r, h, m, pre):
        t, eps = self.t, float(self.cfg["norm"]["eps"])
        H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        S = self.kept[r] if self.kept[r] is not None else np.zeros((H, D, V))
        k, v = (h @ t[pre + "k"].T).reshape(H, D), (h @ t[pre + "v"].T).reshape(H, V)
        S = key_decays(h, m, t, pre)[0][:, :, None] * S + k[:, :, None] * v[:, None, :]
        self.kept[r] = S
        o = np.einsum("hdv,hd->hv", S, (h @ t[pre + "q"].T).reshape(H, D) * D ** -0.5)
        o = rms_divide(o, eps) * t[pre + "norm"]
        return (o.reshape(1, -1) * silu(h @ t[pre + "g"].T)) @ t[pre + "o"].T

    def step(self, token, watch=None):
        cfg, t, eps = self.cfg, self.t, float(self.cfg["norm"]["eps"])
        start = embed(t, [token], self.n)
        x = start.copy()
        for r, (i, again) in enumerate(self.runs):
            layer, pre = cfg["layers"][i], f"l{i}."
            if again:
                x = x + start
            h = centred_norm(x, t[pre + "norm1"], eps)
            one = self._latent if layer["type"] == "latent_attention" else self._gla
            x = x + centred_norm(one(r, h, layer["mixer"], pre + "mix."), t[pre + "norm1b"], eps)
            if layer.get("mlp") is not None:
                h = centred_norm(x, t[pre + "norm2"], eps)
                if watch is not None:
                    watch(i, h)
                x = x + centred_norm(feed_forward(h, layer["mlp"], t, pre + "mlp."), t[pre + "norm2b"], eps)
        self.n += 1
        return (centred_norm(x, t["final.norm"], eps) @ t["embed"].T)[0]


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")
