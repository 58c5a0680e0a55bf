"""Shared by the Nekotar tests: small configurations that differ from one another in every size and
option, weights at a scale where every mechanism matters, model folders in temporary places, and the
plain implementation's results."""
from __future__ import annotations

import functools
from pathlib import Path

import numpy as np

from helpers import tmp_root
from plain import nekotar_plain as NP
from senotar_helpers import to_bf16_values, write_folder


def latent(heads, dim, vdim, kv_rank, rot_dim, scale, base=10000.0, kv_from=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, rot_dim=rot_dim, scale=scale, rot=dict(base=base, dims=rot_dim))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def windowed(heads, kv_heads, dim, vdim, dims, scale, window=None, keep=0, base=10000.0):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dims))
    if window is not None:
        m["mask"] = dict(size=window, keep_first=keep)
    return m


def _layer(kind, mixer, ff):
    return dict(type={"latent": "latent_attention", "win": "attention", "wkv": "wkv"}[kind], mixer=mixer,
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def _config(width, vocab, streams, mult, eps, layers):
    return dict(architecture="Nekotar", width=width, vocab=vocab, streams=streams, residual_mult=mult, norm=dict(eps=eps),
                layers=layers)


CONFIGS = {
    # time mixing first and last, once with and once without a feed-forward; latents of 40 + 8; a window of 20 behind
    # which three tokens stay; another head count, key and value size on the latents of a layer three places back
    "s": _config(64, 211, 3, 0.7, 1e-6, [
        _layer("wkv", dict(heads=3, dim=20), 40),
        _layer("latent", latent(3, 24, 16, 40, 8, 0.3), None),
        _layer("win", windowed(4, 2, 24, 16, 16, 0.35, 20, 3), 72),
        _layer("wkv", dict(heads=2, dim=32), None),
        _layer("latent", latent(2, 12, 8, 40, 8, 0.45, kv_from=1), 56),
    ]),
    # one stream; rows of 128 (104 + 24) and of 64 (40 + 24), the sizes the tensor-core kernels take; as many key heads as
    # query heads; value heads larger than key heads; a window longer than a page; a key size that takes 32 lanes
    "t": _config(96, 300, 1, 1.0, 1e-5, [
        _layer("latent", latent(2, 48, 32, 104, 24, 0.2, 500.0), 72),
        _layer("win", windowed(3, 3, 64, 104, 64, 0.15, 70, 1, 1e5), None),
        _layer("wkv", dict(heads=1, dim=136), 56),
        _layer("latent", latent(5, 64, 64, 40, 24, 0.15), None),
        _layer("latent", latent(4, 16, 24, 40, 24, 0.2, kv_from=3), 40),
    ]),
    # a width that is no multiple of 8, sizes that are none either; a window of the token itself; one key head; a layer
    # that sees everything; four streams; a lender with two borrowers
    "u": _config(60, 130, 4, 0.4, 1e-6, [
        _layer("win", windowed(5, 1, 10, 14, 4, 0.6, 1, 2), 36),
        _layer("latent", latent(1, 10, 14, 20, 2, 0.6), 20),
        _layer("wkv", dict(heads=3, dim=7), 24),
        _layer("latent", latent(4, 8, 12, 20, 2, 0.5, kv_from=1), None),
        _layer("win", windowed(6, 3, 12, 10, 12, 0.4), None),
        _layer("latent", latent(2, 6, 5, 20, 2, 0.5, kv_from=1), 28),
    ]),
}
SEEDS = {"s": 61, "t": 62, "u": 63}
DECAY_RANK = {"s": 5, "t": 16, "u": 9}


def mixer_weights(rng, kind, m, d, pre="", decay_rank=16):
    """The tensors of one mixer, name -> array, at a scale where scores, decays and gates matter."""
    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)
    W = {}
    H, D = m["heads"], m["dim"]
    if kind == "latent_attention":
        V, r, rot = m["vdim"], m["kv_rank"], m["rot_dim"]
        W[pre + "q"] = mat(H * (D + rot), d)
        if m.get("kv_from") is None:
            W[pre + "dkv"], W[pre + "dkv.norm"] = mat(r + rot, d), 1 + 0.3 * rng.standard_normal(r)
        W[pre + "uk"], W[pre + "uv"] = mat(H * D, r), mat(H * V, r)
        W[pre + "g"], W[pre + "o"] = mat(H * V, d, 2.0), mat(d, H * V, 1.5)
    elif kind == "attention":
        V, G = m["vdim"], m["kv_heads"]
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
            W[pre + n], W[pre + n + ".b"] = mat(rows, d), 0.5 * rng.standard_normal(rows)
        W[pre + "g"], W[pre + "o"] = mat(H * V, d, 2.0), mat(d, H * V, 1.5)
    elif kind == "wkv":
        n = H * D
        for c in "rkvgw":
            W[pre + "mu." + c] = rng.random(d) * 1.4 - 0.2
        for c in "rkv":
            W[pre + c] = mat(n, d)
        W[pre + "g"], W[pre + "o"] = mat(n, d, 2.0), mat(d, n, 1.5)
        W[pre + "w1"], W[pre + "w2"] = mat(decay_rank, d, 1.5), mat(n, decay_rank, 2.0)
        W[pre + "w0"] = rng.standard_normal(n) * 1.5 - 2.0
        W[pre + "u"], W[pre + "norm"] = rng.standard_normal((H, D)) * 1.5, 1 + 0.3 * rng.standard_normal(n)
    else:
        raise ValueError(kind)
    return W


def mlp_weights(rng, ff, d, pre=""):
    return {pre + "up": rng.standard_normal((ff, d)) * 2.0 / np.sqrt(d), pre + "down": rng.standard_normal((d, ff)) * 1.5 / np.sqrt(ff)}


def make_weights(cfg: dict, seed: int, decay_rank: int = 16) -> dict:
    """name -> float32 array whose values bfloat16 holds exactly."""
    rng = np.random.default_rng(seed)
    d, s = cfg["width"], cfg["streams"]
    W = {"embed": rng.standard_normal((cfg["vocab"], d)) * 3.0, "embed.norm": 1 + 0.3 * rng.standard_normal(d),
         "final.norm": 1 + 0.3 * rng.standard_normal(d), "head": rng.standard_normal((cfg["vocab"], d)) / np.sqrt(d)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        for q in (1, 2) if layer["mlp"] is not None else (1,):
            W[f"{p}norm{q}"] = 1 + 0.3 * rng.standard_normal(d)
            W[f"{p}hc{q}.in"] = (1 + 0.5 * rng.standard_normal(s)) / s
            W[f"{p}hc{q}.out"] = 1 + 0.5 * rng.standard_normal(s)
            W[f"{p}hc{q}.mix"] = np.eye(s) + 0.25 * rng.standard_normal((s, s))
        W.update(mixer_weights(rng, layer["type"], layer["mixer"], d, p + "mix.", decay_rank))
        if layer["mlp"] is not None:
            W.update(mlp_weights(rng, layer["mlp"]["ff"], d, p + "mlp."))
    return {k: to_bf16_values(v) for k, v in W.items()}


@functools.lru_cache(maxsize=None)
def weights(name: str):
    return {k: v.astype(np.float64) for k, v in make_weights(CONFIGS[name], SEEDS[name], DECAY_RANK[name]).items()}


@functools.lru_cache(maxsize=None)
def model_folder(name: str, storage: str = "bfloat16") -> Path:
    return write_folder(tmp_root() / f"nekotar_{name}_{storage}", CONFIGS[name],
                        make_weights(CONFIGS[name], SEEDS[name], DECAY_RANK[name]), storage)


def random_tokens(name: str, n: int, seed: int) -> list:
    return np.random.default_rng(9000 + seed).integers(0, CONFIGS[name]["vocab"], n).tolist()


_plain: dict = {}


def plain_logits(name: str, tokens) -> np.ndarray:
    from threadpoolctl import threadpool_limits
    key = (name, tuple(tokens))
    if key not in _plain:
        with threadpool_limits(1):                        # many small products: threads only get in each other's way
            _plain[key] = NP.forward(CONFIGS[name], weights(name), list(tokens))
    return _plain[key]
