"""Shared by the Kubedra tests: small configurations that differ from one another in every size and
option, weights at a scale where every mechanism matters, model folders in temporary places, token
sequences whose routing choices are clear, and the plain implementation's results."""
from __future__ import annotations

import functools
from pathlib import Path

import numpy as np

from helpers import tmp_root
from plain import kubedra_plain as KP
from senotar_helpers import to_bf16_values, write_folder


def _latent(heads, dim, vdim, q_rank, kv_rank, scale, window=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)
    if window is not None:
        m["mask"] = dict(size=window)
    return m


def _gla(heads, dim, vdim, tau):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(ff, experts, top, limit, shared=None):
    m = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if shared is not None:
        m["shared"] = dict(ff=shared[0], limit=shared[1])
    return m


def _layer(kind, mixer, mlp):
    return dict(type={"latent": "latent_attention", "gla": "gla"}[kind], mixer=mixer, mlp=mlp)


def _config(width, vocab, positions, eps, layers, loop=None):
    c = dict(architecture="Kubedra", width=width, vocab=vocab, max_positions=positions, norm=dict(eps=eps), layers=layers)
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


CONFIGS = {
    # gated linear attention first; a window of 20; latents of 40 (padded to 64 in 16 bits) under queries from 24;
    # the two layers in the middle three times; a layer whose latents are more than four times a head (its
    # up-projections stay products of their own); a decay rank of 5
    "s": _config(64, 211, 192, 1e-6, [
        _layer("gla", _gla(3, 20, 12, 4.0), _dense(40)),
        _layer("latent", _latent(3, 24, 16, 24, 40, 0.35, 20), _moe(24, 5, 3, 1.5, (40, 3.0))),
        _layer("gla", _gla(2, 16, 24, 16.0), None),
        _layer("latent", _latent(2, 12, 8, 40, 56, 0.5, 33), _dense(56)),
    ], (1, 3, 3)),
    # latents of 64 and 128 (the sizes the tensor-core kernels take), a window longer than a page and a layer that
    # sees everything; a key size that takes 16 lanes; a router with a single choice and no shared expert; no loop
    "t": _config(96, 300, 400, 1e-5, [
        _layer("latent", _latent(2, 48, 32, 64, 128, 0.2, 70), _moe(40, 3, 1, 2.5)),
        _layer("gla", _gla(1, 136, 40, 8.0), _dense(72)),
        _layer("latent", _latent(5, 64, 64, 32, 64, 0.15, None), None),
        _layer("gla", _gla(4, 32, 64, 1.0), _moe(56, 6, 2, 0.75, (24, 0.5))),
    ]),
    # a width that is no multiple of 8, ranks and sizes that are none either, key sizes that are no multiple of 4; a
    # window of the token itself; every expert chosen; the whole model twice; a table of positions that the longest
    # test sequence fills to its last row
    "u": _config(60, 130, 181, 1e-6, [
        _layer("latent", _latent(1, 10, 14, 12, 20, 0.6, 1), _moe(20, 4, 4, 1.0, (12, 2.0))),
        _layer("gla", _gla(3, 7, 5, 2.0), _dense(36)),
        _layer("latent", _latent(4, 8, 12, 18, 12, 0.5, 9), _moe(16, 6, 2, 4.0)),
    ], (0, 3, 2)),
}
SEEDS = {"s": 51, "t": 52, "u": 53}
DECAY_RANK = {"s": 5, "t": 16, "u": 9}


def mixer_weights(rng, kind, m, d, pre="", decay_rank=16):
    """The tensors of one mixer, name -> array, at a scale where scores, decays and gates matter."""
    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)
    W = {}
    H, D, V = m["heads"], m["dim"], m["vdim"]
    if kind == "latent_attention":
        qr, r = m["q_rank"], m["kv_rank"]
        W[pre + "dq"], W[pre + "uq"] = mat(qr, d), mat(H * D, qr)
        W[pre + "dkv"], W[pre + "uk"], W[pre + "uv"] = mat(r, d), mat(H * D, r), mat(H * V, r)
        W[pre + "dq.norm"], W[pre + "dkv.norm"] = 1 + 0.3 * rng.standard_normal(qr), 1 + 0.3 * rng.standard_normal(r)
        W[pre + "o"] = mat(d, H * V)
    elif kind == "gla":
        W[pre + "q"], W[pre + "k"], W[pre + "v"] = mat(H * D, d), mat(H * D, d), mat(H * V, d)
        W[pre + "g"], W[pre + "o"] = mat(H * V, d, 2.0), mat(d, H * V)
        W[pre + "a1"], W[pre + "a2"] = mat(decay_rank, d), mat(H * D, decay_rank, 2.0)
        W[pre + "a2.b"] = rng.standard_normal(H * D) * 2.0
        W[pre + "norm"] = 1 + 0.3 * rng.standard_normal(V)
    else:
        raise ValueError(kind)
    return W


def mlp_weights(rng, mlp, d, pre=""):
    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def glu(p, ff):
        return {p + "gate": mat(ff, d, 2.0), p + "up": mat(ff, d, 2.0), p + "down": mat(d, ff)}
    if mlp is None:
        return {}
    if mlp["kind"] == "dense":
        return glu(pre, mlp["ff"])
    E = mlp["router"]["experts"]
    W = {pre + "router": mat(E, d, 2.0), pre + "router.b": rng.standard_normal(E)}
    for e in range(E):
        W.update(glu(f"{pre}e{e}.", mlp["expert"]["ff"]))
    if mlp.get("shared"):
        W.update(glu(pre + "shared.", mlp["shared"]["ff"]))
    return W


def make_weights(cfg: dict, seed: int, decay_rank: int = 16) -> dict:
    """name -> float32 array whose values bfloat16 holds exactly."""
    rng = np.random.default_rng(seed)
    d = cfg["width"]
    W = {"embed": rng.standard_normal((cfg["vocab"], d)), "pos": rng.standard_normal((cfg["max_positions"], d)) * 0.7,
         "final.norm": 0.2 * rng.standard_normal(d)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] is not None else ()):
            W[p + n] = 0.2 * rng.standard_normal(d)
        W.update(mixer_weights(rng, layer["type"], layer["mixer"], d, p + "mix.", decay_rank))
        W.update(mlp_weights(rng, layer["mlp"], d, p + "mlp."))
    return {k: to_bf16_values(v) for k, v in W.items()}


@functools.lru_cache(maxsize=None)
def weights(name: str):
    return {k: v.astype(np.float64) for k, v in make_weights(CONFIGS[name], SEEDS[name], DECAY_RANK[name]).items()}


@functools.lru_cache(maxsize=None)
def model_folder(name: str, storage: str = "bfloat16") -> Path:
    return write_folder(tmp_root() / f"kubedra_{name}_{storage}", CONFIGS[name],
                        make_weights(CONFIGS[name], SEEDS[name], DECAY_RANK[name]), storage)


CLEAR = 0.12     # how far the last chosen logit must stand above the best one left out


@functools.lru_cache(maxsize=None)
def clear_tokens(name: str, n: int, seed: int) -> tuple:
    """``n`` random tokens, each redrawn until every routed layer run's choice at its position stands ``CLEAR`` above the
    best logit left out: a 16-bit run then makes the same choices as the plain one, and the comparison is about
    arithmetic, not about the side of a tie."""
    from threadpoolctl import threadpool_limits
    rng = np.random.default_rng(8000 + seed)
    cfg, W = CONFIGS[name], weights(name)
    model = KP.Stepper(cfg, W)
    out = []
    with threadpool_limits(1):                            # many small products: threads only get in each other's way
        for _ in range(n):
            snap = model.snapshot()
            for _ in range(300):
                tok, margins = int(rng.integers(0, cfg["vocab"])), [np.inf]

                def watch(i, h):
                    mlp = cfg["layers"][i]["mlp"]
                    if mlp["kind"] == "moe":
                        z = KP.router_logits(h, W, f"l{i}.mlp.")[0]
                        margins.append(KP.routing_margin(z, mlp["router"]["top"]))
                model.step(tok, watch)
                if min(margins) > CLEAR:
                    break
                model.restore(snap)
            else:
                raise AssertionError("no token with a clear routing choice found")
            out.append(tok)
    return tuple(out)


_plain: dict = {}


def plain_logits(name: str, tokens) -> np.ndarray:
    from threadpoolctl import threadpool_limits
    key = (name, tuple(tokens))
    if key not in _plain:
        with threadpool_limits(1):
            _plain[key] = KP.forward(CONFIGS[name], weights(name), list(tokens))
    return _plain[key]
