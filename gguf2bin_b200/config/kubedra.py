"""Kubedra: the configuration read from ``config.json`` and its translation into a ``ModelSpec``.

The design: a token embedding plus a learned vector per position; layers of the ``sandwich_norm`` arrangement (an RMS
norm on either side of each sublayer, the weights stored around zero); two kinds of mixer, chosen per layer; a dense or
a routed feed-forward, or none; a run of layers that may be repeated with the same weights; a final norm and a head tied
to the embedding.

* ``latent_attention``: queries from a normed latent of ``q_rank`` numbers, keys and values from a normed latent of
  ``kv_rank`` numbers that is all a token leaves behind; no positions; the last ``mask.size`` tokens are seen.
* ``gla``: gated linear attention, a decay per head and key channel from a low-rank product whose rank is the
  checkpoint's.
* ``dense`` feed-forward: ``swiglu`` with the tanh form of GELU.
* ``moe`` feed-forward: ``routed_experts`` with the capped gate (``expert.limit``), a bias in the router's logits,
  weights that are the softmax over the chosen logits, and an optional shared expert of the same form with an ``ff`` and
  ``limit`` of its own.
* ``loop``: layers ``start`` .. ``stop`` - 1 run ``times`` times in a row, every pass with storage of its own and, from
  the second on, with the embedding's output added to the stream in front of it.

config.json: ``width``, ``vocab``, ``max_positions``, ``norm.eps`` and a list ``layers`` whose entries give ``type``,
``mixer`` and ``mlp``.  Every size and constant comes from there (or from a tensor's shape); ``loop``, ``mask``, ``mlp`` and
``mlp.shared`` may be absent or null (every layer once, every key, no feed-forward, no shared expert); a type or kind this
reader does not know is refused, never skipped.
"""
from __future__ import annotations

from typing import Any, Mapping

from .senotar import _float, _get, _int
from .specs import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Kubedra"
GLU_SLOPE = 1.702                # slope of the sigmoid in the experts' gate


def _positive(d, path: str, where: str) -> float:
    v = _float(d, path)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.{path} must be positive")
    return v


def _latent_attention(m, where: str, eps: float) -> PartSpec:
    mask = m.get("mask")
    return PartSpec.make(
        "latent_attention", n_heads=_int(m, "heads"), qk_dim=_int(m, "dim"), v_dim=_int(m, "vdim"),
        kv_rank=_int(m, "kv_rank"), q_rank=_int(m, "q_rank"), scale=_float(m, "scale"), eps=eps,
        window=_int(mask, "size") if mask is not None else 0, pad_rank=True,
        names=(("q_down", "mix.dq"), ("q_down_norm", "mix.dq.norm"), ("q", "mix.uq"), ("down", "mix.dkv"),
               ("down_norm", "mix.dkv.norm"), ("up_k", "mix.uk"), ("up_v", "mix.uv"), ("o", "mix.o")))


def _gla(m, where: str, eps: float) -> PartSpec:
    return PartSpec.make(
        "gla", n_heads=_int(m, "heads"), qk_dim=_int(m, "dim"), v_dim=_int(m, "vdim"),
        tau=_positive(m, "tau", where + ".mixer"), eps=eps,
        names=(("q", "mix.q"), ("k", "mix.k"), ("v", "mix.v"), ("gate", "mix.g"), ("o", "mix.o"), ("norm", "mix.norm"),
               ("a1", "mix.a1"), ("a2", "mix.a2"), ("a_bias", "mix.a2.b")))


_MIXERS = {"latent_attention": _latent_attention, "gla": _gla}


def _mixer(kind, m, where: str, eps: float) -> PartSpec:
    if kind not in _MIXERS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of {ARCHITECTURE} "
                          f"(known: {', '.join(repr(k) for k in _MIXERS)})")
    if not isinstance(m, Mapping):
        raise ConfigError(f"config.json: {where}.mixer must be an object")
    return _MIXERS[kind](m, where, eps)


def _glu(pre: str, ff: int, **more) -> PartSpec:
    return PartSpec.make("swiglu", intermediate_size=ff,
                         names=(("gate", pre + "gate"), ("up", pre + "up"), ("down", pre + "down")), **more)


def _feed_forward(mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind == "dense":
        return _glu("mlp.", _int(mlp, "ff"), activation="gelu_tanh")
    if kind == "moe":
        experts, top = _int(mlp, "router.experts"), _int(mlp, "router.top")
        if top > experts:
            raise ConfigError(f"config.json: {where}.mlp.router: {top} choices among {experts} experts")
        shared = mlp.get("shared")
        return PartSpec.make(
            "routed_experts", n_experts=experts, n_identity=0, top=top, intermediate_size=_int(mlp, "expert.ff"),
            limit=_positive(mlp, "expert.limit", where + ".mlp"), alpha=GLU_SLOPE, router_bias=True, correction=False,
            renormalise=True,
            shared=None if shared is None else _glu(
                "mlp.shared.", _int(shared, "ff"), limit=_positive(shared, "limit", where + ".mlp.shared"), alpha=GLU_SLOPE),
            names=(("router", "mlp.router"), ("router_bias", "mlp.router.b"), ("gate", "mlp.e{}.gate"),
                   ("up", "mlp.e{}.up"), ("down", "mlp.e{}.down")))
    raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is not a feed-forward of {ARCHITECTURE} "
                      "(known: 'dense', 'moe', or null for none)")


def _schedule(loop, n: int) -> tuple:
    """The layers in the order they run; the first entry of every further pass adds the embedding's output."""
    if loop is None:
        return tuple(ScheduleEntry(i) for i in range(n))
    start, stop, times = _int(loop, "start", 0), _int(loop, "stop"), _int(loop, "times")
    if not start < stop <= n:
        raise ConfigError(f"config.json: loop runs layers {start} to {stop} (exclusive) of {n}")
    out = [ScheduleEntry(i) for i in range(start)]
    for turn in range(times):
        out += [ScheduleEntry(i, add_embedding=turn > 0 and i == start) for i in range(start, stop)]
    return tuple(out + [ScheduleEntry(i) for i in range(stop, n)])


def kubedra_model_spec(d: Mapping[str, Any]) -> ModelSpec:
    width, vocab, positions = _int(d, "width"), _int(d, "vocab"), _int(d, "max_positions")
    eps = _float(d, "norm.eps")
    if not eps > 0:
        raise ConfigError("config.json: 'norm.eps' must be positive")
    norm = PartSpec.make("rmsnorm", eps=eps, offset=1.0)         # weights are stored around zero
    layers_in = _get(d, "layers")
    if not isinstance(layers_in, (list, tuple)) or not layers_in:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    block = PartSpec.make("sandwich_norm", names=(("mixer_norm", "norm1"), ("mixer_out_norm", "norm1b"),
                                                  ("ffn_norm", "norm2"), ("ffn_out_norm", "norm2b")))
    layers = []
    for i, entry in enumerate(layers_in):
        where = f"layers[{i}]"
        if not isinstance(entry, Mapping):
            raise ConfigError(f"config.json: {where} must be an object")
        layers.append(LayerSpec(block=block, mixer=_mixer(entry.get("type"), entry.get("mixer"), where, eps),
                                feed_forward=_feed_forward(entry.get("mlp"), where), norm=norm, prefix=f"l{i}."))
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab, max_positions=positions,
        layers=tuple(layers), schedule=_schedule(d.get("loop"), len(layers)),
        embedding=PartSpec.make("token_embedding", name="embed", positions="pos", n_positions=positions),
        final_norm=PartSpec.make("rmsnorm", eps=eps, offset=1.0, name="final.norm"),
        head=PartSpec.make("lm_head", tied=True, name="head"), stop_token_ids=(), source=dict(d))
    spec.validate()
    return spec
