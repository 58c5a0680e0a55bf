"""Nekotar: the configuration read from ``config.json`` and its translation into a ``ModelSpec``.

The design: a token embedding divided by its root mean square, times a weight; ``streams`` residual streams that all
start as that row; layers of the ``hyper_prenorm`` arrangement, whose sublayers read a weighted sum of the streams and
whose results, times ``residual_mult``, join a mix of them; three kinds of mixer, chosen per layer; a feed-forward of two
matrices around the tanh form of GELU, or none; the streams' sum, a final norm and a head of its own.

* ``wkv``: time mixing with a matrix state per head, a decay per key channel and a bonus for the token's own key; the
  decay's rank is the checkpoint's.
* ``latent_attention``: attention over normed latents of ``kv_rank`` numbers and one rotated key part of ``rot_dim``
  (neighbouring pairs) that all heads share; a gate for every element of the heads; with ``kv_from`` a layer reads the
  rows of an earlier such layer instead of making its own.
* ``attention``: grouped queries with biases, rotation of halves, a window (``mask.size``) behind which the first
  ``mask.keep_first`` positions stay visible, the same gate.

config.json: ``width``, ``vocab``, ``streams``, ``residual_mult``, ``norm.eps`` and a list ``layers`` whose entries give
``type``, ``mixer`` and ``mlp``.  Every size and constant comes from there (or from a tensor's shape); ``mlp`` may be null
(no feed-forward), ``mask`` absent or null (every key); a type or kind this reader does not know is refused, never
skipped.
"""
from __future__ import annotations

from typing import Any, Mapping

from .kubedra import _positive
from .senotar import _float, _get, _int
from .specs import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Nekotar"
MAX_POSITIONS = 1 << 30          # no table of positions, so no limit of its own


def _rotation(m, where: str, kind: str, limit: int) -> PartSpec:
    dims = _int(m, "rot.dims", 2)
    if dims % 2 or dims > limit:
        raise ConfigError(f"config.json: {where}.mixer.rot.dims {dims} must be even and at most {limit}")
    return PartSpec.make(kind, theta=_positive(m, "rot.base", where + ".mixer"), rotary_dim=dims)


def _wkv(m, where: str, eps: float) -> PartSpec:
    return PartSpec.make(
        "wkv", n_heads=_int(m, "heads"), head_dim=_int(m, "dim"), eps=eps,
        names=(("mu_r", "mix.mu.r"), ("mu_k", "mix.mu.k"), ("mu_v", "mix.mu.v"), ("mu_gate", "mix.mu.g"), ("mu_w", "mix.mu.w"),
               ("r", "mix.r"), ("k", "mix.k"), ("v", "mix.v"), ("gate", "mix.g"), ("w1", "mix.w1"), ("w2", "mix.w2"),
               ("w0", "mix.w0"), ("bonus", "mix.u"), ("norm", "mix.norm"), ("o", "mix.o")))


def _latent_attention(m, where: str, eps: float) -> PartSpec:
    rot = _int(m, "rot_dim", 2)
    if _int(m, "rot.dims", 2) != rot:
        raise ConfigError(f"config.json: {where}.mixer: rot.dims and rot_dim must be equal")
    return PartSpec.make(
        "latent_attention", n_heads=_int(m, "heads"), qk_dim=_int(m, "dim"), v_dim=_int(m, "vdim"),
        kv_rank=_int(m, "kv_rank"), rot_dim=rot, position=_rotation(m, where, "rope_interleaved", rot),
        scale=_float(m, "scale"), eps=eps, out_gate="sigmoid", pad_rank=True, shared_kv=m.get("kv_from") is not None,
        names=(("q", "mix.q"), ("down", "mix.dkv"), ("down_norm", "mix.dkv.norm"), ("up_k", "mix.uk"), ("up_v", "mix.uv"),
               ("gate", "mix.g"), ("o", "mix.o")))


def _attention(m, where: str, eps: float) -> PartSpec:
    heads, kv_heads, dim = _int(m, "heads"), _int(m, "kv_heads"), _int(m, "dim")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.mixer: {heads} heads are not a multiple of {kv_heads} kv_heads")
    mask = m.get("mask")
    return PartSpec.make(
        "gqa_attention", n_heads=heads, n_kv_heads=kv_heads, head_dim=dim, v_dim=_int(m, "vdim"), bias=True,
        scale=_float(m, "scale"), position=_rotation(m, where, "rope_neox", dim), out_gate="sigmoid", pad_heads=True,
        window=_int(mask, "size") if mask is not None else 0,
        keep_first=_int(mask, "keep_first", 0) if mask is not None and mask.get("keep_first") is not None else 0,
        names=(("q", "mix.q"), ("k", "mix.k"), ("v", "mix.v"), ("q_bias", "mix.q.b"), ("k_bias", "mix.k.b"),
               ("v_bias", "mix.v.b"), ("gate", "mix.g"), ("o", "mix.o")))


_MIXERS = {"wkv": _wkv, "latent_attention": _latent_attention, "attention": _attention}


def _feed_forward(mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is not a feed-forward of {ARCHITECTURE} "
                          "(known: 'dense', or null for none)")
    return PartSpec.make("act_mlp", intermediate_size=_int(mlp, "ff"), activation="gelu_tanh",
                         names=(("up", "mlp.up"), ("down", "mlp.down")))


def _lender(layers, i: int):
    """The layer whose latents layer ``i`` reads, checked; None: its own."""
    m = layers[i]["mixer"]
    if layers[i]["type"] != "latent_attention" or m.get("kv_from") is None:
        return None
    j = _int(m, "kv_from", 0)
    other = layers[j] if j < i else None
    if other is None or other["type"] != "latent_attention" or other["mixer"].get("kv_from") is not None:
        raise ConfigError(f"config.json: layers[{i}].mixer.kv_from {j} must name an earlier latent_attention layer that "
                          "makes latents of its own")
    for key in ("kv_rank", "rot_dim", "rot.base"):
        if _get(m, key) != _get(other["mixer"], key):
            raise ConfigError(f"config.json: layers[{i}].mixer.{key} differs from layers[{j}]'s, whose latents it reads")
    return j


def nekotar_model_spec(d: Mapping[str, Any]) -> ModelSpec:
    width, vocab, streams = _int(d, "width"), _int(d, "vocab"), _int(d, "streams")
    eps = _positive(_get(d, "norm"), "eps", "norm")
    mult = _float(d, "residual_mult")
    norm = PartSpec.make("rmsnorm", eps=eps)
    layers_in = _get(d, "layers")
    if not isinstance(layers_in, (list, tuple)) or not layers_in:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    block = PartSpec.make("hyper_prenorm", streams=streams, residual_mult=mult, names=(
        ("mixer_norm", "norm1"), ("mixer_in", "hc1.in"), ("mixer_mix", "hc1.mix"), ("mixer_out", "hc1.out"),
        ("ffn_norm", "norm2"), ("ffn_in", "hc2.in"), ("ffn_mix", "hc2.mix"), ("ffn_out", "hc2.out")))
    layers, schedule = [], []
    for i, entry in enumerate(layers_in):
        where = f"layers[{i}]"
        if not isinstance(entry, Mapping):
            raise ConfigError(f"config.json: {where} must be an object")
        kind, m = entry.get("type"), entry.get("mixer")
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of {ARCHITECTURE} "
                              f"(known: {', '.join(repr(k) for k in _MIXERS)})")
        if not isinstance(m, Mapping):
            raise ConfigError(f"config.json: {where}.mixer must be an object")
        layers.append(LayerSpec(block=block, mixer=_MIXERS[kind](m, where, eps),
                                feed_forward=_feed_forward(entry.get("mlp"), where), norm=norm, prefix=f"l{i}."))
        schedule.append(ScheduleEntry(i, cache_of=_lender(layers_in, i)))
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab, max_positions=MAX_POSITIONS, streams=streams,
        layers=tuple(layers), schedule=tuple(schedule),
        embedding=PartSpec.make("token_embedding", name="embed", norm_name="embed.norm", eps=eps),
        final_norm=PartSpec.make("rmsnorm", eps=eps, name="final.norm"),
        head=PartSpec.make("lm_head", tied=False, name="head"), stop_token_ids=(), source=dict(d))
    spec.validate()
    return spec
