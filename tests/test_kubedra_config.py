"""Kubedra without a device: the configuration reader and its refusals, the schedule of repeated layers, the
tensor list with a size that only the checkpoint knows, and facts about the plain mechanisms that the
device tests lean on."""
import copy
import math

import numpy as np
import pytest

from kubedra_helpers import CONFIGS, DECAY_RANK, SEEDS, clear_tokens, make_weights, model_folder, weights
from plain import kubedra_plain as KP


def spec_of(cfg):
    from gguf2bin_b200.config import model_spec_from_dict
    return model_spec_from_dict(cfg)


def test_reader_takes_every_size_and_constant_from_the_configuration():
    spec = spec_of(CONFIGS["s"])
    assert (spec.architecture, spec.hidden_size, spec.vocab_size, spec.max_positions, len(spec.layers)) == \
        ("Kubedra", 64, 211, 192, 4)
    assert spec.final_norm.kind == "rmsnorm" and spec.final_norm["offset"] == 1.0 and spec.head["tied"] is True
    assert (spec.embedding["positions"], spec.embedding["n_positions"]) == ("pos", 192)
    g = spec.layers[0]
    assert g.block.kind == "sandwich_norm" and g.norm["eps"] == 1e-6 and g.norm["offset"] == 1.0 and g.prefix == "l0."
    assert (g.mixer.kind, g.mixer["n_heads"], g.mixer["qk_dim"], g.mixer["v_dim"], g.mixer["tau"]) == ("gla", 3, 20, 12, 4.0)
    assert (g.feed_forward.kind, g.feed_forward["intermediate_size"], g.feed_forward["activation"]) == ("swiglu", 40, "gelu_tanh")
    m = spec.layers[1].mixer
    assert (m.kind, m["n_heads"], m["qk_dim"], m["v_dim"], m["q_rank"], m["kv_rank"]) == ("latent_attention", 3, 24, 16, 24, 40)
    assert (m["scale"], m["window"], m["eps"], m.get("sink"), m.get("out_gate")) == (0.35, 20, 1e-6, None, None)
    r = spec.layers[1].feed_forward
    assert (r.kind, r["n_experts"], r["top"], r["intermediate_size"]) == ("routed_experts", 5, 3, 24)
    assert (r["limit"], r["alpha"], r["router_bias"], r["renormalise"], r["correction"]) == (1.5, 1.702, True, True, False)
    assert (r["shared"].kind, r["shared"]["intermediate_size"], r["shared"]["limit"]) == ("swiglu", 40, 3.0)
    assert spec.layers[2].feed_forward is None
    other = spec_of(CONFIGS["t"])
    assert other.layers[2].mixer["window"] == 0 and other.layers[0].feed_forward["shared"] is None
    assert other.layers[3].mixer["tau"] == 1.0 and other.layers[0].norm["eps"] == 1e-5


def test_a_loop_repeats_its_layers_and_adds_the_embedding_before_every_further_pass():
    def order(cfg):
        return [(e.layer, e.add_embedding) for e in spec_of(cfg).schedule]
    F, A = False, True
    assert order(CONFIGS["s"]) == [(0, F), (1, F), (2, F), (1, A), (2, F), (1, A), (2, F), (3, F)]
    assert order(CONFIGS["t"]) == [(0, F), (1, F), (2, F), (3, F)]
    assert order(CONFIGS["u"]) == [(0, F), (1, F), (2, F), (0, A), (1, F), (2, F)]
    one = dict(CONFIGS["t"], loop=dict(start=2, stop=3, times=4))
    assert order(one) == [(0, F), (1, F), (2, F), (2, A), (2, A), (2, A), (3, F)]
    assert order(dict(CONFIGS["t"], loop=dict(start=1, stop=4, times=1))) == order(CONFIGS["t"])
    assert order(dict(CONFIGS["t"], loop=None)) == order(CONFIGS["t"])
    for cfg in list(CONFIGS.values()) + [one]:
        assert order(cfg) == KP.layer_runs(cfg)
        assert all(e.cache_of is None for e in spec_of(cfg).schedule)       # every pass has storage of its own


def test_tensor_list_matches_the_checkpoint_names():
    from gguf2bin_b200.engine.model import expected_tensors
    from gguf2bin_b200.weights.loader import check_names_and_shapes
    for name, cfg in CONFIGS.items():
        exp = expected_tensors(spec_of(cfg))
        have = make_weights(cfg, SEEDS[name], DECAY_RANK[name])
        optional = {k for k, e in exp.items() if e.optional}
        assert set(exp) - optional == set(have) - optional
        check_names_and_shapes(exp, {k: v.shape for k, v in have.items()})
    exp = expected_tensors(spec_of(CONFIGS["s"]))
    assert exp["l1.mix.uq"].shape == (3 * 24, 24) and exp["l1.mix.uv"].shape == (3 * 16, 40)
    assert exp["l1.mlp.router.b"].shape == (5,) and exp["l0.mix.norm"].shape == (12,) and exp["pos"].shape == (192, 64)
    assert exp["l2.norm2b"].optional and not exp["l1.norm2b"].optional


def test_a_size_that_only_the_checkpoint_knows():
    """The rank of the decay's matrices: any size fits where the shape is free, and nothing else does."""
    from gguf2bin_b200.engine.model import expected_tensors
    from gguf2bin_b200.weights.loader import FreeSize, check_names_and_shapes
    from gguf2bin_b200.weights.safetensors_io import WeightsError
    exp = expected_tensors(spec_of(CONFIGS["t"]))
    assert isinstance(exp["l1.mix.a1"].shape[0], FreeSize) and exp["l1.mix.a1"].shape == (16, 96)
    for rank in (1, 5, 64):
        check_names_and_shapes(exp, {k: v.shape for k, v in make_weights(CONFIGS["t"], 1, rank).items()})
    shapes = {k: v.shape for k, v in make_weights(CONFIGS["t"], 1, 16).items()}
    for bad in ((16, 95), (16,), (0, 96)):
        with pytest.raises(WeightsError, match="l1.mix.a1"):
            check_names_and_shapes(exp, dict(shapes, **{"l1.mix.a1": bad}))


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="retention"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "not a feed-forward"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "choices among"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0), "must be positive"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0), "must be positive"),
    (lambda c: c["layers"][0].update(mixer=None), "must be an object"),
    (lambda c: c.update(loop=dict(start=3, stop=3, times=2)), "loop runs"),
    (lambda c: c.update(loop=dict(start=1, stop=5, times=2)), "loop runs"),
    (lambda c: c.update(loop=dict(start=1, stop=3, times=0)), "at least 1"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c.pop("norm"), "norm.eps"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_reader_refuses_what_it_cannot_build(change, message):
    from gguf2bin_b200.config import ConfigError
    cfg = copy.deepcopy(CONFIGS["s"])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        spec_of(cfg)


def test_random_weights_for_the_design_can_be_written_and_read(tmp_path):
    from gguf2bin_b200.weights import write_random_model
    write_random_model(tmp_path / "m", CONFIGS["u"], 5, "float32")
    W = KP.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert W["l1.mix.a1"].shape == (16, 60) and W["l1.mix.a2"].shape == (21, 16)
    logits = KP.forward(CONFIGS["u"], W, [3, 1, 4, 1, 5, 9, 2, 6])
    assert logits.shape == (8, 130) and np.isfinite(logits).all()


def test_gate_forms():
    """The one form with four numbers is each of the gates that the parts name."""
    from gguf2bin_b200.config import ConfigError
    from gguf2bin_b200.parts.feed_forward import gate_form
    z, u = np.linspace(-9, 9, 181), np.linspace(-5, 5, 181)[::-1]

    def value(f):
        g, v = np.minimum(z, f.limit), np.clip(u, -f.limit, f.limit)
        return g * KP.sigmoid(g * (f.c1 + f.c3 * g * g)) * (v + f.offset)
    assert np.allclose(value(gate_form("x", None, 0.0, 1.0)), KP.silu(z) * u)
    assert np.allclose(value(gate_form("x", "gelu_tanh", 0.0, 1.0)), KP.gelu_tanh(z) * u, atol=1e-12)
    g = np.minimum(z, 2.5)
    assert np.allclose(value(gate_form("x", None, 2.5, 1.702)), g * KP.sigmoid(1.702 * g) * (np.clip(u, -2.5, 2.5) + 1))
    for bad in (("relu", 0.0), ("gelu_tanh", 1.0), (None, -1.0)):
        with pytest.raises(ConfigError):
            gate_form("x", bad[0], bad[1], 1.702)


# ---- facts about the plain mechanisms -------------------------------------------------------------
def test_window_rule():
    assert KP.visible(25, 6, 20) and not KP.visible(26, 6, 20) and KP.visible(7, 7, 1) and not KP.visible(7, 6, 1)
    assert KP.visible(500, 0) and not KP.visible(3, 4)
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((12, 2, n)) for n in (3, 3, 4))
    for window in (0, 1, 5, 12, 40):
        out = KP.attend(q, k, v, 0.7, window)
        for i in range(12):
            js = [j for j in range(12) if KP.visible(i, j, window)]
            for h in range(2):
                e = np.exp(0.7 * k[js, h] @ q[i, h])
                assert np.allclose(out[i, h], (e / e.sum()) @ v[js, h])


def test_decay_acts_on_the_rows_of_key_channels():
    """One head of two key channels with decays of their own: the closed form of the read-out."""
    T, a = 6, np.array([0.5, 0.9])
    q, k, v = np.ones((T, 1, 2)), np.zeros((T, 1, 2)), np.arange(1.0, 1.0 + T)[:, None, None]
    k[0] = 1.0                                             # the first token alone writes
    out = KP.recurrence(q, k, v, np.broadcast_to(a, (T, 1, 2)))
    assert np.allclose(out[:, 0, 0], [a[0] ** i + a[1] ** i for i in range(T)])
    m = dict(heads=1, dim=2, tau=4.0)
    t = {"a1": np.eye(2), "a2": np.eye(2), "a2.b": np.array([0.3, -1.0])}
    h = np.array([[0.5, 2.0]])
    assert np.allclose(KP.key_decays(h, m, t, "")[0, 0], KP.sigmoid(np.array([0.8, 1.0])) ** 0.25)


def test_router_weights_are_a_softmax_over_the_chosen_logits():
    chosen, w = KP.route(np.array([0.1, 2.0, -1.0, 1.0]), 2)
    assert list(chosen) == [1, 3] and np.allclose(w, [1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])
    assert KP.routing_margin(np.array([0.1, 2.0, -1.0, 1.0]), 2) == pytest.approx(0.9)
    assert KP.routing_margin(np.array([1.0, 2.0]), 2) == np.inf


def test_whole_prompts_and_single_steps_of_the_plain_model_agree():
    for name in CONFIGS:
        toks = clear_tokens(name, 30, 3)
        whole = KP.forward(CONFIGS[name], weights(name), toks)
        model = KP.Stepper(CONFIGS[name], weights(name))
        assert np.allclose([model.step(t) for t in toks], whole, atol=1e-9)


def test_model_folder_reads_back():
    cfg, W = KP.load(model_folder("s"))
    assert cfg["loop"] == dict(start=1, stop=3, times=3) and W["l0.mix.a1"].shape == (5, 64)
    assert all(np.array_equal(W[k], v) for k, v in weights("s").items())
