"""Nekotar without a device: the configuration reader and its refusals, the tensor list with a size that only
the checkpoint knows, random weights, and facts about the plain mechanisms that the device tests lean on."""
import copy

import numpy as np
import pytest

from nekotar_helpers import CONFIGS, DECAY_RANK, SEEDS, make_weights, model_folder, plain_logits, random_tokens, weights
from plain import nekotar_plain as NP


def spec_of(cfg):
    from gguf2bin_b200.config import model_spec_from_dict
    return model_spec_from_dict(cfg)


def test_reader_takes_every_size_and_constant_from_the_configuration():
    spec = spec_of(CONFIGS["s"])
    assert (spec.architecture, spec.hidden_size, spec.vocab_size, spec.streams, len(spec.layers)) == ("Nekotar", 64, 211, 3, 5)
    assert spec.final_norm.kind == "rmsnorm" and spec.final_norm["eps"] == 1e-6 and spec.head["tied"] is False
    assert (spec.embedding["norm_name"], spec.embedding["eps"]) == ("embed.norm", 1e-6)
    w = spec.layers[0]
    assert w.block.kind == "hyper_prenorm" and (w.block["streams"], w.block["residual_mult"]) == (3, 0.7)
    assert w.norm["eps"] == 1e-6 and w.prefix == "l0."
    assert (w.mixer.kind, w.mixer["n_heads"], w.mixer["head_dim"], w.mixer["eps"]) == ("wkv", 3, 20, 1e-6)
    assert (w.feed_forward.kind, w.feed_forward["intermediate_size"], w.feed_forward["activation"]) == ("act_mlp", 40, "gelu_tanh")
    m = spec.layers[1].mixer
    assert (m.kind, m["n_heads"], m["qk_dim"], m["v_dim"], m["kv_rank"], m["rot_dim"]) == ("latent_attention", 3, 24, 16, 40, 8)
    assert (m["scale"], m["out_gate"], m["shared_kv"]) == (0.3, "sigmoid", False) and m.get("window") is None
    assert (m["position"].kind, m["position"]["theta"], m["position"]["rotary_dim"]) == ("rope_interleaved", 10000.0, 8)
    assert spec.layers[1].feed_forward is None
    a = spec.layers[2].mixer
    assert (a.kind, a["n_heads"], a["n_kv_heads"], a["head_dim"], a["v_dim"]) == ("gqa_attention", 4, 2, 24, 16)
    assert (a["scale"], a["window"], a["keep_first"], a["bias"], a["out_gate"]) == (0.35, 20, 3, True, "sigmoid")
    assert (a["position"].kind, a["position"]["theta"], a["position"]["rotary_dim"]) == ("rope_neox", 10000.0, 16)
    assert [e.cache_of for e in spec.schedule] == [None, None, None, None, 1] and spec.layers[4].mixer["shared_kv"] is True
    u = spec_of(CONFIGS["u"])
    assert [e.cache_of for e in u.schedule] == [None, None, None, 1, None, 1]
    assert (u.layers[4].mixer["window"], u.layers[4].mixer["keep_first"]) == (0, 0)
    t = spec_of(CONFIGS["t"])
    assert t.streams == 1 and t.layers[0].mixer["position"]["theta"] == 500.0 and t.layers[1].mixer["position"]["theta"] == 1e5


def test_tensor_list_matches_the_checkpoint_names():
    from gguf2bin_b200.engine.model import expected_tensors
    from gguf2bin_b200.weights.loader import FreeSize, check_names_and_shapes
    for name, cfg in CONFIGS.items():
        exp = expected_tensors(spec_of(cfg))
        have = make_weights(cfg, SEEDS[name], DECAY_RANK[name])
        assert set(exp) == set(have)
        check_names_and_shapes(exp, {k: v.shape for k, v in have.items()})
    exp = expected_tensors(spec_of(CONFIGS["s"]))
    assert exp["l1.mix.q"].shape == (3 * 32, 64) and exp["l1.mix.dkv"].shape == (48, 64) and exp["l1.mix.g"].shape == (48, 64)
    assert exp["l0.hc2.mix"].shape == (3, 3) and exp["l2.mix.v.b"].shape == (32,) and exp["l0.mix.u"].shape == (3, 20)
    assert "l4.mix.dkv" not in exp and "l1.hc2.in" not in exp and "l1.norm2" not in exp
    assert isinstance(exp["l0.mix.w1"].shape[0], FreeSize)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="retention"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not a feed-forward"),
    (lambda c: c["layers"][0].update(mixer=None), "must be an object"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=7), "must be equal"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=7, rot=dict(base=10.0, dims=7)), "must be even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=0), "must be positive"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26), "at most 24"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(keep_first=-1), "at least 0"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=0), "must name an earlier"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=4), "must name an earlier"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=4), "must name an earlier"),
    (lambda c: c["layers"][4]["mixer"].update(kv_rank=48), "kv_rank differs"),
    (lambda c: c["layers"][4]["mixer"]["rot"].update(base=77.0), "rot.base differs"),
    (lambda c: c.update(streams=0), "at least 1"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c["norm"].update(eps=0.0), "must be positive"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_reader_refuses_what_it_cannot_build(change, message):
    from gguf2bin_b200.config import ConfigError
    cfg = copy.deepcopy(CONFIGS["s"])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        spec_of(cfg)


def test_several_streams_exclude_what_assumes_one():
    import dataclasses
    from gguf2bin_b200.config import ConfigError, ScheduleEntry
    spec = spec_of(CONFIGS["s"])
    with pytest.raises(ConfigError, match="several streams"):
        dataclasses.replace(spec, schedule=spec.schedule + (ScheduleEntry(0, add_embedding=True),)).validate()
    with pytest.raises(ConfigError, match="at least one"):
        dataclasses.replace(spec, streams=0).validate()


def test_random_weights_for_the_design_can_be_written_and_read(tmp_path):
    from gguf2bin_b200.weights import write_random_model
    write_random_model(tmp_path / "m", CONFIGS["u"], 5, "float32")
    W = NP.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert W["l2.mix.w1"].shape == (16, 60) and W["l2.mix.w2"].shape == (21, 16)
    mix = W["l0.hc1.mix"]                      # the streams of a random model stay apart: near the identity
    assert np.abs(mix - np.eye(4)).max() < 0.6 and np.abs(np.diag(mix) - 1).max() > 0
    logits = NP.forward(CONFIGS["u"], W, [3, 1, 4, 1, 5, 9, 2, 6])
    assert logits.shape == (8, 130) and np.isfinite(logits).all()


# ---- facts about the plain mechanisms -------------------------------------------------------------
def test_window_with_kept_first_tokens():
    assert NP.visible(25, 6, 20) and not NP.visible(26, 6, 20) and NP.visible(26, 2, 20, 3) and not NP.visible(26, 3, 20, 3)
    assert NP.visible(7, 7, 1) and not NP.visible(7, 6, 1) and NP.visible(500, 0) and not NP.visible(3, 4, 20, 9)
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((12, 4, 3)), rng.standard_normal((12, 2, 3)), rng.standard_normal((12, 2, 5))
    out = NP.attend(q, k, v, 0.7, 4, 2)
    for i in range(12):
        js = [j for j in range(i + 1) if i - j < 4 or j < 2]
        for h in range(4):
            e = np.exp(0.7 * k[js, h // 2] @ q[i, h])
            assert np.allclose(out[i, h], (e / e.sum()) @ v[js, h // 2])


def test_rotations_depend_on_distance_alone_and_leave_the_rest():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    Q, K = np.repeat(q[None, None], 30, 0), np.repeat(k[None, None], 30, 0)
    for f in (lambda x: NP.rotate_halves(x, 6, 100.0), lambda x: NP.rotate_neighbours(x, 100.0)):
        a, b = f(Q)[:, 0], f(K)[:, 0]
        assert np.allclose(a[20] @ b[13], a[9] @ b[2]) and not np.allclose(a[20] @ b[13], a[20] @ b[12])
        assert np.allclose(a[0], q)
    assert np.array_equal(NP.rotate_halves(Q, 6, 100.0)[:, 0, 6:], Q[:, 0, 6:])
    one = NP.rotate_neighbours(np.array([[[0.0, 0.0, 0.0, 0.0]], [[1.0, 0.0, 0.0, 2.0]]]), 4.0)[1, 0]
    assert np.allclose(one, [np.cos(1), np.sin(1), -2 * np.sin(0.5), 2 * np.cos(0.5)])
    two = NP.rotate_halves(np.array([[[0.0] * 4], [[1.0, 0.0, 0.0, 2.0]]]), 4, 4.0)[1, 0]
    assert np.allclose(two, [np.cos(1), -2 * np.sin(0.5), np.sin(1), 2 * np.cos(0.5)])


def test_the_bonus_counts_for_the_current_token_only():
    """One head of two channels with decays of their own, written by the first token alone."""
    T, w, u = 5, np.array([0.5, 0.9]), np.array([[3.0, -1.0]])
    r, k, v = np.ones((T, 1, 2)), np.zeros((T, 1, 2)), np.ones((T, 1, 1))
    k[0] = 1.0
    out = NP.recurrence(r, k, v, np.broadcast_to(w, (T, 1, 2)), u)[:, 0, 0]
    assert np.allclose(out, [3.0 - 1.0] + [w[0] ** (i - 1) + w[1] ** (i - 1) for i in range(1, T)])
    t = {"w1": np.eye(2), "w2": np.eye(2), "w0": np.array([0.3, -1.0])}
    h = np.array([[0.5, 2.0]])
    assert np.allclose(NP.key_decays(h, t, ""), np.exp(-np.exp(np.tanh(h) + t["w0"])))
    x = np.arange(6.0).reshape(3, 2)
    assert np.allclose(NP.shifted(x, np.array([1.0, 0.5])), [[0, 0.5], [0, 2], [2, 4]])


def test_streams_are_mixed_from_to():
    X = np.arange(1.0, 4.0)[:, None, None]
    mix = np.array([[1.0, 10.0, 0.0], [0.0, 0.0, 2.0], [5.0, 0.0, 0.0]])
    out = NP.write_streams(X, np.array([[100.0]]), mix, np.array([1.0, 0.0, -2.0]), 0.5)[:, 0, 0]
    assert np.allclose(out, [1 + 15 + 50, 10.0, 4.0 - 100.0])
    assert NP.read_streams(X, np.array([1.0, 0.0, 2.0]))[0, 0] == 7.0


def test_a_prompt_of_the_plain_model_does_not_look_ahead():
    for name in CONFIGS:
        toks = random_tokens(name, 30, 3)
        whole = plain_logits(name, toks)
        assert np.allclose(whole[:20], plain_logits(name, toks[:20]), atol=1e-9) and np.abs(whole).max() > 1.0


def test_model_folder_reads_back():
    cfg, W = NP.load(model_folder("s"))
    assert cfg["streams"] == 3 and W["l0.mix.w1"].shape == (5, 64)
    assert all(np.array_equal(W[k], v) for k, v in weights("s").items())
