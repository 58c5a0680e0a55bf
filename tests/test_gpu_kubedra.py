"""Kubedra on the device against the plain implementation: each mechanism's part alone (with weights
or inputs made so that a far key, a window's edge or a lost state shows), then whole models of three
small configurations in every way of cutting the work (whole prompts, token by token, portions down to
two tokens, unequal batches, slots and pages used again, long decoding over page and window borders),
and greedy generation through the library's entry point, its command line and trace replay."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from helpers import assert_close
from kubedra_helpers import CONFIGS, clear_tokens, mixer_weights, mlp_weights, model_folder, plain_logits, weights
from levolix_helpers import assert_rows_close
from part_runner import DEV, DTYPES, bf, close, dev, i32, run_part, step_ctx
from plain import kubedra_plain as KP

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
EPS = 1e-5

CUTS = [([], []), ([1] * 199, [1] * 99), ([2] * 99, [2] * 50), ([3, 1, 1, 2, 30], [17, 2]),
        ([63, 1, 2, 62, 1, 1], [1, 1, 1]), ([64, 64, 1], [2, 2, 2])]


def bind(part, W, dtype, pre="mix."):
    part.bind({pre + k: dev(v, DTYPES[dtype]) for k, v in W.items()})
    return part


# ----------------------------------------------------------------------------
# embedding with positions, the join between two sublayers
# ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_adds_the_position_row(dtype):
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(0)
    table, pos = bf(rng.standard_normal((50, 37))), bf(rng.standard_normal((9, 37)))
    ids, at = [3, 49, 0, 7], [8, 0, 5, 200]            # the last one counts past the table: its last row
    out, again = (torch.empty((4, 37), dtype=torch.float32, device=DEV) for _ in range(2))
    kernels.embed_rows(dev(table, DTYPES[dtype]), i32(ids), out, 0.5, dev(pos, DTYPES[dtype]), i32(at), again)
    ref = table[ids] * 0.5 + pos[[8, 0, 5, 8]]
    close(out.cpu().numpy(), ref, "float32", "embedding")
    assert torch.equal(out, again)
    kernels.embed_rows(dev(table, DTYPES[dtype]), i32(ids), out)
    close(out.cpu().numpy(), table[ids], "float32", "embedding without positions")


@pytest.mark.parametrize("T,H", [(5, 64), (3, 61), (70, 256), (4, 1500), (3, 4096), (2, 8192), (2, 9000), (2, 2050)])
def test_norm_join(T, H):
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(T + H)
    x, y, e = (rng.standard_normal((T, H)) * s for s in (2.0, 5.0, 1.0))
    w, w2 = 1 + 0.3 * rng.standard_normal(H), 1 + 0.3 * rng.standard_normal(H)
    for add in (None, e):
        joined = x + KP.rms_divide(y, 1e-3) * w + (0 if add is None else add)
        xs = dev(x)
        kernels.norm_join(xs, dev(y), dev(w), 1e-3, add32=None if add is None else dev(add))
        close(xs.cpu().numpy(), joined, "float32", "join")
        for dtype in ("float32", "bfloat16"):
            xs, out = dev(x), torch.empty((T, H), dtype=DTYPES[dtype], device=DEV)
            kernels.norm_join(xs, dev(y), dev(w), 1e-3, (dev(w2), 1e-2), out, None if add is None else dev(add))
            close(xs.cpu().numpy(), joined, "float32", "join in front of a norm")
            close(out.float().cpu().numpy(), KP.rms_divide(joined, 1e-2) * w2, dtype, "norm behind a join", loose=0.5)
    # routed experts: two choices a token, the second without a row (it reads the token's own x), on top of a base
    rows, weight = rng.standard_normal((2 * T, H)), rng.random((T, 2))
    pair_row = np.stack([np.arange(T)[::-1], np.full(T, -1)], 1)
    total = e + weight[:, :1] * rows[pair_row[:, 0]] + weight[:, 1:] * x
    joined = x + KP.rms_divide(total, 1e-3) * w + y
    for dtype in ("float32", "bfloat16"):
        xs, out = dev(x), torch.empty((T, H), dtype=DTYPES[dtype], device=DEV)
        kernels.moe_combine_join(dev(rows), i32(pair_row), dev(weight), dev(e), 2, xs, dev(w), 1e-3, (None, 1e-2), out, dev(y))
        close(xs.cpu().numpy(), joined, "float32", "experts' join")
        close(out.float().cpu().numpy(), KP.rms_divide(joined, 1e-2), dtype, "norm behind the experts' join", loose=0.5)


# ----------------------------------------------------------------------------
# feed-forwards: gates in the products' epilogues, routed experts
# ----------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["gelu", "capped"])
@pytest.mark.parametrize("M,ff,K", [(1, 96, 64), (7, 40, 256), (12, 512, 1024), (40, 1024, 1024), (50, 128, 96),
                                    (100, 2304, 1024), (130, 264, 128), (300, 520, 256), (700, 2048, 512), (4100, 1280, 256),
                                    (3, 4096, 2048), (33, 48, 4096)])
def test_gates_in_the_products_epilogues(M, ff, K, kind):
    """Every product kernel that takes a gate (few rows whole and streamed, rows over a cluster, tiles, persistent
    tiles, pairs of CTAs), in bfloat16, against the gate of the 32-bit product."""
    from gguf2bin_b200 import kernels
    form = kernels.GluForm.gelu_tanh() if kind == "gelu" else kernels.GluForm.capped(1.5, 1.702)
    g = torch.Generator(device=DEV).manual_seed(M + ff)
    h = torch.randn((M, K), device=DEV, generator=g).to(torch.bfloat16)
    w = (torch.randn((2 * ff, K), device=DEV, generator=g) * 2.0 / K ** 0.5).to(torch.bfloat16)
    mid = torch.full((M, ff), 7.0, dtype=torch.bfloat16, device=DEV)
    assert kernels.gate_up_fused(h, w, mid, 8, form)
    z = (h.double() @ w.double().t()).view(M, ff // 8, 2, 8)
    gate, up = z[:, :, 0].reshape(M, ff).cpu().numpy(), z[:, :, 1].reshape(M, ff).cpu().numpy()
    if kind == "gelu":
        ref = KP.gelu_tanh(gate) * up
    else:
        ref = np.minimum(gate, 1.5) * KP.sigmoid(1.702 * np.minimum(gate, 1.5)) * (np.clip(up, -1.5, 1.5) + 1)
    err = np.abs(mid.float().cpu().numpy() - ref)
    assert err.max() <= 0.006 * np.abs(ref).max() and (err <= 0.01 * np.abs(ref) + 2e-3).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,width", [(40, 64), (36, 60), (72, 96)])
def test_gelu_feed_forward(ff, width, dtype):
    from gguf2bin_b200.config.kubedra import _feed_forward
    from gguf2bin_b200.parts.feed_forward import SwiGLU
    rng = np.random.default_rng(ff)
    W = {k: bf(v) for k, v in mlp_weights(rng, dict(kind="dense", ff=ff), width).items()}
    part = bind(SwiGLU(_feed_forward(dict(kind="dense", ff=ff), "test"), width, DTYPES[dtype], DEV), W, dtype, "mlp.")
    for n in (1, 77):
        h = bf(rng.standard_normal((n, width)))
        ref = KP.gelu_ff(h, W, "")
        ctx = step_ctx([n], [0], [0], dtype)
        y = torch.full((n, width), 2.0, dtype=torch.float32, device=DEV)
        part.forward(dev(h, DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref + 2.0, dtype, "gelu feed-forward, added")
        part.forward_into(dev(h, DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref, dtype, "gelu feed-forward, stored")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,ff,limit,shared,rows", [
    (5, 3, 24, 1.5, (40, 3.0), 77), (4, 4, 20, 1.0, (12, 2.0), 77), (3, 1, 40, 2.5, None, 77), (16, 2, 48, 0.5, (24, 4.0), 77),
    (3, 2, 64, 2.0, (64, 1.0), 300), (1, 1, 16, 3.0, None, 200)])
def test_routed_experts(experts, top, ff, limit, shared, rows, dtype):
    """Choices and weights as the plain router makes them, limits that bend most values, a row alone, two rows,
    and enough rows for each of the grouped products."""
    from gguf2bin_b200.config.kubedra import _feed_forward
    from gguf2bin_b200.parts.feed_forward import RoutedExperts
    rng = np.random.default_rng(experts * 10 + top)
    width = 48
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if shared:
        mlp["shared"] = dict(ff=shared[0], limit=shared[1])
    W = {k: bf(v) for k, v in mlp_weights(rng, mlp, width).items()}
    part = bind(RoutedExperts(_feed_forward(mlp, "test"), width, DTYPES[dtype], DEV), W, dtype, "mlp.")
    h = []
    while len(h) < rows:                                # rows whose choice is clear in 16 bits too
        row = bf(rng.standard_normal(width))
        if KP.routing_margin(KP.router_logits(row, W, ""), top) > 0.1:
            h.append(row)
    h = np.array(h)
    ref = KP.routed_ff(h, mlp, W, "")
    x0, add = rng.standard_normal((rows, width)), rng.standard_normal((rows, width))
    w, w2 = 1 + 0.3 * rng.standard_normal(width), 1 + 0.3 * rng.standard_normal(width)
    for sel in (slice(0, rows), slice(5, 6), slice(40, 42)):
        n = sel.stop - sel.start
        ctx = step_ctx([n], [0], [0], dtype)
        y = torch.zeros((n, width), dtype=torch.float32, device=DEV)
        part.forward(dev(h[sel], DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref[sel], dtype, f"routed rows {sel}")
        y = torch.full((n, width), 9.0, dtype=torch.float32, device=DEV)
        part.forward_into(dev(h[sel], DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref[sel], dtype, f"routed rows {sel}, stored")
        xs, out = dev(x0[sel]), torch.empty((n, width), dtype=DTYPES[dtype], device=DEV)
        assert part.forward_norm_join(dev(h[sel], DTYPES[dtype]), ctx, y, xs, dev(w), EPS, (dev(w2), EPS), out, dev(add[sel]))
        joined = x0[sel] + KP.rms_divide(ref[sel], EPS) * w + add[sel]
        close(xs.cpu().numpy(), joined, dtype, f"routed rows {sel}, joined")
        close(out.float().cpu().numpy(), KP.rms_divide(joined, EPS) * w2, dtype, f"routed rows {sel}, next norm")


# ----------------------------------------------------------------------------
# latent attention with a query latent and a window
# ----------------------------------------------------------------------------
def latent_part(m, W, width, dtype):
    from gguf2bin_b200.config.kubedra import _latent_attention
    from gguf2bin_b200.parts.latent import LatentAttention
    return bind(LatentAttention(_latent_attention(m, "test", EPS), width, DTYPES[dtype], DEV), W, dtype)


def latent_config(H, D, V, qr, r, window, scale=None):
    m = dict(heads=H, dim=D, vdim=V, q_rank=qr, kv_rank=r, scale=scale if scale is not None else 1.5 / np.sqrt(D))
    if window:
        m["mask"] = dict(size=window)
    return m


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V,qr,r,window", [
    (3, 24, 16, 24, 40, 20),         # latents padded to 64 in 16 bits, up-projections multiplied into their neighbours
    (2, 8, 12, 40, 56, 33),          # heads so small that the up-projections stay products of their own
    (2, 48, 32, 64, 128, 70),        # a rank the tensor-core kernels take, a window longer than a page
    (4, 64, 64, 32, 64, 0),          # everything seen
    (1, 10, 14, 12, 20, 1),          # the token itself
    (5, 40, 24, 20, 100, 64),        # padded to 128, a window of one page, a query rank that is no multiple of 8
    (2, 32, 16, 16, 160, 9),         # more than the tensor-core kernels take
    (16, 16, 8, 24, 96, 65),
])
def test_latent_attention_part(H, D, V, qr, r, window, dtype):
    rng = np.random.default_rng(H * 1000 + r)
    width = 40
    m = latent_config(H, D, V, qr, r, window)
    W = {k: bf(v) for k, v in mixer_weights(rng, "latent_attention", m, width).items()}
    part = latent_part(m, W, width, dtype)
    hs = [bf(rng.standard_normal((n, width))) for n in (200, 37)]
    ref = [KP.latent_attention(h, m, W, "", EPS) for h in hs]
    edge = max(window, 1)
    for cuts in CUTS + [([edge - 1, 1, 1, 1], [edge, 2]), ([edge + 1, 1, 1, 2, 5], [2, 2, 2])]:
        cuts = tuple([c for c in one if c > 0] for one in cuts)
        got = run_part(part, part.cache_need(), hs, cuts, dtype)
        for b in range(2):
            close(got[b], ref[b], dtype, f"latent attention {cuts[0][:4]} sequence {b}", loose=2.0)


def flagged_latents(H, D, V, qr, r, window, bump=14.0, width=24, seed=1):
    """Latent attention whose scores get ``bump`` more for a key whose input row has channel 0 set to one: that channel
    feeds latent entry 0 and nothing else does, the key's last entry is that latent entry alone, and the query's last
    entry is a constant that comes from channel 1 (one in every row).  A flagged token takes nearly all the weight of
    every query that sees it, and its value points in a direction of its own."""
    rng = np.random.default_rng(seed)
    m = latent_config(H, D, V, qr, r, window, scale=0.25)
    W = mixer_weights(rng, "latent_attention", m, width)
    for k in ("dq", "dkv"):
        W[k][:, :2] = 0.0
        W[k][0] = 0.0
        W[k + ".norm"][0] = 1.0
    W["dkv"][0, 0], W["dq"][0, 1] = 12.0, 12.0
    c0, q0 = (12.0 / np.sqrt((144.0 + n) / n) for n in (r, qr))        # what entry 0 is after the norm, about
    W["uq"] *= 0.3
    W["uk"] *= 0.3
    W["uk"][:, 0] = 0.0                                    # (the score's other entries do not move with the flag)
    for h in range(H):
        at = h * D + D - 1
        W["uq"][at], W["uk"][at] = 0.0, 0.0
        W["uq"][at, 0], W["uk"][at, 0] = 1.0, bump / (c0 * q0 * m["scale"])
    return m, {k: bf(v) for k, v in W.items()}, width


def flagged_rows(rng, n, width, targets):
    h = rng.standard_normal((n, width))
    h[:, 0], h[:, 1] = 0.0, 1.0
    for t in targets:
        h[t, 0] = 1.0
    return bf(h)


SIZES = [("float32", (2, 16, 16, 20, 24)), ("bfloat16", (2, 16, 16, 20, 24)), ("bfloat16", (3, 64, 32, 64, 128)),
         ("bfloat16", (2, 16, 8, 24, 136))]


@pytest.mark.parametrize("dtype,sizes", SIZES)
@pytest.mark.parametrize("target", [0, 1, 63, 64, 127, 300])
def test_a_far_key_among_hundreds(target, dtype, sizes):
    """One key of 700 takes the weight, at the first positions, at page borders and far back, with nothing masked."""
    m, W, width = flagged_latents(*sizes, window=0)
    part = latent_part(m, W, width, dtype)
    h = flagged_rows(np.random.default_rng(target), 700, width, [target])
    ref = KP.latent_attention(h, m, W, "", EPS)
    without = KP.latent_attention(flagged_rows(np.random.default_rng(target), 700, width, []), m, W, "", EPS)
    assert np.abs(ref[699] - without[699]).max() > 0.2 * np.abs(ref).max()          # the key does matter at the far end
    for cuts in ([[]], [[690] + [1] * 10], [[target + 1, 650] + [1] * 49]):
        got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(2,), pages_per_seq=11)
        close(got[0], ref, dtype, f"far key at {target}, cuts {cuts[0][:3]}", loose=2.0)


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype,sizes", SIZES)
@pytest.mark.parametrize("window", [1, 7, 63, 64, 65, 130])
def test_window_edges_stand_out(window, dtype, sizes, decode):
    """A flagged token just inside the window takes a query's weight, just outside it takes none: rows of the prompt and
    rows decoded one by one, flags at page borders and elsewhere, the window's edges in pages of their own."""
    m, W, width = flagged_latents(*sizes, window=window)
    part = latent_part(m, W, width, dtype)
    n = 3 * window + 150
    flags = [2, 63, 64 + window, 100 + 2 * window]
    h = flagged_rows(np.random.default_rng(window), n, width, flags)
    ref = KP.latent_attention(h, m, W, "", EPS)
    for off in (window - 1, window + 1):
        if off:
            other = KP.latent_attention(h, dict(m, mask=dict(size=off)), W, "", EPS)
            assert np.abs(other - ref).max() > 0.3 * np.abs(ref).max()              # one token off is no small thing
    start = 60 + window
    cuts = [[start] + [1] * (n - start)] if decode else [[start, 1, 1, 2]]
    got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(4,), pages_per_seq=9)[0]
    close(got, ref, dtype, f"window {window}", loose=2.0)


# ----------------------------------------------------------------------------
# gated linear attention
# ----------------------------------------------------------------------------
def gla_part(m, W, width, dtype):
    from gguf2bin_b200.config.kubedra import _gla
    from gguf2bin_b200.parts.recurrent import GatedLinearAttention
    return bind(GatedLinearAttention(_gla(m, "test", EPS), width, DTYPES[dtype], DEV), W, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V,tau,rank", [
    (3, 20, 12, 4.0, 5), (2, 16, 24, 16.0, 16), (1, 136, 40, 8.0, 16), (4, 32, 64, 1.0, 3), (3, 7, 5, 2.0, 9),
    (2, 64, 33, 16.0, 24), (1, 96, 130, 3.0, 1), (1, 260, 10, 16.0, 40), (1, 130, 6, 5.0, 8), (2, 1, 3, 2.0, 2),
    (1, 512, 9, 20.0, 16), (1, 300, 70, 16.0, 64), (2, 128, 256, 16.0, 16), (2, 256, 48, 16.0, 16), (1, 402, 4, 9.0, 7)])
def test_gla_part(H, D, V, tau, rank, dtype):
    """Key sizes of 1 to 512 (8 to 32 lanes a column, with and without 16-byte rows), column counts that fill no block,
    decay ranks that are no multiple of eight; the first token is made large, so that a state that is lost or not cleared
    shows later on; the prompts' segments and single tokens in every order."""
    rng = np.random.default_rng(D * 10 + V)
    width = 40
    m = dict(heads=H, dim=D, vdim=V, tau=tau)
    W = {k: bf(v) for k, v in mixer_weights(rng, "gla", m, width, decay_rank=rank).items()}
    part = gla_part(m, W, width, dtype)
    hs = [bf(rng.standard_normal((n, width))) for n in (200, 37)]
    hs[0][0] *= 6.0
    ref = [KP.gla(h, m, W, "", EPS) for h in hs]
    for cuts in CUTS + [([15, 1, 16, 17, 1, 1], [1, 1, 1]), ([129, 2], [16, 16, 5]), ([5, 130], [])]:
        got = run_part(part, part.cache_need(), hs, cuts, dtype)
        for b in range(2):
            close(got[b], ref[b], dtype, f"gla {cuts[0][:4]} sequence {b}", loose=3.0)


@pytest.mark.parametrize("wide", [False, True])
def test_a_state_carried_over_hundreds_of_tokens(wide, monkeypatch):
    """700 tokens in one step (eleven segments, or six of twice the size), then 20 one by one: channels that forget
    slowly still hold the first token, those that forget at once hold nothing of it."""
    from gguf2bin_b200 import kernels
    if wide:
        monkeypatch.setattr(kernels, "CHANNEL_TILES_WIDE_FROM", 2)
    rng = np.random.default_rng(9)
    width, m = 32, dict(heads=2, dim=24, vdim=16, tau=16.0)
    W = mixer_weights(rng, "gla", m, width)
    W["a2"] *= 0.2
    W["a2.b"][:] = 6.0                                     # a decay of about 0.9998 a token
    W["a2.b"][::3] = -80.0                                 # and of about 0.007
    W = {k: bf(v) for k, v in W.items()}
    h = bf(rng.standard_normal((720, width)))
    h[0] *= 20.0
    ref = KP.gla(h, m, W, "", EPS)
    calm = h.copy()
    calm[0] /= 20.0
    assert np.abs(ref[719] - KP.gla(calm, m, W, "", EPS)[719]).max() > 1e-2         # still the first token's doing
    part = gla_part(m, W, width, "float32")
    for cuts in ([[700] + [1] * 20], [[64, 2, 634] + [1] * 20], [[]]):
        got = run_part(part, part.cache_need(), [h], cuts, "float32", slots=(2,), pages_per_seq=12)[0]
        close(got, ref, "float32", f"long state {cuts[0][:3]}", loose=2.0)


def test_prompts_of_many_lengths_in_one_step():
    """Sequences of one token, of less than a segment, of exactly one, of one and a token, of several, side by side,
    each going on from a state of its own."""
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(17)
    H, D, V, R = 2, 20, 12, 8
    lens, pasts = [1, 70, 64, 65, 200, 3, 128], [0, 5, 64, 1, 0, 100, 7]
    slots = [6, 2, 0, 5, 1, 3, 4]
    T = sum(lens)
    q, k, v, low = (bf(rng.standard_normal((T, n))) for n in (H * D, H * D, H * V, R))
    w, b = bf(rng.standard_normal((H * D, R))), rng.standard_normal(H * D)
    S0 = rng.standard_normal((8, H, V, D))
    state = dev(S0)
    out = torch.empty((T, H * V), dtype=torch.float32, device=DEV)
    kernels.channel_scan(dev(q), dev(k), dev(v), dev(low), dev(w), dev(b), state, step_ctx(lens, pasts, slots, "float32"), out,
                         H, D, V, 0.3, 5.0)
    alpha = np.exp(-np.logaddexp(0.0, -(low @ w.T + b)) / 5.0).reshape(T, H, D)
    at = 0
    for n, s in zip(lens, slots):
        S = S0[s].transpose(0, 2, 1).copy()                # [H, D, V]
        for t in range(at, at + n):
            S = alpha[t][:, :, None] * S + k[t].reshape(H, D, 1) * v[t].reshape(H, 1, V)
            ref = np.einsum("hdv,hd->hv", S, q[t].reshape(H, D) * 0.3).reshape(-1)
            close(out[t:t + 1].cpu().numpy(), ref[None], "float32", f"token {t}", loose=2.0)
        close(state[s].cpu().numpy(), S.transpose(0, 2, 1), "float32", f"state of slot {s}", loose=2.0)
        at += n
    assert np.array_equal(state[7].cpu().numpy(), S0[7].astype(np.float32))         # a slot outside the step is untouched


# ----------------------------------------------------------------------------
# whole models
# ----------------------------------------------------------------------------
CASES = [(n, d) for n in ("s", "t", "u") for d in ("float32", "bfloat16")]
LENGTHS = {"s": [70, 9, 131, 1, 33], "t": [80, 1, 140, 17], "u": [131, 2, 64, 65, 23]}


@pytest.fixture(scope="module")
def engines():
    from gguf2bin_b200.engine import Engine, Model
    made = {}

    def get(name, dtype, max_tokens=2048):
        key = (name, dtype, max_tokens)
        if key not in made:
            made[key] = Engine(Model.from_folder(model_folder(name), dtype=dtype), max_tokens=max_tokens)
        return made[key]
    return get


def requests_of(name):
    return [list(clear_tokens(name, n, i)) for i, n in enumerate(LENGTHS[name])]


def run_in_portions(eng, toks, sizes):
    from gguf2bin_b200.engine import StepEntry
    seq, got, done = eng.open_sequence(), [], 0
    sizes = list(sizes)
    while done < len(toks):
        n = min(sizes.pop(0) if sizes else len(toks), len(toks) - done)
        got.append(eng.step([StepEntry(seq, toks[done:done + n], range(n))]).cpu().numpy())
        done += n
    eng.close_sequence(seq)
    return np.concatenate(got)


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompts(engines, name, dtype):
    eng, reqs = engines(name, dtype), requests_of(name)
    got, ref = [run_in_portions(eng, toks, []) for toks in reqs], [plain_logits(name, toks) for toks in reqs]
    # (the 16-bit rule speaks of the median row: a request of one or two tokens has none to speak of)
    assert_rows_close(np.concatenate(got), np.concatenate(ref), dtype, f"kubedra {name}/{dtype} whole")


@pytest.mark.parametrize("name,dtype", CASES)
def test_the_stream_after_every_layer_run(engines, name, dtype):
    """The residual stream behind every execution of a layer, looped ones each time, before the embedding is added
    again: where a difference would begin."""
    from gguf2bin_b200.engine import StepEntry
    eng, toks = engines(name, dtype), requests_of(name)[0][:40]
    ref, got = [], []
    KP.forward(CONFIGS[name], weights(name), toks, layers_out=ref)
    model, graphs = eng.model, eng.step_graphs
    cls = type(model.blocks[0])
    forward = cls.forward

    def watched(self, x, ctx, view):
        add = ctx.next_add
        if not cls.takes_stream_add:           # a block that knows nothing of the addition
            ctx.next_add = None
        forward(self, x, ctx, view)
        if not cls.takes_stream_add:
            ctx.next_add = add
        taken = add is not None and ctx.next_add is None
        got.append((x - add if taken else x)[:len(toks)].cpu().numpy())
    try:
        eng.step_graphs, cls.forward = False, watched
        for one_launch in (True, False):       # the addition and the next norm in the layer's last launch, or by themselves
            got.clear()
            cls.takes_stream_add = one_launch
            seq = eng.open_sequence()
            eng.step([StepEntry(seq, toks, [0])])
            eng.close_sequence(seq)
            assert len(got) == len(ref)
            for i, (a, b) in enumerate(zip(got, ref)):
                assert np.abs(a - b).max() <= (3e-5 if dtype == "float32" else 0.06) * np.abs(b).max(), f"layer run {i}"
    finally:
        cls.forward, cls.takes_stream_add, eng.step_graphs = forward, True, graphs


@pytest.mark.parametrize("name,dtype", CASES)
def test_token_by_token_and_portions(engines, name, dtype):
    """The same logits however the prompt is cut: every token alone from the first one on; portions
    of two; mixed portions that end on, before and behind page and window borders."""
    eng = engines(name, dtype)
    toks = requests_of(name)[2 if name != "u" else 0][:110]
    ref = plain_logits(name, toks)
    whole = run_in_portions(eng, toks, [])
    for what, sizes in [("one by one", [1] * len(toks)), ("twos", [2] * len(toks)), ("mixed", [3, 2, 5, 1, 2, 50, 1, 2, 2]),
                        ("window edge", [19, 1, 1, 4, 1, 6, 1, 1, 36, 1]), ("page edge", [63, 1, 1, 2]), ("page", [64, 2, 2])]:
        got = run_in_portions(eng, toks, sizes)
        assert_rows_close(got, ref, dtype, f"kubedra {name}/{dtype} {what}")
        if dtype == "float32":       # the cut changes nothing but the order of a few additions
            assert np.abs(got - whole).max() <= 2e-5 * max(1.0, np.abs(ref).max()), what


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_batches_with_reuse(engines, name, dtype):
    """Batches of up to three requests: prompts (all but the last 6 tokens, at least one) in one step,
    then one token each, shorter requests ending earlier; the cache holds one batch, so every batch
    gets the slots, states and pages that the one before gave back."""
    from gguf2bin_b200.engine import StepEntry
    reqs = requests_of(name)
    batches = [reqs[i:i + 3] for i in range(0, len(reqs), 3)] * 2
    need = max(sum(-(-len(t) // 64) * 64 for t in b) for b in batches)
    eng = engines(name, dtype, need)
    every, refs = [], []
    for batch in batches:
        seqs = [eng.open_sequence() for _ in batch]
        heads = [max(1, len(t) - 6) for t in batch]
        got = [[] for _ in batch]
        out = eng.step([StepEntry(s, t[:h], range(h)) for s, t, h in zip(seqs, batch, heads)]).cpu().numpy()
        o = 0
        for j, h in enumerate(heads):
            got[j].append(out[o:o + h])
            o += h
        done = list(heads)
        live = [j for j in range(len(batch)) if done[j] < len(batch[j])]
        for j in range(len(batch)):
            if j not in live:
                eng.close_sequence(seqs[j])
        while live:
            out = eng.step([StepEntry(seqs[j], [batch[j][done[j]]], [0]) for j in live]).cpu().numpy()
            for r, j in enumerate(live):
                got[j].append(out[r:r + 1])
                done[j] += 1
            for j in [j for j in live if done[j] == len(batch[j])]:
                eng.close_sequence(seqs[j])
            live = [j for j in live if done[j] < len(batch[j])]
        every += [row for rows in got for row in rows]
        refs += [plain_logits(name, toks) for toks in batch]
    assert_rows_close(np.concatenate(every), np.concatenate(refs), dtype, f"kubedra {name}/{dtype} batches")
    assert eng.cache.table.pages.n_held == 0 and eng.cache.table.slots.n_held == 0


@pytest.mark.parametrize("name,dtype", [("s", "float32"), ("t", "bfloat16"), ("u", "bfloat16"), ("u", "float32")])
def test_long_decoding(engines, name, dtype):
    """A short prompt, then 120 tokens one by one: the window passes over decoded tokens, pages begin, positions reach
    the table's last row; beside a second sequence that started elsewhere."""
    from gguf2bin_b200.engine import StepEntry, StepError
    eng = engines(name, dtype)
    a, b = list(clear_tokens(name, 150, 70)), list(clear_tokens(name, 181, 71))
    sa, sb = eng.open_sequence(), eng.open_sequence()
    out = eng.step([StepEntry(sa, a[:30], range(30)), StepEntry(sb, b[:61], range(61))]).cpu().numpy()
    ga, gb = [out[:30]], [out[30:]]
    for t in range(120):
        out = eng.step([StepEntry(sa, [a[30 + t]], [0]), StepEntry(sb, [b[61 + t]], [0])]).cpu().numpy()
        ga.append(out[:1])
        gb.append(out[1:])
    if CONFIGS[name]["max_positions"] == 181:              # no row of the table is left for another token
        with pytest.raises(StepError, match="positions"):
            eng.step([StepEntry(sb, [1], [0])])
    eng.close_sequence(sa)
    eng.close_sequence(sb)
    assert_rows_close(np.concatenate(ga), plain_logits(name, a), dtype, f"kubedra {name}/{dtype} long decoding a")
    assert_rows_close(np.concatenate(gb), plain_logits(name, b), dtype, f"kubedra {name}/{dtype} long decoding b")


def plain_greedy(name, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(plain_logits(name, toks)[-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["s", "u"])
def test_greedy_generation_through_the_entry_point(name):
    """LLM.generate (scheduler, decode session with its graph) against the plain implementation's
    argmax, several unequal prompts at once."""
    from gguf2bin_b200.api import LLM
    llm = LLM(model_folder(name), dtype="float32", max_tokens=2048)
    prompts = [list(clear_tokens(name, n, 90 + i)) for i, n in enumerate([9, 1, 66, 30])]
    for _ in range(2):                         # the second call finds slots, pages and graphs of the first
        outs = llm.generate(prompts, n=30, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0)
        for p, o in zip(prompts, outs):
            toks = list(p)
            for t in o.tokens:
                row = plain_logits(name, toks)[-1]
                assert row[t] >= row.max() - 2e-5 * max(1.0, np.abs(row).max())
                toks.append(t)
            assert len(o.tokens) == 30
    a = llm.generate(prompts[:2], n=12, seed=5)
    b = llm.generate(prompts[:2], n=12, seed=5)
    assert [o.tokens for o in a] == [o.tokens for o in b]
    assert llm.engine.cache.table.pages.n_held == 0 and llm.engine.cache.table.slots.n_held == 0


def test_the_programs(tmp_path):
    """info and run of the command line, random weights for the design's config.json, and trace replay."""
    folder = model_folder("s")
    exe = [sys.executable, str(ROOT / "bin" / "gguf2bin_b200")]
    out = subprocess.run(exe + ["info", str(folder)], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0 and "Kubedra" in out.stdout + out.stderr, out.stderr[-2000:]
    prompt = list(clear_tokens("s", 7, 40))
    out = subprocess.run(exe + ["run", str(folder), "--tokens", ",".join(map(str, prompt)), "-n", "6", "-t", "0",
                                "--repeat-penalty", "1", "--dtype", "float32", "--ignore-eos"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert [int(t) for t in out.stdout.split()] == prompt + plain_greedy("s", prompt, 6)
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(CONFIGS["u"]))
    made = tmp_path / "made"
    out = subprocess.run(exe + ["synth", str(made), "--config", str(cfg_file), "--seed", "3", "--dtype", "float32"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    W = KP.read_safetensors(made / "model.safetensors")
    toks = np.random.default_rng(4).integers(0, CONFIGS["u"]["vocab"], 9).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:6], "want": [0, 5]},
                                     {"id": "b", "tokens": toks[:1], "want": [0]}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[6:7], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[7:8], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[8:], "want": [0]}], "end": ["a"]}]
    out_dir = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(made), "--dtype", "float32",
                           "--out", str(out_dir), "--max-tokens", "64"],
                          input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out_dir / "1.f32").exists()
    got = np.concatenate([np.fromfile(out_dir / f"{i}.f32", "<f4").reshape(-1, CONFIGS["u"]["vocab"]) for i in (0, 2, 3)])
    ref = KP.forward(CONFIGS["u"], W, toks)
    assert_close(got, ref[[0, 5, 0, 7, 8]], "float32", "kubedra trace replay")
