"""Nekotar on the device against the plain implementation: each mechanism's part alone (with weights
or inputs made so that a far key, a window's edge, a kept first token or a lost state shows), then whole
models of three small configurations in every way of cutting the work (whole prompts, token by token,
portions down to two tokens, unequal batches, slots and pages used again, long decoding over page and
window borders), and greedy generation through the library's entry point, its command line and trace replay."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from helpers import assert_close
from levolix_helpers import assert_rows_close
from nekotar_helpers import (CONFIGS, latent, mixer_weights, mlp_weights, model_folder, plain_logits, random_tokens, weights,
                             windowed)
from part_runner import DEV, DTYPES, bf, close, dev, i32, run_part, step_ctx
from plain import nekotar_plain as NP

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
EPS = 1e-5
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])

CUTS = [([], []), ([1] * 199, [1] * 99), ([2] * 99, [2] * 50), ([3, 1, 1, 2, 30], [17, 2]),
        ([63, 1, 2, 62, 1, 1], [1, 1, 1]), ([64, 64, 1], [2, 2, 2])]


def bind(part, W, dtype, pre="mix."):
    part.bind({pre + k: dev(v, DTYPES[dtype]) for k, v in W.items()})
    return part


# ----------------------------------------------------------------------------
# embedding with a norm, several streams
# ----------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("copies,H", [(1, 37), (3, 64), (4, 600)])
def test_embedding_with_a_norm_and_copies(copies, H, dtype):
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(H)
    table, w = bf(rng.standard_normal((50, H)) * 0.02), 1 + 0.3 * rng.standard_normal(H)
    ids = [3, 49, 0, 7, 7]
    out = torch.empty((5, copies, H), dtype=torch.float32, device=DEV)
    kernels.embed_norm_rows(dev(table, DTYPES[dtype]), i32(ids), dev(w), 1e-4, out, 1.5)
    ref = NP.rms_norm(table[ids] * 1.5, w, 1e-4)
    for c in range(copies):
        close(out[:, c].cpu().numpy(), ref, "float32", f"copy {c}")


@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("T,H", [(5, 64), (3, 61), (70, 256), (4, 1500), (3, 4096), (2, 8192), (2, 9000), (2, 2050)])
def test_streams_read_and_join(T, H, S):
    """Every variant of the kernel: widths for each number of registers, widths that are no multiple of four, more
    streams than it is specialised on; with and without a reader behind the join; rows picked for the head."""
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(T + H + S)
    X, y = rng.standard_normal((S, T, H)) * np.arange(1, S + 1)[:, None, None], rng.standard_normal((T, H)) * 4
    mix, out, a = rng.standard_normal((S, S)), rng.standard_normal(S), rng.standard_normal(S)
    w = 1 + 0.3 * rng.standard_normal(H)
    new = NP.write_streams(X, y, mix, out, 0.6)
    Xd = dev(X.transpose(1, 0, 2)).contiguous()
    xs = Xd.clone()
    kernels.streams_join(xs, dev(y), dev(mix), dev(out), 0.6)
    close(xs.cpu().numpy().transpose(1, 0, 2), new, "float32", "join")
    rows = i32([T - 1, 0, T - 1])
    for dtype in ("float32", "bfloat16"):
        h = torch.empty((T, H), dtype=DTYPES[dtype], device=DEV)
        kernels.streams_read(Xd, dev(a), dev(w), 1e-2, h)
        close(h.float().cpu().numpy(), NP.rms_norm(NP.read_streams(X, a), w, 1e-2), dtype, "read", loose=0.5)
        picked = torch.empty((3, H), dtype=DTYPES[dtype], device=DEV)
        kernels.streams_read(Xd, None, dev(w), 1e-2, picked, rows)
        close(picked.float().cpu().numpy(), NP.rms_norm(X.sum(0), w, 1e-2)[[T - 1, 0, T - 1]], dtype, "the sum's rows", loose=0.5)
        xs = Xd.clone()
        kernels.streams_join(xs, dev(y), dev(mix), dev(out), 0.6, (dev(a), dev(w), 1e-2), h)
        close(xs.cpu().numpy().transpose(1, 0, 2), new, "float32", "join in front of a reader")
        close(h.float().cpu().numpy(), NP.rms_norm(NP.read_streams(new, a), w, 1e-2), dtype, "reader behind a join", loose=0.5)


# ----------------------------------------------------------------------------
# feed-forward
# ----------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("ff,width", [(40, 64), (36, 60), (72, 96), (21, 40), (1024, 256)])
def test_gelu_feed_forward(ff, width, dtype):
    from gguf2bin_b200.config.nekotar import _feed_forward
    from gguf2bin_b200.parts.feed_forward import ActMLP
    rng = np.random.default_rng(ff)
    W = {k: bf(v) for k, v in mlp_weights(rng, ff, width).items()}
    part = bind(ActMLP(_feed_forward(dict(kind="dense", ff=ff), "test"), width, DTYPES[dtype], DEV), W, dtype, "mlp.")
    for n in (1, 9, 77, 300):
        h = bf(rng.standard_normal((n, width)))
        ref = NP.gelu_mlp(h, W, "")
        ctx = step_ctx([n], [0], [0], dtype)
        y = torch.full((n, width), 2.0, dtype=torch.float32, device=DEV)
        part.forward(dev(h, DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref + 2.0, dtype, "gelu feed-forward, added")
        part.forward_into(dev(h, DTYPES[dtype]), ctx, y)
        close(y.cpu().numpy(), ref, dtype, "gelu feed-forward, stored")


@pytest.mark.parametrize("M,N,K", [(1, 96, 64), (7, 40, 256), (12, 512, 1024), (40, 1024, 1024), (50, 128, 96), (100, 2304, 1024),
                                   (130, 264, 128), (300, 520, 256), (700, 2048, 512), (4100, 1280, 256), (3, 4096, 2048),
                                   (33, 48, 4096), (16, 4096, 4096), (2048, 1024, 4096)])
def test_an_activation_in_the_products_epilogues(M, N, K):
    """Every product kernel (few rows whole and streamed, rows over a cluster, tiles, persistent tiles, parts of K,
    pairs of CTAs) with the activation on its way out, against that of the 32-bit product; columns of a wider output."""
    from gguf2bin_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(M + N)
    a = torch.randn((M, K), device=DEV, generator=g).to(torch.bfloat16)
    w = (torch.randn((N, K), device=DEV, generator=g) * 2.0 / K ** 0.5).to(torch.bfloat16)
    wide = torch.full((M, N + 16), 7.0, dtype=torch.bfloat16, device=DEV)
    for out in (torch.full((M, N), 7.0, dtype=torch.bfloat16, device=DEV), wide[:, 8:8 + N]):
        assert kernels.linear_act(a, w, out, kernels.GluForm.gelu_tanh())
        ref = NP.gelu_tanh((a.double() @ w.double().t()).cpu().numpy())
        err = np.abs(out.float().cpu().numpy() - ref)
        assert err.max() <= 0.006 * np.abs(ref).max() and (err <= 0.01 * np.abs(ref) + 2e-3).all()
    assert (wide[:, :8] == 7.0).all() and (wide[:, 8 + N:] == 7.0).all()


@pytest.mark.parametrize("G,M,N,K", [(4, 1, 64, 72), (3, 8, 48, 1024), (4, 8, 2048, 2048), (2, 13, 128, 256), (5, 40, 272, 512),
                                     (4, 3, 1024, 2048), (3, 100, 256, 512), (4, 300, 512, 256), (2, 2048, 768, 512),
                                     (3, 4200, 256, 256), (4, 130, 96, 64), (2, 7, 20, 64), (4, 16, 4096, 4096)])
def test_products_of_several_inputs_side_by_side(G, M, N, K):
    """A stack of inputs, each for a range of the output's columns, in one launch where a kernel takes the case (few rows
    whole and streamed, rows over a cluster, tiles, persistent tiles, pairs of CTAs) and one by one where none does."""
    from gguf2bin_b200 import kernels
    gen = torch.Generator(device=DEV).manual_seed(M + N)
    a = torch.randn((G, M, K), device=DEV, generator=gen).to(torch.bfloat16)
    w = (torch.randn((G, N, K), device=DEV, generator=gen) / K ** 0.5).to(torch.bfloat16)
    out = torch.full((M, G * N), 7.0, dtype=torch.bfloat16, device=DEV)
    kernels.linear_stacked(a, w, out)
    ref = torch.einsum("gmk,gnk->mgn", a.double(), w.double()).reshape(M, G * N).cpu().numpy()
    assert np.abs(out.float().cpu().numpy() - ref).max() <= 0.006 * np.abs(ref).max()
    out32 = torch.empty((M, G * N), dtype=torch.float32, device=DEV)
    kernels.linear_stacked(a.float(), w.float(), out32)
    assert np.abs(out32.cpu().numpy() - ref).max() <= 1e-4 * np.abs(ref).max()


@pytest.mark.parametrize("T,heads,n,r", [(65, 3, 16, 48), (200, 2, 128, 128), (70, 5, 72, 64), (300, 1, 8, 8), (129, 4, 64, 512),
                                         (66, 16, 136, 40)])
def test_products_of_small_matrices_per_head(T, heads, n, r):
    """One launch for all heads, with no gate, a gate per head and a gate per output; rows of wider buffers."""
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(n + r)
    x, w, g1, g2 = (bf(rng.standard_normal(s)) for s in ((T, heads * r), (heads, n, r), (T, heads), (T, heads * n)))
    w = bf(w / np.sqrt(r))
    ref = np.einsum("thr,hnr->thn", x.reshape(T, heads, r), w)
    wide = torch.zeros((T, heads * r + 24), dtype=torch.bfloat16, device=DEV)
    wide[:, 16:16 + heads * r] = dev(x, torch.bfloat16)
    for gate, factor in ((None, 1.0), (g1, NP.sigmoid(g1)[:, :, None]), (g2, NP.sigmoid(g2).reshape(T, heads, n))):
        gd = dev(gate, torch.bfloat16) if gate is not None else None
        for xs in (dev(x, torch.bfloat16), wide[:, 16:16 + heads * r]):
            out = torch.full((T, heads * n), 5.0, dtype=torch.bfloat16, device=DEV)
            assert kernels.head_expand_tiles(xs, dev(w.reshape(heads * n, r), torch.bfloat16), out, heads, gd)
            close(out.float().cpu().numpy(), (ref * factor).reshape(T, -1), "bfloat16", "per-head product", loose=0.3)
        few = torch.full((9, heads * n), 5.0, dtype=torch.bfloat16, device=DEV)
        kernels.head_product(dev(x[:9], torch.bfloat16), dev(w.reshape(heads * n, r), torch.bfloat16), few, heads, True,
                             gd[:9] if gd is not None else None)
        close(few.float().cpu().numpy(), (ref * factor).reshape(T, -1)[:9], "bfloat16", "per-head product of few rows", loose=0.3)


# ----------------------------------------------------------------------------
# latent attention with rotated entries and a gate per element
# ----------------------------------------------------------------------------
def latent_part(m, W, width, dtype):
    from gguf2bin_b200.config.nekotar import _latent_attention
    from gguf2bin_b200.parts.latent import LatentAttention
    return bind(LatentAttention(_latent_attention(m, "test", EPS), width, DTYPES[dtype], DEV), W, dtype)


LATENT_SIZES = [
    (3, 24, 16, 40, 8),          # rows of 48 padded to 64 in 16 bits, U_k multiplied into the query matrix
    (2, 48, 32, 104, 24),        # rows of 128
    (4, 64, 64, 40, 24),         # rows of 64
    (1, 10, 14, 20, 2),          # a single rotated pair; one head
    (5, 40, 24, 70, 30),         # padded to 128; a rotated part that is no multiple of 8
    (2, 8, 12, 100, 16),         # heads so small that U_k stays a product of its own
    (3, 9, 7, 130, 32),          # more than the tensor-core kernels take, sizes that are no multiple of 8
    (16, 16, 8, 56, 8),
]


@BOTH
@pytest.mark.parametrize("H,D,V,r,rot", LATENT_SIZES)
def test_latent_attention_part(H, D, V, r, rot, dtype):
    rng = np.random.default_rng(H * 1000 + r)
    width = 40
    m = latent(H, D, V, r, rot, 1.5 / np.sqrt(D + rot), base=50.0)
    W = {k: bf(v) for k, v in mixer_weights(rng, "latent_attention", m, width).items()}
    part = latent_part(m, W, width, dtype)
    hs = [bf(rng.standard_normal((n, width))) for n in (200, 37)]
    ref = [NP.latent_attention(h, m, W, "", EPS) for h in hs]
    for cuts in CUTS:
        got = run_part(part, part.cache_need(), hs, cuts, dtype)
        for b in range(2):
            close(got[b], ref[b], dtype, f"latent attention {cuts[0][:4]} sequence {b}", loose=2.0)


@pytest.mark.parametrize("fold", [False, True])
def test_up_projections_multiplied_in_or_not(fold, monkeypatch):
    """The same part with U_k in the query matrix and as a product of its own, for few rows and for many."""
    from gguf2bin_b200.parts import latent as L
    monkeypatch.setattr(L, "folds", lambda *a: fold)
    rng = np.random.default_rng(3)
    m = latent(4, 32, 24, 48, 16, 0.2, base=50.0)
    W = {k: bf(v) for k, v in mixer_weights(rng, "latent_attention", m, 64).items()}
    part = latent_part(m, W, 64, "bfloat16")
    assert part.fold_k == fold and not part.fold_v
    h = bf(rng.standard_normal((210, 64)))
    for cuts in ([[]], [[130, 70] + [1] * 10], [[5] * 42]):
        close(run_part(part, part.cache_need(), [h], cuts, "bfloat16", slots=(1,))[0], NP.latent_attention(h, m, W, "", EPS),
              "bfloat16", f"{cuts[0][:2]}", loose=2.0)


@BOTH
def test_a_layer_that_reads_another_layers_latents(dtype):
    """The borrower has its own queries, up-projections, gate and head sizes, and writes nothing."""
    rng = np.random.default_rng(8)
    width = 48
    m0 = latent(3, 24, 16, 40, 8, 0.3)
    m1 = latent(2, 12, 20, 40, 8, 0.4, kv_from=0)
    W0, W1 = ({k: bf(v) for k, v in mixer_weights(rng, "latent_attention", m, width).items()} for m in (m0, m1))
    lender, borrower = latent_part(m0, W0, width, dtype), latent_part(m1, W1, width, dtype)
    assert borrower.cache_need() is None
    h = bf(rng.standard_normal((150, width)))
    ref = NP.latent_attention(h, m1, W1, "", EPS, kept=NP.latents(h, m0, W0, "", EPS))

    def both(u, ctx, view, y):
        lender.forward(u, ctx, view, torch.zeros_like(y))
        before = view.pages.clone()
        borrower.forward(u, ctx, view, y)
        assert torch.equal(before, view.pages)
    for cuts in ([[]], [[1] * 150], [[63, 1, 2, 2]]):
        got = run_part(lender, lender.cache_need(), [h], cuts, dtype, slots=(2,), call=both)
        close(got[0], ref, dtype, f"borrowed latents {cuts[0][:3]}", loose=2.0)


def flagged_latents(H, D, V, r, rot, bump=14.0, width=24, seed=1):
    """Latent attention whose scores get ``bump`` more for a key whose input row has channel 0 set to one: that channel
    feeds latent entry 0 and nothing else does, the unrotated key's last entry is that latent entry alone, and the query's
    is a constant that comes from channel 1 (one in every row)."""
    rng = np.random.default_rng(seed)
    m = latent(H, D, V, r, rot, 0.25)
    W = mixer_weights(rng, "latent_attention", m, width)
    W["dkv"][:, :2] = 0.0
    W["dkv"][0] = 0.0
    W["dkv"][0, 0], W["dkv.norm"][0] = 12.0, 1.0
    c0 = 12.0 / np.sqrt((144.0 + r) / r)                   # what entry 0 is after the norm, about
    W["q"][:, :2] = 0.0
    W["q"] *= 0.3
    W["uk"] *= 0.3
    W["uk"][:, 0] = 0.0                                    # (the score's other entries do not move with the flag)
    for h in range(H):
        k_at, q_at = h * D + D - 1, h * (D + rot) + D - 1
        W["q"][q_at], W["uk"][k_at] = 0.0, 0.0
        W["q"][q_at, 1], W["uk"][k_at, 0] = 1.0, bump / (c0 * m["scale"])
    return m, {k: bf(v) for k, v in W.items()}, width


def flagged_rows(rng, n, width, targets):
    h = rng.standard_normal((n, width))
    h[:, 0], h[:, 1] = 0.0, 1.0
    for t in targets:
        h[t, 0] = 1.0
    return bf(h)


LATENT_FAST = [("float32", (2, 16, 16, 24, 6)), ("bfloat16", (2, 16, 16, 24, 6)), ("bfloat16", (3, 64, 32, 104, 24)),
               ("bfloat16", (2, 16, 8, 136, 8))]


@pytest.mark.parametrize("dtype,sizes", LATENT_FAST)
@pytest.mark.parametrize("target", [0, 1, 63, 64, 127, 300])
def test_a_far_latent_among_hundreds(target, dtype, sizes):
    """One key of 700 takes the weight: at the first positions, at page borders and far back."""
    m, W, width = flagged_latents(*sizes)
    part = latent_part(m, W, width, dtype)
    h = flagged_rows(np.random.default_rng(target), 700, width, [target])
    ref = NP.latent_attention(h, m, W, "", EPS)
    without = NP.latent_attention(flagged_rows(np.random.default_rng(target), 700, width, []), m, W, "", EPS)
    assert np.abs(ref[699] - without[699]).max() > 0.2 * np.abs(ref).max()          # the key does matter at the far end
    for cuts in ([[]], [[690] + [1] * 10], [[target + 1, 650] + [1] * 49]):
        got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(2,), pages_per_seq=11)
        close(got[0], ref, dtype, f"far latent at {target}, cuts {cuts[0][:3]}", loose=2.0)


@BOTH
def test_rotated_entries_alone_decide(dtype):
    """Scores that come from the rotated entries alone (U_k is zero), so large that a key one position off, a pair
    turned the wrong way or a part that is not turned is another result altogether; at positions in the hundreds."""
    rng = np.random.default_rng(5)
    width, m = 32, latent(3, 8, 16, 24, 16, 1.2, base=30.0)
    W = mixer_weights(rng, "latent_attention", m, width)
    W["uk"][:] = 0.0
    W["q"] *= 1.3
    W = {k: bf(v) for k, v in W.items()}
    h = bf(rng.standard_normal((300, width)))
    ref = NP.latent_attention(h, m, W, "", EPS)
    other = NP.latent_attention(h, dict(m, rot=dict(base=32.0, dims=16)), W, "", EPS)
    assert np.abs(other - ref).max() > 0.3 * np.abs(ref).max()
    part = latent_part(m, W, width, dtype)
    for cuts in ([[]], [[280] + [1] * 20], [[2] * 150]):
        got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(2,))
        close(got[0], ref, dtype, f"rotated part, cuts {cuts[0][:2]}", loose=3.0)


# ----------------------------------------------------------------------------
# attention behind a window that keeps the first tokens
# ----------------------------------------------------------------------------
def windowed_part(m, W, width, dtype):
    from gguf2bin_b200.config.nekotar import _attention
    from gguf2bin_b200.parts.mixers import GQAAttention
    return bind(GQAAttention(_attention(m, "test", EPS), width, DTYPES[dtype], DEV), W, dtype)


@BOTH
@pytest.mark.parametrize("H,G,D,V,dims,window,keep", [
    (4, 2, 24, 16, 16, 20, 3),       # padded to 64 in 16 bits, part of a head turned
    (3, 3, 64, 104, 64, 70, 1),      # padded to 128; value heads larger than key heads; a key head per query head
    (6, 1, 10, 14, 4, 1, 2),         # one key head; a window of the token itself
    (4, 4, 128, 128, 128, 64, 0),    # nothing padded, nothing kept
    (8, 2, 40, 40, 40, None, 0),     # everything seen
    (2, 1, 130, 30, 64, 33, 70),     # larger than the tensor-core kernels take; kept tokens beyond the window and a page
    (12, 3, 16, 64, 2, 130, 5),
])
def test_windowed_attention_part(H, G, D, V, dims, window, keep, dtype):
    rng = np.random.default_rng(H * 1000 + D)
    width = 40
    m = windowed(H, G, D, V, dims, 1.5 / np.sqrt(D), window, keep, base=60.0)
    W = {k: bf(v) for k, v in mixer_weights(rng, "attention", m, width).items()}
    part = windowed_part(m, W, width, dtype)
    hs = [bf(rng.standard_normal((n, width))) for n in (200, 37)]
    ref = [NP.windowed_attention(h, m, W, "") for h in hs]
    edge = window or 50
    for cuts in CUTS + [([max(edge - 1, 1), 1, 1, 1], [edge, 2]), ([edge + 1, 1, 1, 2, 5], [2, 2, 2])]:
        got = run_part(part, part.cache_need(), hs, cuts, dtype)
        for b in range(2):
            close(got[b], ref[b], dtype, f"windowed attention {cuts[0][:4]} sequence {b}", loose=2.0)


def flagged_keys(H, G, D, V, dims, window, keep, bump=14.0, width=24, seed=1):
    """Scores get ``bump`` more for a key whose input row has channel 0 set to one: the key's last entry is that channel,
    the query's is its bias; what turns of that entry turns too slowly to matter."""
    rng = np.random.default_rng(seed)
    m = windowed(H, G, D, V, dims, 0.25, window, keep, base=1e9)
    W = mixer_weights(rng, "attention", m, width)
    for n, heads in (("q", H), ("k", G)):
        W[n][:, :2] = 0.0
        W[n] *= 0.3
        W[n + ".b"] *= 0.3
        for h in range(heads):
            W[n][h * D + D - 1], W[n + ".b"][h * D + D - 1] = 0.0, (1.0 if n == "q" else 0.0)
    for g in range(G):
        W["k"][g * D + D - 1, 0] = bump / m["scale"]
    return m, {k: bf(v) for k, v in W.items()}, width


WINDOWED_FAST = [("float32", (4, 2, 24, 16, 16)), ("bfloat16", (4, 2, 24, 16, 16)), ("bfloat16", (3, 1, 64, 96, 64)),
                 ("bfloat16", (2, 2, 136, 40, 8))]


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype,sizes", WINDOWED_FAST)
@pytest.mark.parametrize("window,keep", [(1, 1), (7, 0), (63, 64), (64, 3), (65, 0), (130, 65)])
def test_window_edges_and_kept_tokens_stand_out(window, keep, dtype, sizes, decode):
    """A flagged token just inside the window or among the kept ones takes a query's weight, just outside it takes none:
    rows of the prompt and rows decoded one by one, flags at page borders, on the last kept token and on the next."""
    n = 3 * window + 150
    start = 60 + window
    cuts = [[start] + [1] * (n - start)] if decode else [[start, 1, 1, 2]]
    edges = [f for f in (2, 63, 64 + window, 100 + 2 * window) if f >= keep]        # none that stays visible anyway
    for flags in (edges, [max(keep - 1, 0)], [keep]):
        m, W, width = flagged_keys(*sizes, window=window, keep=keep)
        part = windowed_part(m, W, width, dtype)
        h = flagged_rows(np.random.default_rng(window), n, width, flags)
        ref = NP.windowed_attention(h, m, W, "")
        if flags[-1] == keep:                              # one token more or fewer that is kept is no small thing
            for off in (keep + 1,) + ((keep - 1,) if keep and flags[0] < keep else ()):
                other = NP.windowed_attention(h, dict(m, mask=dict(size=window, keep_first=off)), W, "")
                assert np.abs(other - ref).max() > 0.2 * np.abs(ref).max()
        elif len(flags) > 1:
            for off in (window - 1, window + 1):
                if off:
                    other = NP.windowed_attention(h, dict(m, mask=dict(size=off, keep_first=keep)), W, "")
                    assert np.abs(other - ref).max() > 0.2 * np.abs(ref).max()
        got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(4,), pages_per_seq=9)[0]
        close(got, ref, dtype, f"window {window}, kept {keep}, flags {flags}", loose=2.0)


# ----------------------------------------------------------------------------
# time mixing
# ----------------------------------------------------------------------------
def wkv_part(m, W, width, dtype):
    from gguf2bin_b200.config.nekotar import _wkv
    from gguf2bin_b200.parts.recurrent import WKVMixer
    return bind(WKVMixer(_wkv(m, "test", EPS), width, DTYPES[dtype], DEV), W, dtype)


@BOTH
@pytest.mark.parametrize("H,D,rank,width", [(3, 20, 5, 40), (2, 16, 16, 64), (1, 136, 16, 40), (4, 32, 3, 64), (3, 7, 9, 60),
                                            (2, 64, 24, 40), (1, 260, 40, 40), (1, 130, 8, 41), (2, 1, 2, 40), (1, 402, 7, 40),
                                            (5, 64, 12, 104), (1, 512, 16, 24)])
def test_wkv_part(H, D, rank, width, dtype):
    """Key sizes of 1 to 512, ranks that are no multiple of eight, widths that are none of four; the first token is made
    large, so that a state, or a token before, that is lost or not cleared shows later on; segments and single tokens
    in every order."""
    rng = np.random.default_rng(D * 10 + rank)
    m = dict(heads=H, dim=D)
    W = {k: bf(v) for k, v in mixer_weights(rng, "wkv", m, width, decay_rank=rank).items()}
    part = wkv_part(m, W, width, dtype)
    hs = [bf(rng.standard_normal((n, width))) for n in (200, 37)]
    hs[0][0] *= 6.0
    ref = [NP.wkv(h, m, W, "", EPS) for h in hs]
    for cuts in CUTS + [([15, 1, 16, 17, 1, 1], [1, 1, 1]), ([129, 2], [16, 16, 5]), ([5, 130], [])]:
        got = run_part(part, part.cache_need(), hs, cuts, dtype)
        for b in range(2):
            if dtype == "bfloat16":
                # a head's read-out is divided by its own size: where it nearly cancels its rounding grows with it
                rows = np.abs(got[b] - ref[b]).max(-1) / np.abs(ref[b]).max()
                assert np.median(rows) < 0.02 and (rows > 0.06).mean() < 0.05 and rows.max() < 0.5, (cuts[0][:4], rows.max())
            else:
                close(got[b], ref[b], dtype, f"wkv {cuts[0][:4]} sequence {b}", loose=5.0)


@BOTH
def test_the_token_before_and_the_bonus_stand_out(dtype):
    """Every mix looks at the token before alone, and the bonus is what the token's own key counts: a row off by one, a
    kept row that is lost between steps, or a bonus that stays in the state is another result altogether."""
    rng = np.random.default_rng(12)
    width, m = 32, dict(heads=2, dim=24)
    W = mixer_weights(rng, "wkv", m, width)
    for c in "rkvgw":
        W["mu." + c][:] = 1.0
    W["u"][:] = 8.0
    W = {k: bf(v) for k, v in W.items()}
    h = bf(rng.standard_normal((140, width)))
    ref = NP.wkv(h, m, W, "", EPS)
    assert np.array_equal(ref[0], 0 * ref[0])                  # nothing in front of the first token
    part = wkv_part(m, W, width, dtype)
    for cuts in ([[]], [[1] * 140], [[2] * 70], [[64, 1, 63, 2]]):
        got = run_part(part, part.cache_need(), [h], cuts, dtype, slots=(2,))[0]
        close(got, ref, dtype, f"cuts {cuts[0][:3]}", loose=3.0)


@pytest.mark.parametrize("wide", [False, True])
def test_a_state_carried_over_hundreds_of_tokens(wide, monkeypatch):
    """700 tokens in one step (eleven segments, or six of twice the size), then 20 one by one: channels that forget
    slowly still hold the first token, those that forget at once hold nothing of it."""
    from gguf2bin_b200 import kernels
    if wide:
        monkeypatch.setattr(kernels, "CHANNEL_TILES_WIDE_FROM", 2)
    rng = np.random.default_rng(9)
    width, m = 32, dict(heads=2, dim=24)
    W = mixer_weights(rng, "wkv", m, width)
    W["w2"] *= 0.2
    W["w0"][:] = -8.5                                      # a decay of about 0.9998 a token
    W["w0"][::3] = 5.0                                     # and one that is zero in 32 bits
    W = {k: bf(v) for k, v in W.items()}
    h = bf(rng.standard_normal((720, width)))
    h[0] *= 20.0
    ref = NP.wkv(h, m, W, "", EPS)
    calm = h.copy()
    calm[0] /= 20.0
    assert np.abs(ref[719] - NP.wkv(calm, m, W, "", EPS)[719]).max() > 1e-2         # still the first token's doing
    part = wkv_part(m, W, width, "float32")
    for cuts in ([[700] + [1] * 20], [[64, 2, 634] + [1] * 20], [[]]):
        got = run_part(part, part.cache_need(), [h], cuts, "float32", slots=(2,), pages_per_seq=12)[0]
        close(got, ref, "float32", f"long state {cuts[0][:3]}", loose=5.0)


@BOTH
def test_sequences_of_many_lengths_in_one_step(dtype):
    """Sequences of one token, of less than a segment, of exactly one, of one and a token, of several, side by side, each
    going on from a state and a token before of its own: the mixed rows, the read-outs, the states left behind."""
    from gguf2bin_b200 import kernels
    rng = np.random.default_rng(17)
    H, D, R, width, n_mix = 2, 20, 8, 44, 3
    lens, pasts = [1, 70, 64, 65, 200, 3, 128], [0, 5, 64, 1, 0, 100, 7]
    slots = [6, 2, 0, 5, 1, 3, 4]
    T, dt = sum(lens), DTYPES[dtype]
    h, kept0, mu = bf(rng.standard_normal((T, width))), bf(rng.standard_normal((8, width))), bf(rng.random((n_mix, width)))
    ctx = step_ctx(lens, pasts, slots, dtype)
    kept, mixed = dev(kept0, dt), torch.empty((n_mix, T, width), dtype=dt, device=DEV)
    kernels.shift_mix(dev(h, dt), dev(mu), kept, ctx, mixed)
    r, k, v = (bf(rng.standard_normal((T, n))) for n in (H * D, H * D, H * D))
    low = rng.standard_normal((T, R)).astype(np.float32).astype(np.float64)
    w, b, u = bf(rng.standard_normal((H * D, R))), rng.standard_normal(H * D) - 1, rng.standard_normal((H, D))
    S0 = rng.standard_normal((8, H, D, D))
    state, own = dev(S0), torch.empty((T, H * D), dtype=torch.float32, device=DEV)
    kernels.channel_scan(dev(r, dt), dev(k, dt), dev(v, dt), dev(low), dev(w, dt), dev(b), state, ctx, own, H, D, D, 1.0,
                         decay="double_exp", low_tanh=True, bonus=dev(u))
    alpha = np.exp(-np.exp(np.tanh(low) @ w.T + b)).reshape(T, H, D)
    at = 0
    for n, s, past in zip(lens, slots, pasts):
        rows = slice(at, at + n)
        for i in range(n_mix):
            ref = NP.shifted(h[rows], mu[i], kept0[s] if past else None)
            close(mixed[i, rows].float().cpu().numpy(), ref, dtype, f"mix {i} of slot {s}")
        S = S0[s].transpose(0, 2, 1)
        ref = NP.recurrence(r[rows].reshape(n, H, D), k[rows].reshape(n, H, D), v[rows].reshape(n, H, D), alpha[rows], u, S)
        close(own[rows].cpu().numpy(), ref.reshape(n, -1), "float32", f"read-out of slot {s}", loose=3.0)
        for t in range(at, at + n):
            S = alpha[t][:, :, None] * S + k[t].reshape(H, D, 1) * v[t].reshape(H, 1, D)
        close(state[s].cpu().numpy(), S.transpose(0, 2, 1), "float32", f"state of slot {s}", loose=3.0)
        assert np.array_equal(kept[s].float().cpu().numpy(), h[at + n - 1].astype(np.float32))
        at += n
    assert np.array_equal(state[7].cpu().numpy(), S0[7].astype(np.float32))         # a slot outside the step is untouched
    assert np.array_equal(kept[7].float().cpu().numpy(), kept0[7].astype(np.float32))


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
    return [random_tokens(name, n, i) for i, n in enumerate(LENGTHS[name])]


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
    assert_rows_close(np.concatenate(got), np.concatenate(ref), dtype, f"nekotar {name}/{dtype} whole")


@pytest.mark.parametrize("name,dtype", CASES)
def test_the_streams_after_every_layer(engines, name, dtype):
    """The sum of the streams behind every layer: where a difference would begin; with the next layer's norm in the
    layer's last launch, and with every layer reading the streams by itself."""
    from gguf2bin_b200.engine import StepEntry
    eng, toks = engines(name, dtype), requests_of(name)[0][:40]
    ref, got = [], []
    NP.forward(CONFIGS[name], weights(name), toks, layers_out=ref)
    model, graphs = eng.model, eng.step_graphs
    cls = type(model.blocks[0])
    forward = cls.forward

    def watched(self, x, ctx, view):
        if apart:
            ctx.next_block = None
        forward(self, x, ctx, view)
        got.append(x.view(x.shape[0], -1, model.hidden).sum(1)[:len(toks)].cpu().numpy())
    try:
        eng.step_graphs, cls.forward = False, watched
        for apart in (False, True):
            got.clear()
            seq = eng.open_sequence()
            eng.step([StepEntry(seq, toks, [0])])
            eng.close_sequence(seq)
            assert len(got) == len(ref)
            for i, (a, b) in enumerate(zip(got, ref)):
                assert np.abs(a - b).max() <= (3e-5 if dtype == "float32" else 0.06) * np.abs(b).max(), f"layer {i}"
    finally:
        cls.forward, eng.step_graphs = forward, graphs


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
        assert_rows_close(got, ref, dtype, f"nekotar {name}/{dtype} {what}")
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
    assert_rows_close(np.concatenate(every), np.concatenate(refs), dtype, f"nekotar {name}/{dtype} batches")
    assert eng.cache.table.pages.n_held == 0 and eng.cache.table.slots.n_held == 0


@pytest.mark.parametrize("name,dtype", CASES)
def test_one_decodes_while_another_brings_a_prompt(engines, name, dtype):
    """Steps in which one sequence goes on by one token, another by two, and a third begins."""
    from gguf2bin_b200.engine import StepEntry
    eng, reqs = engines(name, dtype), [t for t in requests_of(name) if len(t) > 12][:3]
    seqs, done, got = [eng.open_sequence() for _ in reqs], [0] * 3, [[], [], []]
    plan = [(5, 0, 0), (1, 3, 0), (1, 2, 0), (1, 2, 11), (2, 1, 1), (1, 1, 1), (100, 200, 100)]
    for sizes in plan:
        part = [(j, min(n, len(reqs[j]) - done[j])) for j, n in enumerate(sizes)]
        part = [(j, n) for j, n in part if n > 0]
        out = eng.step([StepEntry(seqs[j], reqs[j][done[j]:done[j] + n], range(n)) for j, n in part]).cpu().numpy()
        o = 0
        for j, n in part:
            got[j].append(out[o:o + n])
            done[j] += n
            o += n
    for j in range(3):
        eng.close_sequence(seqs[j])
    assert_rows_close(np.concatenate([r for g in got for r in g]),
                      np.concatenate([plain_logits(name, reqs[j])[:done[j]] for j in range(3)]), dtype, f"nekotar {name} mixed")


@pytest.mark.parametrize("name,dtype", [("s", "float32"), ("t", "bfloat16"), ("u", "bfloat16"), ("u", "float32")])
def test_long_decoding(engines, name, dtype):
    """A short prompt, then 120 tokens one by one: the window passes over decoded tokens, pages begin; beside a second
    sequence that started elsewhere."""
    from gguf2bin_b200.engine import StepEntry
    eng = engines(name, dtype)
    a, b = random_tokens(name, 150, 70), random_tokens(name, 181, 71)
    sa, sb = eng.open_sequence(), eng.open_sequence()
    out = eng.step([StepEntry(sa, a[:30], range(30)), StepEntry(sb, b[:61], range(61))]).cpu().numpy()
    ga, gb = [out[:30]], [out[30:]]
    for t in range(120):
        out = eng.step([StepEntry(sa, [a[30 + t]], [0]), StepEntry(sb, [b[61 + t]], [0])]).cpu().numpy()
        ga.append(out[:1])
        gb.append(out[1:])
    eng.close_sequence(sa)
    eng.close_sequence(sb)
    assert_rows_close(np.concatenate(ga), plain_logits(name, a), dtype, f"nekotar {name}/{dtype} long decoding a")
    assert_rows_close(np.concatenate(gb), plain_logits(name, b), dtype, f"nekotar {name}/{dtype} long decoding b")


@pytest.mark.parametrize("streams,batch", [(2, 8), (1, 1), (4, 20)])
def test_replayed_steps_are_the_plain_steps_at_real_widths(streams, batch):
    """Layers wide enough for the products that stream their weights, split K over a cluster or take stacked inputs in
    tiles: steps replayed from graphs, where launches overlap most, give the bits of steps launched one by one."""
    from gguf2bin_b200.engine import Engine, Model, StepEntry
    W, V = 2048, 700
    layers = [dict(type="wkv", mixer=dict(heads=32, dim=64), mlp=dict(kind="dense", ff=9216)),
              dict(type="latent_attention", mixer=latent(16, 128, 128, 104, 24, 0.08), mlp=None),
              dict(type="attention", mixer=windowed(16, 4, 128, 128, 128, 0.09, 90, 5), mlp=dict(kind="dense", ff=6144))]
    model = Model.random(dict(architecture="Nekotar", width=W, vocab=V, streams=streams, residual_mult=0.8, norm=dict(eps=1e-5),
                              layers=layers), 3)
    rng = np.random.default_rng(streams)
    prompts = [[rng.integers(0, V, 300).tolist() for _ in range(batch)] for _ in range(4)]     # the same shape, four times
    nxt = rng.integers(0, V, (6, batch)).tolist()
    runs = []
    for graphs in (True, False):
        eng, rows = Engine(model, max_tokens=64 * 6 * batch, step_graphs=graphs), []
        for p in prompts:
            seqs = [eng.open_sequence() for _ in p]
            rows.append(eng.step([StepEntry(s, t, [0, 299]) for s, t in zip(seqs, p)]).cpu())
            for toks in nxt:
                rows.append(eng.step([StepEntry(s, [t], [0]) for s, t in zip(seqs, toks)]).cpu())
            for s in seqs:
                eng.close_sequence(s)
        assert (eng.graph_captures > 0) == graphs
        runs.append(rows)
    for i, (a, b) in enumerate(zip(*runs)):
        assert torch.isfinite(a).all() and torch.equal(a, b), f"step {i}: {(a - b).abs().max()}"


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
    prompts = [random_tokens(name, n, 90 + i) for i, n in enumerate([9, 1, 66, 30])]
    for _ in range(2):                         # the second call finds slots, pages and graphs of the first
        outs = llm.generate(prompts, n=30, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0)
        for p, o in zip(prompts, outs):
            toks = list(p) + list(o.tokens)
            rows = plain_logits(name, toks)[len(p) - 1:-1]       # a prompt's rows do not depend on what follows
            for row, t in zip(rows, o.tokens):
                assert row[t] >= row.max() - 2e-5 * max(1.0, np.abs(row).max())
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
    assert out.returncode == 0 and "Nekotar" in out.stdout + out.stderr, out.stderr[-2000:]
    prompt = random_tokens("s", 7, 40)
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
    W = NP.read_safetensors(made / "model.safetensors")
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
    ref = NP.forward(CONFIGS["u"], W, toks)
    assert_close(got, ref[[0, 5, 0, 7, 8]], "float32", "nekotar trace replay")


def test_weights_made_on_the_device_are_those_of_a_written_folder(tmp_path):
    """Among them the streams' mixing matrices, which lie around the identity."""
    from gguf2bin_b200.weights import write_random_model
    from gguf2bin_b200.weights.random_init import random_tensors_on_device
    from gguf2bin_b200.config import model_spec_from_dict
    from gguf2bin_b200.engine.model import expected_tensors
    exp = expected_tensors(model_spec_from_dict(CONFIGS["s"]))
    write_random_model(tmp_path / "m", CONFIGS["s"], 4, "bfloat16", on_device=False)
    W = NP.read_safetensors(tmp_path / "m" / "model.safetensors")
    made = random_tensors_on_device(exp, 4, torch.bfloat16, torch.bfloat16, DEV)
    assert set(W) == set(made) and all(np.array_equal(W[k], made[k].float().cpu().numpy()) for k in W)
