"""``latent_attention``: causal attention over cached low-rank latents, without positions or with rotated entries
beside the latent.

Per token the mixer projects its input u to queries q (``n_heads`` x ``qk_dim``) and to a latent
c = rmsnorm(W_down u) * w of ``kv_rank`` numbers, which is ALL it caches.  Keys and values are
projections of the latents, k_j = U_k c_j and v_j = U_v c_j per head.  Since
q . (U_k c_j) = (U_k^T q) . c_j and sum_j p_j U_v c_j = U_v (sum_j p_j c_j), a step never builds
keys or values: it takes U_k into the query (``kv_rank`` numbers per head), attends over the
latents themselves, which then are keys and values at once for every head (one kv head, one
panel per page: ``KVNeed(planes=1)``), and applies U_v to each head's weighted sum of latents.
Options, each a parameter of the spec: ``sink`` (a learned logit per head that joins the
softmax's denominator and nothing else), ``out_gate`` (each head's output times the sigmoid of
a linear function of u), ``shared_kv`` (no down-projection: the layer attends over the latents
that the schedule entry's ``cache_of`` layer stored), ``scale``, ``q_rank`` (queries come from a latent of their own
of that many numbers, c_q = rmsnorm(W_dq u) * w_q, q = W_uq c_q; names ``q_down``, ``q_down_norm``, and ``q`` for W_uq),
``window`` (a token sees the last ``window`` positions, its own among them), ``pad_rank`` (bfloat16: latents of a rank
below a size that the tensor-core attention kernels take lie in rows of that size, zero-filled, as do the
up-projections' columns; scores and sums are what they were), ``rot_dim`` with ``position`` (each head of q has
``rot_dim`` more entries behind its ``qk_dim`` ones, the down-projection as many more rows; those entries are turned by
the token's position, are not normed, and the key's are one part for all heads: score = q . k + q_rot . k_rot.  A
cached row is the latent with the rotated key behind it, a query in latent coordinates its rotated part behind it, so
that attention over the rows is still one panel for keys and values; U_v has zeros in those columns),
``out_gate`` = "sigmoid" (an element of the gate for every element of the concatenated heads instead of one per head).

Scores, softmax and the latent's norm are 32-bit; products accumulate in 32-bit.

Where a head's rank is not much more than its key (value) size, or the matrices are small,
bfloat16 compute multiplies U_k into the query matrix (U_v into the output matrix) once, when
the weights are bound (``folds``): the per-head products then cost nothing at run time, at the price of a query
(output) product that is rank / size times as large, and of one more rounding of the matrix to
bfloat16.  The output gate is a number per head, so it commutes with U_v and is applied to
the weighted latents, by the attention kernel itself; the queries, which then come out of the
input product in latent coordinates, are read by the attention in place.  The 32-bit path keeps the formula's order.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.storage import KVNeed, KVView
from ..config.specs import ConfigError, PartSpec
from ..weights.loader import Expected
from .registry import position_class, register_mixer

HEAD_PRODUCT_ROWS = 64       # steps of more rows multiply per head on the tensor cores (bfloat16)
FOLD_UP_TO = 1.5             # rank / head size up to which an up-projection is always multiplied into its neighbour
FOLD_SMALL_UP_TO = 4.0       # ... and up to which it is while the matrix grows by no more than FOLD_SMALL_BYTES
FOLD_SMALL_BYTES = 4 << 20


def folds(rank: int, size: int, heads: int, width: int) -> bool:
    """Whether a head's up-projection [size, rank] is multiplied into the [heads * size, width] matrix
    beside it, which then has heads * rank rows.  Always while that costs at most half as much again;
    for small matrices up to four times as much: a decode step reads the extra bytes in less time than
    the launch of the per-head product takes, and a prompt's per-head products are one launch a head."""
    if rank <= FOLD_UP_TO * size:
        return True
    extra = heads * (rank - size) * width * 2
    return rank <= FOLD_SMALL_UP_TO * size and extra <= FOLD_SMALL_BYTES


class LatentAttention:
    graph_safe = True          # its step only launches kernels: may be replayed from a CUDA graph

    def __init__(self, spec: PartSpec, hidden_size: int, dtype: torch.dtype, device):
        self.nh, self.dk, self.dv = int(spec["n_heads"]), int(spec["qk_dim"]), int(spec["v_dim"])
        self.rank = int(spec["kv_rank"])
        self.hidden = int(hidden_size)
        self.scale = float(spec["scale"])
        self.eps = float(spec["eps"])
        self.shared_kv = bool(spec.get("shared_kv") or False)
        self.has_sink = bool(spec.get("sink") or False)
        gate = spec.get("out_gate")
        if gate not in (None, False, True, "sigmoid"):
            raise ConfigError("latent_attention: out_gate is true (a number a head), 'sigmoid' (one an element) or absent")
        self.has_gate, self.wide_gate = bool(gate), gate == "sigmoid"
        self.rot = int(spec.get("rot_dim") or 0)
        self.position = None
        if self.rot:
            pos = spec["position"]
            self.position = position_class(pos)(pos, self.rot, device)
            if self.rot < 0 or not hasattr(self.position, "table_rotation") or self.position.table_rotation()[0] is None \
                    or self.position.table_rotation()[1] != self.rot:
                raise ConfigError("latent_attention: rot_dim goes with a position part that turns all of it by a table")
        if min(self.nh, self.dk, self.dv, self.rank) <= 0:
            raise ConfigError("latent_attention: heads, sizes and rank must be positive")
        if self.rank + self.rot > 512:
            raise ConfigError(f"latent_attention: kv_rank {self.rank} (+ {self.rot}) is more than the attention kernels' 512")
        self.q_rank = int(spec.get("q_rank") or 0)
        self.window = int(spec.get("window") or 0)
        if spec.get("pad_rank") and not self.q_rank and not self.rot:
            raise ConfigError("latent_attention: padded ranks go with a query latent or rotated entries")
        if self.rot and self.q_rank:
            raise ConfigError("latent_attention: rotated entries do not go with a query latent")
        if self.q_rank < 0 or self.window < 0 or (self.q_rank and (self.shared_kv or self.has_gate)):
            raise ConfigError("latent_attention: q_rank and window are positive or absent; a query latent goes with "
                              "neither shared latents nor a gate")
        self.dtype, self.device = dtype, device
        self.names = dict(spec["names"])
        self.own_rank = self.rank                 # the latent's entries; ``rank``: a row of the pages
        self.rank += self.rot
        if spec.get("pad_rank") and dtype == torch.bfloat16:
            self.rank = kernels.padded_head_size(self.rank)
        # columns of the fused input product: queries (or their latent), then the latent (unless shared), then the gates
        self.n_q = self.q_rank or self.nh * (self.dk + self.rot)
        self.n_c = 0 if self.shared_kv else self.own_rank + self.rot
        self.n_g = 0 if not self.has_gate else self.nh * (self.dv if self.wide_gate else 1)
        self.w_in = self.w_o = self.w_uk = self.w_uv = self.c_norm = self.sink = self.w_uq = self.q_norm = None
        self.fold_k = self.fold_v = False

    # ---- weights -------------------------------------------------------------
    @classmethod
    def expected(cls, spec: PartSpec, hidden_size: int) -> dict:
        n = dict(spec["names"])
        nh, dk, dv, r = spec["n_heads"], spec["qk_dim"], spec["v_dim"], spec["kv_rank"]
        qr, rot = spec.get("q_rank"), int(spec.get("rot_dim") or 0)
        out = {n["q"]: Expected((nh * (dk + rot), qr or hidden_size)), n["up_k"]: Expected((nh * dk, r)),
               n["up_v"]: Expected((nh * dv, r)), n["o"]: Expected((hidden_size, nh * dv))}
        if qr:
            out[n["q_down"]] = Expected((qr, hidden_size))
            out[n["q_down_norm"]] = Expected((qr,), init="scale")
        if not (spec.get("shared_kv") or False):
            out[n["down"]] = Expected((r + rot, hidden_size))
            out[n["down_norm"]] = Expected((r,), init="scale")
        if spec.get("sink"):
            out[n["sink"]] = Expected((nh,))
        if spec.get("out_gate"):
            out[n["gate"]] = Expected((nh * dv if spec["out_gate"] == "sigmoid" else nh, hidden_size))
        return out

    def bind(self, tensors: dict) -> None:
        n = self.names
        w_q, w_o = tensors[n["q"]], tensors[n["o"]]
        up_k, up_v = tensors[n["up_k"]], tensors[n["up_v"]]
        if self.rank != self.own_rank:             # columns of zeros behind the rank
            up_k, up_v = (torch.nn.functional.pad(t, (0, self.rank - self.own_rank)) for t in (up_k, up_v))
        q_in = self.q_rank or self.hidden          # what the queries are a product of
        folding = self.dtype == torch.bfloat16 and w_q.dtype == torch.bfloat16 and w_o.dtype == torch.bfloat16
        self.fold_k = folding and folds(self.rank, self.dk, self.nh, q_in)
        # (a gate per element does not commute with U_v)
        self.fold_v = folding and not self.wide_gate and folds(self.rank, self.dv, self.nh, self.hidden)
        w_rot = None
        if self.rot:                               # rows head by head [qk_dim, rot_dim]: the two kinds apart
            w_q = w_q.view(self.nh, self.dk + self.rot, q_in)
            w_q, w_rot = w_q[:, :self.dk].reshape(self.nh * self.dk, q_in), w_q[:, self.dk:]
        if self.fold_k:
            # W_q'[h] = U_k[h]^T W_q[h]: [rank, qk_dim] x [qk_dim, width] per head; the queries then
            # come out of the input product in latent coordinates, `rank` numbers per head
            uk = up_k.double().view(self.nh, self.dk, self.rank)
            wq = w_q.double().view(self.nh, self.dk, q_in)
            w_q = torch.einsum("hdr,hdw->hrw", uk, wq)
            if self.rot:                           # a head's rotated entries lie behind its latent coordinates
                w_q[:, self.own_rank:self.own_rank + self.rot] = w_rot.double()
            w_q = w_q.reshape(self.nh * self.rank, q_in).to(torch.bfloat16).contiguous()
            if not self.q_rank:
                self.n_q = self.nh * self.rank
        elif self.rot:                             # all heads' unrotated rows, then all heads' rotated ones
            w_q = torch.cat([w_q, w_rot.reshape(self.nh * self.rot, q_in)], dim=0)
        parts = [w_q]
        if self.q_rank:
            self.w_uq = w_q.contiguous()
            self.q_norm = tensors[n["q_down_norm"]].to(torch.float32).contiguous()
            parts = [tensors[n["q_down"]]]
        if not self.shared_kv:
            parts.append(tensors[n["down"]])
            self.c_norm = tensors[n["down_norm"]].to(torch.float32).contiguous()
        if self.has_gate:
            parts.append(tensors[n["gate"]])
        common = torch.float32 if any(p.dtype == torch.float32 for p in parts) else parts[0].dtype
        rows = sum(p.shape[0] for p in parts)
        pad = -rows % 8                         # rows of the product's output start on 16 bytes
        if pad:
            parts.append(torch.zeros((pad, self.hidden), dtype=common, device=parts[0].device))
        self.w_in = torch.cat([p.to(common) for p in parts], dim=0).contiguous()
        if self.fold_v:
            # W_o'[:, h] = W_o[:, h] U_v[h]: [width, v_dim] x [v_dim, rank] per head
            uv = up_v.double().view(self.nh, self.dv, self.rank)
            wo = w_o.double().view(self.hidden, self.nh, self.dv)
            self.w_o = torch.einsum("whv,hvr->whr", wo, uv).reshape(self.hidden, self.nh * self.rank) \
                .to(torch.bfloat16).contiguous()
        else:
            self.w_o = w_o.contiguous()
            self.w_uv = up_v.to(self.dtype).contiguous()
        if not self.fold_k:
            self.w_uk = up_k.to(self.dtype).contiguous()
        if self.has_sink:
            self.sink = tensors[n["sink"]].to(torch.float32).contiguous()

    def weights(self):
        return [t for t in (self.w_in, self.w_o, self.w_uk, self.w_uv, self.c_norm, self.sink, self.w_uq, self.q_norm)
                if t is not None]

    def notices(self) -> list:
        from ..cache.storage import PAGE_SIZE
        return (kernels.product_notices("latent attention input", self.w_in, self.dtype)
                + kernels.product_notices("latent attention queries", self.w_uq, self.dtype)
                + kernels.product_notices("latent attention output", self.w_o, self.dtype)
                + kernels.attention_notices("latent attention", self.rank, PAGE_SIZE, self.dtype))

    # ---- cache ---------------------------------------------------------------
    def cache_need(self):
        return None if self.shared_kv else KVNeed(1, self.rank, self.window, planes=1)

    # ---- step ----------------------------------------------------------------
    def forward(self, u: torch.Tensor, ctx, view: KVView, residual32: torch.Tensor) -> None:
        self._run(u, ctx, view, residual32, True, None)

    def forward_store(self, u: torch.Tensor, ctx, view: KVView, out32: torch.Tensor) -> None:
        """Stores the mixer's result instead of adding it."""
        self._run(u, ctx, view, out32, False, None)

    def forward_into(self, u: torch.Tensor, ctx, view: KVView, out32: torch.Tensor, keep=None) -> None:
        """Stores the mixer's result instead of adding it.  ``keep`` = (rows, ring, taps): the
        block's wish to have the last rows of every sequence written to its ring, which rides
        on the launch that writes the latents."""
        self._run(u, ctx, view, out32, False, keep)

    def _per_head(self, x, w, out, expand: bool, gate) -> None:
        """out[:, h] = w_h^T x[:, h] (absorb) or w_h x[:, h] (expand, then the gate)."""
        T = x.shape[0]
        n, r = w.shape[0] // self.nh, w.shape[1]
        fast = (self.dtype == torch.bfloat16 and T > HEAD_PRODUCT_ROWS and n % 8 == 0 and r % 8 == 0
                and x.stride(0) % 8 == 0 and out.stride(0) % 8 == 0)
        if not fast:
            kernels.head_product(x, w, out, self.nh, expand, gate)
            return
        if kernels.head_expand_tiles(x, w if expand else self._uk_t.view(self.nh * r, n), out, self.nh, gate):
            return
        for h in range(self.nh):
            wh = w[h * n:(h + 1) * n]
            if expand:
                kernels.linear(x[:, h * r:(h + 1) * r], wh, out[:, h * n:(h + 1) * n])
            else:
                kernels.linear(x[:, h * n:(h + 1) * n], self._uk_t[h], out[:, h * r:(h + 1) * r])
        if expand and gate is not None:
            if self.wide_gate:
                kernels.gate_mul(out, n, gate, self.nh, n, 1.0, out)       # in place: an element is read and written by one thread
            else:
                kernels.head_gate(out, gate, self.nh)

    @property
    def _uk_t(self):
        """U_k of each head transposed ([rank, qk_dim] per head), for the tensor-core products
        that want the contraction index innermost; made when a long step first asks."""
        t = getattr(self, "_uk_t_cache", None)
        if t is None:
            t = self._uk_t_cache = self.w_uk.view(self.nh, self.dk, self.rank).transpose(1, 2).contiguous()
        return t

    def _run(self, u, ctx, view: KVView, out32, accumulate: bool, keep) -> None:
        T = u.shape[0]
        ws = ctx.workspace
        if view is None or view.planes != 1:
            raise kernels.KernelError("latent_attention: needs latent pages (one panel per page)")
        proj = ws.buffer("latent.in", (T, self.w_in.shape[0]), self.dtype)
        kernels.linear(u, self.w_in, proj)
        q = proj[:, :self.n_q]
        d = proj[:, self.n_q:self.n_q + self.n_c] if self.n_c else None
        gate = proj[:, self.n_q + self.n_c:self.n_q + self.n_c + self.n_g] if self.n_g else None
        rows, ring, taps = keep if keep is not None else (None, None, 0)
        if self.q_rank:
            if ring is not None:
                kernels.latent_keep(None, None, 0.0, None, rows, ring, taps, ctx)
            cq = ws.buffer("latent.cq", (T, self.q_rank), self.dtype)
            kernels.latent_pair(d, self.rank, self.c_norm, view.pages, q, self.q_norm, cq, self.eps, ctx)
            q = ws.buffer("latent.uq", (T, self.w_uq.shape[0]), self.dtype)
            kernels.linear(cq, self.w_uq, q)
        elif self.rot:
            if ring is not None:
                kernels.latent_keep(None, None, 0.0, None, rows, ring, taps, ctx)
        elif d is not None or ring is not None:
            kernels.latent_keep(d, self.c_norm, self.eps, view.pages if d is not None else None,
                                rows, ring, taps, ctx)
        if self.fold_k:
            qa = q                          # columns of the product's output: the attention reads them in place
        else:
            qa = ws.buffer("latent.q", (T, self.nh * self.rank), self.dtype)
            self._per_head(q[:, :self.nh * self.dk], self.w_uk, qa, False, None)
        if self.rot:
            inv_freq, _, interleaved = self.position.table_rotation()
            at = self.own_rank                     # where a head's rotated entries begin in latent coordinates
            src, step = (qa[:, at:], self.rank) if self.fold_k else (q[:, self.nh * self.dk:], self.rot)
            kernels.latent_rope(d, self.own_rank, self.rank, self.c_norm, self.eps, view.pages, src, step, qa[:, at:], self.rank,
                                self.nh, self.rot, ctx.rope_table(inv_freq), interleaved, ctx)
        mix = ws.buffer("latent.mix", (T, self.nh * self.rank), self.dtype)
        # with U_v folded into the output matrix the heads' gate is the attention's last step
        kernels.attention(qa, mix, view.pages, ctx, self.nh, 1, self.rank, view.page_size, self.window, self.scale,
                          sink=self.sink, planes=1, gate=gate if self.fold_v else None)
        if self.fold_v:
            o = mix
        else:
            o = ws.buffer("latent.o", (T, self.nh * self.dv), self.dtype)
            self._per_head(mix, self.w_uv, o, True, gate)
        kernels.linear(o, self.w_o, out32, accumulate=accumulate)


register_mixer("latent_attention", LatentAttention)
