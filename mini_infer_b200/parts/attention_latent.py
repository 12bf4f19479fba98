"""Attention through a latent: per token the cache holds ONE row that all heads share.

With ``h`` the layer's input, ``c_q = norm(W_dq h)`` and ``q_h = W_uq,h c_q = [q_h^plain | q_h^rot]`` per head (or,
without a latent for the queries, ``q_h = W_q,h h``);
``[c | k^rot] = W_dkv h`` with ``c`` brought to unit root mean square (times a gain) and ``k^rot`` rotated by
position; key and value of head ``h`` are ``W_uk,h c`` and ``W_uv,h c``;
``score = (q_h^plain . W_uk,h c + rot(q_h^rot) . rot(k^rot)) * scale``; softmax over a window of keys; the
heads' outputs times ``sigmoid(W_g h)`` (or as they are); then ``W_o``.

Only ``[c | rot(k^rot)]`` is cached (``LatentNeed``).  Two forms of the attention follow from that:

*folded* (decode steps and short portions): ``q_h' = W_uk,h^T q_h^plain`` (so ``q_h^plain . W_uk,h c = q_h' . c``), and
the value matrices after the weighted sum (``sum_j p_j W_uv,h c_j = W_uv,h sum_j p_j c_j``): the attention itself runs
over one shared key/value head whose keys are the cached rows and whose values are their first ``kv_rank`` numbers.
The float32 path takes this form for every step (``ops.functional.attention_mix``, or ``attention_shared_plain`` for
sizes that it does not take).  The bfloat16 path takes ``attention_shared_tc``, whose tensor-core tiles are rows of
(query, head) pairs; steps of few tokens fold and unfold in kernels of their own (``latent_fold``, ``latent_values``)
and split the keys; portions below the threshold of the unfolded form take the tcgen05 kernel with (query, head) rows
(``prefill_attention_tc_shared``) where the sizes allow.

*unfolded* (prompt portions of the bfloat16 path): the latents of the whole context are gathered from their pages, one
library product forms the keys and values of all heads, and the tcgen05 kernel runs over them
(``prefill_attention_tc_unfolded``): ``d + r + e`` products per pair of query and key instead of ``2 c + r``.

A step that brings prompt portions beside decoding requests (which stand first) takes both.  A layer may read the rows
another layer caches (``shares_cache``): it then has no ``W_dkv`` of its own.

The rotation pairs neighbouring dimensions (``2i`` with ``2i + 1``).
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config.registry import part_class, register_part
from ..config.spec import PartSpec
from ..ops import functional as F
from .base import CacheBinding, LatentNeed, Mixer, Runtime, StepContext, TensorDecl, linear
from .tuning import TUNING


class LatentAttention(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``head_dim`` (unrotated query/key size per head), ``rot_dim``
    (rotated size), ``value_dim``, ``kv_rank``, ``q_rank`` (0: queries straight from the input), ``window`` (0 = all
    keys), ``scale``, ``eps`` (of the latent norms), ``position`` (a ``PartSpec`` of category ``position`` whose table
    has ``rot_dim / 2`` frequencies; its ``magnitude`` stretches queries' and keys' rotated parts), ``output_gate``
    (default True), ``shares_cache`` (reads another layer's cached rows; no ``dkv`` tensors).

    Tensors below the prefix: ``dq [q_rank, hidden]``, ``dq.norm [q_rank]``, ``uq [heads*(head_dim+rot_dim),
    q_rank]`` (or, without ``q_rank``, ``q [heads*(head_dim+rot_dim), hidden]``), ``dkv [kv_rank+rot_dim, hidden]``, ``dkv.norm [kv_rank]``, ``uk [heads*head_dim, kv_rank]``,
    ``uv [heads*value_dim, kv_rank]``, ``g [heads*value_dim, hidden]``, ``o [hidden, heads*value_dim]``."""

    graph_safe = True
    kernel_files = ("attention_latent.cu", "attention_mix.cu", "attention_prefill_tc.cu", "attention_shared.cu",
                    "dense_f32.cu", "elementwise.cu")
    launches_follow_context = True      # a captured prompt portion is launched for a bucket of context lengths

    def __init__(self, params, prefix):
        super().__init__(params, prefix)
        p = self.params
        self.W = int(p["hidden_size"])
        self.nh = int(p["num_heads"])
        self.d = int(p["head_dim"])
        self.r = int(p["rot_dim"])
        self.e = int(p["value_dim"])
        self.c = int(p["kv_rank"])
        self.qr = int(p.get("q_rank", 0))
        self.gated = bool(p.get("output_gate", True))
        self.window = int(p.get("window", 0))
        self.scale = float(p.get("scale", (self.d + self.r) ** -0.5))
        self.eps = float(p["eps"])
        self.shares_cache = bool(p.get("shares_cache", False))
        pos: PartSpec = p.get("position") or PartSpec("none")
        self.position = part_class("position", pos.kind)(pos.params, prefix)
        if self.r % 2:
            raise ValueError(f"latent attention: the rotated part ({self.r}) must be even")

    def tensor_decls(self) -> List[TensorDecl]:
        p = self.prefix
        if self.qr:
            out = [TensorDecl(p + "dq", (self.qr, self.W)), TensorDecl(p + "dq.norm", (self.qr,), "norm"),
                   TensorDecl(p + "uq", (self.nh * (self.d + self.r), self.qr))]
        else:
            out = [TensorDecl(p + "q", (self.nh * (self.d + self.r), self.W))]
        if not self.shares_cache:
            out += [TensorDecl(p + "dkv", (self.c + self.r, self.W)), TensorDecl(p + "dkv.norm", (self.c,), "norm")]
        out += [TensorDecl(p + "uk", (self.nh * self.d, self.c)), TensorDecl(p + "uv", (self.nh * self.e, self.c)),
                TensorDecl(p + "o", (self.W, self.nh * self.e))]
        if self.gated:
            out.append(TensorDecl(p + "g", (self.nh * self.e, self.W)))
        return out

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        m, dev, p = rt.precision.matrix, rt.device, self.prefix
        f32 = lambda t: t.to(device=dev, dtype=torch.float32).contiguous()      # norms are float arithmetic
        # one product of the input: the gate, the latent (unless the rows come from another layer) and the queries
        # (unless they have a latent of their own)
        rows, at = [], 0
        self.g_col = self.kv_col = self.q_col = 0
        self.w_dq = self.dkv_gain = None
        if self.gated:
            rows.append(m(tensors[p + "g"], dev))
            at = rows[-1].shape[0]
        if not self.shares_cache:
            self.kv_col = at
            rows.append(m(tensors[p + "dkv"], dev))
            self.dkv_gain = f32(tensors[p + "dkv.norm"])
            at += rows[-1].shape[0]
        if self.qr:
            self.w_dq = m(tensors[p + "dq"], dev)
            self.dq_gain = f32(tensors[p + "dq.norm"])
            self.w_uq = m(tensors[p + "uq"], dev)
        else:
            self.q_col = at
            rows.append(m(tensors[p + "q"], dev))
        self.w_in = torch.cat(rows, dim=0).contiguous() if rows else None
        # the heads' key matrices [H, d, c], then their value matrices [H, e, c], as rows of one matrix
        self.w_ukv = torch.cat([m(tensors[p + "uk"], dev), m(tensors[p + "uv"], dev)], dim=0).contiguous()
        self.w_uk = self.w_ukv[:self.nh * self.d].view(self.nh, self.d, self.c)
        self.w_uv = self.w_ukv[self.nh * self.d:].view(self.nh, self.e, self.c)
        if rt.act == torch.float32:
            self.w_uk_fold = self.w_uk.transpose(1, 2).contiguous()  # [H, c, d]: q' = w . q_plain
        self.w_o = m(tensors[p + "o"], dev)
        self.inv_freq = self.position.table(dev)
        if self.r and (self.inv_freq is None or self.inv_freq.numel() != self.r // 2):
            raise ValueError(f"latent attention: a rotated part of {self.r} needs {self.r // 2} frequencies")
        dk = self.c + self.r
        f32 = rt.act == torch.float32
        self._mix = f32 and F.attention_mix_supported(self.nh, 1, dk, self.c, rt.act)
        if not self._mix and not F.attention_shared_plain_supported(dk, self.c):
            raise ValueError(f"latent attention: rows of {dk} with values of {self.c} are more than one block of the "
                             f"kernel holds")
        self._tensor_cores = not f32 and F.attention_shared_tc_supported(dk, self.c)
        self._small = self._tensor_cores and F.latent_fold_takes(self.d, self.r, self.c)
        self._small_max = min(TUNING.latent_small_max_tokens, F.latent_fold_max_tokens()) if self._small else 0
        self._unfold = (not f32 and self.c % 8 == 0
                        and F.prefill_attention_tc_unfolded_supported(self.d, self.r, self.e))
        # prompt portions on the tensor-memory attention: its blocks want whole SMs (a block arrangement that
        # runs another part beside this one asks)
        self.large_steps_fill_the_device = not f32

    def prefetch_first(self, ctx: StepContext, cache: Optional[CacheBinding]) -> None:
        for w in (self.w_dq, self.w_in):
            if w is not None:
                F.l2_prefetch(w)

    def cache_need(self):
        return LatentNeed(self.c, self.r, self.window)

    def _span(self, max_kv_len: int) -> int:
        return min(self.window, max_kv_len) if self.window > 0 else max_kv_len

    def _context_rows(self, ctx: StepContext, first: int) -> int:
        """Rows that the whole contexts of the requests from ``first`` on take (of one request: the longest context
        this step is launched for, which a captured pass shares with the steps it is replayed for)."""
        if ctx.num_requests - first == 1:
            return ctx.max_kv_len
        return sum(ctx.host_kv_len[first:])

    def _first_unfolded(self, ctx: StepContext) -> int:
        """The first request whose portion takes the unfolded form; the step's number of requests: none does."""
        none = ctx.num_requests
        if not self._unfold or ctx.all_decode:
            return none
        lead = ctx.num_leading_decodes
        if not self._tensor_cores:
            lead = 0                    # no form of the tensor cores for the decoding requests alone
        if ctx.num_tokens - lead < TUNING.latent_unfold_min_tokens:
            return none
        rows = self._context_rows(ctx, lead)
        if self.window > 0 and rows > 4 * (ctx.num_tokens + self.window * (none - lead)):
            return none                 # most of those rows lie below every window
        size = rows * self.nh * (self.d + self.e) * 2
        return lead if size <= TUNING.latent_unfold_max_mbytes << 20 else none

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheBinding) -> torch.Tensor:
        view = ctx.kv_groups[cache.group]
        rows = view.tensors["latent"][cache.layer_slot]              # [pages, 1, page_size, c + r]
        # gate, this token's cached row, queries
        y = linear(x, self.w_in, torch.float32) if self.w_in is not None else None
        q = y
        if self.qr:
            cq = F.add_rmsnorm(linear(x, self.w_dq, torch.float32), None, self.dq_gain, self.eps, self.rt.act)
            q = linear(cq, self.w_uq, torch.float32)
        store = None
        if not self.shares_cache:
            if not cache.writes:
                raise RuntimeError("latent attention: a layer with a latent projection of its own must own its cache")
            store = (y, self.kv_col, self.dkv_gain, self.eps, view.slot_mapping, rows)
        if self.rt.act == torch.float32:
            v = self._forward_f32(q, y, store, ctx, view, rows)
        else:
            v = self._forward_bf16(q, y, store, ctx, view, rows)
        return linear(v, self.w_o, torch.float32)

    def _forward_f32(self, q, y, store, ctx: StepContext, view, rows) -> torch.Tensor:
        T, H, d, r, e, c = ctx.num_tokens, self.nh, self.d, self.r, self.e, self.c
        q_full, _ = F.latent_query(q, ctx.positions, self.inv_freq, H, d, r, c, torch.float32, False, col0=self.q_col,
                                   magnitude=self.position.magnitude, store=store)
        F.dense_f32_heads(q, self.w_uk_fold, out=q_full, x_col=self.q_col, x_head_stride=d + r, out_head_stride=c + r)
        # one shared key/value head: keys are the cached rows, values their first c numbers
        if self._mix:
            a = F.attention_mix(q_full, rows, rows, None, view.block_table, ctx.q_start, ctx.kv_len, ctx.max_q_len,
                                self.window, self.scale, 0.0, value_dim=c)
        else:
            a = F.attention_shared_plain(q_full, rows, view.block_table, ctx.q_start, ctx.kv_len, ctx.max_q_len,
                                         self.window, self.scale, c)
        v = F.dense_f32_heads(a.view(T, H * c), self.w_uv)
        return F.sigmoid_gate(v, False, y, self.g_col, H, e) if self.gated else v

    def _forward_bf16(self, q, y, store, ctx: StepContext, view, rows) -> torch.Tensor:
        T, H, B = ctx.num_tokens, self.nh, ctx.num_requests
        first = self._first_unfolded(ctx)
        v = torch.empty(T, H * self.e, dtype=self.rt.act, device=q.device)
        if first == B:
            self._folded(q, y, store, ctx, view, rows, v, T, B, ctx.max_q_len, ctx.max_kv_len)
            return v
        if first:
            # the decoding requests in front (a token each); the rows of all tokens are cached by this launch
            if store is not None:
                F.latent_rows(ctx.positions, self.inv_freq, self.c, self.r, store=store,
                              magnitude=self.position.magnitude)
                store = None
            self._folded(q, y, None, ctx, view, rows, v, first, first, 1, ctx.leading_decodes_max_kv_len)
        self._unfolded(q, y, store, ctx, view, rows, v, first)
        return v

    def _folded(self, q, y, store, ctx: StepContext, view, rows, out, T, B, max_q_len, max_kv_len) -> None:
        """The first ``B`` requests, which bring the first ``T`` tokens of the step, into ``out[:T]``."""
        H, d, r, e, c = self.nh, self.d, self.r, self.e, self.c
        q, out, positions = q[:T], out[:T], ctx.positions[:T]
        gate = y[:T] if self.gated else None
        table, q_start, kv_len = view.block_table[:B], ctx.q_start[:B + 1], ctx.kv_len[:B]
        mag = self.position.magnitude
        if T <= self._small_max:
            q_full = F.latent_fold(q, self.q_col, H, d, self.w_uk, positions, self.inv_freq, r, mag, store)
            splits = F.attention_shared_splits(B, max_q_len, H, c + r, c, self._span(max_kv_len))
            part_o, part_ml = F.attention_shared_tc(q_full, rows, table, q_start, kv_len, max_q_len, self.window,
                                                    self.scale, c, splits, partial=True)
            F.latent_values(part_o, part_ml, self.w_uv, gate, self.g_col, out)
            return
        q_full, q_plain = F.latent_query(q, positions, self.inv_freq, H, d, r, c, self.rt.act, True, col0=self.q_col,
                                         magnitude=mag, store=store)
        # written head by head into its place before the rotated parts (rows H * (c + r) apart)
        torch.bmm(q_plain.transpose(0, 1), self.w_uk, out=q_full.transpose(0, 1)[:, :, :c])
        if max_q_len > 1 and F.prefill_attention_tc_shared_supported(H, c + r, c, view.page_size):
            # prompt portions (and what decodes beside them): the tensor-memory attention with (query, head)
            # pairs as the rows of a tile
            a = F.prefill_attention_tc_shared(q_full, rows, table, q_start, kv_len, max_q_len, self.window, self.scale, c)
        elif self._tensor_cores:
            splits = F.attention_shared_splits(B, max_q_len, H, c + r, c, self._span(max_kv_len))
            a = F.attention_shared_tc(q_full, rows, table, q_start, kv_len, max_q_len, self.window, self.scale, c, splits)
        else:
            a = F.attention_shared_plain(q_full, rows, table, q_start, kv_len, max_q_len, self.window, self.scale, c)
        # values of the heads from the weighted latents, gate
        if gate is not None:
            F.sigmoid_gate(torch.bmm(a.transpose(0, 1), self.w_uv.transpose(1, 2)), True, gate, self.g_col, H, e, out=out)
        else:
            torch.bmm(a.transpose(0, 1), self.w_uv.transpose(1, 2), out=out.view(T, H, e).transpose(0, 1))

    def _unfolded(self, q, y, store, ctx: StepContext, view, rows, out, first: int) -> None:
        """The requests from ``first`` on (every one before brings one token), into ``out[first:]``."""
        T, H, d, r, e = ctx.num_tokens, self.nh, self.d, self.r, self.e
        cols, rot_at = F.unfolded_query_layout(d, r)
        q_pad = torch.empty(T, H, cols, dtype=self.rt.act, device=q.device)
        mine = q_pad[first:]
        if store is not None and first:
            raise RuntimeError("latent attention: the cached rows of all tokens belong to one launch")
        F.latent_rows(ctx.positions[first:], self.inv_freq, self.c, r, store=store,
                      query=(q[first:], self.q_col, H, d, mine, -(-d // 16) * 16, mine, rot_at, -(-r // 16) * 16),
                      magnitude=self.position.magnitude)
        kv_len = ctx.kv_len[first:]
        lat, k_rot = F.latent_gather(rows, view.block_table[first:], kv_len, self._context_rows(ctx, first), self.c, r)
        kv = torch.mm(lat, self.w_ukv.t())
        F.prefill_attention_tc_unfolded(q_pad, kv, k_rot, ctx.q_start[first:], kv_len, ctx.max_q_len, d, r, e,
                                        self.window, self.scale, out, y if self.gated else None, self.g_col)


register_part("mixer", "latent_attention", LatentAttention)
