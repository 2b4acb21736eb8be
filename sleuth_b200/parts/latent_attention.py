"""Causal attention through low-rank latents over the paged latent cache, as a mixer part.

With h the layer's normed input:

* queries: c_q = RMSNorm(W_dq h) (gain ``dq_norm``), q = W_uq c_q, laid out head by head as ``plain_dim``
  unrotated values followed by ``rot_dim`` rotated ones;
* keys and values: W_dkv h has ``kv_rank + rot_dim`` rows; the first ``kv_rank``, RMS-normed (gain ``dkv_norm``),
  are the token's latent c, the rest (not normed) is one rotated key part that all heads share. Head n's
  unrotated key is W_uk[n] c and its value W_uv[n] c;
* score = (q_plain . k_plain + q_rot . k_rot) * scale, causal softmax, the heads' outputs side by side, times
  sigmoid(W_g h), then W_o, added into the stream.

The cache keeps c and the rotated key part only (``LatentRequest``), and the per-head keys and values are never
formed: the key up-projection is applied to the query instead (q_lat[n] = W_uk[n]^T q_plain[n], so that
q_plain . (W_uk c) = q_lat . c), the softmax-weighted sum runs over the latents, and the value up-projection is
applied to that sum (value[n] = W_uv[n] sum_j p_j c_j). One kernel then serves prompts, single tokens and chunks
alike, and a token costs ``kv_rank + rot_dim`` cache values per layer whatever the number of heads.

A bfloat16 step in which every sequence starts at position 0 (whole prompts of 64 tokens and more) takes another
way to the same result: its keys are its own tokens, so one product forms every head's unrotated keys and values
from the step's latents and ``head_prompt_attention`` runs ordinary per-head attention, which multiplies
``plain_dim + rot_dim + value_dim`` values per head and pair of tokens instead of ``2 * kv_rank + rot_dim``. The cache
is written the same way, and later portions and single tokens read it through the latent form. Heads without a rotated part
whose keys and values have the same width, 64 or 128, run on the tcgen05 attention kernel of the key/value cache when the
prompts fill its tiles: the product that forms their keys and values stores them straight into pages of scratch memory
(``gemm_tc_qkv``), ``latent_post`` writes those pages' block table, and the output gate is applied in the epilogue of the
gate's own product.

Options of the spec: ``q_rank`` 0 (the queries are W_q h, no query latent); ``window`` (a query sees the ``window`` most
recent tokens, its own included); ``sinks`` (a learned score per head in the softmax denominator: the attention kernels join
it to a row's maximum and mass once, at the row's end, or where the key slices are merged); ``rot_dim`` 0 (no rotated part:
the cache row is the latent alone); ``gate_span="head"`` (W_g gives one gate value per head; its rows then ride in the
stacked down-projection and the gate is read from that product's float32 result); a position part that pairs
neighbouring channels (2i with 2i + 1): the rows of the query and key projections that produce the rotated parts are
reordered once at load time so that pair i sits at channels i and i + rot/2, which the kernels turn; a dot product
does not care about the order of its channels as long as query and key agree.

Launches of a step (latent form): the stacked down-projections (float32 result), the gate projection, ``latent_post`` (both
norms, the key part's rotation, the cache write), the query up-projection, the per-head carry into the latent
space (a batched library product), ``latent_attention`` (which turns the queries' rotated part as it loads them),
the per-head value up-projection (batched library product), ``latent_gate``, the output projection.
"""

from __future__ import annotations

import os

import torch

from ..cache.paged import LatentRequest
from ..kernels import ops
from .attention import use_tc_attention
from .base import BuildContext, Normed, ParamDecl, Part, build_position, register_mixer, result_target
from .linear import Linear, use_tc
from .spec import LatentAttentionSpec


# From this many tokens of its longest sequence on, a bfloat16 step in which every sequence starts at position 0 (whole
# prompts) forms each head's keys and values from its own tokens' latents and runs ordinary per-head attention: that
# multiplies plain_dim + rot_dim + value_dim values per head and token pair instead of 2 * kv_rank + rot_dim.
PER_HEAD_PROMPT_TOKENS = 64


# Up to this many sequences a bfloat16 single-token step runs on the kernels of ``csrc/latent_decode.cu``: five launches a layer
# (projections, queries and cache rows, attention, values with the gate, output product). SLEUTH_B200_LATENT_STEP=0 keeps
# the launches that steps of many tokens take.
STEP_ROWS = 32 if os.environ.get("SLEUTH_B200_LATENT_STEP", "1") != "0" else 0


class LatentAttention(Part):
    stores_result = True
    accepts_normed = True       # a single-token step normalises in the prologue of its first product
    accepts_rider = True        # a layer's own rows ride at the end of the stacked down-projection

    def __init__(self, spec: LatentAttentionSpec, ctx: BuildContext):
        if spec.rot_dim % 2:
            raise ValueError(f"rot_dim {spec.rot_dim} must be even")
        if spec.gate_span not in ("channel", "head"):
            raise ValueError(f"latent_attention: gate_span {spec.gate_span!r} is not 'channel' or 'head'")
        if spec.q_rank < 0 or spec.window < 0:
            raise ValueError(f"latent_attention: q_rank {spec.q_rank}, window {spec.window}")
        self.spec, self.ctx = spec, ctx
        self._step_ok = None            # whether the single-token kernels take these sizes (asked once)
        self.head_gate = spec.output_gate and spec.gate_span == "head"
        self.position = build_position(spec.position, ctx)
        self.down = self.down_all = self.gate = self.uq = self.o = None
        self.w_ukt = self.w_uv = self.q_gain = self.c_gain = self.sinks = None

    def declare(self):
        s = self.spec
        if s.q_rank:
            d = {"dq.weight": ParamDecl((s.q_rank, s.hidden)),
                 "dq_norm.weight": ParamDecl((s.q_rank,), "vector", init="gain"),
                 "uq.weight": ParamDecl((s.heads * (s.plain_dim + s.rot_dim), s.q_rank))}
        else:
            d = {"q.weight": ParamDecl((s.heads * (s.plain_dim + s.rot_dim), s.hidden))}
        d.update({
             "dkv.weight": ParamDecl((s.kv_rank + s.rot_dim, s.hidden)),
             "dkv_norm.weight": ParamDecl((s.kv_rank,), "vector", init="gain"),
             "uk.weight": ParamDecl((s.heads * s.plain_dim, s.kv_rank)),
             "uv.weight": ParamDecl((s.heads * s.value_dim, s.kv_rank)),
             "o.weight": ParamDecl((s.hidden, s.heads * s.value_dim))})
        if s.output_gate:
            d["g.weight"] = ParamDecl((s.heads if self.head_gate else s.heads * s.value_dim, s.hidden))
        if s.sinks:
            d["sinks"] = ParamDecl((s.heads,), "vector")
        return d

    def _paired_halves(self, w: torch.Tensor, first: int, step: int, count: int) -> torch.Tensor:
        """``w`` with the rows that produce rotated channels reordered from neighbouring pairs (2i, 2i + 1) to halves
        (i, i + rot/2): ``count`` runs of rotated channels, the first starting at row ``first``, ``step`` rows apart."""
        rot = self.position.rot_dim
        if not getattr(self.position, "neighbours", False) or rot < 4:
            return w
        order = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)]).to(w.device)
        rows = torch.arange(w.shape[0], device=w.device)
        for k in range(count):
            at = first + k * step
            rows[at:at + rot] = at + order
        return w[rows]

    def bind(self, t):
        s, dt = self.spec, self.ctx.dtype
        dn, P = s.plain_dim, s.rot_dim
        stack = ([t["dq.weight"]] if s.q_rank else []) + [self._paired_halves(t["dkv.weight"], s.kv_rank, 0, 1)]
        if self.head_gate:
            stack.append(t["g.weight"])         # a gate value per head: its few rows ride in the stacked product
        self.rider_rows = 0
        if t.get("rider.weight") is not None:
            stack.append(t["rider.weight"])
            self.rider_rows = t["rider.weight"].shape[0]
        # one product with a float32 result; a gate value per channel has a product of its own in steps of many tokens
        # (behind the attention, which its epilogue then gates) and rides at the end of this one in single-token steps
        rows = sum(w.shape[0] for w in stack)
        channel_gate = s.output_gate and not self.head_gate
        self.down_all = Linear(torch.cat(stack + ([t["g.weight"]] if channel_gate else []), dim=0), dt)
        self.down = Linear(self.down_all.weight[:rows], dt)
        self.gate = Linear(self.down_all.weight[rows:], dt) if channel_gate else None
        self.uq = Linear(self._paired_halves(t["uq.weight" if s.q_rank else "q.weight"], dn, dn + P, s.heads), dt)
        self.o = Linear(t["o.weight"], dt)
        self.ukv = Linear(torch.cat([t["uk.weight"], t["uv.weight"]], dim=0), dt)      # whole prompts: keys and values per head
        self.w_ukt = t["uk.weight"].to(dt).view(s.heads, s.plain_dim, s.kv_rank).transpose(1, 2).contiguous()   # [H, rank, plain]
        self.w_uv = t["uv.weight"].to(dt).view(s.heads, s.value_dim, s.kv_rank).contiguous()
        self.q_gain, self.c_gain = t.get("dq_norm.weight"), t["dkv_norm.weight"]
        self.sinks = t["sinks"].to(torch.float32).contiguous() if s.sinks else None

    def cache_request(self):
        s = self.spec
        return LatentRequest(s.kv_rank + s.rot_dim, s.window)

    def lead_weight(self):
        return self.down_all.weight if self.down_all is not None else None

    def forward(self, h, x, b, view, ws):
        s, dt = self.spec, self.ctx.dtype
        if b.max_count == 1 and b.T <= STEP_ROWS and self._step_takes(dt):
            self._single_tokens(h, x, b, view, ws)
            return
        if isinstance(h, Normed):
            h = h.tensor()
        T, H, R, P, dn, dv = h.shape[0], s.heads, s.kv_rank, s.rot_dim, s.plain_dim, s.value_dim
        table = b.tables[view.group]
        tables = self.position.tables()
        cos, sin = tables if tables is not None else (None, None)
        rotated = self.position.rot_dim
        mark = ws.mark()
        lat = self.down.forward(h, ws=ws, stream=b.stream, out_dtype=torch.float32)
        if self.rider_rows:
            b.rider = lat[:, lat.shape[1] - self.rider_rows:]        # (a channel gate's rows are not part of this product)
        cq = ws.take((T, s.q_rank), dt) if s.q_rank else None
        fresh = getattr(b, "fresh", False) and b.max_count >= PER_HEAD_PROMPT_TOKENS
        paged = fresh and self._prompt_takes_pages(b, T)
        per_head = fresh and (paged or ops.head_prompt_supported(dn, P, dv, dt))
        c_out = ws.take((T, R), dt) if per_head else None
        k_out = ws.take((T, P), dt) if per_head else None
        own = None
        if paged:
            shape = (ops.prompt_pages(T, b.n), H, 64, dn)
            k_pages, v_pages = ws.take(shape, dt), ws.take(shape, dt)
            own = (ws.take((b.n, -(-b.max_count // 64)), torch.int32), b.seq_start, v_pages)
        ops.latent_post(lat, self.q_gain, self.c_gain, cos, sin, cq, view.pool if view.writes else None, b.tok_seq,
                        b.tok_pos, table, s.q_rank, R, P, rotated, s.norm_eps, b.stream, c_out, k_out, dtype=dt, pages=own)
        q = self.uq.forward(cq if s.q_rank else h, ws=ws, stream=b.stream).view(T, H, dn + P)
        if paged:
            # the up-projection's epilogue puts every head's keys and values into pages of the step's own, and the tcgen05
            # attention reads them there as it reads a key/value cache
            ops.gemm_tc_qkv(c_out, self.ukv.weight, 0, H, dn, None, None, None, None, None, 1e-6, None, k_pages, v_pages,
                            b.tok_seq, b.tok_pos, own[0], b.stream)
            y = ws.take((T, H * dv), dt)
            ops.attention_tc(q, k_pages, v_pages, y, b.seq_start, b.past, b.counts, own[0], b.max_count, H, H, dn, view.window,
                             s.scale, b.stream, max_keys=b.max_count, sinks=self.sinks)
            if self.gate is not None:
                self.gate.gate_values(h, y, ws=ws, stream=b.stream)
            self.o.forward(y, ws=ws, stream=b.stream, next_read=getattr(b, "next_read", None), **result_target(b, x))
            ws.release(mark)
            return
        if self.head_gate:
            g = lat[:, s.q_rank + R + P:s.q_rank + R + P + H]
        else:
            g = self.gate.forward(h, ws=ws, stream=b.stream) if self.gate is not None else None
        if per_head:
            kv = self.ukv.forward(c_out, ws=ws, stream=b.stream)
            val = ws.take((H, T, dv), dt)
            ops.head_prompt_attention(q, kv, k_out, val, cos, sin, b.seq_start, b.counts, b.max_count, H, dn, P, dv, rotated,
                                      view.window, s.scale, b.stream, sinks=self.sinks)
            self._gate_and_project(val, g, x, b, ws, T, H, dv, dt)
            ws.release(mark)
            return
        q_lat = ws.take((H, T, R), dt)
        torch.bmm(q[:, :, :dn].transpose(0, 1), self.w_ukt.transpose(1, 2), out=q_lat)
        o_lat = ws.take((H, T, R), dt)
        # the number of key slices follows the batch and the longest sequence allowed, never the lengths of the
        # moment: a recorded step stays valid as its sequences grow
        splits = ops.latent_splits(b.n, H, b.max_count, table.shape[1] * 64)
        floats = ops.latent_scratch_floats(T, H, R, splits)
        scratch = ws.take((floats,), torch.float32) if floats else None
        ops.latent_attention(q_lat, q, view.pool, o_lat, cos, sin, b.seq_start, b.past, b.counts, table, b.max_count,
                             H, R, P, dn, rotated, view.window, s.scale, splits, scratch, b.stream, sinks=self.sinks)
        val = ws.take((H, T, dv), dt)
        torch.bmm(o_lat, self.w_uv.transpose(1, 2), out=val)
        self._gate_and_project(val, g, x, b, ws, T, H, dv, dt)
        ws.release(mark)

    def _prompt_takes_pages(self, b, T: int) -> bool:
        """Whether the step's whole prompts run on the tcgen05 attention: heads without a rotated part, keys and values of
        the same width that kernel takes, sequences that fill its tiles."""
        s = self.spec
        return (s.rot_dim == 0 and s.plain_dim == s.value_dim and not self.head_gate
                and use_tc_attention(s.heads, s.heads, s.plain_dim, self.ctx.dtype, b.max_count, s.scale)
                and use_tc(T, 2 * s.heads * s.plain_dim, s.kv_rank))

    def _step_takes(self, dt) -> bool:
        s = self.spec
        if self._step_ok is None:
            self._step_ok = ops.latent_decode_supported(s.heads, s.kv_rank, s.rot_dim, s.plain_dim, s.q_rank or s.hidden, dt)
        return self._step_ok

    def _single_tokens(self, h, x, b, view, ws):
        """A step that brings one token a sequence, few sequences: the down-projections with every gate row (the norm in
        their prologue where that pays), queries into the latent space and cache rows, attention in slices, slices joined,
        values up-projected and gated, output product."""
        s, dt = self.spec, self.ctx.dtype
        n, H, R, P, dn, dv = b.T, s.heads, s.kv_rank, s.rot_dim, s.plain_dim, s.value_dim
        table = b.tables[view.group]
        tables = self.position.tables()
        cos, sin = tables if tables is not None else (None, None)
        rotated = self.position.rot_dim
        mark = ws.mark()
        if isinstance(h, Normed) and not s.q_rank:
            h = h.tensor()              # the queries read it too
        lat = self.down_all.forward(h, ws=ws, stream=b.stream, out_dtype=torch.float32, next_read=self.uq.weight)
        rows = self.down.out_features
        if self.rider_rows:
            b.rider = lat[:, rows - self.rider_rows:rows]
        g = None
        if self.head_gate:
            g = lat[:, s.q_rank + R + P:s.q_rank + R + P + H]
        elif self.gate is not None:
            g = lat[:, rows:]
        q_lat = ws.take((H, n, R), dt)
        q_raw = ws.take((n, H, dn + P), dt) if P else None
        ops.latent_query(lat, self.q_gain, self.c_gain, None if s.q_rank else h, self.uq.weight, self.w_ukt, cos, sin, q_lat, q_raw,
                         view.pool if view.writes else None, b.tok_pos, table, s.q_rank, R, P, dn, rotated, s.norm_eps, b.stream)
        # the number of slices follows the batch and the longest sequence allowed: a recorded step stays valid
        splits = ops.latent_decode_splits(n, H, R, P, table.shape[1] * 64)
        floats = ops.latent_scratch_floats(n, H, R, splits)
        parts = ws.take((floats,), torch.float32) if floats else None
        o_lat = ws.take((H, n, R), dt) if splits == 1 else None
        ops.latent_decode_attention(q_lat, q_raw, view.pool, o_lat, parts, cos, sin, b.past, table, R, P, dn, rotated, view.window,
                                    s.scale, splits, sinks=self.sinks, stream=b.stream)
        y = ws.take((n, H * dv), dt)
        ops.latent_value(parts, o_lat, self.w_uv, g, y, splits, sinks=self.sinks, stream=b.stream)
        self.o.forward(y, ws=ws, stream=b.stream, next_read=getattr(b, "next_read", None), **result_target(b, x))
        ws.release(mark)

    def _gate_and_project(self, val, g, x, b, ws, T, H, dv, dt):
        y = ws.take((T, H * dv), dt)
        if g is not None and self.head_gate:
            ops.latent_head_gate(val, g, y, b.stream)
        elif g is not None:
            ops.latent_gate(val, g, y, b.stream)
        else:
            y.view(T, H, dv).copy_(val.transpose(0, 1))
        self.o.forward(y, ws=ws, stream=b.stream, next_read=getattr(b, "next_read", None), **result_target(b, x))


register_mixer("latent_attention", LatentAttention)
