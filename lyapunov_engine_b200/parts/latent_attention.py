"""Latent attention: every head's keys and values are linear maps of one
normed latent vector per token, and only that vector is cached.

With x the mixer's input (width H), nh heads, d query/key size, e value size
and r the latent size:

    q_h = Wq_h x                     c = rmsnorm(Wdkv x) * w_c           (r values, 32-bit norm)
    k_h(j) = Wuk_h c_j               v_h(j) = Wuv_h c_j
    score_h(i, j) = (q_h(i) . k_h(j)) * scale,   j <= i (optionally a window or chunks)
    out = Wo concat_h( sigmoid(g_h . x) * sum_j softmax_j(score_h) v_h(j) )

No positions enter.  Because k and v are linear in c, the step never builds
them: q_h . (Wuk_h c) = (Wuk_h^T q_h) . c, so each head's query is carried into
the latent space (one small product per head), attention runs over the cached
latents as both keys and values -- all heads share the one "key/value head" of
size r, the existing paged kernels serve it -- and each head's attended latent
is carried out through Wuv_h (again one small product per head, with the
head's output gate in its epilogue).  The cache holds r values per token and
layer, in one pool that the kernels read as keys and as values (the pool's rows
are padded with zeros to a multiple of 16).

Options beyond that:

* ``rot_dim`` > 0: beside the latent every token has one rotated key part of
  rot_dim entries, shared by all heads (the last rot_dim rows of the down
  projection, not normed), and every head's query has rot_dim more entries
  behind its head_dim unrotated ones; both turn in neighbouring pairs by
  position * rot_base^(-2i / rot_dim) (``rot_scaling``: rates and a factor on
  cosine and sine as rope.ramped_rates makes them), and the score is (q_unrotated .
  k_unrotated + q_rotated . k_rotated) * scale.  The cached row is [latent |
  rotated part]; a head's query in the latent space gets its own turned part
  behind it, so the one dot product over the row gives the score; the way out
  of the latent space reads the latent's columns only.
  ``rot_halves``: entry i turns with entry i + rot_dim / 2 instead.  A score
  does not change when the same order of entries is chosen for queries and
  keys, so the projections' rows are put in the order of neighbouring pairs at
  load and the same kernels serve both layouts.
* ``gate_per_entry``: the gate's tensor is [nh * e, H] and every entry of the
  heads' outputs has a gate of its own.
* ``q_rank`` > 0: the queries go through a latent of their own, q = Wuq
  rmsnorm(Wdq x) * w_q (``q_down_name``, ``q_norm_name``; ``q_name`` is then
  Wuq, [heads * (head_dim + rot_dim), q_rank]).

Per-head products: the package's FP32-pipe kernel (float32, and bfloat16 steps
of few rows); bfloat16 steps of many rows go to the library's batched product,
as the other many-row products do.
"""
from __future__ import annotations

import os

import torch

from .. import ops
from . import attention_kernels
from .attention import signed_scale
from .base import KVNeed, Mixer, TensorDecl, register_mixer
from .rope import pair_rates, ramped_rates

LIBRARY_ROWS = 64       # bfloat16 steps with more rows than this run the per-head products in the library
# The most ways a decoded token's latents are cut.  (Capping it at 8, the most that merge inside a thread-block
# cluster without a second kernel, was measured and is slower: all heads of a request share one pool, so a request is
# two blocks before splitting, and 512 keys a block cost more than the merge kernel: 1.03 against 0.93 ms a step.)
MAX_DECODE_SPLITS = int(os.environ.get("LYAPUNOV_LATENT_SPLITS", str(attention_kernels.DECODE_MAX_SPLITS)))


@register_mixer("latent_attention")
class LatentAttentionMixer(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, latent_dim: int, scale: float,
                 norm_eps: float, q_name: str, down_name: str, latent_norm_name: str, up_k_name: str, up_v_name: str,
                 o_name: str, gate_name: str | None = None, window: int | None = None, chunk: int | None = None,
                 rot_dim: int = 0, rot_base: float | None = None, q_rank: int = 0, q_down_name: str | None = None,
                 q_norm_name: str | None = None, rot_halves: bool = False, rot_scaling: dict | None = None,
                 gate_per_entry: bool = False):
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.qk_dim, self.value_dim, self.latent_dim = int(head_dim), int(value_dim), int(latent_dim)
        self.rot_dim, self.rot_base, self.q_rank = int(rot_dim), rot_base, int(q_rank)
        self.rot_halves, self.rot_scaling = bool(rot_halves), (dict(rot_scaling) if rot_scaling else None)
        if self.rot_dim and (self.rot_dim % 2 or rot_base is None):
            raise ValueError(f"a rotated part needs an even size and a base, got {rot_dim} and {rot_base}")
        if self.rot_dim and self.q_rank and self.latent_dim % 2:
            raise ValueError(f"a rotated part behind a query latent needs an even latent, got {latent_dim}")
        if self.q_rank and not (q_down_name and q_norm_name):
            raise ValueError("queries through a latent need the names of its projection and of its norm's weight")
        self.q_names = (q_down_name, q_norm_name)
        self.q_head = self.qk_dim + self.rot_dim                         # a head's query: unrotated, then rotated
        self.padded_latent = (self.latent_dim + self.rot_dim + 15) // 16 * 16   # the head size of kernels and pages
        if not 16 <= self.padded_latent <= attention_kernels.MAX_HEAD_DIM:
            raise ValueError(f"latent attention takes latent sizes up to {attention_kernels.MAX_HEAD_DIM} "
                             f"(with the rotated part), got {latent_dim} and {rot_dim}")
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.reach = ops.reach_code(window, chunk)
        self.window, self.chunk = (int(window) if window else None), (int(chunk) if chunk else None)
        self.names = (q_name, down_name, latent_norm_name, up_k_name, up_v_name, o_name)
        self.gate_name = gate_name
        self.gate_per_entry = bool(gate_per_entry) and bool(gate_name)
        self.gates = 0                                    # columns of the projection that are gates
        if gate_name:
            self.gates = self.num_heads * self.value_dim if self.gate_per_entry else self.num_heads
        self.gate_rows = (self.gates + 7) // 8 * 8
        self.runtime = None

    def cache_need(self):
        return KVNeed(1, self.padded_latent, self.window, self.chunk, values=False)

    def tile_sizes(self):
        return attention_kernels.tile_sizes()

    def decode_variant(self, fill, num_decode, context_bound):
        if self.runtime is None or self.runtime.dtype != torch.bfloat16:
            return None
        return attention_kernels.decode_variant(fill, self.num_heads, 1, self.padded_latent, context_bound, self.reach,
                                                MAX_DECODE_SPLITS)

    def tensors(self):
        q, down, norm, uk, uv, o = self.names
        H, nh, d, e, r = self.hidden_size, self.num_heads, self.qk_dim, self.value_dim, self.latent_dim
        decls = [TensorDecl(q, (nh * self.q_head, self.q_rank or H)), TensorDecl(down, (r + self.rot_dim, H)),
                 TensorDecl(norm, (r,), role="vector", init="ones_jitter"),
                 TensorDecl(uk, (nh * d, r)), TensorDecl(uv, (nh * e, r)), TensorDecl(o, (H, nh * e))]
        if self.gate_name:
            decls.append(TensorDecl(self.gate_name, (self.gates, H)))
        if self.q_rank:
            decls += [TensorDecl(self.q_names[0], (self.q_rank, H)),
                      TensorDecl(self.q_names[1], (self.q_rank,), role="vector", init="ones_jitter")]
        return decls

    def bind(self, get, runtime):
        q, down, norm, uk, uv, o = self.names
        nh, d, e, r, rp = self.num_heads, self.qk_dim, self.value_dim, self.latent_dim, self.padded_latent
        rd, qh = self.rot_dim, self.q_head
        # the projection's first rows: the queries themselves, or their latent
        w_q, w_down = get(q), get(down)
        if self.rot_halves and rd:
            # row 2i from row i, row 2i + 1 from row i + rd / 2 (of every head's rotated part, and of the keys')
            pairs = torch.arange(rd, device=w_q.device).view(2, rd // 2).t().reshape(-1)
            order = torch.cat([torch.arange(d, device=w_q.device), d + pairs])
            w_q = w_q.view(nh, qh, -1)[:, order].reshape(nh * qh, -1)
            w_down = torch.cat([w_down[:r], w_down[r:][pairs]])
        rows = [get(self.q_names[0]) if self.q_rank else w_q, w_down]
        self.q_width = self.q_rank or nh * qh
        self.w_up_q = w_q.contiguous() if self.q_rank else None
        self.q_norm_weight = get(self.q_names[1]) if self.q_rank else None
        self.rates, self.magnitude = None, 1.0
        if rd:
            # (plain pairs: rates, and so angles, of 32 bits)
            if self.rot_halves or self.rot_scaling:
                rates, self.magnitude = ramped_rates(rd, self.rot_base, self.rot_scaling)
            else:
                rates = pair_rates(rd, self.rot_base)
            self.rates = rates.to(runtime.device).contiguous()
        # the latent's columns start on a 16-byte boundary of the projection's rows, and so do the gate's
        self.latent_col = (self.q_width + 7) // 8 * 8
        if self.latent_col != self.q_width:
            rows.insert(1, torch.zeros((self.latent_col - self.q_width, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.gate_col = (self.latent_col + r + rd + 7) // 8 * 8
        if self.gate_col != self.latent_col + r + rd:
            rows.append(torch.zeros((self.gate_col - self.latent_col - r - rd, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        if self.gate_name:
            gate = get(self.gate_name)
            rows += [gate, torch.zeros((self.gate_rows - self.gates, self.hidden_size), dtype=gate.dtype, device=gate.device)]
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.norm_weight = get(norm)
        # into the latent space: [nh, r (padded), d], head h's key map transposed.  A rotated part of the projection's
        # queries goes its own way to the columns behind the latent, and the product ends at the latent's; behind a
        # query latent the rotated entries pass through the product (with ones and zeros it is exact) and turn there.
        through = rd if self.q_rank else 0
        into = torch.zeros((nh, r if rd and not through else rp, d + through), dtype=runtime.dtype, device=runtime.device)
        into[:, :r, :d] = get(uk).view(nh, d, r).transpose(1, 2)
        for j in range(through):
            into[:, r + j, d + j] = 1.0
        self.w_into = into.contiguous()
        # out of it: [nh, e, r (padded)]
        out_of = torch.zeros((nh, e, rp), dtype=runtime.dtype, device=runtime.device)
        out_of[:, :, :r] = get(uv).view(nh, e, r)
        self.w_out_of = out_of.contiguous()
        self.w_o = get(o)
        self.runtime = runtime
        self.kernel_scale, self.head_scale, self.head_scale_positive = signed_scale(self.scale, None, nh, runtime.device)
        attention_kernels.prepare(rp)

    def _per_head(self, out, a, w, gate, heads, a_head=None, out_head=None):
        """out[t, h, :] = w[h] @ a[t, h, :] (times the head's gate, or its
        entries' gates); ``a_head`` / ``out_head``: columns from head to head
        where those are more than the product's."""
        T, K, N = a.shape[0], w.shape[2], w.shape[1]
        if a.dtype == torch.bfloat16 and T > LIBRARY_ROWS:
            ops.counters["library_products"] += 1
            torch.bmm(a.unflatten(1, (heads, a_head or K))[:, :, :K].transpose(0, 1), w.transpose(1, 2),
                      out=out.unflatten(1, (heads, out_head or N))[:, :, :N].transpose(0, 1))
            if gate is not None and self.gate_per_entry:
                ops.sigmoid_gate(out, out, gate)
            elif gate is not None:
                ops.head_gate(out, gate, heads, N)
            return
        ops.gemm_heads(out, a, w, gate, a_head=a_head, out_head=out_head)

    def _queries_through_latent(self, q_latent, proj, ctx, kv, write):
        """The queries' own latent: norm and up projection, then as the others."""
        rt, ws = self.runtime, ctx.workspace
        nh, r, rp, T = self.num_heads, self.latent_dim, self.padded_latent, proj.shape[0]
        table = ctx.block_tables[kv.group]
        q_normed = ws.get("latent_q_normed", (T, self.q_rank), rt.dtype)
        # the latent's norm, the rotated part's turn and the cache write, and the norm of the queries' latent
        ops.latent_rope_store(proj, self.latent_col, r, self.rot_dim, rp, self.norm_weight, self.norm_eps, self.rates,
                              kv.k if write else None, ctx.positions, ctx.request_of_token, table, kv.page_size, ctx.status,
                              second=(0, self.q_rank, self.q_norm_weight, q_normed), magnitude=self.magnitude)
        queries = ws.get("latent_queries", (T, nh * self.q_head), rt.dtype)
        ops.linear(queries, q_normed, self.w_up_q, ctx.status)
        self._per_head(q_latent, queries, self.w_into, None, nh)
        if self.rot_dim:
            ops.rope_norm_store(q_latent, None, None, self.rates, ctx.positions, ctx.request_of_token, table, nh, 0, rp,
                                r, self.rot_dim, None, rp, kv.page_size, False, False, ctx.status, magnitude=self.magnitude)

    def forward(self, x, ctx, cache):
        rt = self.runtime
        nh, r, rp, e, rd = self.num_heads, self.latent_dim, self.padded_latent, self.value_dim, self.rot_dim
        T = x.shape[0]
        ws = ctx.workspace
        proj = ws.get("latent_proj", (T, self.w_in.shape[0]), rt.dtype)
        ops.linear(proj, x, self.w_in, ctx.status)
        kv = cache.kv
        pool = kv.k if cache.write else None
        q_latent = ws.get("latent_q", (T, nh * rp), rt.dtype)
        place = (ctx.positions, ctx.request_of_token, ctx.block_tables[kv.group], kv.page_size, ctx.status)
        if self.q_rank:
            self._queries_through_latent(q_latent, proj, ctx, kv, cache.write)
        elif ops.latent_prepare_applies(proj, self.qk_dim, rd):
            # few rows: the latent's norm and store, the turns of rotated parts and the queries' way into the latent
            # space as one launch
            ops.latent_prepare(q_latent, proj, self.w_into, self.latent_col, r, self.norm_weight, self.norm_eps, pool, *place,
                               rot=rd, rates=self.rates, magnitude=self.magnitude)
        elif rd:
            ops.latent_rope_store(proj, self.latent_col, r, rd, rp, self.norm_weight, self.norm_eps, self.rates, pool, *place,
                                  magnitude=self.magnitude, queries=(self.qk_dim, self.q_head, nh, q_latent))
            self._per_head(q_latent, proj[:, :self.q_width], self.w_into, None, nh, a_head=self.q_head, out_head=rp)
        else:
            if cache.write:
                ops.latent_norm_store(proj, self.latent_col, r, self.norm_weight, self.norm_eps, pool, *place)
            self._per_head(q_latent, proj[:, :self.q_width], self.w_into, None, nh)
        attended = ws.get("latent_attn", (T, nh * rp), rt.dtype)
        attention_kernels.run(attended, q_latent, ctx, kv, nh, 1, rp, self.reach, self.kernel_scale, self.head_scale,
                              self.head_scale_positive, max_splits=MAX_DECODE_SPLITS)
        heads_out = ws.get("attn", (T, nh * e), rt.dtype)
        gate = proj[:, self.gate_col:self.gate_col + self.gates] if self.gate_name else None
        self._per_head(heads_out, attended, self.w_out_of, gate, nh)
        return ops.linear_for_residual(heads_out, self.w_o, ws, "mixer_out", ctx.status)
