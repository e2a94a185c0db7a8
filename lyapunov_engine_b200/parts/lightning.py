"""Lightning attention: a linear recurrence with one fixed decay per head.

With x the mixer's input, H heads, d the query/key size and e the value size:

    q = silu(Wq x),  k = silu(Wk x)  [H, d]      v = silu(Wv x)  [H, e]
    S <- decay_h S + k v^T                       o = S^T q                     per head
    y = Wo ( o / sqrt(mean(o^2) + eps) * w * sigmoid(Wg x) )                   over all heads together

S is carried from token to token in 32 bits, per request and head
(``state_need``).  One product makes all four projections, and silu on q, k and
v comes with it (ops.activated_linear).  Decoded tokens (and whatever the tensor-core form does
not take: 32-bit runs, heads of more than 128 entries) run token by token
(ops.lightning_scan); requests that bring several tokens in bfloat16 run over
chunks on the tensor cores (ops.lightning_chunks).  The norm and the gate are one kernel (ops.head_norm_gate, the heads
taken as one).
"""
from __future__ import annotations

import os

import torch

from .. import ops
from .base import Mixer, StateNeed, TensorDecl, register_mixer

SEGMENT = 256      # tokens of a request that a block of the chunked form takes
# 0: every request goes token by token
USE_CHUNKS = os.environ.get("LYAPUNOV_LIGHTNING_CHUNKS", "1") not in ("0", "")


@register_mixer("lightning")
class LightningMixer(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, decay, norm_eps: float, q_name: str,
                 k_name: str, v_name: str, gate_name: str, norm_name: str, o_name: str):
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.value_dim = int(head_dim), int(value_dim)
        self.decay, self.norm_eps = tuple(float(d) for d in decay), float(norm_eps)
        if len(self.decay) != self.num_heads:
            raise ValueError(f"{len(self.decay)} decays for {num_heads} heads")
        if not 1 <= self.head_dim <= ops.LIGHTNING_MAX_DIM:
            raise ValueError(f"lightning attention takes heads of up to {ops.LIGHTNING_MAX_DIM} entries, got {head_dim}")
        self.names = (q_name, k_name, v_name, gate_name)
        self.norm_name, self.o_name = norm_name, o_name
        H, d, e = self.num_heads, self.head_dim, self.value_dim
        self.q_col, self.k_col, self.v_col, self.gate_col = 0, H * d, 2 * H * d, 2 * H * d + H * e
        self.width = (self.gate_col + H * e + 7) // 8 * 8
        self.runtime = None

    def _in_chunks(self) -> bool:
        return USE_CHUNKS and self.runtime.dtype == torch.bfloat16 and self.head_dim <= ops.LIGHTNING_CHUNK_MAX_DIM

    def state_need(self):
        return StateNeed((self.num_heads, self.value_dim, self.head_dim), torch.float32)

    def tile_sizes(self):
        return [SEGMENT]

    def tensors(self):
        q, k, v, g = self.names
        W, H, d, e = self.hidden_size, self.num_heads, self.head_dim, self.value_dim
        return [TensorDecl(q, (H * d, W)), TensorDecl(k, (H * d, W)), TensorDecl(v, (H * e, W)), TensorDecl(g, (H * e, W)),
                TensorDecl(self.norm_name, (H * e,), role="vector", init="ones_jitter"), TensorDecl(self.o_name, (W, H * e))]

    def bind(self, get, runtime):
        rows = [get(n) for n in self.names]
        pad = self.width - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.norm_weight = get(self.norm_name).contiguous()
        self.w_o = get(self.o_name)
        self.decay_parts, self.powers = ops.lightning_tables(self.decay, runtime.device)
        if ops.lightning_segment() != SEGMENT:
            raise RuntimeError(f"the kernels' segments have {ops.lightning_segment()} tokens, the mixer lists {SEGMENT}")
        self.runtime = runtime

    def inner_width(self) -> int:
        return self.num_heads * self.value_dim

    def output_weight(self):
        return self.w_o

    def forward(self, x, ctx, cache):
        return ops.linear_for_residual(self.forward_inner(x, ctx, cache), self.w_o, ctx.workspace, "mixer_out", ctx.status)

    def forward_inner(self, x, ctx, cache, out=None, scale: float = 1.0):
        """The normed, gated heads before the output projection [T, H * e],
        into ``out`` where given, times ``scale``."""
        rt, ws = self.runtime, ctx.workspace
        H, d, e = self.num_heads, self.head_dim, self.value_dim
        T = x.shape[0]
        proj = ws.get("lightning_proj", (T, self.width), rt.dtype)
        ops.activated_linear(proj, x, self.w_in, ops.ACT_SILU_COLUMNS, ctx.status, columns=self.gate_col)
        o = ws.get("lightning_out", (T, H * e), torch.float32)
        request, q0, _, segments = ctx.tiles[SEGMENT]
        columns = (self.q_col, self.k_col, self.v_col)
        if segments and self._in_chunks():
            # (a step in which no request has a second segment goes from state row to state row)
            scratch = None
            if segments > ctx.num_requests - ctx.num_decode:
                scratch = ws.get("lightning_scratch", (segments, H, e, d), torch.float32)
            ops.lightning_chunks(o, proj, *columns, self.powers, cache.state, scratch, ctx.state_slots, ctx.cu_q, request, q0,
                                 segments, H, d, e)
            if ctx.num_decode:
                ops.lightning_scan(o, proj, *columns, self.decay_parts, cache.state, ctx.state_slots, ctx.cu_q, ctx.num_decode,
                                   H, d, e, requests=ctx.decode_requests, single=True)
        else:
            ops.lightning_scan(o, proj, *columns, self.decay_parts, cache.state, ctx.state_slots, ctx.cu_q, ctx.num_requests,
                               H, d, e, single=ctx.max_q_len == 1)
        if out is None:
            out = ws.get("lightning_gated", (T, H * e), rt.dtype)
        ops.head_norm_gate(out, o, proj[:, self.gate_col:self.gate_col + H * e], self.norm_weight, self.norm_eps, 1, H * e,
                           sigmoid=True, out_scale=scale)
        return out
