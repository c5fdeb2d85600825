"""Gated delta rule: a mixer that carries a float32 state [key size, value size] per head from token to token and writes
into it what the state does not yet say, S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.

forward = one fused input projection [q; k; v; gate; b; a] -> a kernel that makes the recurrence's float32 operands
(short convolution with its memory in the cache's state storage, SiLU, unit keys and queries, decays, step sizes) -> the
recurrence over the state in the cache's state storage -> each head over its root mean square, times the weight, times
SiLU of the gate -> the output projection. Runs as a branch of a ``ParallelMixer`` (``mix``).
"""
import torch

from ..cache.requests import StateRequest
from ..config.specs import GatedDeltaSpec
from ..csrc import api
from .base import ParamDecl, Part, register_part
from .linear import linear


class GatedDelta(Part):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        s = spec
        if s.num_heads % s.num_kv_heads or s.head_dim > 256 or not 1 <= s.conv_taps <= api.SHORT_CONV_MAX_TAPS:
            raise ValueError(f"{s.num_heads} heads on {s.num_kv_heads} key heads of {s.head_dim} (up to 256), {s.conv_taps} taps "
                             f"(up to {api.SHORT_CONV_MAX_TAPS})")
        self.n_qk = s.num_kv_heads * s.head_dim
        self.n_mid = s.num_heads * s.v_head_dim
        self.n_conv = 2 * self.n_qk + self.n_mid            # the channels that pass the convolution: q, k, v
        # filled up with zero rows, so that rows of the product stay aligned
        self.n_in = (self.n_conv + self.n_mid + 2 * s.num_heads + 7) // 8 * 8

    def param_decls(self):
        s = self.spec
        sizes = (("q", self.n_qk), ("k", self.n_qk), ("v", self.n_mid))
        return [ParamDecl(n, (rows, s.hidden_size)) for n, rows in sizes] + \
            [ParamDecl(n + ".conv", (rows, s.conv_taps), init="taps") for n, rows in sizes] + \
            [ParamDecl("g", (self.n_mid, s.hidden_size)), ParamDecl("b", (s.num_heads, s.hidden_size)),
             ParamDecl("a", (s.num_heads, s.hidden_size)), ParamDecl("A_log", (s.num_heads,), init="unit", keep_float32=True),
             ParamDecl("dt_bias", (s.num_heads,), init="unit", keep_float32=True),
             ParamDecl("norm", (s.v_head_dim,), init="norm", keep_float32=True), ParamDecl("o", (s.hidden_size, self.n_mid))]

    def bind(self, tensors):
        rows = [tensors.pop(n) for n in ("q", "k", "v", "g", "b", "a")]
        fill = self.n_in - sum(w.shape[0] for w in rows)
        rows.append(torch.zeros((fill, self.spec.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, 0).contiguous()
        self.w_conv = torch.cat([tensors.pop(n + ".conv") for n in ("q", "k", "v")], 0).contiguous()
        self.a_log = tensors.pop("A_log").to(torch.float32).contiguous()
        self.dt_bias = tensors.pop("dt_bias").to(torch.float32).contiguous()
        self.norm_weight = tensors.pop("norm").to(torch.float32).contiguous()
        self.w_o = tensors.pop("o").contiguous()

    def step_weights(self):
        return [self.w_in, self.w_o]

    def cache_requests(self):
        s = self.spec
        r = [StateRequest((s.num_heads, s.head_dim, s.v_head_dim), torch.float32)]
        if s.conv_taps > 1:     # the convolution's memory: the last taps - 1 projected rows [q | k | v] of a sequence
            r.append(StateRequest((s.conv_taps - 1, self.n_conv), self.rt.dtype))
        return r

    def mix(self, ctx, views, proj, mid, scale, writes=True):
        s, dev, T = self.spec, self.rt.device, ctx.n_tok
        if not writes:
            raise ValueError("a recurrent layer cannot read another layer's state")
        sizes = (s.num_heads, s.num_kv_heads, s.head_dim, s.v_head_dim)
        rows, c = proj[:, :self.n_conv], self.n_conv + self.n_mid
        gate, b, a = proj[:, self.n_conv:c], proj[:, c:c + s.num_heads], proj[:, c + s.num_heads:c + 2 * s.num_heads]
        memory = views[1].state if s.conv_taps > 1 else None
        cu_q, pos0, n_seq = ctx.sequences()
        qkv, scal = api.delta_operands(T, *sizes, dev)
        api.delta_prepare(rows, a, b, memory, self.w_conv, s.conv_taps, self.a_log, self.dt_bias, s.unit_eps, ctx.row_pos,
                          ctx.row_seq, pos0, ctx.seq_slot, qkv, scal, *sizes)
        if s.conv_taps > 1:
            api.conv_state_update(rows, memory, s.conv_taps, cu_q, pos0, ctx.seq_slot, n_seq)
        o = torch.empty((T, self.n_mid), dtype=torch.float32, device=dev)
        api.delta_rule(qkv, scal, o, views[0].state, cu_q, pos0, ctx.seq_slot, n_seq, *sizes)
        api.norm_gate(o, self.norm_weight, s.norm_eps, gate, scale, mid, group=s.v_head_dim, gate_act="silu")

    def forward(self, ctx, views, a, writes=True):
        proj = linear(a, self.w_in)
        mid = torch.empty((ctx.n_tok, self.n_mid), dtype=self.rt.dtype, device=self.rt.device)
        self.mix(ctx, views, proj, mid, 1.0, writes)
        return linear(mid, self.w_o, allow_partial=True)


register_part(GatedDeltaSpec, GatedDelta)
