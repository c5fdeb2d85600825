"""Matrix memory with exponential gates (mLSTM): a mixer that carries a float32 state [key size, value size] per head, a sum of
keys and a running maximum of the gates' exponents from token to token.

forward = one fused input projection [q; k; v; gate; i; f] -> for portions a kernel that turns the gate rows into the
recurrence's factors, the recurrence over the states in the cache's state storage, and a kernel for quotient, norm, weight and
gate (bfloat16: chunks of tokens side by side on the tensor cores, with the last steps in the outputs' kernel); for single tokens one kernel that does all of it -> the output projection. Runs as a branch of a ``ParallelMixer``
too (``mix``).
"""
import numpy as np
import torch

from ..cache.requests import StateRequest
from ..config.specs import MatrixMemorySpec
from ..csrc import api
from .base import ParamDecl, Part, StepPlan, register_part
from .linear import linear


MIN_CHUNKED = 16       # tokens a sequence must bring, in the mean, for its step to run in chunks rather than token by token


class MemoryChunks(StepPlan):
    """A portion's chunks of ``tokens`` tokens: int32 [sequences + chunks, 4], per sequence (its first chunk, how many, 0, 0), then
    per chunk (sequence, first row of the chunk in the step, its rows, its number within the sequence). Empty for single tokens
    and for portions too short for it."""

    def __init__(self, tokens):
        self.tokens = tokens
        self.key = ("memory_chunks", tokens)

    def build(self, lens, pos0, is_decode):
        lens = np.asarray(lens, dtype=np.int64)
        if is_decode or lens.sum() < MIN_CHUNKED * len(lens):
            return np.zeros((0, 4), np.int32)
        per = (lens + self.tokens - 1) // self.tokens
        first = np.cumsum(per) - per
        seq = np.repeat(np.arange(len(lens)), per)
        k = np.arange(int(per.sum())) - first[seq]
        row = (np.cumsum(lens) - lens)[seq] + k * self.tokens
        rows = np.minimum(lens[seq] - k * self.tokens, self.tokens)
        zero = np.zeros_like(per)
        return np.concatenate([np.stack([first, per, zero, zero], 1), np.stack([seq, row, rows, k], 1)]).astype(np.int32)


class MatrixMemory(Part):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        s = spec
        if s.head_dim > 256 or s.v_head_dim > 4096:
            raise ValueError(f"a matrix memory takes keys up to 256 and values up to 4096, not {s.head_dim} / {s.v_head_dim}")
        if not s.gate_cap > 0:
            raise ValueError(f"a gate cap of {s.gate_cap}")
        self.n_qk, self.n_mid = s.num_heads * s.head_dim, s.num_heads * s.v_head_dim
        # filled up with zero rows, so that rows of the product stay aligned
        self.n_in = (2 * self.n_qk + 2 * self.n_mid + 2 * s.num_heads + 7) // 8 * 8
        self.q_scale = float(s.head_dim) ** -0.5

        self.chunks = MemoryChunks(api.MEMORY_CHUNK) if rt.dtype == torch.bfloat16 and api.memory_chunks_take(s.head_dim, s.v_head_dim) else None

    def step_plans(self):
        return [] if self.chunks is None else [self.chunks]

    def param_decls(self):
        s = self.spec
        return [ParamDecl("q", (self.n_qk, s.hidden_size)), ParamDecl("k", (self.n_qk, s.hidden_size)),
                ParamDecl("v", (self.n_mid, s.hidden_size)), ParamDecl("g", (self.n_mid, s.hidden_size)),
                ParamDecl("i", (s.num_heads, s.hidden_size)), ParamDecl("i.b", (s.num_heads,), init="unit", keep_float32=True),
                ParamDecl("f", (s.num_heads, s.hidden_size)), ParamDecl("f.b", (s.num_heads,), init="unit", keep_float32=True),
                ParamDecl("norm", (self.n_mid,), init="norm", keep_float32=True), ParamDecl("o", (s.hidden_size, self.n_mid))]

    def bind(self, tensors):
        rows = [tensors.pop(n) for n in ("q", "k", "v", "g", "i", "f")]
        fill = self.n_in - sum(w.shape[0] for w in rows)
        rows.append(torch.zeros((fill, self.spec.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, 0).contiguous()
        self.w_o = tensors.pop("o").contiguous()
        self.i_bias = tensors.pop("i.b").to(torch.float32).contiguous()
        self.f_bias = tensors.pop("f.b").to(torch.float32).contiguous()
        self.norm_weight = tensors.pop("norm").to(torch.float32).contiguous()

    def step_weights(self):
        return [self.w_in, self.w_o]

    def cache_requests(self):
        s = self.spec
        return [StateRequest((s.num_heads, s.head_dim, s.v_head_dim), torch.float32), StateRequest((s.num_heads, s.head_dim), torch.float32),
                StateRequest((s.num_heads,), torch.float32)]

    def mix(self, ctx, views, proj, mid, scale, writes=True):
        s = self.spec
        if not writes:
            raise ValueError("a recurrent layer cannot read another layer's state")
        cut = [0]
        for n in (self.n_qk, self.n_qk, self.n_mid, self.n_mid, s.num_heads, s.num_heads):
            cut.append(cut[-1] + n)
        q, k, v, gate, i, f = (proj[:, a:b] for a, b in zip(cut, cut[1:]))
        cu_q, pos0, n_seq = ctx.sequences()
        plan = ctx.plans.get(self.chunks.key) if self.chunks is not None and not ctx.is_decode else None
        api.matrix_memory(q, k, v, gate, i, f, self.i_bias, self.f_bias, s.gate_cap, [w.state for w in views[:3]], self.norm_weight,
                          s.norm_eps, scale, mid, self.q_scale, cu_q, pos0, ctx.seq_slot, ctx.row_pos, n_seq, s.num_heads, s.head_dim,
                          s.v_head_dim, chunks=plan if plan is not None and plan.shape[0] else None)

    def forward(self, ctx, views, a, writes=True):
        proj = linear(a, self.w_in)
        mid = torch.empty((ctx.n_tok, self.n_mid), dtype=self.rt.dtype, device=self.rt.device)
        self.mix(ctx, views, proj, mid, 1.0, writes)
        return linear(mid, self.w_o, allow_partial=True)


register_part(MatrixMemorySpec, MatrixMemory)
