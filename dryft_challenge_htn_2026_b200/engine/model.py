"""A causal language model put together from a ``ModelSpec``: embedding, blocks run in schedule
order, final norm, output head. ``forward`` runs one step over the token rows a ``StepContext``
describes and returns float32 logits at the wanted rows (reference: engine/engine.py:459-503).
"""
import torch

from ..cache.requests import StateRequest
from ..csrc import api
from ..parts import ParamDecl, Runtime, build_part
from ..parts.block import add_norm
from ..parts.linear import STORE_F32, linear, linear_partial
from ..parts.norm import NormedDelta, RMSNorm, StreamReset, norm_args


class CausalLM:
    def __init__(self, spec, dtype=torch.bfloat16, device="cuda"):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"dtype must be torch.float32 or torch.bfloat16, not {dtype}")
        self.spec = spec
        self.rt = Runtime(torch.device(device), dtype)
        self.blocks = [build_part(ls, self.rt) for ls in spec.layers]
        self.final_norm = build_part(spec.final_norm, self.rt)
        n_entries = max(e.cache for e in spec.schedule) + 1
        owners = {}
        for e in spec.schedule:
            if not 0 <= e.layer < len(self.blocks):
                raise ValueError(f"schedule names layer {e.layer}, the model has {len(self.blocks)}")
            if e.writes:
                if e.cache in owners:
                    raise ValueError(f"cache entry {e.cache} is written by two schedule entries")
                owners[e.cache] = e.layer
        for e in spec.schedule:
            if e.cache not in owners:
                raise ValueError(f"cache entry {e.cache} is read but never written")
            if self.blocks[e.layer].cache_requests() != self.blocks[owners[e.cache]].cache_requests():
                raise ValueError(f"layer {e.layer} cannot use cache entry {e.cache}: its owner stores something else")
        self._entry_requests = [self.blocks[owners[c]].cache_requests() for c in range(n_entries)]
        self.bigram = None       # the table of token pairs (ModelSpec.embed_bigram); its memory is a cache entry behind the layers'
        if spec.embed_bigram is not None:
            if spec.embed_position is not None or any(e.add_embedding for e in spec.schedule):
                raise ValueError("an embedding with token pairs goes without a position vector and is not taken in again")
            self._entry_requests.append([StateRequest((1,), torch.int32)])
        self.embed = self.head = None
        self.tied = None
        self.position = build_part(spec.embed_position, self.rt) if spec.embed_position is not None else None
        if self.position is not None and not getattr(self.position, "added_to_embedding", False):
            raise TypeError(f"{type(self.position).__name__} is not a position vector the embedding can add")
        self.tables = {}         # the model's own learned tables (ModelSpec.tables), float32, by name
        names = {n for n, _ in spec.tables}
        for e in spec.schedule:
            if e.add_row is not None and e.add_row[0] not in names:
                raise ValueError(f"schedule adds a row of {e.add_row[0]!r}, which is not a table of the model")
        self.matrices = {}       # the model's own learned matrices (ModelSpec.matrices), by name
        wide = {n for n, shape in spec.matrices if tuple(shape) == (spec.hidden_size, 2 * spec.hidden_size)}
        for e in spec.schedule:
            if e.take_in is not None and (e.take_in not in wide or e.add_embedding):
                raise ValueError(f"a run takes the embedding in by {e.take_in!r}, which is not a matrix [hidden, 2 hidden] of the "
                                 "model, or adds it as well")
        self._keeps_embedding = any(e.add_embedding for e in spec.schedule)
        self._takes_in = any(e.take_in is not None for e in spec.schedule)
        # index arrays the parts' kernels want built for every step (engine.batch.build_context), once per key
        self.step_plans = list({p.key: p for b in self.blocks for p in b.step_plans()}.values())
        self.prepared = 0        # positions the parts' tables reach
        self.generation = 0      # counts the times they were rebuilt: captured graphs hold the old tables' addresses

    # -- parameters --------------------------------------------------------------------------
    def param_decls(self, tied):
        """Checkpoint name -> ParamDecl for the whole model."""
        s = self.spec
        out = {s.embed_name: ParamDecl(s.embed_name, (s.vocab_size, s.hidden_size), "matrix")}
        if s.embed_bigram is not None:
            b = s.embed_bigram
            out[b.tensor] = ParamDecl(b.tensor, (b.buckets + 1, s.hidden_size), "matrix")
        for ls, blk in zip(s.layers, self.blocks):
            for p in blk.param_decls():
                out[ls.prefix + p.name] = p
        for p in self.final_norm.param_decls():
            out[s.final_norm_prefix + p.name] = p
        for name, shape in s.tables:
            out[name] = ParamDecl(name, tuple(shape), "matrix", keep_float32=True)
        for name, shape in s.matrices:
            out[name] = ParamDecl(name, tuple(shape), "matrix")
        if not tied:
            out[s.head_name] = ParamDecl(s.head_name, (s.vocab_size, s.hidden_size), "matrix")
        return out

    def bind(self, tensors, tied):
        s = self.spec
        self.tied = tied
        self.embed = tensors.pop(s.embed_name).contiguous()
        self.head = self.embed if tied else tensors.pop(s.head_name).contiguous()
        if s.embed_bigram is not None:
            self.bigram = tensors.pop(s.embed_bigram.tensor).contiguous()
        self.tables = {name: tensors.pop(name).to(torch.float32).contiguous() for name, _ in s.tables}
        self.matrices = {name: tensors.pop(name).contiguous() for name, _ in s.matrices}
        for ls, blk in zip(s.layers, self.blocks):
            n = len(ls.prefix)
            blk.bind({k[n:]: tensors.pop(k) for k in [k for k in tensors if k.startswith(ls.prefix)]})
        n = len(s.final_norm_prefix)
        self.final_norm.bind({k[n:]: tensors.pop(k) for k in [k for k in tensors if k.startswith(s.final_norm_prefix)]})

    def entry_requests(self):
        return self._entry_requests

    def prepare(self, max_positions):
        """Makes the parts' tables (rotation angles) reach ``max_positions``; they grow by doubling.
        Returns ``generation``, which changes whenever they were rebuilt."""
        if max_positions > self.prepared:
            self.prepared = max(max_positions, 2 * self.prepared, 256)
            for b in self.blocks:
                b.prepare(self.prepared)
            self.generation += 1
        return self.generation

    def weight_bytes_per_step(self):
        """Bytes of weights a decode step reads: what every part says it streams once a step, for
        every run of a layer in the schedule, and the head (the embedding is read by row only, so it
        counts only where it is also the head)."""
        total = self.head.numel() * self.head.element_size()
        for e in self.spec.schedule:
            total += sum(w.numel() * w.element_size() for w in self.blocks[e.layer].step_weights())
            if e.take_in is not None:
                total += self.matrices[e.take_in].numel() * self.matrices[e.take_in].element_size()
        return total

    # -- one step ----------------------------------------------------------------------------
    def _take_in(self, h, pending, both, matrix, row):
        """The stream x (``h`` with what is still ``pending``) becomes M [x; x0] (+ ``row``): ``both`` [rows, 2 hidden] holds x0
        in its second half, in the storage type, and gets x in its first. -> the ``StreamReset`` the next block starts from."""
        norm = None
        if isinstance(pending, NormedDelta):
            pending, norm = pending.delta, norm_args(pending.norm)
        api.sublayer_add(h, pending, norm, both[:, :self.spec.hidden_size])
        return StreamReset(linear_partial(both, matrix), row)

    def forward(self, ctx, cache, tap=None):
        """``tap(k, h)``: called after the k-th schedule entry with the residual stream as it then
        stands (that entry's feed-forward output added in): for dumps that look for the layer where
        two runs part ways. It costs a launch and a copy per entry, so it is for debugging only."""
        s, rt = self.spec, self.rt
        h = torch.empty((ctx.n_tok, s.hidden_size), dtype=torch.float32, device=rt.device)
        a = torch.empty((ctx.n_tok, s.hidden_size), dtype=rt.dtype, device=rt.device)
        first = self.blocks[s.schedule[0].layer]
        # the embedding kernel computes RMSNorm and nothing else, and only of the embedding as it leaves the kernel
        fused = isinstance(getattr(first, "norm_in", None), RMSNorm) and not (
            s.schedule[0].add_embedding or s.schedule[0].add_row or s.schedule[0].take_in)
        norm_w, eps = (first.norm_in.weight, first.norm_in.spec.eps) if fused else (None, 0.0)
        ctx.carry = {}           # what one layer of the step leaves for later ones (e.g. values that layers share)
        ctx.stream_copy = None   # the stream in the storage type, where a kernel has left it (blocks with the norm after the sum)
        plain = getattr(first, "reads_stream", False) and not (
            s.schedule[0].add_embedding or s.schedule[0].add_row or s.schedule[0].take_in)
        ctx.stream = None        # the stream, where a block has written it to another buffer than the one it was given
        if self.bigram is not None:
            b = s.embed_bigram
            api.embed_bigram(ctx.tok, self.embed, s.embed_scale, self.bigram, b.mul_prev, b.mul_cur,
                             cache.views(len(self._entry_requests) - 1)[0].state, ctx.sequence_rows(), h)
            fused = False
        elif self.position is None and s.embed_scale == 1.0:
            api.embed_rmsnorm(ctx.tok, self.embed, norm_w, eps, h, a if (fused or plain) else None)
            if plain:
                ctx.stream_copy = a
        else:
            api.embed_position_rmsnorm(ctx.tok, self.embed, s.embed_scale, ctx.row_pos,
                                       self.position.inv_freq if self.position is not None else None, norm_w, eps, h, a)
        e0 = h.clone() if self._keeps_embedding else None     # the embedding's output, for the runs that take it in again
        both = None
        if self._takes_in:       # [x | x0] for the runs that take the embedding in by a matrix: x0 stays in its half
            both = torch.empty((ctx.n_tok, 2 * s.hidden_size), dtype=rt.dtype, device=rt.device)
            api.sublayer_add(h, None, None, both[:, s.hidden_size:])
        pending = None
        for i, e in enumerate(s.schedule):
            if e.take_in is not None:
                pending = self._take_in(h, pending, both, self.matrices[e.take_in],
                                        self.tables[e.add_row[0]][e.add_row[1]] if e.add_row is not None else None)
                ctx.stream_copy = None
            elif e.add_embedding or e.add_row is not None:
                api.stream_add(h, e0 if e.add_embedding else None,
                               self.tables[e.add_row[0]][e.add_row[1]] if e.add_row is not None else None)
                ctx.stream_copy = None
            pending = self.blocks[e.layer].forward(ctx, h, pending, cache.views(e.cache), e.writes,
                                                   a if (i == 0 and fused) else None)
            if ctx.stream is not None:
                h, ctx.stream = ctx.stream, None
            if tap is not None:
                tap(i, h.clone() if pending is None else
                    h + (pending.to_float32() if hasattr(pending, "to_float32") else
                         pending.ws.sum(0) if isinstance(pending, api.Partial) else pending.to(torch.float32)))
        if ctx.n_want == 0:
            return torch.empty((0, s.vocab_size), dtype=torch.float32, device=rt.device)
        an = add_norm(self.final_norm, h, pending, rt.dtype, rows=ctx.want_rows)
        logits = linear(an, self.head, STORE_F32)
        if s.logit_cap or s.logit_scale != 1.0:
            api.softcap(logits, s.logit_cap, s.logit_scale)
        return logits
