"""Mozutar without a GPU: config keys and their errors, the specification that comes out of a config (tensor names and shapes,
cache requests, the loop's runs), what does not go together, the chunks a portion is cut into, and the plain implementation's
mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

import dryft_challenge_htn_2026_b200 as dk
import plain_mozutar as plain
from dryft_challenge_htn_2026_b200.cache import Cache, KVRequest, StateRequest
from dryft_challenge_htn_2026_b200.config.specs import (GatedLinearAttentionSpec, GatedMLPSpec, GroupRMSNormSpec, LayerNormSpec, MaskedAttentionSpec,
                                                        MatrixMemorySpec, ParallelMixerSpec, RMSNormSpec, RotaryPartSpec, RoutedMLPSpec,
                                                        SandwichLayerSpec, ScheduleEntry)
from dryft_challenge_htn_2026_b200.engine.model import CausalLM
from dryft_challenge_htn_2026_b200.parts import Runtime, build_part
from dryft_challenge_htn_2026_b200.parts.matrix_memory import MemoryChunks

F = torch.float64
MEM = {"type": "mlstm", "mixer": {"heads": 3, "dim": 10, "vdim": 14, "gate_cap": 6.0}, "mlp": {"kind": "dense", "ff": 56}}
MOE = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 7, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 2}}}
PAR = {"type": "parallel", "mixer": {"left": {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 12, "scale": 0.25, "softcap": 9.0, "rot": {"dims": 8, "base": 50.0}},
                                     "right": {"heads": 4, "dim": 10, "vdim": 8, "tau": 4.0}}, "mlp": MOE}
CFG = {"architecture": "Mozutar", "vocab": 120, "width": 40, "norm": {"eps": 2e-5}, "embedding": {"scale": 2.5},
       "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [PAR, MEM, dict(MEM, mlp=None)]}


def test_config_round_trip_and_what_may_be_left_out():
    cfg = dk.config_from_dict(copy.deepcopy(CFG))
    assert isinstance(cfg, dk.MozutarConfig) and dk.config_from_dict(cfg.to_dict()) == cfg
    small = {"architecture": "Mozutar", "vocab": 50, "width": 16, "norm": {"eps": 1e-6},
             "layers": [{"type": "mlstm", "mixer": {"heads": 2, "dim": 8, "gate_cap": 3.0}, "mlp": None},
                        {"type": "parallel", "mixer": {"left": {"heads": 2, "dim": 8, "scale": 0.3}, "right": {"heads": 2, "dim": 4}},
                         "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 4, "top": 1}}}]}
    spec = dk.config_from_dict(small).to_spec()
    m, p = spec.layers[0].mixer, spec.layers[1].mixer
    left, right = p.branches[0][1], p.branches[1][1]
    assert m.v_head_dim == 8 and (left.num_kv_heads, left.v_head_dim, left.softcap, left.position) == (2, 8, None, None)
    assert (right.v_head_dim, right.tau) == (4, 1.0)
    ff = spec.layers[1].feed_forward
    assert (ff.identity, ff.groups, ff.keep_groups) == (0, 1, 1) and spec.layers[0].feed_forward is None
    assert spec.embed_scale == 1.0 and spec.tables == () and spec.matrices == () and all(e.take_in is None for e in spec.schedule)


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=10), "values are the keys"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "not be negative"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14), "even and at most"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=3), "even and at most"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0.0), "must be positive"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "'right' must be an object"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "'gate_cap' is missing"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0), "must be positive"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=3), "do not fit together"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "do not fit together"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "do not fit together"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "do not fit together"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "not implemented"),
    (lambda c: c["loop"].update(stop=4), "does not lie within"),
    (lambda c: c["loop"].update(times=0), "must be positive"),
    (lambda c: c.update(decay_rank=[4]), "one entry per layer"),
    (lambda c: c.update(layers=[]), "non-empty list"),
    (lambda c: c.pop("norm"), "'norm' must be an object"),
])
def test_config_errors(change, text):
    c = copy.deepcopy(CFG)
    change(c)
    with pytest.raises(dk.ConfigError, match=text):
        dk.config_from_dict(c)


def test_specification_tensors_and_cache_requests():
    cfg = dk.config_from_dict(copy.deepcopy(CFG)).with_shapes({"l0.mix.right.a1": (5, 40), "l1.mix.q": (30, 40)})
    assert cfg.decay_rank == (5, None, None) and dk.config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.to_spec()
    norm = LayerNormSpec(40, 2e-5, bias=".b")
    assert all(isinstance(l, SandwichLayerSpec) and l.layer_scale == ("ls1", "ls2") and l.norm_in == norm and l.norm_mix_out == norm for l in spec.layers)
    assert spec.final_norm == norm and spec.tie_embeddings is True and spec.embed_scale == 2.5
    p = spec.layers[0].mixer
    assert isinstance(p, ParallelMixerSpec) and p.out_norm_eps == 2e-5 and [b[2] for b in p.branches] == [0.5, 0.5]
    left, right = p.branches[0][1], p.branches[1][1]
    assert isinstance(left, MaskedAttentionSpec) and left.keys_as_values and left.qk_norm == RMSNormSpec(12, 2e-5) and left.softcap == 9.0 \
        and left.position == RotaryPartSpec(8, 50.0) and not left.norm_after_rotation and left.scale == 0.25
    assert isinstance(right, GatedLinearAttentionSpec) and (right.decay_rank, right.tau) == (5, 4.0)
    assert spec.layers[1].mixer == MatrixMemorySpec(40, 3, 10, 14, 6.0, 2e-5)
    assert spec.layers[0].feed_forward == RoutedMLPSpec(40, 24, 7, 2, 3, 2, renorm=False, scores="softmax", group_top=1, identity=2)
    assert spec.layers[1].feed_forward == GatedMLPSpec(40, 56, "silu", names=("gate", "up", "down")) and spec.layers[2].feed_forward is None
    model = CausalLM(spec, dtype=torch.float32, device="cpu")
    shapes = {n: d.shape for n, d in model.param_decls(True).items()}
    want = {"embed": (120, 40), "final.norm": (40,), "final.norm.b": (40,), "loop.in": (40, 80), "loop.step": (2, 40)}
    for i in range(3):
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if i < 2 else ()):
            want.update({f"l{i}.{n}": (40,), f"l{i}.{n}.b": (40,)})
        want.update({f"l{i}.ls1": (40,)})
    want.update({"l0.ls2": (40,), "l1.ls2": (40,)})
    want.update({"l0.mix.left." + n: s for n, s in (("q", (72, 40)), ("k", (36, 40)), ("q.norm", (12,)), ("k.norm", (12,)), ("o", (40, 72)), ("out", (40,)))})
    want.update({"l0.mix.right." + n: s for n, s in (("q", (40, 40)), ("k", (40, 40)), ("v", (32, 40)), ("g", (32, 40)), ("o", (40, 32)), ("norm", (8,)),
                                                     ("a1", (5, 40)), ("a2", (40, 5)), ("a2.b", (40,)), ("out", (40,)))})
    want.update({f"l0.mlp.e{e}.{n}": s for e in range(7) for n, s in (("gate", (24, 40)), ("up", (24, 40)), ("down", (40, 24)))})
    want.update({"l0.mlp.router": (9, 40), "l0.mlp.correction": (9,)})
    for i in (1, 2):
        want.update({f"l{i}.mix." + n: s for n, s in (("q", (30, 40)), ("k", (30, 40)), ("v", (42, 40)), ("g", (42, 40)), ("o", (40, 42)), ("norm", (42,)),
                                                      ("i", (3, 40)), ("i.b", (3,)), ("f", (3, 40)), ("f.b", (3,)))})
    want.update({"l1.mlp.gate": (56, 40), "l1.mlp.up": (56, 40), "l1.mlp.down": (40, 56)})
    assert shapes == want
    # two passes of layers 0 and 1, each with an entry of its own, then layer 2
    assert [(e.layer, e.cache, e.take_in, e.add_row) for e in spec.schedule] == [
        (0, 0, "loop.in", ("loop.step", 0)), (1, 1, None, None), (0, 2, "loop.in", ("loop.step", 1)), (1, 3, None, None), (2, 4, None, None)]
    req = model.entry_requests()
    par = [KVRequest(3, 12, None, torch.float32, 12), StateRequest((4, 10, 8), torch.float32)]
    mem = [StateRequest((3, 10, 14), torch.float32), StateRequest((3, 10), torch.float32), StateRequest((3,), torch.float32)]
    assert req == [par, mem, par, mem, mem]
    cache = Cache(req, 64 * 4, 2, "cpu")
    assert [v.state.shape for v in cache.views(1)] == [(2, 3, 10, 14), (2, 3, 10), (2, 3)] and float(cache.views(1)[2].state.abs().max()) == 0.0


def test_a_loop_without_layers_has_its_tensors_and_no_passes():
    c = dict(copy.deepcopy(CFG), loop={"start": 2, "stop": 2, "times": 3})
    spec = dk.config_from_dict(c).to_spec()
    assert [(e.layer, e.take_in) for e in spec.schedule] == [(0, None), (1, None), (2, None)]
    assert spec.tables == (("loop.step", (3, 40)),) and spec.matrices == (("loop.in", (40, 80)),)


def test_what_does_not_go_together_is_refused():
    rt = Runtime(torch.device("cpu"), torch.float32)
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, scale=1.0, keys_as_values=True)
    for bad in (dict(v_head_dim=4), dict(v_head_dim=8, conv_taps=3), dict(v_head_dim=8, bias=True), dict(v_head_dim=8, value_mix="source")):
        with pytest.raises(ValueError):
            build_part(MaskedAttentionSpec(**base, **bad), rt)
    for bad in (dict(gate_cap=0.0), dict(head_dim=300)):
        with pytest.raises(ValueError):
            build_part(MatrixMemorySpec(**{**dict(hidden_size=16, num_heads=2, head_dim=8, v_head_dim=8, gate_cap=1.0, norm_eps=1e-5), **bad}), rt)
    for bad in (dict(scores="linear"), dict(group_top=3), dict(identity=1), dict(identity=-2), dict(identity=2, top=8, groups=4, keep_groups=1)):
        with pytest.raises(ValueError):
            build_part(RoutedMLPSpec(**{**dict(hidden_size=16, expert_ff=8, num_experts=6, top=2, groups=2, keep_groups=1), **bad}), rt)
    norm, rms, mem = LayerNormSpec(16, 1e-5), RMSNormSpec(16, 1e-5), MatrixMemorySpec(16, 2, 8, 8, 1.0, 1e-5)
    for n_in, n_out in ((rms, norm), (GroupRMSNormSpec(16, 1e-5, 2), norm)):       # what follows a sum takes such an output norm, or is refused
        with pytest.raises(TypeError):
            build_part(SandwichLayerSpec("l0.", n_in, mem, n_out, None, None, None), rt)
    # a run that takes the embedding in wants a matrix of the model of that shape, and does not add it as well
    spec = dk.config_from_dict(copy.deepcopy(CFG)).to_spec()
    for entry, matrices in ((ScheduleEntry(0, 0, take_in="loop.in"), (("loop.in", (40, 40)),)), (ScheduleEntry(0, 0, take_in="other"), spec.matrices),
                            (ScheduleEntry(0, 0, take_in="loop.in", add_embedding=True), spec.matrices)):
        from dataclasses import replace
        with pytest.raises(ValueError):
            CausalLM(replace(spec, schedule=(entry,), matrices=matrices), dtype=torch.float32, device="cpu")


@pytest.mark.parametrize("lens", [[1], [255], [256], [257], [600, 3, 256, 1], [16, 16], [4, 200, 900]])
def test_chunks_of_a_portion_cover_every_row_once(lens):
    plan = MemoryChunks(256).build(np.array(lens), np.zeros(len(lens)), False)
    if sum(lens) < 16 * len(lens):
        assert plan.shape == (0, 4)
        return
    firsts, chunks = plan[:len(lens)], plan[len(lens):]
    seen = []
    for s, n in enumerate(lens):
        start = sum(lens[:s])
        own = chunks[firsts[s, 0]:firsts[s, 0] + firsts[s, 1]]
        assert (own[:, 0] == s).all() and own[:, 3].tolist() == list(range(len(own))) and (own[:, 2] > 0).all() and (own[:, 2] <= 256).all()
        assert ((own[:, 1] - start) % 256 == 0).all()
        seen += [r for _, a, k, _ in own.tolist() for r in range(a, a + k)]
    assert seen == list(range(sum(lens))) and len(chunks) == firsts[:, 1].sum()
    assert MemoryChunks(256).build(np.ones(3), np.zeros(3), True).shape == (0, 4)


def test_plain_mechanisms_against_closed_forms():
    t = lambda *v: torch.tensor(v, dtype=F)
    # layer norm: mean off, over the deviation, eps inside, weight, then bias
    x = t(1.0, 3.0, 5.0, 7.0)[None]
    assert torch.allclose(plain.layer_norm(x, 3 * torch.ones(4, dtype=F), t(1.0, 0.0, 0.0, -1.0), 4.0), t(-2.0, -1.0, 1.0, 2.0)[None])
    # half the head turns by position times base^(-2i/dims), the rest passes
    v = t(1.0, 0.0, 0.0, 2.0, 9.0).reshape(1, 1, 5)
    y = plain.rotate_halves(v, torch.tensor([3]), 4, 100.0)[0, 0]
    assert torch.allclose(y, t(math.cos(3.0), -2 * math.sin(0.3), math.sin(3.0), 2 * math.cos(0.3), 9.0))
    # values are the keys ahead of norm and rotation: one token returns its raw key
    p = {"q": torch.eye(2, dtype=F), "k": torch.eye(2, dtype=F), "q.norm": t(1.0, 1.0), "k.norm": t(5.0, 7.0), "o": torch.eye(2, dtype=F)}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    assert torch.allclose(plain.keys_as_values_attention(t(3.0, -4.0)[None], p, m, 1e-9), t(3.0, -4.0)[None])
    # the log gates: capped, the forget gate below zero
    p = {"i": t(1.0)[None], "i.b": t(0.5), "f": t(-1.0)[None], "f.b": t(0.0)}
    i, f = plain.exponential_gates(t(1e9, -0.5)[:, None], p, 4.0)
    assert abs(float(i[0, 0]) - 4.0) < 1e-12 and float(i[1, 0]) == 0.0 and abs(float(f[0, 0]) - math.log(1 / (1 + math.exp(4.0)))) < 1e-12
    # the memory's first token: the maximum starts at zero, so a weak write is small beside exp(-m) = 1 and is not blown up
    q = k = t(1.0, 0.0).reshape(1, 1, 2)
    val = t(6.0).reshape(1, 1, 1)
    o, (S, n, mx) = plain.matrix_memory(q, k, val, t(-3.0)[None], t(-0.1)[None])
    assert abs(float(mx) + 0.1) < 1e-12                                   # max(f + 0, i)
    assert abs(float(o) - 6.0 * math.exp(-2.9) / (math.exp(0.1) + 1e-6)) < 1e-9
    # a strong write: the maximum takes it, the quotient is the value
    o, (S, n, mx) = plain.matrix_memory(q, k, val, t(9.0)[None], t(-0.1)[None])
    assert float(mx) == 9.0 and abs(float(o) - 6.0 / (1 + 1e-6)) < 1e-9 and float(n[0, 0]) == 1.0
    # the running maximum changes nothing but the floor and the 1e-6: without them the quotient is the plain weighted mean
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F)
    T = 7
    k, val = r(T, 1, 3).abs(), r(T, 1, 2)
    q = r(T, 1, 3).abs() * 50
    i, f = r(T, 1) + 5, -r(T, 1).abs()
    o, _ = plain.matrix_memory(q, k, val, i, f)
    w = torch.tensor([math.exp(float(f[s + 1:].sum() + i[s])) for s in range(T)], dtype=F) * (k[:, 0] @ q[-1, 0])
    assert torch.allclose(o[-1, 0], (w[:, None] * val[:, 0]).sum(0) / w.sum(), rtol=1e-6)
    # the router: negative choice scores, a group left out, weights without the correction, not renormalized
    p = {"router": torch.eye(4, dtype=F), "correction": t(-2.0, -9.0, -1.5, -9.0)}
    z = t(0.0, 3.0, 0.0, 3.0)
    s = torch.softmax(z, 0)
    assert plain.route(z[None], p, {"experts": 3, "identity": 1, "top": 2, "groups": {"count": 2, "keep": 1}}) == [([2, 3], [float(s[2]), float(s[3])])]
    assert plain.route(z[None], p, {"experts": 4, "top": 2}) == [([2, 0], [float(s[2]), float(s[0])])]
    # an identity expert passes the input on, times its score
    y = plain.mixture(z[None], p, {"experts": 0, "identity": 4, "top": 1})
    assert torch.allclose(y, float(s[2]) * z[None])
    # what opens a pass
    assert torch.allclose(plain.take_in(t(1.0)[None], t(10.0)[None], t(2.0, 3.0)[None], t(0.5)), t(32.5)[None])


def test_plain_recurrences_do_not_depend_on_how_a_sequence_is_cut():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F) * 0.5
    W, H, D, V, R = 12, 2, 6, 3, 4
    p = {"q": r(H * D, W), "k": r(H * D, W), "v": r(H * V, W), "g": r(H * V, W), "o": r(W, H * V), "norm": 1 + r(H * V), "i": r(H, W), "i.b": r(H),
         "f": r(H, W), "f.b": r(H), "a1": r(R, W), "a2": r(H * D, R), "a2.b": r(H * D)}
    x = r(9, W)
    for run, m, norm in ((plain.mlstm, {"heads": H, "dim": D, "vdim": V, "gate_cap": 5.0}, p["norm"]),
                         (plain.gated_linear_attention, {"heads": H, "dim": D, "vdim": V, "tau": 3.0}, p["norm"][:V])):
        q = {**p, "norm": norm}
        whole, _ = run(x, q, m, 1e-5)
        state, got = None, []
        for a, b in ((0, 4), (4, 5), (5, 7), (7, 9)):
            y, state = run(x[a:b], q, m, 1e-5, state)
            got.append(y)
        assert torch.allclose(torch.cat(got), whole, atol=1e-12)


def test_plain_loop_runs_its_span_again_with_a_vector_and_the_embedding_for_each_pass():
    assert plain.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert plain.runs({"layers": [0] * 2}) == [(0, None), (1, None)] and plain.runs({"layers": [0], "loop": {"start": 0, "stop": 1, "times": 1}}) == [(0, 0)]
