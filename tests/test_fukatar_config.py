"""Fukatar without a GPU: config keys and their errors, the specification that comes out of a config (tensor names and shapes,
cache requests), and the plain implementation's mechanisms against closed forms."""
import copy
import math

import pytest
import torch

import dryft_challenge_htn_2026_b200 as dk
import plain_fukatar as plain
from dryft_challenge_htn_2026_b200.cache import Cache, KVRequest, StateRequest
from dryft_challenge_htn_2026_b200.config.specs import (BigramSpec, DenseMLPSpec, GatedDeltaSpec, LatentAttentionSpec, LayerNormSpec,
                                                        MaskedAttentionSpec, OutputNormLayerSpec, ParallelMixerSpec, RMSNormSpec,
                                                        RotaryPairsSpec, RotaryPartSpec, UnitRMSNormSpec)
from dryft_challenge_htn_2026_b200.engine.model import CausalLM
from dryft_challenge_htn_2026_b200.parts import Runtime, build_part

F = torch.float64
FF = {"kind": "dense", "ff": 56}
ATT = {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.3, "softcap": 20.0,
                                      "rot": {"dims": 12, "base": 700.0, "scaling": {"factor": 3.0, "original": 90, "fast": 6.0, "slow": 1.5}}}, "mlp": FF}
LAT = {"type": "latent_attention", "mixer": {"heads": 3, "dim": 10, "vdim": 14, "kv_rank": 20, "scale": 0.4}, "mlp": None}
PAR = {"type": "parallel", "mixer": {"left": {"heads": 4, "kv_heads": 1, "dim": 8, "vdim": 12, "scale": 0.25, "rot": {"dims": 4, "base": 50.0}},
                                     "right": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 8, "conv": 3}}, "mlp": FF}
CFG = {"architecture": "Fukatar", "vocab": 120, "width": 40, "norm": {"eps": 2e-5}, "logit_softcap": 9.0,
       "embedding": {"scale": 2.5, "bigram": {"buckets": 37, "mul_prev": 11, "mul_cur": 3}}, "layers": [PAR, LAT, ATT]}


def test_config_round_trip_and_what_may_be_left_out():
    cfg = dk.config_from_dict(copy.deepcopy(CFG))
    assert isinstance(cfg, dk.FukatarConfig) and dk.config_from_dict(cfg.to_dict()) == cfg
    small = {"architecture": "Fukatar", "vocab": 50, "width": 16, "norm": {"eps": 1e-6},
             "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 8, "scale": 0.3, "rot": {"dims": 0, "base": 10.0}}, "mlp": None},
                        {"type": "parallel", "mixer": {"left": {"heads": 2, "dim": 8, "scale": 0.3, "rot": {"dims": 8, "base": 10.0}},
                                                       "right": {"heads": 2, "dim": 4, "conv": 1}}}]}
    spec = dk.config_from_dict(small).to_spec()
    a, p = spec.layers[0].mixer, spec.layers[1].mixer
    assert (a.num_kv_heads, a.v_head_dim, a.softcap, a.position) == (2, 8, None, None) and a.value_position == RotaryPartSpec(8, 10.0)
    assert (p.branches[1][1].num_kv_heads, p.branches[1][1].v_head_dim) == (2, 4) and spec.layers[1].feed_forward is None
    assert spec.embed_scale == 1.0 and spec.embed_bigram is None and spec.logit_cap is None


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=23), "must be even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=18), "even and at most"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "'slow' is missing"),
    (lambda c: c["layers"][2]["mixer"].update(softcap=-1.0), "not be negative"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("rot"), "'rot' must be an object"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("conv"), "'conv' is missing"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "'kv_rank' is missing"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not implemented"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "must be positive"),
    (lambda c: c["embedding"]["bigram"].update(mul_prev=-1), "not be negative"),
    (lambda c: c.update(layers=[]), "non-empty list"),
    (lambda c: c.pop("norm"), "'norm' must be an object"),
])
def test_config_errors(change, text):
    c = copy.deepcopy(CFG)
    change(c)
    with pytest.raises(dk.ConfigError, match=text):
        dk.config_from_dict(c)


def test_specification_tensors_and_cache_requests():
    spec = dk.config_from_dict(copy.deepcopy(CFG)).to_spec()
    assert all(isinstance(l, OutputNormLayerSpec) and l.shift == "shift" and l.norm_mix == LayerNormSpec(40, 2e-5) for l in spec.layers)
    assert spec.final_norm == LayerNormSpec(40, 2e-5) and spec.tie_embeddings is False and spec.embed_bigram == BigramSpec(37, 11, 3)
    p, l, a = (x.mixer for x in spec.layers)
    assert isinstance(p, ParallelMixerSpec) and p.out_norm_eps == 2e-5 and [b[2] for b in p.branches] == [0.5, 0.5]
    left, right = p.branches[0][1], p.branches[1][1]
    assert isinstance(left, MaskedAttentionSpec) and left.position == RotaryPairsSpec(4, 50.0) and left.norm_after_rotation \
        and left.qk_norm == UnitRMSNormSpec(8, 2e-5) and left.softcap is None and not left.head_gate
    assert isinstance(right, GatedDeltaSpec) and (right.num_heads, right.num_kv_heads, right.conv_taps, right.unit_eps) == (6, 3, 3, 1e-6)
    assert isinstance(l, LatentAttentionSpec) and l.sink and l.q_rank is None and l.rot_dim == 0 and l.position is None
    assert a.qk_norm == RMSNormSpec(96, 2e-5) and a.qk_norm_whole and a.head_gate and a.softcap == 20.0
    assert a.position == RotaryPartSpec(12, 700.0, (3.0, 90.0, 6.0, 1.5)) and a.value_position == RotaryPartSpec(24, 700.0)
    assert spec.layers[0].feed_forward == DenseMLPSpec(40, 56, "relu2") and spec.layers[1].feed_forward is None
    model = CausalLM(spec, dtype=torch.float32, device="cpu")
    shapes = {n: d.shape for n, d in model.param_decls(False).items()}
    want = {"embed": (120, 40), "bigram": (38, 40), "head": (120, 40), "final.norm": (40,)}
    for i in range(3):
        want.update({f"l{i}.norm1": (40,), f"l{i}.shift": (40,)})
    for i in (0, 2):
        want.update({f"l{i}.norm2": (40,), f"l{i}.mlp.up": (56, 40), f"l{i}.mlp.down": (40, 56)})
    want.update({"l0.mix.left." + n: s for n, s in (("q", (32, 40)), ("k", (8, 40)), ("v", (12, 40)), ("o", (40, 48)), ("out", (40,)))})
    want.update({"l0.mix.right." + n: s for n, s in (
        ("q", (30, 40)), ("k", (30, 40)), ("v", (48, 40)), ("q.conv", (30, 3)), ("k.conv", (30, 3)), ("v.conv", (48, 3)), ("b", (6, 40)),
        ("a", (6, 40)), ("A_log", (6,)), ("dt_bias", (6,)), ("norm", (8,)), ("g", (48, 40)), ("o", (40, 48)), ("out", (40,)))})
    want.update({"l1.mix." + n: s for n, s in (("q", (30, 40)), ("dkv", (20, 40)), ("dkv.norm", (20,)), ("uk", (30, 20)), ("uv", (42, 20)),
                                               ("sink", (3,)), ("o", (40, 42)))})
    want.update({"l2.mix." + n: s for n, s in (("q", (96, 40)), ("k", (32, 40)), ("v", (48, 40)), ("q.norm", (96,)), ("k.norm", (32,)),
                                               ("g", (6, 40)), ("o", (40, 144)))})
    assert shapes == want
    req = model.entry_requests()
    shift = StateRequest((40,), torch.float32)
    assert req[0] == [KVRequest(1, 8, None, torch.float32, 12), StateRequest((6, 10, 8), torch.float32), StateRequest((2, 108), torch.float32), shift]
    assert req[1] == [KVRequest(1, 20, None, torch.float32, 20, values_in_keys=True), shift]
    assert req[2] == [KVRequest(2, 16, None, torch.float32, 24), shift]
    assert req[3] == [StateRequest((1,), torch.int32)]           # the last token of a sequence: the model's own entry
    cache = Cache(req, 64 * 4, 2, "cpu")
    assert cache.views(3)[0].state.shape == (2, 1) and cache.views(1)[0].v is None


def test_what_does_not_go_together_is_refused():
    rt = Runtime(torch.device("cpu"), torch.float32)
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, v_head_dim=8, scale=1.0)
    for bad in (dict(position=RotaryPairsSpec(4, 10.0), bias=True), dict(qk_norm_whole=True), dict(head_gate=True, output_gate=True),
                dict(value_position=RotaryPartSpec(4, 10.0)), dict(value_position=RotaryPartSpec(8, 10.0), conv_taps=3)):
        with pytest.raises(ValueError):
            build_part(MaskedAttentionSpec(**base, **bad), rt)
    with pytest.raises(ValueError):
        build_part(ParallelMixerSpec(16, tuple((f"{i}.", MaskedAttentionSpec(**base), 0.3 * i) for i in range(2)), out_norm_eps=1e-5), rt)
    with pytest.raises(ValueError):
        build_part(GatedDeltaSpec(16, 4, 3, 8, 8, 4, 1e-5), rt)


def test_stretched_positions_keep_fast_pairs_and_divide_slow_ones():
    part = build_part(RotaryPartSpec(32, 10000.0, (4.0, 256, 32.0, 1.0)), Runtime(torch.device("cpu"), torch.float32))
    cos, sin = part.tables(200)
    f = [10000.0 ** (-2 * i / 32) for i in range(16)]
    at = lambda turns: 32 * math.log(256 / (2 * math.pi * turns)) / (2 * math.log(10000.0))
    lo, hi = math.floor(at(32.0)), math.ceil(at(1.0))
    assert 0 <= lo < hi < 16
    mag = 1 + 0.1 * math.log(4.0)
    for i, want in ((0, f[0]), (lo, f[lo]), (hi, f[hi] / 4), (15, f[15] / 4), (lo + 1, f[lo + 1] * (1 - 1 / (hi - lo)) + f[lo + 1] / 4 / (hi - lo))):
        for p in (1, 199):
            assert abs(float(cos[p, i]) - mag * math.cos(p * want)) < 3e-5 and abs(float(sin[p, i]) - mag * math.sin(p * want)) < 3e-5, i
    fp, m = plain.frequencies(32, 10000.0, {"factor": 4.0, "original": 256, "fast": 32.0, "slow": 1.0})
    assert m == mag and abs(fp[hi] - f[hi] / 4) < 1e-12 and fp[0] == f[0]


def test_plain_mechanisms_against_closed_forms():
    # layer norm: mean off, over the deviation, eps inside
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F)
    assert torch.allclose(plain.layer_norm(x, torch.ones(4, dtype=F), 4.0), torch.tensor([[-1.0, -1 / 3, 1 / 3, 1.0]], dtype=F))
    # the shift: a share of one reads the token before, of zero this one; zeros ahead of the first
    x = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]], dtype=F)
    assert plain.token_shift(x, torch.tensor([1.0, 0.25], dtype=F)).tolist() == [[0.0, 7.5], [1.0, 17.5], [2.0, 27.5]]
    assert plain.token_shift(x[1:], torch.ones(2, dtype=F), x[0]).tolist() == x[:2].tolist()
    # pairs of tokens: the last row first, then (previous * a + this * b) mod buckets
    p = {"embed": torch.zeros(10, 1, dtype=F), "bigram": torch.arange(8, dtype=F)[:, None]}
    cfg = {"embedding": {"scale": 2.0, "bigram": {"buckets": 7, "mul_prev": 3, "mul_cur": 5}}}
    assert plain.embed([4, 9, 0], p, cfg).flatten().tolist() == [7.0, (12 + 45) % 7, 27 % 7]
    # a rotation by pairs and by halves is the same up to the order of the coordinates, and turning back undoes it
    v = torch.randn(3, 2, 8, generator=torch.Generator().manual_seed(0), dtype=F)
    f, pos = plain.frequencies(6, 5.0)[0], torch.tensor([0, 4, 9])
    order = [0, 2, 4, 1, 3, 5, 6, 7]
    assert torch.allclose(plain.turn(v, pos, 6, f, pairs=True)[..., order], plain.turn(v[..., order], pos, 6, f))
    for pairs in (False, True):
        assert torch.allclose(plain.turn(plain.turn(v, pos, 6, f, pairs=pairs), pos, 6, f, pairs=pairs, back=True), v)
    # values that turn: with one key of all the weight the output is that value turned by j - i
    w = plain.softmax_causal(torch.tensor([[0.0, 0.0], [50.0, -50.0]], dtype=F))
    assert torch.allclose(w[1], torch.tensor([1.0, 0.0], dtype=F)) and w[0].tolist() == [1.0, 0.0]
    # a sink takes its share and gives nothing; a large one takes all
    w = plain.softmax_causal(torch.zeros(3, 3, dtype=F), torch.tensor(math.log(2.0), dtype=F))
    assert torch.allclose(w.sum(-1), torch.tensor([1 / 3, 2 / 4, 3 / 5], dtype=F))
    assert float(plain.softmax_causal(torch.zeros(3, 3, dtype=F), torch.tensor(800.0, dtype=F)).sum()) < 1e-9
    # the cap holds scores inside it and is the identity near zero
    assert abs(float(plain.soft_cap(torch.tensor(1e9, dtype=F), 5.0)) - 5.0) < 1e-12 and abs(float(plain.soft_cap(torch.tensor(1e-4, dtype=F), 5.0)) - 1e-4) < 1e-12
    assert plain.squared_relu(torch.tensor([-2.0, 0.0, 3.0], dtype=F)).tolist() == [0.0, 0.0, 9.0]
    # the delta rule with unit orthogonal keys, no decay and full steps is a table of values, the last write of a key wins
    k = torch.eye(2, dtype=F)[[0, 1, 0]][:, None]
    v = torch.tensor([[1.0, 2.0], [3.0, 4.0], [5.0, 6.0]], dtype=F)[:, None]
    one = torch.ones(3, 1, dtype=F)
    o, S = plain.delta_rule(k, k, v, one, one, torch.zeros(1, 2, 2, dtype=F))
    assert o[:, 0].tolist() == v[:, 0].tolist() and S[0].tolist() == [[5.0, 6.0], [3.0, 4.0]]
    o, S = plain.delta_rule(k, k, v, 0.5 * one, 0.5 * one, torch.zeros(1, 2, 2, dtype=F))
    assert S[0, 0].tolist() == [0.25 * 0.5 + 0.5 * (5.0 - 0.25 * 0.5), 0.25 + 0.5 * (6.0 - 0.25)]     # decayed twice, then halfway to the new value


def test_plain_recurrence_does_not_depend_on_how_a_sequence_is_cut():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F) * 0.5
    W, H, G, D, V, taps = 12, 4, 2, 6, 3, 3
    p = {"q": r(G * D, W), "k": r(G * D, W), "v": r(H * V, W), "q.conv": r(G * D, taps), "k.conv": r(G * D, taps), "v.conv": r(H * V, taps),
         "b": r(H, W), "a": r(H, W), "A_log": r(H), "dt_bias": r(H), "norm": 1 + r(V), "g": r(H * V, W), "o": r(W, H * V)}
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V}
    x = r(9, W)
    whole, _ = plain.gated_delta(x, p, m, 1e-5)
    state, got = None, []
    for a, b in ((0, 4), (4, 5), (5, 7), (7, 9)):
        y, state = plain.gated_delta(x[a:b], p, m, 1e-5, state)
        got.append(y)
    assert torch.allclose(torch.cat(got), whole, atol=1e-12)
