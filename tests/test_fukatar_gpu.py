"""The Fukatar decoder in the library against the plain implementation (``plain_fukatar``): every mechanism alone, then whole
models of several small shapes through the step function, the cache, the decode state and the entry points. The shapes differ
in every size and option: layers in any order, layers without feed-forward (also the last), key/value groups of 1 to 4, key
and value sizes that differ, rotations over the whole head, a part of it and none, with and without stretched positions and
capped scores, latents narrower and wider than the heads and wider than 256, convolutions of 1 to 7 taps, models without
token pairs, embedding scale or capped logits, head sizes the tensor-core kernels take and ones they do not."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import dryft_challenge_htn_2026_b200 as dk
import plain_fukatar as plain
from dryft_challenge_htn_2026_b200.config.specs import (DenseMLPSpec, GatedDeltaSpec, LatentAttentionSpec, LayerNormSpec,
                                                        MaskedAttentionSpec, ParallelMixerSpec, RMSNormSpec, RotaryPairsSpec,
                                                        RotaryPartSpec, UnitRMSNormSpec)
from dryft_challenge_htn_2026_b200.csrc import api
from dryft_challenge_htn_2026_b200.engine import DecodeLoop, Runner, load_model
from dryft_challenge_htn_2026_b200.parts import Runtime, build_part
from helpers import ROOT, random_tokens
from part_helpers import DEV, Errors, bound_part, close, dev, rnd, run_cut, tol, whole

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
CUTS = [131, 2, 1, 1, 40, 1, 1, 1, 90]
EPS = 1e-5


def dense(ff):
    return {"kind": "dense", "ff": ff}


def heads_of(H, G, D, V, scale, rot, cap):
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "rot": {"dims": rot[0], "base": rot[1]}}
    if len(rot) > 2:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2:]))
    if cap:
        m["softcap"] = cap
    return m


def att(H, G, D, V, scale, rot, cap, mlp):
    return {"type": "attention", "mixer": heads_of(H, G, D, V, scale, rot, cap), "mlp": mlp}


def lat(H, D, V, rank, scale, mlp):
    return {"type": "latent_attention", "mixer": {"heads": H, "dim": D, "vdim": V, "kv_rank": rank, "scale": scale}, "mlp": mlp}


def par(left, right, mlp):
    return {"type": "parallel", "mixer": {"left": heads_of(*left),
                                          "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))}, "mlp": mlp}


SHAPES = {
    # sizes the mma.sync kernels take; a last layer without feed-forward; more value than key size on one layer, less on another
    "A": dict(architecture="Fukatar", vocab=200, width=64, norm={"eps": 1e-5}, logit_softcap=12.0,
              embedding={"scale": 3.0, "bigram": {"buckets": 97, "mul_prev": 13, "mul_cur": 5}},
              layers=[lat(4, 16, 32, 48, 0.3, dense(80)), att(4, 2, 32, 48, 0.5, (16, 500.0, 4.0, 60, 8.0, 1.0), 9.0, dense(96)),
                      par((6, 2, 48, 16, 0.4, (48, 1000.0), 15.0), (6, 2, 16, 32, 3), None),
                      att(3, 1, 64, 16, 0.2, (64, 10000.0), None, None), par((2, 2, 16, 32, 0.3, (8, 50.0), None), (3, 3, 32, 16, 2), None)]),
    # sizes that no tensor-core kernel takes; no pairs, no scale, no caps; a convolution of one tap (no memory)
    "B": dict(architecture="Fukatar", vocab=136, width=44, norm={"eps": 3e-4},
              layers=[par((3, 1, 20, 10, 0.5, (6, 30.0), 5.0), (4, 1, 12, 10, 1), dense(52)),
                      att(3, 3, 12, 6, 0.6, (0, 100.0), None, dense(36)), lat(3, 10, 6, 20, 0.7, None),
                      att(4, 1, 22, 14, 0.3, (22, 200.0, 2.0, 40, 1.0, 1.0), 7.0, dense(44))]),
    # sizes of the tcgen05 kernels on both kinds of attention, a latent wider than 256, keys of 128 in the delta rule, 7 taps
    "C": dict(architecture="Fukatar", vocab=320, width=128, norm={"eps": 1e-6}, logit_softcap=40.0,
              embedding={"scale": 0.7, "bigram": {"buckets": 1, "mul_prev": 3, "mul_cur": 1}},
              layers=[att(4, 1, 64, 64, 0.4, (32, 10000.0, 8.0, 100, 16.0, 2.0), 30.0, dense(192)), lat(3, 64, 48, 288, 0.2, dense(160)),
                      par((2, 1, 128, 128, 0.3, (128, 1e6), 25.0), (2, 1, 128, 64, 7), dense(128)),
                      lat(8, 32, 16, 112, 0.4, None), att(2, 2, 128, 128, 0.1, (64, 300.0), None, dense(64))]),
    # only recurrences' neighbours without a cap, as many key heads as heads, state sizes in between
    "D": dict(architecture="Fukatar", vocab=264, width=96, norm={"eps": 1e-5}, logit_softcap=5.0, embedding={"scale": 2.0},
              layers=[par((4, 4, 32, 64, 0.3, (2, 7.0), None), (4, 4, 48, 24, 4), dense(72)),
                      par((8, 2, 64, 64, 0.2, (64, 5000.0), 50.0), (6, 3, 100, 36, 5), dense(88)), lat(1, 16, 16, 16, 1.0, dense(104))]),
}


def make_model(tmp_path, name, seed=0):
    cfg = dk.config_from_dict(SHAPES[name])
    folder = str(tmp_path / f"fukatar{name}_{seed}")
    dk.write_random_model(cfg, folder, seed=seed, dtype=torch.float32, matrix_std=0.08)
    return folder, cfg


# ------------------------------------------------------------------------------------ the stream
def sequence_case(lens, cached):
    """Rows of sequences that bring ``lens`` tokens after ``cached`` ones, on slots 2, 3, ..: what the kernels take."""
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    pos = [c + j for n, c in zip(lens, cached) for j in range(n)]
    seq = [s for s, n in enumerate(lens) for _ in range(n)]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return i32(pos), i32(seq), i32(cu), i32([2 + s for s in range(len(lens))])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [48, 50, 1000, 2560, 4100, 9000])
def test_a_sublayers_output_normed_added_and_mixed_with_the_token_before(dtype, W):
    """x = h + norm(d), then x + (x_prev - x) share: with one output, with two each normed first, as split-K partial sums, with
    none; rows at the start, in the middle and at the end of runs of rows and sequences."""
    lens = [3, 1, 9, 700] if W <= 1000 else [3, 1, 9]
    seqs = sequence_case(lens, [0, 5, 64, 2])
    n = sum(lens)
    h0, d0, d1 = rnd(n, W, seed=1, scale=3.0).float().double(), rnd(n, W, seed=2, scale=0.4) + 0.7, rnd(n, W, seed=3, scale=5.0)
    d0, d1 = d0.to(dtype).double(), d1.to(dtype).double()
    w, w0, w1, share = ((1 + 0.2 * rnd(W, seed=s)).float().double() for s in (4, 5, 6, 7))
    state = rnd(8, W, seed=8).float().double()
    f32 = lambda x: dev(x, torch.float32)
    first = [0]
    for k in lens[:-1]:
        first.append(first[-1] + k)

    def shifted(x):
        return torch.cat([plain.token_shift(x[a:a + k], share, state[2 + s]) for s, (a, k) in enumerate(zip(first, lens))])

    halves = torch.stack([f32(d0 * 0.25), f32(d0 * 0.75)]).contiguous()
    both = plain.side_by_side(d0, d1, {"left.out": w0, "right.out": w1}, EPS)
    cases = [("one", dev(d0, dtype), plain.layer_norm(d0, w, EPS), (f32(w), EPS, True)),
             ("rms", dev(d0, dtype), plain.rms(d0, EPS) * w, (f32(w), EPS, False)),
             ("partial sums", api.Partial(halves), plain.layer_norm(d0, w, EPS), (f32(w), EPS, True)),
             ("two", api.NormedSum([dev(d0, dtype), dev(d1, dtype)], [f32(w0), f32(w1)], EPS, 0.5), plain.layer_norm(both, w, EPS), (f32(w), EPS, True)),
             ("two without a norm", api.NormedSum([api.Partial(halves), dev(d1, dtype)], [f32(w0), f32(w1)], EPS, 0.5), both, None),
             ("none", None, torch.zeros_like(h0), None)]
    for what, delta, add, norm in cases:
        h, x, a = f32(h0), torch.empty(n, W, device=DEV), torch.empty(n, W, dtype=dtype, device=DEV)
        api.sublayer_add_shift(h, delta, norm, f32(share), f32(state), seqs, a, h_out=None if delta is None else x)
        if delta is not None:
            close(x, h0 + add, torch.float32, what + ": stream", slack=0.1)
        assert torch.equal(h.cpu().double(), h0)
        close(a, shifted(h0 + add), dtype, what + ": shifted", slack=0.25)
        # the same sum in place; the state takes the stream as it stood before, at every sequence's last row
        st = f32(state)
        api.sublayer_add(h, delta, norm, a, h_out=h, save=st, seqs=seqs)
        close(h, h0 + add, torch.float32, what + ": in place", slack=0.1)
        close(a, h0 + add, dtype, what + ": as the next sublayer reads it", slack=0.25)
        want = state.clone()
        for s, (a0, k) in enumerate(zip(first, lens)):
            want[2 + s] = h0[a0 + k - 1]
        assert torch.equal(st.cpu().double(), want), what
        # gathered rows with a norm behind the sum; the stream stays
        rows = torch.tensor([n - 1, 0, 3], dtype=torch.int32, device=DEV)
        h, few = f32(h0), torch.empty(3, W, dtype=dtype, device=DEV)
        api.sublayer_add(h, delta, norm, few, rows=rows, next_norm=(f32(w1), EPS, True))
        close(few, plain.layer_norm((h0 + add)[[n - 1, 0, 3]], w1, EPS), dtype, what + ": wanted rows", slack=0.25)
        assert torch.equal(h.cpu().double(), h0)
    # single tokens: no list of first rows, every row reads its own state; a padding row leaves the states alone
    pos, seq, _, slots = sequence_case([1, 1, 1], [4, 0, 9])
    pos[1] = -1
    a, st = torch.empty(3, W, dtype=dtype, device=DEV), f32(state)
    api.sublayer_add_shift(f32(h0[:3]), dev(d0[:3], dtype), (f32(w), EPS, True), f32(share), st, (pos, seq, None, slots), a, h_out=torch.empty(3, W, device=DEV))
    x = h0[:3] + plain.layer_norm(d0[:3], w, EPS)
    close(a[[0, 2]], (x + (state[2:5] - x) * share)[[0, 2]], dtype, "single tokens", slack=0.25)
    api.stream_save(f32(x), st, None, pos, slots, 3)
    assert torch.equal(st[3].cpu().double(), state[3])
    close(st[[2, 4]], x[[0, 2]], torch.float32, "saved", slack=0.1)


def test_layer_norm_takes_the_mean_off_before_it_squares_and_eps_stands_inside():
    """A row far from zero with small deviations (squares minus the squared mean would lose them), and one where eps decides."""
    x = torch.stack([1000.0 + 0.01 * rnd(64, seed=1), 1e-3 * rnd(64, seed=2), rnd(64, seed=3)]).float().double()
    part, p = bound_part(LayerNormSpec(64, 1e-5), torch.float32)
    out = part.add_forward(dev(x, torch.float32), None, torch.empty(3, 64, device=DEV))
    ref = plain.layer_norm(x, p[""], 1e-5)
    assert float((out.cpu().double() - ref).abs().max()) < 2e-2 and float((out[1:].cpu().double() - ref[1:]).abs().max()) < 1e-5
    assert float(out[1].abs().max()) < 1.5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,mul_prev,mul_cur,vocab", [(97, 13, 5, 200), (1, 7, 3, 40), (100003, 92821, 68917, 150000), (64, 0, 1, 64), (31, 1, 0, 90)])
def test_rows_of_token_pairs_in_prompts_portions_and_single_tokens(dtype, buckets, mul_prev, mul_cur, vocab):
    W, scale = 24, 1.7
    e, b = rnd(vocab, W, seed=1).to(dtype), rnd(buckets + 1, W, seed=2).to(dtype)
    tokens = [random_tokens(vocab, n, s) for s, n in enumerate([12, 9])]
    tokens[0][3] = tokens[0][4] = vocab - 1
    cfg = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    ref = [plain.embed(t, {"embed": e.double(), "bigram": b.double()}, cfg) for t in tokens]
    state = torch.full((6, 1), 17, dtype=torch.int32, device=DEV)
    at = [0, 0]
    for lens in ([4, 3], [1, 1], [2, 1], [1, 1], [4, 3]):
        pos, seq, cu, slots = sequence_case(lens, at)
        tok = torch.tensor([t for i in range(2) for t in tokens[i][at[i]:at[i] + lens[i]]], dtype=torch.int32, device=DEV)
        h = torch.empty(sum(lens), W, device=DEV)
        api.embed_bigram(tok, e.to(DEV), scale, b.to(DEV), mul_prev, mul_cur, state,
                         (pos, seq, None if lens == [1, 1] else cu, slots), h)
        close(h, torch.cat([ref[i][at[i]:at[i] + lens[i]] for i in range(2)]), torch.float32, f"from {at}", slack=0.1)
        at = [a + n for a, n in zip(at, lens)]
    assert state[:2].flatten().tolist() == [17, 17] and state[2:4].flatten().tolist() == [tokens[0][-1], tokens[1][-1]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,Fw", [(64, 104), (44, 52), (128, 384)])
def test_feed_forward_with_the_squared_relu(dtype, W, Fw):
    part, p = bound_part(DenseMLPSpec(W, Fw, "relu2"), dtype, scale=0.2)
    for rows in (1, 5, 33, 70, 200):          # the row counts that pick the library's different products
        a = rnd(rows, W, seed=7, scale=1.5).to(dtype).double()
        close(whole(part.forward(None, dev(a, dtype))), plain.squared_relu(a @ p["up"].T) @ p["down"].T, dtype, f"{rows} rows", slack=1.0)


# ------------------------------------------------------------------------------------ positions
@pytest.mark.parametrize("cls", [RotaryPartSpec, RotaryPairsSpec])
@pytest.mark.parametrize("dims,base,scaling", [(16, 500.0, (4.0, 60, 8.0, 1.0)), (40, 30000.0, (2.5, 4096, 24.0, 1.0)), (2, 10.0, (3.0, 100, 1.0, 1.0)),
                                               (64, 1e6, (8.0, 100, 16.0, 2.0)), (22, 200.0, (1.0, 40, 1.0, 1.0)), (30, 7.0, None)])
def test_angle_tables_of_stretched_positions(cls, dims, base, scaling):
    part = build_part(cls(dims, base, scaling), Runtime(DEV, torch.float32))
    cos, sin = part.tables(3000)
    f, mag = plain.frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None)
    for p in (0, 1, 63, 64, 1000, 2999):
        a = p * torch.tensor(f, dtype=torch.float64)
        assert float((cos[p].cpu().double() - a.cos() * mag).abs().max()) < 3e-4 and float((sin[p].cpu().double() - a.sin() * mag).abs().max()) < 3e-4
    assert (mag == 1.0) == (scaling is None or scaling[0] == 1.0)


ROWS = [(4, 2, 32, 48, 16, True), (3, 1, 20, 10, 6, True), (1, 1, 128, 128, 128, False), (5, 5, 24, 8, 2, True), (2, 1, 250, 256, 250, True), (6, 2, 64, 64, 0, False)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pairs", [False, True])
@pytest.mark.parametrize("H,G,D,V,rot,turned", ROWS)
def test_rows_between_projection_and_cache_and_behind_the_attention(dtype, pairs, H, G, D, V, rot, turned):
    """Norms of whole projections, per head before and behind the rotation; halves and pairs; values turned and turned back."""
    positions = [0, 1, 2, 63, 64, 65, 1000, 300]
    T, base = len(positions), 100.0
    proj = rnd(T, H * D + G * D + G * V + 8, seed=1, scale=2.0).to(dtype).double()
    q, k, v = (proj[:, a:a + n] for a, n in ((0, H * D), (H * D, G * D), (H * D + G * D, G * V)))
    pos = torch.tensor(positions, dtype=torch.int32, device=DEV)
    seq = torch.arange(T, dtype=torch.int32, device=DEV)
    table = torch.arange(T * 16, dtype=torch.int32, device=DEV).reshape(T, 16)
    cls = RotaryPairsSpec if pairs else RotaryPartSpec
    tables = lambda n: (*build_part(cls(n, base), Runtime(DEV, dtype)).tables(1001), n, pairs)
    f, fv = plain.frequencies(rot, base)[0], plain.frequencies(V, base)[0]
    at = torch.tensor(positions)
    turn = lambda x, n: plain.turn(x, at, n, plain.frequencies(n, base)[0], pairs=pairs) if n else x
    for mode in (api.NORM_NONE, api.NORM_BEFORE_ROTATION, api.NORM_AFTER_ROTATION, api.NORM_WHOLE):
        for weighted in ((True, False) if mode else (False,)):
            n_q, n_k = (H * D, G * D) if mode == api.NORM_WHOLE else (D, D)
            wq, wk = (1 + 0.3 * rnd(n_q, seed=2)).float().double(), (1 + 0.3 * rnd(n_k, seed=3)).float().double()
            uq, uk = (wq, wk) if weighted else (torch.ones(n_q).double(), torch.ones(n_k).double())
            heads = lambda x, n: x.reshape(T, -1, n)
            if mode == api.NORM_WHOLE:
                rq, rk = turn(heads(plain.rms(q, EPS) * uq, D), rot), turn(heads(plain.rms(k, EPS) * uk, D), rot)
            elif mode == api.NORM_BEFORE_ROTATION:
                rq, rk = turn(plain.rms(heads(q, D), EPS) * uq, rot), turn(plain.rms(heads(k, D), EPS) * uk, rot)
            elif mode == api.NORM_AFTER_ROTATION:
                rq, rk = plain.rms(turn(heads(q, D), rot), EPS) * uq, plain.rms(turn(heads(k, D), rot), EPS) * uk
            else:
                rq, rk = turn(heads(q, D), rot), turn(heads(k, D), rot)
            ks, vs = torch.zeros(T * 16, G, 64, D, dtype=dtype, device=DEV), torch.zeros(T * 16, G, 64, V, dtype=dtype, device=DEV)
            out = torch.empty(T, H * D, dtype=dtype, device=DEV)
            api.qkv_rows(dev(proj, dtype)[:, :H * D + G * D + G * V], out, mode, dev(wq, torch.float32) if weighted else None,
                         dev(wk, torch.float32) if weighted else None, EPS, tables(rot) if rot else None, tables(V) if turned else None,
                         pos, seq, H, G, D, V, ks, vs, table)
            close(out, rq.reshape(T, -1), dtype, f"q, mode {mode}", slack=0.5 if dtype == torch.float32 else 0.1)
            pick = lambda store: torch.stack([store[16 * t + p // 64, :, p % 64] for t, p in enumerate(positions)])
            close(pick(ks), rk, dtype, f"k, mode {mode}", slack=0.5 if dtype == torch.float32 else 0.1)
            close(pick(vs), turn(heads(v, V), V) if turned else heads(v, V), dtype, f"v, mode {mode}", slack=0.5 if dtype == torch.float32 else 0.1)
    o, gate = rnd(T, H * V, seed=5).to(dtype).double(), rnd(T, H, seed=6, scale=2.0).to(dtype).double()
    for g in (gate, None):
        out = torch.empty(T, H * V + 8, dtype=dtype, device=DEV)
        api.turn_back_gate(dev(o, dtype), out[:, :H * V], dev(g, dtype) if g is not None else None, tables(V) if turned else None, 0.5, pos, H, V)
        ref = plain.turn(o.reshape(T, H, V), at, V, fv, pairs=pairs, back=True) if turned else o.reshape(T, H, V)
        ref = 0.5 * ref * (torch.sigmoid(g)[:, :, None] if g is not None else 1.0)
        close(out[:, :H * V], ref.reshape(T, -1), dtype, "turned back", slack=0.5 if dtype == torch.float32 else 0.1)


# ------------------------------------------------------------------------------------ mixers
def scaling_of(rot):
    return tuple(rot[2:]) if len(rot) > 2 else None


def turned_spec(H, G, D, V, scale, rot, cap, W):
    return MaskedAttentionSpec(hidden_size=W, num_heads=H, num_kv_heads=G, head_dim=D, v_head_dim=V, scale=scale, softcap=cap,
                               qk_norm=RMSNormSpec(H * D, EPS), qk_norm_whole=True, head_gate=True,
                               position=RotaryPartSpec(rot[0], rot[1], scaling_of(rot)) if rot[0] else None, value_position=RotaryPartSpec(V, rot[1]))


def pairs_spec(H, G, D, V, scale, rot, cap, W):
    return MaskedAttentionSpec(hidden_size=W, num_heads=H, num_kv_heads=G, head_dim=D, v_head_dim=V, scale=scale, softcap=cap,
                               qk_norm=UnitRMSNormSpec(D, EPS), norm_after_rotation=True, position=RotaryPairsSpec(rot[0], rot[1]) if rot[0] else None)


ATT_SHAPES = [(4, 2, 32, 48, 0.5, (16, 500.0, 4.0, 60, 8.0, 1.0), 9.0), (3, 1, 20, 10, 0.4, (6, 30.0), 5.0), (2, 2, 64, 64, 0.3, (64, 1e4), 30.0),
              (8, 2, 128, 128, 0.2, (32, 1e4, 8.0, 100, 16.0, 2.0), 20.0), (3, 3, 16, 96, 0.7, (2, 9.0), None), (5, 1, 48, 32, 0.3, (0, 50.0), 3.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,scale,rot,cap", ATT_SHAPES)
def test_attention_with_turning_values_in_prompts_portions_and_single_tokens(dtype, H, G, D, V, scale, rot, cap):
    W = 40
    part, p = bound_part(turned_spec(H, G, D, V, scale, rot, cap, W), dtype, seed=3)
    x = rnd(sum(CUTS), W, seed=4).to(dtype).double()
    ref = plain.turned_value_attention(x, p, heads_of(H, G, D, V, scale, rot, cap), EPS)
    close(run_cut(part, x, CUTS, dtype), ref, dtype, "turning values")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,scale,rot,cap", ATT_SHAPES)
def test_attention_rotated_by_pairs_in_prompts_portions_and_single_tokens(dtype, H, G, D, V, scale, rot, cap):
    W = 40
    part, p = bound_part(pairs_spec(H, G, D, V, scale, rot[:2], cap, W), dtype, seed=3)
    x = rnd(sum(CUTS), W, seed=4).to(dtype).double()
    ref = plain.pairs_attention(x, p, heads_of(H, G, D, V, scale, rot[:2], cap), EPS)
    close(run_cut(part, x, CUTS, dtype), ref, dtype, "pairs")


def latent_spec(H, D, V, rank, scale, W):
    return LatentAttentionSpec(hidden_size=W, num_heads=H, head_dim=D, rot_dim=0, v_head_dim=V, q_rank=None, kv_rank=rank, scale=scale,
                               norm_eps=EPS, sink=True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V,rank", [(4, 16, 32, 48), (3, 10, 6, 20), (6, 64, 48, 288), (1, 16, 16, 16), (20, 32, 16, 512), (5, 24, 40, 256), (2, 8, 8, 300)])
def test_latent_attention_with_a_sink_in_prompts_portions_and_single_tokens(dtype, H, D, V, rank):
    """Rows up to 256 wide in steps of 16 on the mma.sync kernels, 288 and 512 on the one for rows that are key and value at
    once, others on the float32-arithmetic kernel. The sinks are of the scores' size, so leaving them out or scaling them shows."""
    W, scale = 40, 0.3
    part, p = bound_part(latent_spec(H, D, V, rank, scale, W), dtype, seed=5, sink=2.0 + rnd(H, seed=1))
    x = rnd(sum(CUTS), W, seed=6).to(dtype).double()
    m = {"heads": H, "dim": D, "vdim": V, "kv_rank": rank, "scale": scale}
    ref = plain.latent_sink_attention(x, p, m, EPS)
    got = run_cut(part, x, CUTS, dtype)
    close(got, ref, dtype, "latent")
    for other in (p["sink"] * scale, p["sink"] - 20.0):
        wrong = plain.latent_sink_attention(x, {**p, "sink": other}, m, EPS)
        assert float((wrong - ref).abs().max()) > 2 * tol(dtype, ref) * 0.5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["turned", "turned 64", "pairs 128", "pairs 24", "latent 64", "latent 320"])
@pytest.mark.parametrize("where", ["prompt", "decoded"])
@pytest.mark.parametrize("kj", [0, 7, 63, 64, 255, 256, 299], ids=lambda k: f"key {k}")
def test_a_planted_key_far_away_at_page_borders_and_at_the_start_shows(dtype, kind, where, kj):
    """The query at 300 is made of the negative of token kj's input, and W_q of -W_k: that key alone scores high (its own key
    scores as low), about ten where the others are of the order of one, so the output there is nearly the key's value; another
    token at kj changes it by more than the tolerance."""
    W, qi = 48, 300
    x = rnd(qi + 20, W, seed=6)
    x[qi] = -x[kj]
    x = x.to(dtype).double()
    if kind.startswith("latent"):
        H, D, V, rank = 2, 32, 32, int(kind.split()[1])
        dkv, uk = rnd(rank, W, seed=11, scale=0.3), rnd(H * D, rank, seed=12, scale=0.1)
        c = plain.rms(x[kj] @ dkv.T, EPS) @ uk.T
        scale = 14.0 / float((-(x[qi] @ dkv.T) @ uk.T * c).reshape(H, D).sum(-1).min())
        spec, m = latent_spec(H, D, V, rank, scale, W), {"heads": H, "dim": D, "vdim": V, "kv_rank": rank, "scale": scale}
        given = dict(dkv=dkv, uk=uk, q=-(uk @ dkv), sink=torch.zeros(H))
        run = lambda y, p: plain.latent_sink_attention(y, p, m, EPS)
    else:
        D = {"turned": 32, "turned 64": 64, "pairs 128": 128, "pairs 24": 24}[kind]
        V, rot = {32: 48, 64: 64, 128: 128, 24: 10}[D], (2, 10.0)
        make = turned_spec if kind.startswith("turned") else pairs_spec
        spec, m = make(2, 2, D, V, 14.0 / D, rot, 40.0, W), heads_of(2, 2, D, V, 14.0 / D, rot, 40.0)
        wk = rnd(2 * D, W, seed=11, scale=0.3)
        given = dict(k=wk, q=-wk)
        if kind.startswith("turned"):
            given.update({"q.norm": torch.ones(2 * D), "k.norm": torch.ones(2 * D)})
        run = lambda y, p: (plain.turned_value_attention if kind.startswith("turned") else plain.pairs_attention)(y, p, m, EPS)
    part, p = bound_part(spec, dtype, seed=3, **given)
    ref = run(x, p)
    y = x.clone()
    y[kj] = rnd(W, seed=50)
    assert float((run(y, p)[qi] - ref[qi]).abs().max()) > 2 * tol(dtype, ref) * 0.5
    close(run_cut(part, x, [qi + 20] if where == "prompt" else [qi - 10] + [1] * 30, dtype), ref, dtype, kind)


DELTA_SHAPES = [(6, 2, 16, 32, 3), (4, 1, 12, 10, 1), (2, 1, 128, 64, 7), (3, 3, 100, 36, 4), (2, 2, 256, 20, 2), (1, 1, 33, 130, 9), (8, 4, 64, 128, 4)]


def delta_case(H, G, D, V, taps, W, dtype, seed, **given):
    spec = GatedDeltaSpec(hidden_size=W, num_heads=H, num_kv_heads=G, head_dim=D, v_head_dim=V, conv_taps=taps, norm_eps=EPS)
    part, p = bound_part(spec, dtype, seed=seed, **given)
    return part, p, {"heads": H, "kv_heads": G, "dim": D, "vdim": V}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps", DELTA_SHAPES)
def test_gated_delta_rule_in_prompts_portions_and_single_tokens(dtype, H, G, D, V, taps):
    W = 40
    part, p, m = delta_case(H, G, D, V, taps, W, dtype, 11)
    x = rnd(sum(CUTS), W, seed=12).to(dtype).double()
    ref, _ = plain.gated_delta(x, p, m, EPS)
    close(run_cut(part, x, CUTS, dtype), ref, dtype, "delta rule")


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_delta_rule_keeps_what_later_tokens_do_not_write_over(dtype):
    """Decays next to one, and step sizes next to zero for all but the first hundred tokens (the first input coordinate says
    which): what those wrote is what comes out 900 tokens on."""
    H, G, D, V, taps, W = 2, 1, 32, 16, 3, 24
    b = torch.zeros(H, W)
    b[:, 0] = 8.0
    part, p, m = delta_case(H, G, D, V, taps, W, dtype, 13, b=b, A_log=torch.full((H,), -12.0))
    x = rnd(930, W, seed=14)
    x[:, 0] = -1.0
    x[:100, 0] = 1.0
    x = x.to(dtype).double()
    ref, _ = plain.gated_delta(x, p, m, EPS)
    y = x.clone()
    y[:100, 1:] = rnd(100, W - 1, seed=15)
    assert float((plain.gated_delta(y, p, m, EPS)[0][920:] - ref[920:]).abs().max()) > 2 * tol(dtype, ref)
    close(run_cut(part, x, [500, 1, 1, 2, 400, 1, 25], dtype), ref, dtype, "far tokens")


def test_the_read_out_sees_the_current_tokens_write_and_the_step_corrects():
    """A single token: o = beta (k . q) v; the same key again with another value: the state moves by the difference only."""
    H, G, D, V = 1, 1, 16, 8
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)
    k = plain.unit(rnd(1, D, seed=1))
    q, v = rnd(1, D, seed=2), rnd(2, V, seed=3)
    qkv = torch.cat([q.repeat(2, 1), k.repeat(2, 1), v], 1)
    scal = torch.tensor([[0.9, 0.5, float((k * q).sum())], [0.9, 1.0, float((k * q).sum())]], dtype=torch.float64)
    ref, S = plain.delta_rule(q.repeat(2, 1)[:, None], k.repeat(2, 1)[:, None], v[:, None], scal[:, :1], scal[:, 1:2], torch.zeros(1, D, V, dtype=torch.float64))
    assert torch.allclose(ref[0, 0], 0.5 * (k * q).sum() * v[0]) and torch.allclose(S[0].T @ k[0], v[1], atol=1e-6)
    for step in (True, False):
        state = torch.zeros(3, H, D, V, device=DEV)
        out = torch.empty(2, H * V, device=DEV)
        if step:
            for t in range(2):
                api.delta_rule(dev(qkv[t:t + 1], torch.float32), dev(scal[t:t + 1], torch.float32), out[t:t + 1], state, None, i32(t), i32(2), 1, H, G, D, V)
        else:
            api.delta_rule(dev(qkv, torch.float32), dev(scal, torch.float32), out, state, i32(0, 2), i32(0), i32(2), 1, H, G, D, V)
        close(out, ref.reshape(2, -1), torch.float32, "outputs", slack=0.1)
        close(state[2], S, torch.float32, "state", slack=0.1)
        assert float(state[:2].abs().max()) == 0.0
    # a padding row: nothing comes out and no state moves
    before = state.clone()
    api.delta_rule(dev(qkv[:1], torch.float32), dev(scal[:1], torch.float32), out[:1], state, None, i32(-1), i32(2), 1, H, G, D, V)
    assert torch.equal(before, state) and float(out[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("left,right", [((6, 2, 48, 16, 0.4, (48, 1000.0), 15.0), (6, 2, 16, 32, 3)), ((2, 1, 128, 128, 0.3, (128, 1e6), None), (2, 1, 128, 64, 4)),
                                        ((3, 1, 20, 10, 0.5, (6, 30.0), 5.0), (4, 1, 12, 10, 1))])
def test_two_mixers_side_by_side_with_normed_outputs(dtype, left, right):
    W = 40
    r = dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))
    spec = ParallelMixerSpec(hidden_size=W, out_norm_eps=EPS, branches=(
        ("left.", pairs_spec(*left, W), 0.5),
        ("right.", GatedDeltaSpec(hidden_size=W, num_heads=r["heads"], num_kv_heads=r["kv_heads"], head_dim=r["dim"], v_head_dim=r["vdim"],
                                  conv_taps=r["conv"], norm_eps=EPS), 0.5)))
    part, p = bound_part(spec, dtype, seed=21)
    x = rnd(sum(CUTS), W, seed=22).to(dtype).double()
    ref = plain.mixer("parallel", x, p, {"left": heads_of(*left), "right": r}, EPS)
    close(run_cut(part, x, CUTS, dtype), ref, dtype, "side by side")


# ------------------------------------------------------------------------------------ whole models
def plain_logits(folder, tokens):
    cfg, t = plain.read_model(folder)
    return plain.forward(tokens, t, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SHAPES))
def test_the_stream_after_every_layer(tmp_path, name, dtype):
    folder, cfg = make_model(tmp_path, name, seed=1)
    tokens = random_tokens(cfg.vocab, 75, 3)
    pcfg, t = plain.read_model(folder)
    ref = []
    plain.forward(tokens, t, pcfg, ref)
    runner = Runner(load_model(folder, dtype), 64 * 4, 2)
    got = []
    slot = runner.begin()
    runner.step([(slot, tokens, [])], tap=lambda k, h: got.append(h))
    assert len(got) == len(ref) == len(SHAPES[name]["layers"])
    errs = Errors(dtype)
    for k, (g, r) in enumerate(zip(got, ref)):
        for pos in range(len(tokens)):
            errs.add(g[pos], r[pos], f"layer {k} position {pos}", bound_of=r)
    errs.verdict()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SHAPES))
def test_whole_prompts_portions_batches_and_reused_slots(tmp_path, name, dtype):
    folder, cfg = make_model(tmp_path, name)
    runner = Runner(load_model(folder, dtype), 64 * 24, 6)
    lens = [1, 23, 131, 200]
    seqs = [random_tokens(cfg.vocab, n, 40 + i) for i, n in enumerate(lens)]
    ref = [plain_logits(folder, s) for s in seqs]

    errs = Errors(dtype)

    def check(out, pairs, what):
        for row, (i, p) in enumerate(pairs):
            errs.add(out[row], ref[i][p], f"{what}: sequence {i} position {p}", bound_of=ref[i])

    for round_ in range(2):        # the second round runs on the slots, pages and states the first gave back
        for i, s in enumerate(seqs):
            slot = runner.begin()
            want = sorted({0, len(s) // 2, len(s) - 1})
            check(runner.step([(slot, s, want)]), [(i, p) for p in want], "alone")
            runner.end(slot)
        cut = [1, 17, 100, 130]
        slots = [runner.begin() for _ in seqs]
        check(runner.step([(sl, s[:c], [c - 1]) for sl, s, c in zip(slots, seqs, cut)]), [(i, c - 1) for i, c in enumerate(cut)],
              "batch of prompts")
        live, k = [i for i in range(4) if cut[i] < lens[i]], 0
        while live and k < 40:
            out = runner.step([(slots[i], [seqs[i][cut[i] + k]], [0]) for i in live])
            check(out, [(i, cut[i] + k) for i in live], f"decode step {k}")
            k += 1
            for i in [i for i in live if cut[i] + k >= lens[i]]:
                runner.end(slots[i])
                slots[i] = None
            live = [i for i in live if cut[i] + k < lens[i]]
        for sl in slots:
            if sl is not None:
                runner.end(sl)
        slot, at = runner.begin(), 0           # portions of several sizes, down to two tokens and one; some want nothing
        for n in [64, 2, 31, 1, 2, 70, 30]:
            want = [0, n - 1] if n != 31 else []
            check(runner.step([(slot, seqs[3][at:at + n], want)]), [(3, at + w) for w in want], f"portion of {n} at {at}")
            at += n
        runner.end(slot)
    errs.verdict()
    assert runner.cache.slots.n_live == 0 and all(f == runner.cache.num_pages for f in runner.cache.pages_free())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_the_decode_state_and_its_graph(tmp_path, name, dtype):
    folder, cfg = make_model(tmp_path, name, seed=3)
    model = load_model(folder, dtype)
    seqs = [random_tokens(cfg.vocab, n, 60 + i) for i, n in enumerate([150, 90, 120])]
    ref = [plain_logits(folder, s) for s in seqs]
    for use_graph in (False, True):
        errs = Errors(dtype)
        runner = Runner(model, 64 * 12, 4)
        loop = DecodeLoop(runner, use_graph=use_graph)
        slots = [runner.begin() for _ in seqs]
        cut = [30, 5, 1]
        runner.step([(sl, s[:c], []) for sl, s, c in zip(slots, seqs, cut)])
        for k in range(85):                          # three sequences in four rows: a padding row in every step
            out = loop.forced_step([(sl, [s[c + k]], [0]) for sl, s, c in zip(slots, seqs, cut)])
            for i in range(3):
                errs.add(out[i], ref[i][cut[i] + k], f"graph={use_graph} step {k} sequence {i}", bound_of=ref[i])
        errs.verdict()
        for sl in slots:
            runner.end(sl)
    api.gemm_tc_check()


def random_config(rng):
    """A configuration drawn at random: any order of layers, sizes that no kernel was built for."""
    def rot(D):
        r = (rng.choice([d for d in (0, 2, 4, 6, 8, 16, 32, 64, 128) if d <= D]), rng.choice([50.0, 1e4, 1e6]))
        return r + (rng.choice([1.5, 4.0]), rng.choice([30, 500]), rng.choice([4.0, 32.0]), 1.0) if rng.random() < 0.5 else r

    def group():
        G = rng.choice([1, 2, 3])
        return G * rng.choice([1, 2, 3, 4]), G

    def one():
        mlp = dense(rng.choice([20, 48, 64, 130])) if rng.random() < 0.8 else None
        kind = rng.choice(["att", "lat", "par"])
        D = rng.choice([8, 12, 16, 20, 32, 64, 128])
        cap = rng.choice([None, 4.0, 30.0])
        if kind == "lat":
            return lat(rng.choice([1, 2, 3, 5, 8]), D, rng.choice([6, 16, 32, 33]), rng.choice([16, 20, 64, 96, 160, 256, 320]), D ** -0.5, mlp)
        if kind == "att":
            return att(*group(), D, rng.choice([D, 8, 16, 22, 64]), D ** -0.5 * rng.choice([1.0, 2.0]), rot(D), cap, mlp)
        return par((*group(), D, rng.choice([D, 7, 16, 48]), D ** -0.5 * rng.choice([1.0, 3.0]), rot(D)[:2], cap),
                   (*group(), rng.choice([8, 12, 30, 32, 64, 96, 128]), rng.choice([5, 8, 16, 32, 64]), rng.choice([1, 2, 3, 4, 6])), mlp)

    cfg = dict(architecture="Fukatar", vocab=rng.choice([50, 136, 333]), width=rng.choice([40, 52, 60, 100, 128, 160]),
               norm={"eps": rng.choice([1e-6, 1e-5, 1e-4])}, embedding={"scale": rng.choice([1.0, 4.0])}, layers=[one() for _ in range(rng.randint(2, 5))])
    if rng.random() < 0.8:
        cfg["embedding"]["bigram"] = {"buckets": rng.choice([3, 64, 211]), "mul_prev": rng.choice([1, 29]), "mul_cur": rng.choice([1, 23])}
    if rng.random() < 0.7:
        cfg["logit_softcap"] = rng.choice([3.0, 30.0])
    return cfg


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations_through_batches_the_decode_state_and_portions(tmp_path, seed):
    cfg = dk.config_from_dict(random_config(random.Random(2000 + seed)))
    folder = str(tmp_path / "model")
    dk.write_random_model(cfg, folder, seed=seed, dtype=torch.float32, matrix_std=0.08)
    lens = [1, 37, 150, 230]
    seqs = [random_tokens(cfg.vocab, n, 10 * seed + i) for i, n in enumerate(lens)]
    ref = [plain_logits(folder, s) for s in seqs]
    for dtype in DTYPES:
        runner = Runner(load_model(folder, dtype), 64 * 24, 6)

        errs = Errors(dtype)

        def check(out, pairs, what):
            for row, (i, p) in enumerate(pairs):
                errs.add(out[row], ref[i][p], f"seed {seed} {what}: sequence {i} position {p}", bound_of=ref[i])

        for use_graph in (False, True):
            cut = [1, 20, 100, 140]
            slots = [runner.begin() for _ in seqs]
            check(runner.step([(sl, s[:c], [c - 1]) for sl, s, c in zip(slots, seqs, cut)]), [(i, c - 1) for i, c in enumerate(cut)], "prompts")
            loop = DecodeLoop(runner, use_graph=use_graph)
            live, k = [i for i in range(4) if cut[i] < lens[i]], 0
            while live and k < 40:
                check(loop.forced_step([(slots[i], [seqs[i][cut[i] + k]], [0]) for i in live]), [(i, cut[i] + k) for i in live], f"token {k}")
                k += 1
                for i in [i for i in live if cut[i] + k >= lens[i]]:
                    runner.end(slots[i])
                    slots[i] = None
                live = [i for i in live if cut[i] + k < lens[i]]
            for sl in slots:
                if sl is not None:
                    runner.end(sl)
        slot, at = runner.begin(), 0
        for n in [64, 2, 31, 1, 2, 70, 30]:
            check(runner.step([(slot, seqs[3][at:at + n], [0, n - 1])]), [(3, at), (3, at + n - 1)], f"portion of {n} at {at}")
            at += n
        runner.end(slot)
        errs.verdict()


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_entry_point(tmp_path, name):
    folder, cfg = make_model(tmp_path, name, seed=5)
    pcfg, t = plain.read_model(folder)
    prompts = [random_tokens(cfg.vocab, n, 80 + i) for i, n in enumerate([1, 40, 77])]
    n_new = 30
    for dtype in DTYPES:
        eng = dk.Engine(folder, dtype=dtype)
        steps = list(eng.generate(prompts, n_new))
        again = list(dk.Engine(folder, dtype=dtype, use_graph=False, max_prefill_tokens=16).generate(prompts, n_new))
        for i, p in enumerate(prompts):
            emitted = [s[i] for s in steps]
            logits = plain.forward(p + emitted[:-1], t, pcfg)[len(p) - 1:]
            gap = float((logits.max(-1).values - logits.gather(1, torch.tensor(emitted).view(-1, 1)).squeeze(1)).max())
            assert gap <= (1e-4 if dtype == torch.float32 else 0.12 * max(1.0, float(logits.abs().max()))), (name, dtype, i, gap)
            if dtype == torch.float32:               # prompts cut into portions of 16, plain launches: the same tokens
                assert emitted == [s[i] for s in again]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_of_a_ragged_schedule(tmp_path, dtype):
    folder, cfg = make_model(tmp_path, "D", seed=7)
    seqs = {"a": random_tokens(cfg.vocab, 140, 1), "b": random_tokens(cfg.vocab, 9, 2), "c": random_tokens(cfg.vocab, 66, 3)}
    ref = {k: plain_logits(folder, s) for k, s in seqs.items()}
    start = {"a": 130, "b": 1, "c": 60}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seqs["a"][:130], "want": [0, 63, 64, 129]},
                                     {"id": "b", "tokens": seqs["b"][:1], "want": [0]},
                                     {"id": "c", "tokens": seqs["c"][:60], "want": []}], "end": []}]
    for k in range(10):
        ent = [{"id": i, "tokens": [seqs[i][start[i] + k]], "want": [0] if (i != "c" or k % 2) else []}
               for i in ("a", "b", "c") if start[i] + k < len(seqs[i])]
        steps.append({"step": k + 1, "entries": ent, "end": [e["id"] for e in ent if start[e["id"]] + k + 1 == len(seqs[e["id"]])]})
    out_dir = str(tmp_path / "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                           "--out", out_dir, "--max-tokens", "512"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    at = {"a": 0, "b": 0, "c": 0}
    errs = Errors(dtype)
    for s in steps:
        rows = []
        for e in s["entries"]:
            rows += [(e["id"], at[e["id"]] + w) for w in e["want"]]
            at[e["id"]] += len(e["tokens"])
        if rows:
            got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{s['step']}.f32"), dtype="<f4").reshape(len(rows), cfg.vocab))
            for r, (i, p) in enumerate(rows):
                errs.add(got[r], ref[i][p], f"step {s['step']} request {i} position {p}", bound_of=ref[i])
    errs.verdict()


def test_command_line_generates_with_a_fukatar_model(tmp_path):
    """Random weights from a config.json of this design through the command line, the tokens it prints against the
    plain implementation's greedy tokens."""
    from dryft_challenge_htn_2026_b200.cli import random_prompts

    cfg = dk.config_from_dict(SHAPES["A"])
    cfg.save(str(tmp_path))
    model_dir = str(tmp_path / "model")
    env = dict(os.environ, PYTHONPATH=ROOT + os.pathsep + os.environ.get("PYTHONPATH", ""))
    r = subprocess.run([sys.executable, "-m", "dryft_challenge_htn_2026_b200.cli", "--random-weights", str(tmp_path / "config.json"),
                        "--save-model", model_dir, "--seed", "3", "--dtype", "float32", "--shapes", "2,30,6", "--samples", "1",
                        "--print-tokens"], capture_output=True, text=True, env=env, cwd=str(ROOT), timeout=900)
    assert r.returncode == 0, r.stdout + r.stderr
    lines = [l for l in r.stdout.splitlines() if l.startswith("tokens 2,30,6 seq ")]
    assert len(lines) == 2
    pcfg, t = plain.read_model(model_dir)
    prompts = random_prompts(2, 30, 1, cfg.vocab, False)
    for i, line in enumerate(lines):
        emitted = [int(x) for x in line.split(":")[1].split()]
        logits = plain.forward(prompts[i] + emitted[:-1], t, pcfg)[len(prompts[i]) - 1:]
        gap = float((logits.max(-1).values - logits.gather(1, torch.tensor(emitted).view(-1, 1)).squeeze(1)).max())
        assert gap <= 1e-4, (i, gap)
