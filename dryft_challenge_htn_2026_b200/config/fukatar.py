"""Fukatar: a decoder with a layer norm on each sublayer's output alone, x <- x + norm(sublayer(x)), whose mixers read the
stream mixed with the stream of the token before (a learned share per element, at every layer). Its layers mix in one of
three ways: grouped-query attention with q and k normed as whole projections before a rotate-half rotation (with YaRN's
stretched positions where asked), capped scores, values turned by their position and turned back behind the sum, and one
gate per head; attention through one normed latent per token, without positions, with a sink per head; or two mixers side
by side, grouped-query attention (rotation by neighbouring pairs, then q and k over their root mean square, capped scores)
beside the gated delta rule (short convolutions, unit keys and queries), each output normed over the width, half their sum.
The feed-forward is a squared ReLU between two products, or none. The embedding is scaled and a row for the pair of this
token and the one before is added; the head is a table of its own, its logits capped.

config.json keys (every size, and every constant that differs between models of the design):
  architecture "Fukatar"; vocab, width; norm.eps; logit_softcap;
  embedding: {scale, bigram: {buckets, mul_prev, mul_cur}};
  layers[i] = {type: "attention", mixer: {heads, kv_heads, dim, vdim, scale, softcap,
                                          rot: {dims, base, scaling: {factor, original, fast, slow}}}, mlp}
            | {type: "latent_attention", mixer: {heads, dim, vdim, kv_rank, scale}, mlp}
            | {type: "parallel", mixer: {left: {heads, kv_heads, dim, vdim, scale, softcap, rot: {dims, base}},
                                         right: {heads, kv_heads, dim, vdim, conv}}, mlp}
     with mlp = {kind: "dense", ff} | null.
  Left out: kv_heads = heads, vdim = dim, softcap = none, rot.scaling = none, embedding.scale = 1, embedding.bigram = none,
  logit_softcap = none.
Tensors: embed, bigram [buckets + 1, width], head, final.norm, and per layer l<i>.norm1, .shift, .norm2 (the last with a
  feed-forward only), attention: l<i>.mix.{q,k,v,g,o}, .mix.q.norm [heads * dim], .mix.k.norm [kv_heads * dim];
  latent attention: l<i>.mix.{q,dkv,uk,uv,o}, .mix.dkv.norm [kv_rank], .mix.sink [heads];
  parallel: l<i>.mix.left.{q,k,v,o}, l<i>.mix.right.{q,k,v,b,a,g,o}, .right.{q,k,v}.conv [channels, taps],
            .right.{A_log,dt_bias} [heads], .right.norm [vdim], .mix.{left,right}.out [width];
  feed-forward: l<i>.mlp.{up,down}.
"""
from dataclasses import dataclass, field
from typing import Optional, Tuple

from .base import ConfigError, ModelConfig, get
from .nilivik import _freeze, _section, _thaw
from .specs import (BigramSpec, DenseMLPSpec, GatedDeltaSpec, LatentAttentionSpec, LayerNormSpec, MaskedAttentionSpec, ModelSpec,
                    OutputNormLayerSpec, ParallelMixerSpec, RMSNormSpec, RotaryPairsSpec, RotaryPartSpec, UnitRMSNormSpec)

UNIT_EPS = 1e-6          # under the root of the delta rule's unit keys and queries; fixed by the design
BRANCH_SHARE = 0.5       # the two mixers side by side: half the sum of their normed outputs


def _group_heads(m, where):
    H = get(m, "heads", int, positive=True)
    G = get(m, "kv_heads", int, H, positive=True)
    if H % G:
        raise ConfigError(f"config.json: {where}: {H} heads are not a multiple of {G} key/value heads")
    dim = get(m, "dim", int, positive=True)
    return {"heads": H, "kv_heads": G, "dim": dim, "vdim": get(m, "vdim", int, dim, positive=True)}


def _rotation(m, where):
    rot = _section(m, "rot", where)
    out = {"dims": get(rot, "dims", int), "base": get(rot, "base", float, positive=True)}
    if out["dims"] % 2 or not 0 <= out["dims"] <= m["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims {out['dims']} must be even and at most {m['dim']}")
    if rot.get("scaling") is not None:
        sc = _section(rot, "scaling", f"{where}.rot")
        out["scaling"] = {k: get(sc, k, float, positive=True) for k in ("factor", "original", "fast", "slow")}
    return out


def _attention(m, where):
    out = _group_heads(m, where)
    out["scale"] = get(m, "scale", float)
    out["rot"] = _rotation({**m, "dim": out["dim"]}, where)
    cap = get(m, "softcap", float, 0.0)
    if cap < 0:
        raise ConfigError(f"config.json: {where}.softcap must not be negative")
    if cap:
        out["softcap"] = cap
    return out


def _check_mixer(kind, m, where):
    if kind == "attention":
        out = _attention(m, where)
        if out["vdim"] % 2:
            raise ConfigError(f"config.json: {where}.vdim {out['vdim']} must be even (values turn by pairs)")
        return out
    if kind == "latent_attention":
        return {"heads": get(m, "heads", int, positive=True), "dim": get(m, "dim", int, positive=True),
                "vdim": get(m, "vdim", int, positive=True), "kv_rank": get(m, "kv_rank", int, positive=True),
                "scale": get(m, "scale", float)}
    if kind == "parallel":
        r = _section(m, "right", where)
        right = _group_heads(r, f"{where}.right")
        right["conv"] = get(r, "conv", int, positive=True)
        return {"left": _attention(_section(m, "left", where), f"{where}.left"), "right": right}
    raise ConfigError(f"config.json: {where}.type {kind!r} is not implemented (attention, latent_attention, parallel)")


def _check_mlp(mlp, where):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}.mlp must be an object or null")
    if mlp.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}.mlp kind {mlp.get('kind')!r} is not implemented (dense or null)")
    return {"kind": "dense", "ff": get(mlp, "ff", int, positive=True)}


def _scaling(rot):
    sc = rot.get("scaling")
    return (sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None


@dataclass(frozen=True)
class FukatarConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Optional[Tuple[int, int, int]]     # (buckets, mul_prev, mul_cur), or none
    logit_softcap: float                       # 0: logits are not capped
    layers: tuple = field(default=())          # the config's layer entries, checked, frozen

    architecture = "Fukatar"

    @classmethod
    def from_dict(cls, d):
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        checked = []
        for i, lc in enumerate(layers):
            if not isinstance(lc, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = lc.get("type")
            checked.append({"type": kind, "mixer": _check_mixer(kind, _section(lc, "mixer", f"layers[{i}]"), f"layers[{i}].mixer"),
                            "mlp": _check_mlp(lc.get("mlp"), f"layers[{i}]")})
        emb = d.get("embedding") or {}
        if not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object")
        bigram = None
        if emb.get("bigram") is not None:
            b = _section(emb, "bigram", "embedding")
            bigram = (get(b, "buckets", int, positive=True), get(b, "mul_prev", int), get(b, "mul_cur", int))
            if bigram[1] < 0 or bigram[2] < 0:
                raise ConfigError("config.json: embedding.bigram multipliers must not be negative")
        cap = get(d, "logit_softcap", float, 0.0)
        if cap < 0:
            raise ConfigError("config.json: 'logit_softcap' must not be negative")
        return cls(vocab=get(d, "vocab", int, positive=True), width=get(d, "width", int, positive=True),
                   norm_eps=get(_section(d, "norm", "the"), "eps", float, positive=True),
                   embedding_scale=get(emb, "scale", float, 1.0), bigram=bigram, logit_softcap=cap,
                   layers=tuple(_freeze(l) for l in checked))

    def layer_dicts(self):
        return [_thaw(l) for l in self.layers]

    def to_dict(self):
        emb = {"scale": self.embedding_scale}
        if self.bigram:
            emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": emb, "layers": self.layer_dicts()}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d

    def _attention_spec(self, m, rotation, **options):
        rot = m["rot"]
        return MaskedAttentionSpec(
            hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            scale=m["scale"], softcap=m.get("softcap"),
            position=rotation(rot["dims"], rot["base"], _scaling(rot)) if rot["dims"] else None, **options)

    def _mixer_spec(self, kind, m):
        W, eps = self.width, self.norm_eps
        if kind == "attention":
            return self._attention_spec(m, RotaryPartSpec, qk_norm=RMSNormSpec(m["heads"] * m["dim"], eps), qk_norm_whole=True,
                                        value_position=RotaryPartSpec(m["vdim"], m["rot"]["base"]), head_gate=True)
        if kind == "latent_attention":
            return LatentAttentionSpec(hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], rot_dim=0, v_head_dim=m["vdim"],
                                       q_rank=None, kv_rank=m["kv_rank"], scale=m["scale"], norm_eps=eps, sink=True)
        left = self._attention_spec(m["left"], RotaryPairsSpec, qk_norm=UnitRMSNormSpec(m["left"]["dim"], eps),
                                    norm_after_rotation=True)
        r = m["right"]
        right = GatedDeltaSpec(hidden_size=W, num_heads=r["heads"], num_kv_heads=r["kv_heads"], head_dim=r["dim"],
                               v_head_dim=r["vdim"], conv_taps=r["conv"], norm_eps=eps, unit_eps=UNIT_EPS)
        return ParallelMixerSpec(hidden_size=W, branches=(("left.", left, BRANCH_SHARE), ("right.", right, BRANCH_SHARE)),
                                 out_norm_eps=eps)

    def to_spec(self):
        W, eps = self.width, self.norm_eps
        layers = []
        for i, lc in enumerate(self.layer_dicts()):
            ff = DenseMLPSpec(W, lc["mlp"]["ff"], "relu2") if lc["mlp"] else None
            names = (("mixer", "mix."), ("norm_mix", "norm1")) + ((("feed_forward", "mlp."), ("norm_ff", "norm2")) if ff else ())
            layers.append(OutputNormLayerSpec(prefix=f"l{i}.", mixer=self._mixer_spec(lc["type"], lc["mixer"]),
                                              norm_mix=LayerNormSpec(W, eps), feed_forward=ff,
                                              norm_ff=LayerNormSpec(W, eps) if ff else None, shift="shift", names=names))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers),
                         schedule=ModelSpec.identity_schedule(len(layers)), final_norm=LayerNormSpec(W, eps),
                         tie_embeddings=False, max_positions=1 << 20, embed_name="embed", final_norm_prefix="final.norm",
                         head_name="head", embed_scale=self.embedding_scale, logit_cap=self.logit_softcap or None,
                         embed_bigram=BigramSpec(*self.bigram) if self.bigram else None)
