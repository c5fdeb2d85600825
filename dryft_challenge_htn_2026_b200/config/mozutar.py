"""Mozutar: a decoder with a layer norm (weight and bias) before and after each sublayer and a learned scale per element on
what a sublayer adds, x <- x + ls * norm(sublayer(norm(x))). A layer mixes in one of two ways: the matrix memory of the mLSTM
(exponential gates kept in range by a running maximum), or two mixers side by side, grouped-query attention whose values are
its keys as projected (a norm per q and k head before a rotate-half rotation, capped scores) beside gated linear attention (a
decay per key channel and token), each output normed over the width, half their sum. The feed-forward is gated with SiLU:
dense, a mixture of experts (softmax scores, a correction for the choice, groups scored by their best expert, identity experts
that pass their input on, weights not renormalized) or none. A span of layers runs several times with the same weights and a
cache or state for each pass; ahead of a pass the stream takes the embedding in by a matrix, x <- W [x; x0], and a vector of
the pass is added. The head is the embedding table.

config.json keys (every size, and every constant that differs between models of the design):
  architecture "Mozutar"; vocab, width; norm.eps; embedding.scale;
  layers[i] = {type: "mlstm", mixer: {heads, dim, vdim, gate_cap}, mlp}
            | {type: "parallel", mixer: {left: {heads, kv_heads, dim, vdim, scale, softcap, rot: {dims, base}},
                                         right: {heads, dim, vdim, tau}}, mlp}
     with mlp = {kind: "dense", ff} | {kind: "moe", expert: {ff}, router: {experts, identity, top, groups: {count, keep}}} | null;
  loop = {start, stop, times}: layers start .. stop-1 run ``times`` times.
  Left out: kv_heads = heads, vdim = dim, softcap = none, rot = none, tau = 1, identity = 0, groups = one group,
  embedding.scale = 1, loop = none. The left mixer's vdim is its dim.
Tensors: embed, final.norm, final.norm.b, loop.in [width, 2 width], loop.step [times, width], and per layer
  l<i>.norm1, .norm1b, .norm2, .norm2b, each with .b, l<i>.ls1, .ls2 (norm2, norm2b and ls2 with a feed-forward only);
  mlstm: l<i>.mix.{q,k,v,g,o}, .mix.{i,f} [heads, width], .mix.{i,f}.b, .mix.norm [heads * vdim];
  parallel: l<i>.mix.left.{q,k,o}, .left.{q,k}.norm [dim], l<i>.mix.right.{q,k,v,g,o}, .right.norm [vdim],
            .right.a1 [rank, width], .right.a2 [heads * dim, rank], .right.a2.b, .mix.{left,right}.out [width];
  dense: l<i>.mlp.{gate,up,down}; moe: l<i>.mlp.e<k>.{gate,up,down}, .mlp.router, .mlp.correction [experts + identity].
The inner size of the decay's two-step projection is the shape of .right.a1 and not a config key: ``to_spec`` takes it from
``decay_rank`` (set by ``with_shapes`` from a checkpoint, or given).
"""
from dataclasses import dataclass, field, replace
from typing import Optional, Tuple

from .base import ConfigError, ModelConfig, get
from .nilivik import _freeze, _section, _thaw
from .pibulix import DEFAULT_DECAY_RANK
from .specs import (GatedLinearAttentionSpec, GatedMLPSpec, LayerNormSpec, MaskedAttentionSpec, MatrixMemorySpec, ModelSpec,
                    ParallelMixerSpec, RMSNormSpec, RotaryPartSpec, RoutedMLPSpec, SandwichLayerSpec, ScheduleEntry)

BRANCH_SHARE = 0.5       # the two mixers side by side: half the sum of their normed outputs
LOOP_TABLE, LOOP_MATRIX = "loop.step", "loop.in"


def _check_mlp(mlp, where):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}.mlp must be an object or null")
    if mlp.get("kind") == "dense":
        return {"kind": "dense", "ff": get(mlp, "ff", int, positive=True)}
    if mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}.mlp kind {mlp.get('kind')!r} is not implemented (dense, moe or null)")
    r = _section(mlp, "router", f"{where}.mlp")
    g = r.get("groups") or {"count": 1, "keep": 1}
    router = {"experts": get(r, "experts", int, positive=True), "identity": get(r, "identity", int, 0), "top": get(r, "top", int, positive=True),
              "groups": {"count": get(g, "count", int, positive=True), "keep": get(g, "keep", int, positive=True)}}
    n, count, keep = router["experts"] + router["identity"], router["groups"]["count"], router["groups"]["keep"]
    if router["identity"] < 0 or n % count or keep > count or router["top"] > keep * (n // count):
        raise ConfigError(f"config.json: {where}.mlp.router: {router['experts']} experts and {router['identity']} identity experts, "
                          f"{count} groups, {keep} kept, {router['top']} chosen do not fit together")
    return {"kind": "moe", "expert": {"ff": get(_section(mlp, "expert", f"{where}.mlp"), "ff", int, positive=True)}, "router": router}


def _sizes(m):
    dim = get(m, "dim", int, positive=True)
    return {"heads": get(m, "heads", int, positive=True), "dim": dim, "vdim": get(m, "vdim", int, dim, positive=True)}


def _check_left(m, where):
    out = _sizes(m)
    out["kv_heads"] = get(m, "kv_heads", int, out["heads"], positive=True)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}: {out['heads']} heads are not a multiple of {out['kv_heads']} key/value heads")
    if out["vdim"] != out["dim"]:
        raise ConfigError(f"config.json: {where}: values are the keys, so vdim {out['vdim']} must be dim {out['dim']}")
    out["scale"] = get(m, "scale", float)
    cap = get(m, "softcap", float, 0.0)
    if cap < 0:
        raise ConfigError(f"config.json: {where}.softcap must not be negative")
    if cap:
        out["softcap"] = cap
    if m.get("rot") is not None:
        rot = _section(m, "rot", where)
        out["rot"] = {"dims": get(rot, "dims", int), "base": get(rot, "base", float, positive=True)}
        if out["rot"]["dims"] % 2 or not 0 <= out["rot"]["dims"] <= out["dim"]:
            raise ConfigError(f"config.json: {where}.rot.dims {out['rot']['dims']} must be even and at most {out['dim']}")
    return out


def _check_mixer(kind, m, where):
    if kind == "mlstm":
        return {**_sizes(m), "gate_cap": get(m, "gate_cap", float, positive=True)}
    if kind == "parallel":
        r = _section(m, "right", where)
        return {"left": _check_left(_section(m, "left", where), f"{where}.left"),
                "right": {**_sizes(r), "tau": get(r, "tau", float, 1.0, positive=True)}}
    raise ConfigError(f"config.json: {where}.type {kind!r} is not implemented (mlstm, parallel)")


@dataclass(frozen=True)
class MozutarConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    loop: Optional[Tuple[int, int, int]]       # (start, stop, times), or none
    layers: tuple = field(default=())          # the config's layer entries, checked, frozen
    decay_rank: tuple = field(default=())      # per layer: inner size of the decay projection (None where there is none)

    architecture = "Mozutar"

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
        loop = None
        if d.get("loop") is not None:
            s = _section(d, "loop", "the")
            loop = (get(s, "start", int), get(s, "stop", int), get(s, "times", int, positive=True))
            if not 0 <= loop[0] <= loop[1] <= len(checked):
                raise ConfigError(f"config.json: loop {loop[0]}..{loop[1]} does not lie within the {len(checked)} layers")
        emb = d.get("embedding") or {}
        if not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object")
        ranks = d.get("decay_rank")       # not a key of the design's config.json; kept when this library writes one
        if ranks is None:
            ranks = [DEFAULT_DECAY_RANK if lc["type"] == "parallel" else None for lc in checked]
        if not isinstance(ranks, list) or len(ranks) != len(checked):
            raise ConfigError("config.json: 'decay_rank' must give one entry per layer")
        return cls(vocab=get(d, "vocab", int, positive=True), width=get(d, "width", int, positive=True),
                   norm_eps=get(_section(d, "norm", "the"), "eps", float, positive=True), embedding_scale=get(emb, "scale", float, 1.0),
                   loop=loop, layers=tuple(_freeze(l) for l in checked), decay_rank=tuple(ranks))

    def layer_dicts(self):
        return [_thaw(l) for l in self.layers]

    def to_dict(self):
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "layers": self.layer_dicts()}
        if self.loop:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if any(r not in (None, DEFAULT_DECAY_RANK) for r in self.decay_rank):
            d["decay_rank"] = list(self.decay_rank)
        return d

    def with_shapes(self, shapes):
        """The config with what only the checkpoint's tensor shapes say: the inner size of each layer's decay projection
        (rows of l<i>.mix.right.a1). ``shapes``: tensor name -> shape."""
        ranks = list(self.decay_rank)
        for i, lc in enumerate(self.layer_dicts()):
            name = f"l{i}.mix.right.a1"
            if lc["type"] == "parallel" and name in shapes and len(shapes[name]) == 2:
                ranks[i] = int(shapes[name][0])
        return replace(self, decay_rank=tuple(ranks))

    def runs(self):
        """[(layer, pass number or None)] in running order; the number is set on the first layer of a pass of the loop."""
        n = len(self.layers)
        a, b, times = self.loop or (n, n, 0)
        out = [(i, None) for i in range(a)]
        for p in range(times if b > a else 0):
            out += [(i, p if i == a else None) for i in range(a, b)]
        return out + [(i, None) for i in range(b, n)]

    def _mixer_spec(self, kind, m, rank):
        W, eps = self.width, self.norm_eps
        if kind == "mlstm":
            return MatrixMemorySpec(hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], gate_cap=m["gate_cap"],
                                    norm_eps=eps)
        l, r = m["left"], m["right"]
        rot = l.get("rot")
        left = MaskedAttentionSpec(hidden_size=W, num_heads=l["heads"], num_kv_heads=l["kv_heads"], head_dim=l["dim"], v_head_dim=l["vdim"],
                                   scale=l["scale"], softcap=l.get("softcap"), qk_norm=RMSNormSpec(l["dim"], eps), keys_as_values=True,
                                   position=RotaryPartSpec(rot["dims"], rot["base"]) if rot and rot["dims"] else None)
        right = GatedLinearAttentionSpec(hidden_size=W, num_heads=r["heads"], head_dim=r["dim"], v_head_dim=r["vdim"],
                                         decay_rank=rank or DEFAULT_DECAY_RANK, tau=r["tau"], norm_eps=eps)
        return ParallelMixerSpec(hidden_size=W, branches=(("left.", left, BRANCH_SHARE), ("right.", right, BRANCH_SHARE)), out_norm_eps=eps)

    def _feed_forward_spec(self, mlp):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return GatedMLPSpec(self.width, mlp["ff"], "silu", names=("gate", "up", "down"))
        r = mlp["router"]
        return RoutedMLPSpec(hidden_size=self.width, expert_ff=mlp["expert"]["ff"], num_experts=r["experts"], top=r["top"],
                             groups=r["groups"]["count"], keep_groups=r["groups"]["keep"], activation="silu", renorm=False, scores="softmax",
                             group_top=1, identity=r["identity"])

    def to_spec(self):
        W, eps = self.width, self.norm_eps
        norm = LayerNormSpec(W, eps, bias=".b")
        layers = []
        for i, lc in enumerate(self.layer_dicts()):
            ff = self._feed_forward_spec(lc["mlp"])
            names = (("norm_in", "norm1"), ("mixer", "mix."), ("norm_mix_out", "norm1b"))
            if ff:
                names += (("norm_post", "norm2"), ("feed_forward", "mlp."), ("norm_ff_out", "norm2b"))
            layers.append(SandwichLayerSpec(prefix=f"l{i}.", norm_in=norm, mixer=self._mixer_spec(lc["type"], lc["mixer"], self.decay_rank[i]),
                                            norm_mix_out=norm, norm_post=norm if ff else None, feed_forward=ff,
                                            norm_ff_out=norm if ff else None, names=names, layer_scale=("ls1", "ls2")))
        schedule = tuple(ScheduleEntry(layer=i, cache=k, writes=True, add_row=(LOOP_TABLE, p) if p is not None else None,
                                       take_in=LOOP_MATRIX if p is not None else None) for k, (i, p) in enumerate(self.runs()))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers), schedule=schedule,
                         final_norm=norm, tie_embeddings=True, max_positions=1 << 20, embed_name="embed", final_norm_prefix="final.norm",
                         head_name="head", embed_scale=self.embedding_scale,
                         tables=((LOOP_TABLE, (self.loop[2], W)),) if self.loop else (),
                         matrices=((LOOP_MATRIX, (W, 2 * W)),) if self.loop else ())
