"""Typed configuration of Raranex (config.json key "architecture": "Raranex").

A small decoder of parallel layers with two RMS norms, x <- x + (mixer(norm1(x)) + ff(norm2(x))).
config.json lists the layers one by one; `loop` = {start, stop, times} runs layers start .. stop - 1
`times` times in a row with the same weights, each pass with a cache and a state of its own; where a pass
begins the stream is made anew from itself and the embedding's output (`loop.in`) and a vector of the pass
(`loop.step`) is added. A layer's mixer is one of

- "attention": grouped-query softmax attention without biases, rotation of the first rot.dims of a head in
  the interleaved pairing, queries and keys divided by their root mean square without a weight, a sliding
  window (mask.size) beside which the first mask.keep_first tokens stay in sight, a sigmoid gate a head;
- "parallel": two mixers side by side on the same input, each one's output RMS-normed over the model's
  width, half the sum of both. Left (`.left`): grouped-query causal attention without positions but for a
  factor on the queries that grows with the position (q_temp: coef, every), an RMS norm a head with one
  weight for all heads, capped scores (softcap), a sigmoid gate a head. Right (`.right`): RWKV-style time
  mixing, a matrix state a head with a decay a key channel and token.

A layer's feed-forward is a mixture of gated experts (sigmoid-scored, chosen with a correction from the best
groups, weights divided by their sum) beside a shared expert with a gate a token, or absent. config.json
gives every size and constant but the rank of the decays' product, which is the shape of `.right.w1`
(`sized_by` reads it from the checkpoint; a config.json may also name it as `decay_rank`, as the
random-weights mode writes it).
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Dict, Optional, Tuple

from .dabevik import _int, _num, _obj
from .rasezen import UNBOUNDED_POSITIONS
from .registry import eos_ids_of, register_architecture
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _heads(m, where):
    """(heads, kv_heads, dim, vdim, scale) of a softmax attention."""
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}{heads} heads are not a multiple of {kv} kv_heads")
    return heads, kv, _int(m, "dim", where), _int(m, "vdim", where), _num(m, "scale", where)


@dataclass(frozen=True)
class RaranexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                # 0: every earlier token
    keep_first: int
    rot_dims: int              # 0: no rotation
    rot_base: float

    @classmethod
    def from_dict(cls, m, where):
        heads, kv, dim, vdim, scale = _heads(m, where)
        window = keep = 0
        if m.get("mask") is not None:
            mask, w = _obj(m, "mask", where), where + "mask."
            window = _int(mask, "size", w)
            keep = _int(mask, "keep_first", w, 0) if "keep_first" in mask else 0
        dims, base = 0, 1.0
        if m.get("rot") is not None:
            rot, w = _obj(m, "rot", where), where + "rot."
            dims, base = _int(rot, "dims", w, 0), _num(rot, "base", w)
            if dims % 2 or dims > dim:
                raise ConfigError(f"config.json: {w}dims {dims} must be even and at most {dim}")
            if base <= 0:
                raise ConfigError(f"config.json: {w}base must be positive")
        return cls(heads, kv, dim, vdim, scale, window, keep, dims, base)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return d


@dataclass(frozen=True)
class RaranexLeft:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float             # 0: none
    temp_coef: float
    temp_every: float          # 0: no temperature

    @classmethod
    def from_dict(cls, m, where):
        cap = _num(m, "softcap", where) if m.get("softcap") is not None else 0.0
        coef = every = 0.0
        if m.get("q_temp") is not None:
            t, w = _obj(m, "q_temp", where), where + "q_temp."
            coef, every = _num(t, "coef", w), _num(t, "every", w)
            if every <= 0:
                raise ConfigError(f"config.json: {w}every must be positive")
        if cap < 0:
            raise ConfigError(f"config.json: {where}softcap must be positive")
        return cls(*_heads(m, where), cap, coef, every)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.temp_every:
            d["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return d


@dataclass(frozen=True)
class RaranexRight:
    heads: int
    dim: int
    decay_rank: int = 0        # 0: not known yet (the shape of `.w1`)

    @classmethod
    def from_dict(cls, m, where):
        return cls(heads=_int(m, "heads", where), dim=_int(m, "dim", where),
                   decay_rank=_int(m, "decay_rank", where) if "decay_rank" in m else 0)

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim}
        if self.decay_rank:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass(frozen=True)
class RaranexParallel:
    left: RaranexLeft
    right: RaranexRight

    @classmethod
    def from_dict(cls, m, where):
        return cls(left=RaranexLeft.from_dict(_obj(m, "left", where), where + "left."),
                   right=RaranexRight.from_dict(_obj(m, "right", where), where + "right."))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class RaranexExperts:
    experts: int
    top: int
    ff: int
    groups: Tuple[int, int]    # count, keep
    shared_ff: int             # 0: no shared expert

    @classmethod
    def from_dict(cls, m, where):
        if m.get("kind") != "moe":
            raise ConfigError(f"config.json: {where}kind {m.get('kind')!r} is not a feed-forward of this design (known: 'moe')")
        r, w = _obj(m, "router", where), where + "router."
        experts, top, groups = _int(r, "experts", w), _int(r, "top", w), (1, 1)
        if r.get("groups") is not None:
            g = _obj(r, "groups", w)
            groups = (_int(g, "count", w + "groups."), _int(g, "keep", w + "groups."))
        if experts % groups[0] or groups[1] > groups[0] or top > groups[1] * (experts // groups[0]):
            raise ConfigError(f"config.json: {w}{top} choices from {groups[1]} of {groups[0]} groups of {experts} experts")
        shared = _int(_obj(m, "shared", where), "ff", where + "shared.") if m.get("shared") is not None else 0
        return cls(experts=experts, top=top, ff=_int(_obj(m, "expert", where), "ff", where + "expert."), groups=groups,
                   shared_ff=shared)

    def to_dict(self):
        d = {"kind": "moe", "expert": {"ff": self.ff},
             "router": {"experts": self.experts, "top": self.top,
                        "groups": {"count": self.groups[0], "keep": self.groups[1]}}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class RaranexLayer:
    type: str
    mixer: Any
    mlp: Optional[RaranexExperts]


@register_architecture("Raranex")
@dataclass(frozen=True)
class RaranexConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[RaranexLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None             # start, stop, times
    max_positions: int = UNBOUNDED_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    MIXERS = {"attention": RaranexAttention, "parallel": RaranexParallel}

    @classmethod
    def from_dict(cls, d: dict) -> "RaranexConfig":
        for k in ("vocab", "width", "norm", "layers"):
            if k not in d:
                raise ConfigError(f"config.json: missing key '{k}'")
        entries = d["layers"]
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = e.get("type")
            if kind not in cls.MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not a mixer of this design "
                                  f"(known: {sorted(cls.MIXERS)})")
            mixer = cls.MIXERS[kind].from_dict(_obj(e, "mixer", where), where + "mixer.")
            mlp = RaranexExperts.from_dict(_obj(e, "mlp", where), where + "mlp.") if e.get("mlp") is not None else None
            layers.append(RaranexLayer(kind, mixer, mlp))
        loop = None
        if d.get("loop") is not None:
            lp = _obj(d, "loop", "")
            loop = (_int(lp, "start", "loop.", 0), _int(lp, "stop", "loop.", 0), _int(lp, "times", "loop.", 0))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop[0]} .. {loop[1]} - 1 of {len(layers)}")
        known = ("architecture", "vocab", "width", "norm", "layers", "loop", "max_positions", "eos_token_id", "torch_dtype")
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""),
                  norm_eps=_num(_obj(d, "norm", ""), "eps", "norm."), layers=tuple(layers), loop=loop,
                  max_positions=_int(d, "max_positions", "") if "max_positions" in d else UNBOUNDED_POSITIONS,
                  eos_token_ids=eos_ids_of(d.get("eos_token_id"), "config.json"),
                  extra={k: v for k, v in d.items() if k not in known})
        if cfg.norm_eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": "Raranex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [{"type": l.type, "mixer": l.mixer.to_dict(),
                         "mlp": l.mlp.to_dict() if l.mlp is not None else None} for l in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != UNBOUNDED_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    def sized_by(self, shape_of) -> "RaranexConfig":
        """The sizes that only tensors give: `shape_of(name)` is a stored tensor's shape or None."""
        layers = []
        for i, l in enumerate(self.layers):
            if l.type == "parallel" and not l.mixer.right.decay_rank:
                w1 = shape_of(f"l{i}.mix.right.w1")
                if w1:
                    l = replace(l, mixer=replace(l.mixer, right=replace(l.mixer.right, decay_rank=int(w1[0]))))
            layers.append(l)
        return replace(self, layers=tuple(layers))

    # ------------------------------------------------------------ meaning
    def _attention(self, a, prefix, **more):
        return PartSpec("head_norm_attention", {
            "hidden_size": self.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
            "value_dim": a.vdim, "softmax_scale": a.scale, "norm_eps": self.norm_eps, "output_gate": "head",
            "padded_cache": True, **more}, prefix=prefix)

    def model_spec(self) -> ModelSpec:
        D, eps = self.width, self.norm_eps

        def norm(name):
            return PartSpec("rmsnorm", {"size": D, "eps": eps, "tensor": name})

        specs = []
        for i, l in enumerate(self.layers):
            p, m = f"l{i}", l.mixer
            if l.type == "parallel":
                a, b = m.left, m.right
                if not b.decay_rank:
                    raise ConfigError(f"config.json: layers[{i}].mixer.right: the rank of the decays' product is not known "
                                      f"(the shape of {p}.mix.right.w1, or decay_rank)")
                left = self._attention(a, f"{p}.mix.left", softcap=a.softcap, position=PartSpec("none", {}),
                                       **({"query_temperature": (a.temp_coef, a.temp_every)} if a.temp_every else {}))
                right = PartSpec("time_mixing", {"hidden_size": D, "num_heads": b.heads, "head_dim": b.dim,
                                                 "decay_rank": b.decay_rank, "norm_eps": eps}, prefix=f"{p}.mix.right")
                out = lambda side: {"tensor": f"{p}.mix.{side}.out", "eps": eps, "size": D}
                mixer = PartSpec("side_by_side", {"parts": [{"mixer": left, "scale": 0.5, "out_norm": out("left")},
                                                            {"mixer": right, "scale": 0.5, "out_norm": out("right")}]},
                                 prefix=f"{p}.mix")
            else:
                position = PartSpec("none", {})
                if m.rot_dims:
                    position = PartSpec("rotary", {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base,
                                                   "wide_frequencies": True})
                mixer = self._attention(m, f"{p}.mix", window=m.window, keep_first=m.keep_first, qk_norm="unit",
                                        interleaved_rotation=True, position=position)
            ffn, norms = None, {"mixer": norm(f"{p}.norm1")}
            if l.mlp is not None:
                e = l.mlp
                ffn = PartSpec("routed_experts", {
                    "hidden_size": D, "expert_size": e.ff, "num_experts": e.experts, "top": e.top, "router": "sigmoid",
                    "correction": True, "groups": {"count": e.groups[0], "keep": e.groups[1]}, "normalize": True,
                    "shared": {"size": e.shared_ff}, "shared_gate": True, "update_by_place": True}, prefix=f"{p}.mlp")
                norms["ffn"] = norm(f"{p}.norm2")
            specs.append(LayerSpec("parallel", mixer, ffn, norms, prefix=p))
        n = len(specs)
        entries, stream = [ScheduleEntry(i) for i in range(n)], ()
        if self.loop is not None:
            start, stop, times = self.loop
            stream = (PartSpec("loop_input", {"hidden_size": D, "times": times, "tensor": "loop.in",
                                              "step_tensor": "loop.step"}),)
            passes = [ScheduleEntry(i, before=0 if i == start else None, before_index=t if i == start else 0)
                      for t in range(times) for i in range(start, stop)]
            entries = entries[:start] + passes + entries[stop:]
        spec = ModelSpec(
            architecture="Raranex", vocab_size=self.vocab, hidden_size=D, max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D, "tensor": "embed"}),
            layers=tuple(specs), schedule=tuple(entries), final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D, "tensor": "head"}),
            eos_token_ids=self.eos_token_ids, stream_parts=stream)
        spec.validate()
        return spec
