"""Typed configuration of Mefatar (config.json key "architecture": "Mefatar").

A small decoder of pre-norm layers (RMS norm) whose updates are multiplied by learned vectors,
x <- x + ls1 * mixer(norm1(x)), x <- x + ls2 * ff(norm2(x)); the head is the embedding table itself.
config.json lists the layers one by one; `loop` = {start, stop, times} runs layers start .. stop - 1
`times` times in a row with the same weights, each pass with a cache and a state of its own. A layer's
mixer is one of

- "parallel": two mixers side by side on the same input, each one's output RMS-normed over the model's
  width, half the sum of both. Left (`.left`): grouped-query causal softmax attention without biases, a
  short causal convolution over time on every channel of q, k and v, one RMS norm over the whole query
  and one over the whole key projection, rotation of the first rot.dims of a head in the interleaved
  pairing, optionally with frequencies stretched by wavelength (rot.scaling: factor, low, high,
  original), a learned sink a head in the softmax, a sigmoid gate on the output. Right (`.right`): gated
  linear attention, a matrix state a head with a decay for every key channel from a product of low rank;
- "rglru": a recurrent block with a real-gated linear recurrent unit of `width` channels in `blocks`
  blocks.

A layer's feed-forward is dense (a gated unit with the tanh form of GELU) or absent, and then the layer
is its mixer alone. config.json gives every size and constant but the rank of the decays' product, which
is the shape of `.right.a1` (`sized_by` reads it from the checkpoint; a config.json may also name it as
`decay_rank`, as the random-weights mode writes it).
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Dict, Optional, Tuple

from .dabevik import _int, _num, _obj
from .rasezen import UNBOUNDED_POSITIONS
from .registry import eos_ids_of, register_architecture
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

SCALING = ("factor", "low", "high", "original")


def _rot(m, where, limit):
    """(dims, base, scaling or None); dims 0 without a rotation."""
    if m.get("rot") is None:
        return 0, 1.0, None
    rot, w = _obj(m, "rot", where), where + "rot."
    dims, base = _int(rot, "dims", w, 0), _num(rot, "base", w)
    if dims % 2 or dims > limit:
        raise ConfigError(f"config.json: {w}dims {dims} must be even and at most {limit}")
    if base <= 0:
        raise ConfigError(f"config.json: {w}base must be positive")
    if rot.get("scaling") is None:
        return dims, base, None
    sc = _obj(rot, "scaling", w)
    sc = tuple(_num(sc, k, w + "scaling.") for k in SCALING)
    if min(sc) <= 0 or sc[2] < sc[1]:
        raise ConfigError(f"config.json: {w}scaling must be positive numbers with low at most high")
    return dims, base, sc


@dataclass(frozen=True)
class MefatarSoftmaxSide:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    rot_dims: int
    rot_base: float
    rot_scaling: Optional[Tuple[float, float, float, float]]

    @classmethod
    def from_dict(cls, m, where):
        dim = _int(m, "dim", where)
        dims, base, sc = _rot(m, where, dim)
        a = cls(heads=_int(m, "heads", where), kv_heads=_int(m, "kv_heads", where), dim=dim, vdim=_int(m, "vdim", where),
                conv=_int(m, "conv", where), scale=_num(m, "scale", where), rot_dims=dims, rot_base=base, rot_scaling=sc)
        if a.heads % a.kv_heads:
            raise ConfigError(f"config.json: {where}{a.heads} heads are not a multiple of {a.kv_heads} kv_heads")
        return a

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv,
             "scale": self.scale}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                d["rot"]["scaling"] = dict(zip(SCALING, self.rot_scaling))
        return d


@dataclass(frozen=True)
class MefatarGatedSide:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0        # 0: not known yet (the shape of `.a1`)

    @classmethod
    def from_dict(cls, m, where):
        a = cls(heads=_int(m, "heads", where), dim=_int(m, "dim", where), vdim=_int(m, "vdim", where),
                tau=_num(m, "tau", where), decay_rank=_int(m, "decay_rank", where) if "decay_rank" in m else 0)
        if a.tau <= 0:
            raise ConfigError(f"config.json: {where}tau must be positive")
        return a

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}
        if self.decay_rank:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass(frozen=True)
class MefatarParallel:
    left: MefatarSoftmaxSide
    right: MefatarGatedSide

    @classmethod
    def from_dict(cls, m, where):
        return cls(left=MefatarSoftmaxSide.from_dict(_obj(m, "left", where), where + "left."),
                   right=MefatarGatedSide.from_dict(_obj(m, "right", where), where + "right."))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class MefatarRecurrent:
    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, m, where):
        a = cls(width=_int(m, "width", where), blocks=_int(m, "blocks", where), conv=_int(m, "conv", where))
        if a.width % a.blocks:
            raise ConfigError(f"config.json: {where}width {a.width} does not divide into {a.blocks} blocks")
        return a

    def to_dict(self):
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class MefatarLayer:
    type: str
    mixer: Any
    ff: int                    # 0: no feed-forward


@register_architecture("Mefatar")
@dataclass(frozen=True)
class MefatarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[MefatarLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None             # start, stop, times
    max_positions: int = UNBOUNDED_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    MIXERS = {"parallel": MefatarParallel, "rglru": MefatarRecurrent}

    @classmethod
    def from_dict(cls, d: dict) -> "MefatarConfig":
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
            ff = 0
            if e.get("mlp") is not None:
                mlp = _obj(e, "mlp", where)
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind')!r} is not a feed-forward of this "
                                      "design (known: 'dense')")
                ff = _int(mlp, "ff", where + "mlp.")
            layers.append(MefatarLayer(kind, mixer, ff))
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
        d = {"architecture": "Mefatar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [{"type": l.type, "mixer": l.mixer.to_dict(),
                         "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != UNBOUNDED_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    def sized_by(self, shape_of) -> "MefatarConfig":
        """The sizes that only tensors give: `shape_of(name)` is a stored tensor's shape or None."""
        layers = []
        for i, l in enumerate(self.layers):
            if l.type == "parallel" and not l.mixer.right.decay_rank:
                a1 = shape_of(f"l{i}.mix.right.a1")
                if a1:
                    l = replace(l, mixer=replace(l.mixer, right=replace(l.mixer.right, decay_rank=int(a1[0]))))
            layers.append(l)
        return replace(self, layers=tuple(layers))

    # ------------------------------------------------------------ meaning
    def model_spec(self) -> ModelSpec:
        D, eps = self.width, self.norm_eps

        def norm(name):
            return PartSpec("rmsnorm", {"size": D, "eps": eps, "tensor": name})

        specs = []
        for i, l in enumerate(self.layers):
            p, m = f"l{i}", l.mixer
            if l.type == "parallel":
                a, b = m.left, m.right
                position = PartSpec("none", {})
                if a.rot_dims:
                    rot = {"head_dim": a.dim, "rotary_dim": a.rot_dims, "theta": a.rot_base, "wide_frequencies": True}
                    if a.rot_scaling is not None:
                        rot["scaling"] = dict(zip(SCALING, a.rot_scaling))
                    position = PartSpec("rotary", rot)
                if not b.decay_rank:
                    raise ConfigError(f"config.json: layers[{i}].mixer.right: the rank of the decays' product is not known "
                                      f"(the shape of {p}.mix.right.a1, or decay_rank)")
                left = PartSpec("wide_norm_attention", {
                    "hidden_size": D, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
                    "value_dim": a.vdim, "softmax_scale": a.scale, "window": 0, "norm_eps": eps, "bias": False,
                    "taps": a.conv, "sink": True, "output_gate": True, "interleaved_rotation": True,
                    "position": position}, prefix=f"{p}.mix.left")
                right = PartSpec("gated_linear_attention", {
                    "hidden_size": D, "num_heads": b.heads, "head_dim": b.dim, "value_dim": b.vdim, "tau": b.tau,
                    "decay_rank": b.decay_rank, "norm_eps": eps}, prefix=f"{p}.mix.right")
                out = lambda side: {"tensor": f"{p}.mix.{side}.out", "eps": eps, "size": D}
                mixer = PartSpec("side_by_side", {"parts": [{"mixer": left, "scale": 0.5, "out_norm": out("left")},
                                                            {"mixer": right, "scale": 0.5, "out_norm": out("right")}]},
                                 prefix=f"{p}.mix")
            else:
                mixer = PartSpec("real_gated_lru", {"hidden_size": D, "channels": m.width, "blocks": m.blocks,
                                                    "taps": m.conv}, prefix=f"{p}.mix")
            ffn, norms, factors = None, {"mixer": norm(f"{p}.norm1")}, {"mixer": f"{p}.ls1"}
            if l.ff:
                ffn = PartSpec("swiglu", {"hidden_size": D, "intermediate_size": l.ff, "activation": "gelu",
                                          "tensor_names": {"gate": ".gate", "up": ".up", "down": ".down"}},
                               prefix=f"{p}.mlp")
                norms["ffn"], factors["ffn"] = norm(f"{p}.norm2"), f"{p}.ls2"
            specs.append(LayerSpec("pre_norm", mixer, ffn, norms, prefix=p, params={"update_factors": factors}))
        n = len(specs)
        start, stop, times = self.loop or (0, n, 1)
        order = list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))
        spec = ModelSpec(
            architecture="Mefatar", vocab_size=self.vocab, hidden_size=D, max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D, "tensor": "embed"}),
            layers=tuple(specs), schedule=tuple(ScheduleEntry(i) for i in order), final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D, "own_tensor": False,
                                          "tied_to": "embed"}), eos_token_ids=self.eos_token_ids)
        spec.validate()
        return spec
