"""Paditar: typed configuration and its description as parts.

A decoder-only model of layers listed one by one in config.json, of which a stretch is a loop of several passes over the same
weights (`loop`: layers `start` to `stop` - 1, `times` passes, each with its own cache and state).  Before every pass but the
first the embedded tokens join the residual stream again, and before every pass a learned vector of that pass does
(`loop.step`).  Every sublayer has a norm before and a norm after it, x <- x + norm'(f(norm(x))), scale-only root-mean-square
norms whose weight holds the scale minus one.  A layer's `type` names its mixer:

  "attention"  differential attention (`parts/head_attention.py`): two softmaxes per head over the same values, rotary positions
               per map, the difference a_1 - lambda a_2 normed per head, an element-wise sigmoid gate.
  "parallel"   two mixers side by side whose results are added with constants (`parts/mixer_pair.py`).  Left: attention with
               biases, a short convolution on q and k, values that are the keys as they leave it, norms per head, queries scaled
               by a temperature that grows with the position, one in the softmax's denominator and a sigmoid gate per head
               (`parts/head_attention.py`).  Right: the matrix memory of xLSTM (`parts/matrix_memory.py`).

  mlp          kind "dense": W_down max(W_up h, 0)^2 (`parts/feed_forward.py`); null: the layer has a mixer only.

Logits are the final norm's rows times the embedding table.  What the design fixes stands here (which mechanisms exist, the
activations, 1e-6 beside the memory's denominator, q's dim^(-1/2) there); every size and every other constant is read from
config.json.  The design names no longest context; position tables are built for `max_positions` (an optional key of this
library, default 32,768).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple, Union

from .base import Architecture, ConfigReader, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, TensorSpec, looped_schedule

ARCHITECTURE_NAME = "Paditar"
MODEL_TYPE = "paditar"
DEFAULT_MAX_POSITIONS = 32768
MAX_TAPS = 8                # taps the kernels take
MAX_HEAD = 512              # values of a head the kernels take
MEMORY_DEN_EPS = 1e-6


@dataclass(frozen=True)
class RotaryConfig:
    base: float
    dims: int


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: RotaryConfig


@dataclass(frozen=True)
class LeftConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    conv: int
    temp_coef: float
    temp_every: float


@dataclass(frozen=True)
class RightConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelConfig:
    left: LeftConfig
    right: RightConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class PaditarLayer:
    mixer: Union[DifferentialConfig, ParallelConfig]
    ff: Optional[int]                            # the dense feed-forward's inner size; None: no feed-forward


@dataclass(frozen=True)
class PaditarConfig:
    width: int
    vocab: int
    eps: float
    max_positions: int
    layers: Tuple[PaditarLayer, ...]
    loop: Optional[Tuple[int, int, int]]         # start, stop, times

    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "PaditarConfig":
        r = ConfigReader(raw, "Paditar config")
        width = r.integer("width", minimum=1)
        vocab = r.integer("vocab", minimum=1)
        maxpos = r.integer("max_positions", default=DEFAULT_MAX_POSITIONS, minimum=1)
        eps = None
        rn = _sub(raw, "norm", r)
        if rn is not None:
            eps = rn.number("eps", positive=True)
            _fold(r, rn)
        layers: List[PaditarLayer] = []
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            r.problems.append("key 'layers' must list at least one layer")
            listed = []
        for i, entry in enumerate(listed):
            layer, problems = _parse_layer(entry)
            r.problems += [f"layers[{i}]: {p}" for p in problems]
            if layer is not None:
                layers.append(layer)
        loop = None
        rl = _sub(raw, "loop", r, required=False)
        if rl is not None:
            start, stop, times = rl.integer("start", minimum=0), rl.integer("stop", minimum=1), rl.integer("times", minimum=1)
            if None not in (start, stop, times):
                rl.check(start < stop <= len(listed), f"layers {start} to {stop - 1} are not among the {len(listed)} listed")
                loop = (start, stop, times)
            _fold(r, rl)
        r.finish()
        return PaditarConfig(width, vocab, eps, maxpos, tuple(layers), loop)


def _sub(raw, key, reader: ConfigReader, required=True):
    """The object under `key` as a reader of its own, or None (a problem is noted if it is required or ill-typed)."""
    v = raw.get(key)
    if v is None:
        if required:
            reader.problems.append(f"missing key '{key}' (an object)")
        return None
    if not isinstance(v, dict):
        reader.problems.append(f"key '{key}' must be an object")
        return None
    return ConfigReader(v, key)


def _fold(parent: ConfigReader, child: Optional[ConfigReader]):
    if child is not None:
        parent.problems += [f"{child.what}: {p}" for p in child.problems]


def _heads(r: ConfigReader):
    heads = r.integer("heads", minimum=1)
    kv_heads = r.integer("kv_heads", default=heads, minimum=1)
    if None not in (heads, kv_heads):
        r.check(heads % kv_heads == 0, f"heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    dim = r.integer("dim", minimum=1, maximum=MAX_HEAD)
    return heads, kv_heads, dim, r.integer("vdim", default=dim, minimum=1, maximum=MAX_HEAD)


def _parse_differential(r: ConfigReader) -> DifferentialConfig:
    heads, kv_heads, dim, vdim = _heads(r)
    scale, diff = r.number("scale"), r.number("diff")
    rot = None
    rr = _sub(r.raw, "rot", r)
    if rr is not None:
        base, dims = rr.number("base", positive=True), rr.integer("dims", minimum=2)
        if None not in (dims, dim):
            rr.check(dims % 2 == 0 and dims <= dim, f"dims ({dims}) must be even and at most dim ({dim})")
        rot = RotaryConfig(base, dims)
        _fold(r, rr)
    return DifferentialConfig(heads, kv_heads, dim, vdim, scale, diff, rot)


def _parse_left(r: ConfigReader) -> LeftConfig:
    heads, kv_heads, dim, vdim = _heads(r)
    r.check(vdim == dim, f"the values are the keys: vdim ({vdim}) must be dim ({dim})")
    scale = r.number("scale")
    conv = r.integer("conv", minimum=1, maximum=MAX_TAPS)
    coef = every = None
    rt = _sub(r.raw, "q_temp", r)
    if rt is not None:
        coef, every = rt.number("coef"), rt.number("every", positive=True)
        _fold(r, rt)
    return LeftConfig(heads, kv_heads, dim, scale, conv, coef, every)


def _parse_right(r: ConfigReader) -> RightConfig:
    heads, dim = r.integer("heads", minimum=1), r.integer("dim", minimum=1, maximum=MAX_HEAD)
    return RightConfig(heads, dim, r.integer("vdim", default=dim, minimum=1, maximum=MAX_HEAD), r.number("gate_cap", positive=True))


def _parse_layer(entry):
    if not isinstance(entry, dict):
        return None, ["must be an object"]
    r = ConfigReader(entry, "layer")
    kind = r.string("type")
    mixer = None
    if kind is not None and kind not in ("attention", "parallel"):
        r.problems.append(f"type '{kind}' is not known (known: 'attention', 'parallel')")
    elif kind is not None:
        rm = _sub(entry, "mixer", r)
        if rm is not None:
            if kind == "attention":
                mixer = _parse_differential(rm)
            else:
                rl, rr = _sub(rm.raw, "left", rm), _sub(rm.raw, "right", rm)
                left = _parse_left(rl) if rl is not None else None
                right = _parse_right(rr) if rr is not None else None
                _fold(rm, rl)
                _fold(rm, rr)
                mixer = ParallelConfig(left, right, rm.number("left_scale"), rm.number("right_scale"))
            _fold(r, rm)
    ff = None
    if entry.get("mlp") is not None:
        rf = _sub(entry, "mlp", r)
        if rf is not None:
            fk = rf.string("kind")
            rf.check(fk is None or fk == "dense", f"kind '{fk}' is not known (known: 'dense')")
            ff = rf.integer("ff", minimum=1)
            _fold(r, rf)
    if r.problems:
        return None, r.problems
    return PaditarLayer(mixer, ff), []


# ---- the description as parts ----

def _mat(name: str, out_features: int, in_features: int) -> TensorSpec:
    """A matrix [out, in]; random weights are drawn with a standard deviation of in^(-1/2), so that a product keeps the
    size of what it reads and every mechanism of a random model weighs in the logits."""
    return TensorSpec(name, (out_features, in_features), init_std=float(in_features) ** -0.5)


def _vec(name: str, n: int, std: float, mean: float = 0.0) -> TensorSpec:
    return TensorSpec(name, (n,), "vector", init_std=std, init_mean=mean)


def _differential_part(cfg: PaditarConfig, m: DifferentialConfig, p: str) -> PartSpec:
    W, H, G = cfg.width, m.heads, m.kv_heads
    tensors = {"q": _mat(p + "q", H * 2 * m.dim, W), "k": _mat(p + "k", G * 2 * m.dim, W), "v": _mat(p + "v", G * m.vdim, W),
               "g": _mat(p + "g", H * m.vdim, W), "o": _mat(p + "o", W, H * m.vdim)}
    for name in ("lq1", "lk1", "lq2", "lk2"):
        tensors[name] = _vec(p + name, m.dim, 0.15)
    return PartSpec("head_attention", {
        "hidden_size": W, "n_heads": H, "n_kv_heads": G, "head_dim": m.dim, "value_dim": m.vdim, "score_scale": m.scale,
        "differential": {"diff": m.diff, "eps": cfg.eps}, "gate": "value",
        "position": PartSpec("rotary", {"theta": m.rot.base, "head_dim": m.dim, "rotary_dim": m.rot.dims,
                                        "max_positions": cfg.max_positions, "pairing": "half"})}, tensors)


def _left_part(cfg: PaditarConfig, m: LeftConfig, p: str) -> PartSpec:
    W, H, G = cfg.width, m.heads, m.kv_heads
    tensors = {"g": _mat(p + "g", H, W), "o": _mat(p + "o", W, H * m.dim), "o_bias": _vec(p + "o.b", W, 0.1)}
    for name, n in (("q", H * m.dim), ("k", G * m.dim)):
        tensors[name] = _mat(p + name, n, W)
        tensors[name + "_bias"] = _vec(p + name + ".b", n, 0.1)
        tensors[name + "_conv"] = TensorSpec(p + name + ".conv", (n, m.conv), init_std=0.5)
        tensors[name + "_norm"] = _vec(p + name + ".norm", m.dim, 0.1, 1.0)
    return PartSpec("head_attention", {
        "hidden_size": W, "n_heads": H, "n_kv_heads": G, "head_dim": m.dim, "score_scale": m.scale, "values_from_keys": True,
        "head_norm_eps": cfg.eps, "q_temperature": {"coef": m.temp_coef, "every": m.temp_every}, "max_positions": cfg.max_positions,
        "off_by_one": True, "gate": "head"}, tensors)


def _right_part(cfg: PaditarConfig, m: RightConfig, p: str) -> PartSpec:
    W, H = cfg.width, m.heads
    tensors = {"q": _mat(p + "q", H * m.dim, W), "k": _mat(p + "k", H * m.dim, W), "v": _mat(p + "v", H * m.vdim, W),
               "g": _mat(p + "g", H * m.vdim, W), "o": _mat(p + "o", W, H * m.vdim), "norm": _vec(p + "norm", H * m.vdim, 0.1, 1.0),
               "i": _mat(p + "i", H, W), "i_bias": _vec(p + "i.b", H, 1.0, -0.5),
               "f": _mat(p + "f", H, W), "f_bias": _vec(p + "f.b", H, 1.5, 3.0)}
    return PartSpec("matrix_memory", {"hidden_size": W, "n_heads": H, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap,
                                      "q_scale": m.dim ** -0.5, "den_eps": MEMORY_DEN_EPS, "eps": cfg.eps}, tensors)


def build_spec(cfg: PaditarConfig) -> ModelSpec:
    """The model as parts; tensor names are the checkpoint's own ('l<i>.' + 'norm1', 'mix.left.q.conv', 'mlp.up', 'loop.step', ...)."""
    W, V = cfg.width, cfg.vocab

    def norm(name):     # the weight holds the scale minus one (offset 1)
        return PartSpec("rms_norm", {"size": W, "eps": cfg.eps, "offset": 1.0}, {"weight": _vec(name, W, 0.1)})

    layers: List[LayerSpec] = []
    ignored: List[str] = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, DifferentialConfig):
            mixer = _differential_part(cfg, m, p + "mix.")
        else:
            mixer = PartSpec("mixer_pair", {"left": _left_part(cfg, m.left, p + "mix.left."), "right": _right_part(cfg, m.right, p + "mix.right."),
                                            "left_scale": m.left_scale, "right_scale": m.right_scale})
        norms = {"pre_mixer": norm(p + "norm1"), "post_mixer": norm(p + "norm1b")}
        ff = None
        if layer.ff is not None:
            ff = PartSpec("plain_mlp", {"hidden_size": W, "intermediate_size": layer.ff, "activation": "relu2"},
                          {"up": _mat(p + "mlp.up", layer.ff, W), "down": _mat(p + "mlp.down", W, layer.ff)})
            norms.update(pre_feed_forward=norm(p + "norm2"), post_feed_forward=norm(p + "norm2b"))
        else:
            ignored += [p + "norm2", p + "norm2b"]       # a file may carry them; a layer without a feed-forward does not read them
        layers.append(LayerSpec("sandwich", mixer, ff, norms))
    if cfg.loop is not None:
        start, stop, times = cfg.loop
        schedule = looped_schedule(len(layers), start, stop, times, TensorSpec("loop.step", (times, W), "vector", init_std=0.3))
    else:
        schedule = looped_schedule(len(layers), 0, len(layers), 1)
    table = TensorSpec("embed", (V, W), init_std=1.0)
    spec = ModelSpec(
        architecture=ARCHITECTURE_NAME, hidden_size=W, vocab_size=V, max_positions=cfg.max_positions,
        embedding=PartSpec("scaled_embedding", {"vocab_size": V, "hidden_size": W, "scale": 1.0}, {"table": table}),
        layers=tuple(layers), schedule=schedule, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": V, "hidden_size": W, "softcap": None}, {"weight": table}),
        ignored_tensors=tuple(ignored))
    spec.validate()
    return spec


register_architecture(Architecture(ARCHITECTURE_NAME, MODEL_TYPE, PaditarConfig.from_dict, build_spec), replace=True)
