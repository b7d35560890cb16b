"""Kitonex: typed configuration and its description as parts.

A decoder-only model of layers listed one by one in config.json, on a residual stream of `streams` copies
(`parts/hyper.py`): every sublayer reads a weighted sum of the copies through a scale-only root-mean-square norm and
writes its result back into all of them with its own small matrices; the output is formed from the sum of the copies.

  embedding   E[token] plus a learned vector per position (P[p], `max_positions` of them).
  mixer       "attention" (`parts/attention.py`): grouped-query attention without rotation.  q, k and v have biases; a short
              causal convolution (`conv` taps) runs over every channel of the three; the whole query projection and the
              whole key projection are normed; scores times `scale` plus a learned bias per head and bucket of distances
              (`bias_max` is where the last bucket begins); chunks of `mask.size` positions that see only themselves; one is
              added to the softmax's denominator.  With `v_mix` the values are blended with those of the first such layer
              (a learned number per layer); values of `vdim`.
  mlp         kind "dense" (`parts/feed_forward.py`): g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit),
              W_down (g sigmoid(1.702 g) (u + 1)).
              kind "moe" (`parts/routed_experts.py`): `router.experts` experts W_down (silu(W_gate h) (W_up h)) of `expert.ff`,
              of which a token takes `router.top` by sigmoid score, from the `router.groups.keep` best of
              `router.groups.count` groups of neighbours; the chosen scores are divided by their sum; plus an optional shared
              expert of `shared.ff` times sigmoid(W_sg h), a number per token.  null: the layer has a mixer only.

The final norm and an output matrix of its own end the model.  What the design fixes stands here (which mechanisms exist,
the activations, 1e-20 beside the weights' sum); every size and every other constant is read from config.json, the number of
distance buckets from the table's tensor.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple, Union

from .base import Architecture, ConfigReader, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TensorSpec

ARCHITECTURE_NAME = "Kitonex"
MODEL_TYPE = "kitonex"
WEIGHT_SUM_EPS = 1e-20
MAX_TAPS = 8           # taps the kernels take
MAX_STREAMS = 8        # copies the kernels take
FIRST_VALUES = "kitonex.first_values"


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: Optional[int]
    chunk: Optional[int]
    bias_max: float
    bias_buckets: Optional[int]       # optional key of this library: the number of buckets where there is no file
    v_mix: bool


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    limit: float


@dataclass(frozen=True)
class MoEConfig:
    experts: int
    top: int
    ff: int
    groups: Optional[Tuple[int, int]]     # count, keep
    shared_ff: Optional[int]


@dataclass(frozen=True)
class KitonexLayer:
    mixer: AttentionConfig
    mlp: Union[None, DenseConfig, MoEConfig]


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


def _parse_attention(m: Dict[str, Any]):
    r = ConfigReader(m, "mixer")
    heads = r.integer("heads", minimum=1)
    kv_heads = r.integer("kv_heads", default=heads, minimum=1)
    dim = r.integer("dim", minimum=1)
    vdim = r.integer("vdim", default=dim, minimum=1)
    scale = r.number("scale")
    conv = r.integer("conv", default=0, minimum=0, maximum=MAX_TAPS) or None
    bias_max = r.number("bias_max", positive=True)
    buckets = r.integer("bias_buckets", default=0, minimum=0) or None
    v_mix = r.boolean("v_mix", default=False)
    if heads is not None and kv_heads is not None:
        r.check(heads % kv_heads == 0, f"heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    if buckets is not None:
        r.check(buckets % 2 == 0, f"bias_buckets ({buckets}) must be even")
    chunk = None
    rk = _sub(m, "mask", r, required=False)
    if rk is not None:
        chunk = rk.integer("size", minimum=1)
        _fold(r, rk)
    if r.problems:
        return None, r.problems
    return AttentionConfig(heads, kv_heads, dim, vdim, scale, conv, chunk, bias_max, buckets, v_mix), []


def _parse_mlp(f):
    if not isinstance(f, dict):
        return None, ["key 'mlp' must be an object or null"]
    r = ConfigReader(f, "mlp")
    kind = r.string("kind")
    out = None
    if kind == "dense":
        ff = r.integer("ff", minimum=1)
        limit = r.number("limit", positive=True)
        out = DenseConfig(ff, limit)
    elif kind == "moe":
        ff = experts = top = shared = groups = None
        re_ = _sub(f, "expert", r)
        if re_ is not None:
            ff = re_.integer("ff", minimum=1)
            _fold(r, re_)
        rr = _sub(f, "router", r)
        if rr is not None:
            experts = rr.integer("experts", minimum=1)
            top = rr.integer("top", minimum=1)
            choose_from = experts
            rg = _sub(rr.raw, "groups", rr, required=False)
            if rg is not None:
                count, keep = rg.integer("count", minimum=1), rg.integer("keep", minimum=1)
                if None not in (count, keep):
                    rg.check(keep <= count, f"keep ({keep}) exceeds count ({count})")
                    if experts is not None:
                        rg.check(experts % count == 0, f"{experts} experts do not form {count} equal groups")
                        choose_from = keep * (experts // count)
                    groups = (count, keep)
                _fold(rr, rg)
            if choose_from is not None and top is not None:
                rr.check(top <= choose_from, f"top ({top}) of {choose_from} experts cannot be chosen")
            _fold(r, rr)
        rs = _sub(f, "shared", r, required=False)
        if rs is not None:
            shared = rs.integer("ff", minimum=1)
            _fold(r, rs)
        out = MoEConfig(experts, top, ff, groups, shared)
    elif kind is not None:
        r.problems.append(f"kind '{kind}' is not known (known: 'dense', 'moe')")
    if r.problems:
        return None, [f"mlp: {p}" for p in r.problems]
    return out, []


def _parse_layer(entry):
    if not isinstance(entry, dict):
        return None, ["must be an object"]
    r = ConfigReader(entry, "layer")
    kind = r.string("type")
    mixer = mlp = None
    if kind is not None and kind != "attention":
        r.problems.append(f"type '{kind}' is not known (known: 'attention')")
    elif kind is not None:
        if not isinstance(entry.get("mixer"), dict):
            r.problems.append("missing key 'mixer' (an object)")
        else:
            mixer, problems = _parse_attention(entry["mixer"])
            r.problems += [f"mixer: {p}" for p in problems]
    if entry.get("mlp") is not None:
        mlp, problems = _parse_mlp(entry["mlp"])
        r.problems += problems
    if r.problems:
        return None, r.problems
    return KitonexLayer(mixer, mlp), []


@dataclass(frozen=True)
class KitonexConfig:
    width: int
    vocab: int
    eps: float
    streams: int
    max_positions: int
    layers: Tuple[KitonexLayer, ...]

    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "KitonexConfig":
        r = ConfigReader(raw, "Kitonex config")
        width = r.integer("width", minimum=1)
        vocab = r.integer("vocab", minimum=1)
        streams = r.integer("streams", minimum=1, maximum=MAX_STREAMS)
        maxpos = r.integer("max_positions", minimum=1)
        eps = None
        rn = _sub(raw, "norm", r)
        if rn is not None:
            eps = rn.number("eps", positive=True)
            _fold(r, rn)
        layers: List[KitonexLayer] = []
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            r.problems.append("key 'layers' must list at least one layer")
            listed = []
        for i, entry in enumerate(listed):
            layer, problems = _parse_layer(entry)
            r.problems += [f"layers[{i}]: {p}" for p in problems]
            if layer is not None:
                layers.append(layer)
        if len(layers) == len(listed):
            mixed = [(i, l.mixer) for i, l in enumerate(layers) if l.mixer.v_mix]
            for i, m in mixed[1:]:
                first = mixed[0][1]
                r.check(m.kv_heads * m.vdim == first.kv_heads * first.vdim,
                        f"layers[{i}]: {m.kv_heads} x {m.vdim} values cannot be mixed with layer {mixed[0][0]}'s {first.kv_heads} x {first.vdim}")
        r.finish()
        return KitonexConfig(width, vocab, eps, streams, maxpos, tuple(layers))


# ---- the description as parts ----

def _mat(name: str, out_features: int, in_features: int) -> TensorSpec:
    """A matrix [out, in]; random weights are drawn with a standard deviation of in^(-1/2), so that a product keeps the
    size of what it reads and every mechanism of a random model weighs in the logits."""
    return TensorSpec(name, (out_features, in_features), init_std=float(in_features) ** -0.5)


def _vec(name: str, n: int, std: float, mean: float = 0.0) -> TensorSpec:
    return TensorSpec(name, (n,), "vector", init_std=std, init_mean=mean)


def _attention_part(cfg: KitonexConfig, m: AttentionConfig, p: str, first_mixed: bool) -> PartSpec:
    W, H, G = cfg.width, m.heads, m.kv_heads
    sizes = {"q": H * m.dim, "k": G * m.dim, "v": G * m.vdim}
    tensors = {"o": _mat(p + "o", W, H * m.vdim), "rel": TensorSpec(p + "rel", (m.bias_buckets, H), "vector", init_std=0.5)}
    for name, n in sizes.items():
        tensors[name] = _mat(p + name, n, W)
        tensors[name + "_bias"] = _vec(p + name + ".b", n, 0.1)
        if m.conv is not None:
            tensors[name + "_conv"] = TensorSpec(p + name + ".conv", (n, m.conv), init_std=0.4)
        if name != "v":
            tensors[name + "_norm"] = _vec(p + name + ".norm", n, 0.1, 1.0)
    params = {"hidden_size": W, "n_heads": H, "n_kv_heads": G, "head_dim": m.dim, "value_dim": m.vdim, "score_scale": m.scale,
              "proj_norm_eps": cfg.eps, "chunk": m.chunk, "off_by_one": True,
              "distance_bias": {"max": m.bias_max, "longest": min(m.chunk or cfg.max_positions, cfg.max_positions)}}
    if m.v_mix:
        params["v_mix"] = {"name": FIRST_VALUES, "first": first_mixed}
        if not first_mixed:
            tensors["v_mix"] = TensorSpec(p + "vmix", (), "vector", init_std=0.2, init_mean=0.4)
    return PartSpec("attention", params, tensors)


def _dense_part(cfg: KitonexConfig, f: DenseConfig, p: str) -> PartSpec:
    W = cfg.width
    return PartSpec("gated_mlp", {"hidden_size": W, "intermediate_size": f.ff, "activation": "swish_limit", "activation_param": f.limit},
                    {"gate": _mat(p + "gate", f.ff, W), "up": _mat(p + "up", f.ff, W), "down": _mat(p + "down", W, f.ff)})


def _moe_part(cfg: KitonexConfig, f: MoEConfig, p: str) -> PartSpec:
    W = cfg.width
    tensors = {"router": _mat(p + "router", f.experts, W)}

    def expert(roles, name, ff):
        for role, tensor in zip(roles, (_mat(p + name + ".gate", ff, W), _mat(p + name + ".up", ff, W), _mat(p + name + ".down", W, ff))):
            tensors[role] = tensor

    for e in range(f.experts):
        expert((f"gate{e}", f"up{e}", f"down{e}"), f"e{e}", f.ff)
    if f.shared_ff is not None:
        expert(("shared_gate", "shared_up", "shared_down"), "shared", f.shared_ff)
        tensors["shared_sg"] = _mat(p + "shared.sg", 1, W)
    return PartSpec("routed_experts", {"hidden_size": W, "expert_size": f.ff, "n_experts": f.experts, "n_identity": 0, "top": f.top,
                                       "form": "silu", "scoring": "sigmoid", "groups": f.groups, "normalise_eps": WEIGHT_SUM_EPS}, tensors)


def _connection(p: str, q: int, copies: int) -> Dict[str, TensorSpec]:
    """The small matrices of one sublayer's connection to the copies of the stream (random ones keep the copies' size)."""
    return {f"read{q}": _vec(f"{p}hc{q}.in", copies, 0.2, 1.0 / copies), f"write{q}": _vec(f"{p}hc{q}.out", copies, 0.3, 0.8),
            f"mix{q}": TensorSpec(f"{p}hc{q}.mix", (copies, copies), "vector", init_std=0.2, init_mean=0.8 / copies)}


def build_spec(cfg: KitonexConfig) -> ModelSpec:
    """The model as parts; tensor names are the checkpoint's own ('l<i>.' + 'norm1', 'mix.q.conv', 'hc1.in', 'mlp.e<k>.gate', ...)."""
    W, V = cfg.width, cfg.vocab

    def norm(name):
        return PartSpec("rms_norm", {"size": W, "eps": cfg.eps, "offset": 0.0}, {"weight": _vec(name, W, 0.1, 1.0)})

    layers: List[LayerSpec] = []
    ignored: List[str] = []
    seen_mixed = False
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        first_mixed = m.v_mix and not seen_mixed
        seen_mixed = seen_mixed or m.v_mix
        if not m.v_mix or first_mixed:
            ignored.append(p + "mix.vmix")            # the first of the layers that blend has nothing to blend with
        norms, tensors = {"pre_mixer": norm(p + "norm1")}, _connection(p, 1, cfg.streams)
        ff = None
        if layer.mlp is not None:
            ff = _dense_part(cfg, layer.mlp, p + "mlp.") if isinstance(layer.mlp, DenseConfig) else _moe_part(cfg, layer.mlp, p + "mlp.")
            norms["pre_feed_forward"] = norm(p + "norm2")
            tensors.update(_connection(p, 2, cfg.streams))
        else:
            ignored += [p + "norm2", p + "hc2.*"]
        layers.append(LayerSpec("hyper", _attention_part(cfg, m, p + "mix.", first_mixed), ff, norms, {}, tensors))
    spec = ModelSpec(
        architecture=ARCHITECTURE_NAME, hidden_size=W, vocab_size=V, max_positions=cfg.max_positions,
        embedding=PartSpec("scaled_embedding", {"vocab_size": V, "hidden_size": W, "scale": 1.0},
                           {"table": TensorSpec("embed", (V, W), init_std=1.0),
                            "positions": TensorSpec("pos", (cfg.max_positions, W), init_std=0.3)}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i, None) for i in range(len(layers))),
        final_norm=norm("final.norm"), stream=PartSpec("hyper", {"copies": cfg.streams}),
        head=PartSpec("linear_head", {"vocab_size": V, "hidden_size": W, "softcap": None}, {"weight": _mat("head", V, W)}),
        ignored_tensors=tuple(ignored))
    spec.validate()
    return spec


register_architecture(Architecture(ARCHITECTURE_NAME, MODEL_TYPE, KitonexConfig.from_dict, build_spec), replace=True)
