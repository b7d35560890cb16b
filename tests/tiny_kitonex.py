"""Tiny Kitonex configurations for the tests.  They differ from each other in every size and option:
  KA  sizes that are no multiples of 8 (the kernels' plain forms): three copies of the stream, values wider and narrower than
      keys, chunks of 7 and 11 positions and none, 3 and 5 taps and one, few buckets that end inside and outside a chunk, a layer
      without feed-forward, a layer that does not blend its values between layers that do (with other head counts), experts
      in groups and without
  KB  sizes the fast kernels take: two copies, heads of 64, values of 64 and 32, chunks of 33 and 40 positions, four taps, groups
      of which half are kept, a gated shared expert, three query heads a key head and one
  KC  as KB's shapes with four copies and every expert chosen (no choice can flip between number formats), for long runs in bfloat16
"""
import copy


def _attn(heads, kv_heads, dim, vdim, scale, conv, chunk, bias_max, buckets, v_mix):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "bias_buckets": buckets,
         "v_mix": v_mix}
    if conv is not None:
        m["conv"] = conv
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return m


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, groups=None, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


KA = {
    "architecture": "Kitonex", "width": 72, "vocab": 210, "norm": {"eps": 1e-4}, "streams": 3, "max_positions": 400,
    "layers": [
        _layer(_attn(6, 2, 12, 20, 0.4, 3, 7, 5, 6, True), _moe(6, 2, 20, groups=(3, 2), shared=12)),
        _layer(_attn(3, 1, 18, 6, 0.3, 5, 11, 30, 8, False), None),
        _layer(_attn(4, 4, 22, 10, 0.2, 2, None, 24, 10, True), _dense(44, 0.7)),
        _layer(_attn(5, 5, 6, 8, 0.5, 1, 7, 3, 4, True), _moe(3, 1, 28)),
    ],
}
KB = {
    "architecture": "Kitonex", "width": 128, "vocab": 300, "norm": {"eps": 1e-6}, "streams": 2, "max_positions": 1024,
    "layers": [
        _layer(_attn(6, 2, 64, 64, 0.125, 4, 33, 20, 16, True), _dense(96, 1.5)),
        _layer(_attn(6, 2, 64, 64, 0.2, 4, 40, 100, 32, True), _moe(8, 2, 64, groups=(4, 2), shared=32)),
        _layer(_attn(4, 4, 64, 32, 0.125, 4, 33, 33, 16, True), _moe(8, 3, 32, groups=(2, 1))),
    ],
}
KC = copy.deepcopy(KB)
KC["streams"] = 4
KC["layers"][1]["mlp"] = _moe(4, 4, 32, groups=(2, 2), shared=32)
KC["layers"][2]["mlp"] = _moe(2, 2, 48)

CONFIGS = {"KA": (KA, 41), "KB": (KB, 42), "KC": (KC, 43)}


def config(name):
    cfg, seed = CONFIGS[name]
    return copy.deepcopy(cfg), seed
