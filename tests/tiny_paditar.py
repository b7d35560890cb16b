"""Tiny Paditar configurations for the tests.  They differ from each other in every size and option:
  PA  sizes that are no multiples of 8 (the kernels' plain forms): a loop that starts after the first layer and ends before the
      last, two passes; values narrower and wider than keys, part of a map rotated and all of it, 3 and 2 taps, layers without
      feed-forward inside and outside the loop, as many key heads as query heads
  PB  sizes the fast kernels take: a loop over the first two layers, three passes; twelve and sixteen query maps a key head (groups
      that go to several blocks), maps of 32 and 16, heads of 64, a memory with narrow and wide values, four taps
  PC  heads of 128, maps of 64, no loop at all, eight taps and one, for long runs
  PD  one layer in the loop, once (its vector joins, the embedding does not), heads of 96 and 80 values (laid out for the tensor cores
      without being multiples of 64)
"""
import copy


def _attn(heads, kv_heads, dim, vdim, scale, diff, base, dims):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": {"base": base, "dims": dims}}


def _pair(left, right, left_scale, right_scale):
    heads, kv_heads, dim, scale, conv, coef, every = left
    rh, rd, rv, cap = right
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "conv": conv,
                     "q_temp": {"coef": coef, "every": every}},
            "right": {"heads": rh, "dim": rd, "vdim": rv, "gate_cap": cap}, "left_scale": left_scale, "right_scale": right_scale}


def _layer(mixer, ff):
    return {"type": "parallel" if "left" in mixer else "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


PA = {
    "architecture": "Paditar", "width": 76, "vocab": 190, "norm": {"eps": 1e-4}, "max_positions": 400, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        _layer(_attn(4, 2, 10, 14, 0.5, 0.4, 300.0, 6), 50),
        _layer(_pair((6, 2, 12, 0.4, 3, 0.7, 9), (3, 10, 22, 7.0), 0.9, 1.3), None),
        _layer(_attn(3, 3, 6, 30, 0.6, 0.25, 50.0, 6), 44),
        _layer(_pair((5, 5, 18, 0.3, 2, 0.2, 5), (2, 20, 6, 11.0), 1.1, 0.6), None),
    ],
}
PB = {
    "architecture": "Paditar", "width": 128, "vocab": 300, "norm": {"eps": 1e-6}, "max_positions": 1024, "loop": {"start": 0, "stop": 2, "times": 3},
    "layers": [
        _layer(_pair((6, 2, 64, 0.15, 4, 0.4, 16), (2, 32, 48, 13.0), 0.8, 1.2), 160),
        _layer(_attn(6, 1, 32, 64, 0.25, 0.45, 10000.0, 16), 96),
        _layer(_attn(16, 2, 16, 32, 0.3, 0.6, 500.0, 16), None),
        _layer(_pair((9, 1, 32, 0.2, 4, 0.3, 40), (3, 64, 32, 5.0), 1.4, 0.5), 64),
    ],
}
PC = {
    "architecture": "Paditar", "width": 192, "vocab": 260, "norm": {"eps": 1e-5}, "max_positions": 2048,
    "layers": [
        _layer(_pair((2, 1, 128, 0.09, 8, 0.25, 64), (1, 128, 128, 20.0), 1.0, 1.0), 128),
        _layer(_attn(2, 1, 64, 128, 0.125, 0.35, 777.0, 64), None),
        _layer(_pair((4, 4, 16, 0.25, 1, 0.5, 100), (2, 16, 16, 15.0), 0.5, 2.0), 64),
    ],
}
PD = {
    "architecture": "Paditar", "width": 104, "vocab": 150, "norm": {"eps": 1e-6}, "max_positions": 600, "loop": {"start": 1, "stop": 2, "times": 1},
    "layers": [
        _layer(_pair((3, 3, 96, 0.11, 4, 0.6, 30), (2, 80, 16, 15.0), 1.2, 0.7), 72),
        _layer(_attn(4, 2, 40, 48, 0.2, 0.5, 2000.0, 20), 88),
    ],
}

CONFIGS = {"PA": (PA, 51), "PB": (PB, 52), "PC": (PC, 53), "PD": (PD, 54)}


def config(name):
    cfg, seed = CONFIGS[name]
    return copy.deepcopy(cfg), seed
