"""Kitonex without a GPU: the configuration reader, the model's description, the buckets of distances, the cache the chunks
ask for, and the plain implementation's own invariants."""
import copy
import math

import numpy as np
import pytest

import plain_kitonex as plain
import tiny_kitonex
from rust_deeplearning_b200.config.base import ConfigError, architecture_for
from rust_deeplearning_b200.parts.attention import distance_buckets


def _spec(cfg):
    arch = architecture_for(cfg)
    assert arch.name == "Kitonex"
    return arch.build_spec(arch.parse_config(cfg))


def test_configuration_becomes_parts():
    cfg, _ = tiny_kitonex.config("KA")
    spec = _spec(cfg)
    assert [layer.block for layer in spec.layers] == ["hyper"] * 4
    assert spec.stream.kind == "hyper" and spec.stream.params["copies"] == 3
    assert spec.layers[1].feed_forward is None and set(spec.layers[1].norms) == {"pre_mixer"}
    assert set(spec.layers[0].norms) == {"pre_mixer", "pre_feed_forward"}
    a = spec.layers[0].mixer.params
    assert (a["n_heads"], a["n_kv_heads"], a["head_dim"], a["value_dim"], a["chunk"]) == (6, 2, 12, 20, 7)
    assert a["proj_norm_eps"] == 1e-4 and a["off_by_one"] and a["distance_bias"] == {"max": 5.0, "longest": 7}
    assert spec.layers[2].mixer.params["chunk"] is None and spec.layers[2].mixer.params["distance_bias"]["longest"] == 400
    # the first layer that blends has nothing to blend with; the one that does not has no number for it
    assert a["v_mix"]["first"] and "v_mix" not in spec.layers[1].mixer.params and not spec.layers[2].mixer.params["v_mix"]["first"]
    names = spec.tensor_specs()
    assert "l0.mix.vmix" not in names and "l1.mix.vmix" not in names and names["l2.mix.vmix"].shape == ()
    assert names["l0.mix.q.norm"].shape == (72,) and names["l0.mix.k.norm"].shape == (24,) and names["l0.mix.o"].shape == (72, 120)
    assert names["l0.mix.v.conv"].shape == (40, 3) and names["l0.mix.k.b"].shape == (24,) and names["l0.mix.rel"].shape == (6, 6)
    assert names["l0.hc1.in"].shape == (3,) and names["l0.hc2.mix"].shape == (3, 3) and "l1.hc2.mix" not in names and "l1.norm2" not in names
    assert names["pos"].shape == (400, 72) and names["head"].shape == (210, 72) and names["l0.mlp.shared.sg"].shape == (1, 72)
    f = spec.layers[0].feed_forward.params
    assert f["groups"] == (3, 2) and f["scoring"] == "sigmoid" and f["normalise_eps"] == 1e-20 and f["form"] == "silu"
    assert spec.layers[3].feed_forward.params["groups"] is None and "l3.mlp.shared.up" not in names
    d = spec.layers[2].feed_forward.params
    assert d["activation"] == "swish_limit" and d["activation_param"] == 0.7


def test_optional_keys_have_their_meaning():
    """No mask: all keys; kv_heads and vdim missing: as many key heads as query heads, values as wide as keys; no conv: no
    convolution; no v_mix: no blending; the number of buckets comes from the file where the configuration is silent."""
    cfg, _ = tiny_kitonex.config("KB")
    m = cfg["layers"][2]["mixer"]
    for key in ("kv_heads", "vdim", "mask", "conv", "v_mix", "bias_buckets"):
        del m[key]
    spec = _spec(cfg)
    a = spec.layers[2].mixer.params
    assert a["n_kv_heads"] == 4 and a["value_dim"] == 64 and a["chunk"] is None and "v_mix" not in a
    names = spec.tensor_specs()
    assert "l2.mix.q.conv" not in names and names["l2.mix.rel"].shape == (None, 4)


def test_configuration_errors_are_listed_together():
    cfg, _ = tiny_kitonex.config("KA")
    bad = copy.deepcopy(cfg)
    del bad["width"], bad["streams"]
    bad["layers"][0]["mixer"]["kv_heads"] = 4
    bad["layers"][0]["mlp"]["router"]["groups"]["keep"] = 4
    bad["layers"][1]["mixer"]["conv"] = 9
    bad["layers"][2]["mlp"]["limit"] = 0
    bad["layers"][3]["type"] = "convolution"
    with pytest.raises(ConfigError) as e:
        architecture_for(bad).parse_config(bad)
    text = str(e.value)
    for word in ("width", "streams", "kv_heads (4)", "keep (4)", "conv", "limit", "convolution"):
        assert word in text, word
    bad = copy.deepcopy(cfg)
    bad["layers"][2]["mixer"]["vdim"] = 11           # 4 x 11 values cannot be blended with 2 x 20
    with pytest.raises(ConfigError, match="cannot be mixed"):
        architecture_for(bad).parse_config(bad)
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["router"]["groups"] = {"count": 4, "keep": 2}
    with pytest.raises(ConfigError, match="equal groups"):
        architecture_for(bad).parse_config(bad)
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["router"].update(top=3, groups={"count": 3, "keep": 1})
    with pytest.raises(ConfigError, match="cannot be chosen"):
        architecture_for(bad).parse_config(bad)


@pytest.mark.parametrize("buckets,largest,longest", [(32, 120.5, 300), (16, 20, 33), (6, 5, 7), (8, 128, 128), (2, 3, 10), (64, 4096, 5000), (10, 24, 4)])
def test_buckets_of_distances(buckets, largest, longest):
    got = distance_buckets(buckets, largest, longest)
    want = [plain.bucket(n, buckets, largest) for n in range(longest)]
    assert got == want[:len(got)] and all(b == got[-1] for b in want[len(got):])
    if longest > largest:
        assert got[-1] == buckets - 1 and len(got) <= math.ceil(largest) + 1
    # by exact arithmetic: bucket B/2 + k starts where (n / (B/2))^(B - B/2) reaches (largest / (B/2))^k
    from fractions import Fraction
    half = buckets // 2
    for n in range(half, len(got)):
        k = got[n] - half
        r = Fraction(n, half) ** (buckets - half)
        assert r >= (Fraction(largest) / half) ** k and (got[n] == buckets - 1 or r < (Fraction(largest) / half) ** (k + 1))


def test_buckets_that_cannot_be():
    with pytest.raises(ValueError, match="even"):
        distance_buckets(7, 20, 10)
    with pytest.raises(ValueError, match="exceed"):
        distance_buckets(16, 8, 40)


def test_chunks_need_one_chunk_of_keys():
    """The keys a position sees lie in its own chunk: a ring of pages that holds a window of the chunk's length holds them."""
    from rust_deeplearning_b200.cache.cache import ring_pages_for
    for chunk in (1, 7, 33, 64, 120):
        for page in (4, 16, 64):
            rows = ring_pages_for(chunk, page) * page
            for p in range(3 * chunk + 5):
                lo = plain.first_visible(p, chunk)
                # rows of the ring that positions up to p have written last
                last = {q % rows: q for q in range(p + 1)}
                assert all(last[j % rows] == j for j in range(lo, p + 1))


def test_plain_model_invariants(tmp_path):
    """What the plain implementation must satisfy by construction: a token's logits do not depend on later tokens; keys of an
    earlier chunk do not count, the chunk's first key does; one in the denominator takes weight; a convolution of one tap that is
    1 is none; weights of the chosen sum to one; every copy matters; equal connections of one copy are the ordinary residual sum."""
    from rust_deeplearning_b200 import write_random_model
    cfg, seed = tiny_kitonex.config("KA")
    write_random_model(str(tmp_path), cfg, seed, "bfloat16")
    pcfg, w = plain.load_folder(str(tmp_path))
    ids = [int(v) for v in np.random.default_rng(1).integers(0, cfg["vocab"], size=24)]
    full = plain.forward(pcfg, w, ids)
    assert np.allclose(plain.forward(pcfg, w, ids[:11]), full[:11], atol=1e-10)
    rng = np.random.default_rng(2)
    T, H, G, d, e = 16, 4, 2, 6, 5
    q, k, v, rel = rng.normal(size=(T, H, d)), rng.normal(size=(T, G, d)), rng.normal(size=(T, G, e)), rng.normal(size=(8, H))
    base = plain.attend(q, k, v, 0.5, rel, 9, 5)
    moved = k.copy()
    moved[4] += 1.0                  # the last key of the first chunk
    out = plain.attend(q, moved, v, 0.5, rel, 9, 5)
    assert np.array_equal(out[5:], base[5:]) and np.abs(out[4] - base[4]).max() > 1e-6
    moved = k.copy()
    moved[5] += 1.0                  # the first key of the second
    out = plain.attend(q, moved, v, 0.5, rel, 9, 5)
    assert np.abs(out[9] - base[9]).max() > 1e-6 and np.array_equal(out[10:], base[10:]) and np.array_equal(out[:5], base[:5])
    ones = plain.attend(q, k, np.ones_like(v), 0.5, rel, 9, 5)
    assert (ones < 1.0).all() and (ones > 0.0).all()
    s = 0.5 * (q[0, 0] @ k[0, 0]) + rel[0, 0]
    assert np.isclose(ones[0, 0, 0], math.exp(s) / (1.0 + math.exp(s)))
    u = rng.normal(size=(7, 3))
    assert np.allclose(plain.short_conv(u, np.ones((3, 1))), u)
    assert np.allclose(plain.short_conv(u, np.array([[2.0, 0.0, 1.0]] * 3))[1], u[1]) and np.allclose(plain.short_conv(u, np.array([[2.0, 0.0, 1.0]] * 3))[4], u[4] + 2.0 * u[2])
    f = pcfg["layers"][0]["mlp"]
    h = rng.normal(size=(9, cfg["width"]))
    chosen, weight, margin = plain.router(h, w, "l0.mlp.", f["router"])
    assert np.allclose(weight.sum(axis=-1), 1.0) and (weight[:, 0] >= weight[:, 1]).all() and (margin >= 0).all()
    free, _, _ = plain.router(h, w, "l0.mlp.", {"experts": 6, "top": 2})
    one, _, _ = plain.router(h, w, "l0.mlp.", {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert (one // 2 == one[:, :1] // 2).all() and (free != one).any()        # both of one group
    step = np.array([0.1, -0.1, 0.05])           # (where all copies are equal, a common factor on what is read leaves its norm alone)
    for name in ("l1.hc1.in", "l0.hc2.out", "l1.hc1.mix", "l3.hc2.mix"):
        assert np.abs(plain.forward(pcfg, dict(w, **{name: w[name] + step}), ids) - full).max() > 1e-3, name
    x, y = rng.normal(size=(1, 4, 3)), rng.normal(size=(4, 3))
    single = {"c.in": np.ones(1), "c.mix": np.ones((1, 1)), "c.out": np.ones(1)}
    assert np.allclose(plain.write_copies(x, y, single, "c."), x + y) and np.allclose(plain.read_copies(x, single, "c."), x[0])
