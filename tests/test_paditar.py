"""Paditar without a GPU: the configuration reader, the model's description and its loop, the state of two mixers side by side,
shared products, and the plain implementation's own invariants."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_paditar as plain
import tiny_paditar
from rust_deeplearning_b200.cache.cache import Cache, StateRequirement
from rust_deeplearning_b200.config.base import ConfigError, architecture_for
from rust_deeplearning_b200.parts.head_attention import differential_lambda, query_temperature
from rust_deeplearning_b200.parts.joint import ContextMixer, JointProducts, stacked
from rust_deeplearning_b200.parts.spec import PartSpec, StreamEntry, looped_schedule


def _spec(cfg):
    arch = architecture_for(cfg)
    assert arch.name == "Paditar"
    return arch.build_spec(arch.parse_config(cfg))


def test_configuration_becomes_parts():
    cfg, _ = tiny_paditar.config("PA")
    spec = _spec(cfg)
    assert [layer.block for layer in spec.layers] == ["sandwich"] * 4
    assert [layer.mixer.kind for layer in spec.layers] == ["head_attention", "mixer_pair"] * 2
    assert spec.layers[1].feed_forward is None and set(spec.layers[1].norms) == {"pre_mixer", "post_mixer"}
    assert set(spec.layers[0].norms) == {"pre_mixer", "post_mixer", "pre_feed_forward", "post_feed_forward"}
    assert all(n.params["offset"] == 1.0 and n.params["eps"] == 1e-4 for layer in spec.layers for n in layer.norms.values())
    a = spec.layers[0].mixer.params
    assert (a["n_heads"], a["n_kv_heads"], a["head_dim"], a["value_dim"], a["score_scale"]) == (4, 2, 10, 14, 0.5)
    assert a["differential"] == {"diff": 0.4, "eps": 1e-4} and a["gate"] == "value" and "off_by_one" not in a
    assert a["position"].params["theta"] == 300.0 and a["position"].params["rotary_dim"] == 6 and a["position"].params["pairing"] == "half"
    m = spec.layers[1].mixer.params
    assert (m["left_scale"], m["right_scale"]) == (0.9, 1.3)
    left, right = m["left"], m["right"]
    assert left.kind == "head_attention" and left.params["values_from_keys"] and left.params["off_by_one"] and left.params["gate"] == "head"
    assert left.params["q_temperature"] == {"coef": 0.7, "every": 9.0} and left.params["head_norm_eps"] == 1e-4
    assert right.kind == "matrix_memory" and right.params["gate_cap"] == 7.0 and right.params["q_scale"] == 10 ** -0.5 and right.params["den_eps"] == 1e-6
    names = spec.tensor_specs()
    assert names["l0.mix.q"].shape == (80, 76) and names["l0.mix.k"].shape == (40, 76) and names["l0.mix.v"].shape == (28, 76)
    assert names["l0.mix.g"].shape == (56, 76) and names["l0.mix.lq1"].shape == (10,) and names["l0.mix.o"].shape == (76, 56)
    assert names["l1.mix.left.q.conv"].shape == (72, 3) and names["l1.mix.left.k.norm"].shape == (12,) and names["l1.mix.left.o.b"].shape == (76,)
    assert "l1.mix.left.v" not in names and names["l1.mix.left.g"].shape == (6, 76)
    assert names["l1.mix.right.i"].shape == (3, 76) and names["l1.mix.right.f.b"].shape == (3,) and names["l1.mix.right.norm"].shape == (66,)
    assert names["loop.step"].shape == (2, 76) and names["embed"].shape == (190, 76) and "head" not in names
    assert "l1.norm2" not in names and "l1.norm2b" not in names and "l0.norm2b" in names
    f = spec.layers[0].feed_forward
    assert f.kind == "plain_mlp" and f.params["activation"] == "relu2"


def test_the_loop_is_a_schedule():
    cfg, _ = tiny_paditar.config("PA")
    s = _spec(cfg).schedule
    assert [e.layer for e in s] == [0, 1, 2, 1, 2, 3]
    assert [e.enters is not None for e in s] == [False, True, False, True, False, False]
    assert (s[1].enters.embedding, s[1].enters.row) == (False, 0) and (s[3].enters.embedding, s[3].enters.row) == (True, 1)
    cfg, _ = tiny_paditar.config("PC")           # no loop
    assert [(e.layer, e.enters) for e in _spec(cfg).schedule] == [(0, None), (1, None), (2, None)] and "loop.step" not in _spec(cfg).tensor_specs()
    s = looped_schedule(2, 0, 2, 3)              # no vectors: only the embedding joins, from the second pass on
    assert [(e.layer, e.enters) for e in s] == [(0, None), (1, None)] + [(0, StreamEntry(True, None, 1)), (1, None), (0, StreamEntry(True, None, 2)), (1, None)]
    for bad in ((2, 1, 1, 2), (2, 0, 3, 1), (2, 0, 2, 0), (2, -1, 1, 1)):
        with pytest.raises(ValueError):
            looped_schedule(*bad)


def test_optional_keys_have_their_meaning():
    cfg, _ = tiny_paditar.config("PB")
    del cfg["layers"][0]["mixer"]["left"]["kv_heads"], cfg["layers"][0]["mixer"]["left"]["vdim"], cfg["layers"][0]["mixer"]["right"]["vdim"], cfg["max_positions"]
    spec = _spec(cfg)
    m = spec.layers[0].mixer.params
    assert m["left"].params["n_kv_heads"] == 6 and m["right"].params["vdim"] == 32 and spec.max_positions == 32768


def test_configuration_errors_are_listed_together():
    cfg, _ = tiny_paditar.config("PA")
    bad = copy.deepcopy(cfg)
    del bad["width"], bad["norm"]
    bad["layers"][0]["mixer"]["kv_heads"] = 3
    bad["layers"][1]["mixer"]["left"]["conv"] = 9
    bad["layers"][1]["mixer"]["left"]["vdim"] = 13
    bad["layers"][1]["mixer"]["right"]["gate_cap"] = 0
    bad["layers"][2]["mixer"]["rot"]["dims"] = 8
    del bad["layers"][3]["mixer"]["left_scale"]
    bad["layers"][3]["mixer"]["left"]["q_temp"]["every"] = -1
    bad["loop"]["stop"] = 9
    with pytest.raises(ConfigError) as e:
        architecture_for(bad).parse_config(bad)
    text = str(e.value)
    for word in ("width", "norm", "kv_heads (3)", "conv", "vdim (13)", "gate_cap", "dims (8)", "left_scale", "every", "loop"):
        assert word in text, word
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["type"] = "retention"
    with pytest.raises(ConfigError, match="retention"):
        architecture_for(bad).parse_config(bad)
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["kind"] = "moe"
    with pytest.raises(ConfigError, match="moe"):
        architecture_for(bad).parse_config(bad)


def test_every_run_has_cache_and_state_of_its_own():
    """Layer runs of the loop get storage of their own; a pair's run keeps keys, values, the convolution's and the memory's state."""
    from rust_deeplearning_b200.parts.model import Model
    from rust_deeplearning_b200.weights.loader import random_weights
    cfg, seed = tiny_paditar.config("PA")
    spec = _spec(cfg)
    model = Model(spec, random_weights(spec, seed, torch.float32, "cpu"), torch.float32, "cpu")
    needs = model.needs()
    assert len(needs) == 6
    conv, s, n = needs[1].state
    assert conv.shape == (2, 96) and s.shape == (3, 10, 22) and n.shape == (3, 1, 11)
    assert needs[0].state is None and needs[0].kv.n_kv_heads == 2 and needs[0].kv.head_dim == 32
    cache = Cache(needs, max_tokens=64, max_seqs=2, page_size=16, dtype=torch.float32, device="cpu")
    at = set()
    for run in (1, 3):
        rc = cache.run_cache(run)
        at |= {rc.k.data_ptr(), rc.v.data_ptr(), *(t.data_ptr() for t in rc.state)}
    assert len(at) == 10
    pair = model.layers[1].mixer
    left, right = pair._caches(cache.run_cache(1))
    assert tuple(left.state.shape) == (2, 2, 96) and [tuple(t.shape[1:]) for t in right.state] == [(3, 10, 22), (3, 1, 11)]
    for g in cache.state_groups:                 # a slot's state is zero when it is handed out, whatever was left
        g.data.fill_(7.0)
    slot = cache.alloc_slot()
    assert all(float(g.data[:, slot].abs().max()) == 0.0 for g in cache.state_groups)


def test_shared_products_hold_both_mixers():
    """One input matrix, one output matrix with the factors on the biases and, in bfloat16, the bias in two terms."""
    rng = np.random.default_rng(0)

    class One(ContextMixer):
        def __init__(self, n, m, bias, dtype):
            t = lambda *s: torch.tensor(rng.normal(size=s), dtype=torch.float32).to(dtype)
            self.in_matrix, self.out_matrix, self.out_bias = stacked(t(n, 6)), t(6, m), torch.tensor(rng.normal(size=6), dtype=torch.float32) if bias else None

    for dtype in (torch.float32, torch.bfloat16):
        a, b = One(11, 5, True, dtype), One(16, 10, False, dtype)
        wa, wb, ia, ib, bias = a.out_matrix, b.out_matrix, a.in_matrix, b.in_matrix, a.out_bias
        assert ia.shape == (16, 6) and float(ia[11:].abs().max()) == 0.0
        j = JointProducts((a, b), (0.7, 1.3))
        assert torch.equal(j.w_in, torch.cat([ia, ib])) and j.columns == [(0, 16), (16, 32)]
        assert torch.equal(j.w_out[:, :5], wa) and torch.equal(j.w_out[:, 5:15], wb) and j.width % 8 == 0
        assert j.n_ones == (1 if dtype is torch.float32 else 2)
        got = j.w_out[:, 15:15 + j.n_ones].float().sum(dim=1)
        assert torch.allclose(got, bias * 0.7, rtol=0, atol=0.0 if dtype is torch.float32 else 3e-5)
        assert not j.w_out[:, 15 + j.n_ones:].any()
        assert a.in_matrix is None and b.out_matrix is None
        alone = JointProducts([One(8, 8, False, dtype)], [1.0])
        assert alone.n_ones == 0 and alone.width == 8


def test_constants_of_a_layer():
    q = query_temperature(0.5, 7, 40)
    assert q.dtype is torch.float32 and np.allclose(q.numpy(), [plain.temperature(p, 0.5, 7) for p in range(40)], atol=1e-7)
    assert float(q[5]) == 1.0 and float(q[6]) == pytest.approx(1.0 + 0.5 * math.log(2.0)) and float(q[12]) == float(q[6]) < float(q[13])
    assert np.allclose(query_temperature(0.3, 2.5, 9).numpy(), [plain.temperature(p, 0.3, 2.5) for p in range(9)], atol=1e-7)
    rng = np.random.default_rng(1)
    w = {n: rng.normal(size=6) * 0.4 for n in ("lq1", "lk1", "lq2", "lk2")}
    got = differential_lambda(*(torch.tensor(w[n]) for n in ("lq1", "lk1", "lq2", "lk2")), 0.35)
    assert got == pytest.approx(plain.layer_lambda(w, "", 0.35), abs=1e-12)


def test_a_pair_is_normed_or_scaled():
    from rust_deeplearning_b200.parts.mixer_pair import MixerPair

    class Keeps:
        def __init__(self, state):
            self.state = state

        def needs(self):
            return None, self.state
    one, two = StateRequirement((2,)), StateRequirement((3, 4))
    p = MixerPair(Keeps(one), Keeps((two, one)), torch.ones(4), torch.ones(4), 1e-5)
    assert p.needs() == (None, (one, two, one))
    p = MixerPair(Keeps(None), Keeps(two), torch.ones(4), torch.ones(4), 1e-5)
    assert p.needs() == (None, two)
    with pytest.raises(ValueError, match="normed or both"):
        MixerPair(Keeps(one), Keeps(two))
    with pytest.raises(ValueError, match="can be shared"):
        MixerPair(Keeps(one), Keeps(two), scales=(1.0, 1.0))


def test_plain_model_invariants(tmp_path):
    """What the plain implementation must satisfy by construction: a token's logits do not depend on later tokens; one in the
    denominator takes weight; a map against itself cancels; a convolution of one tap that is 1 is none; the memory with the running
    maximum equals the one without it; every tensor of the model moves the logits."""
    from rust_deeplearning_b200 import write_random_model
    cfg, seed = tiny_paditar.config("PA")
    write_random_model(str(tmp_path), cfg, seed, "bfloat16")
    pcfg, w = plain.load_folder(str(tmp_path))
    ids = [int(v) for v in np.random.default_rng(1).integers(0, cfg["vocab"], size=20)]
    full = plain.forward(pcfg, w, ids)
    assert np.allclose(plain.forward(pcfg, w, ids[:9]), full[:9], atol=1e-9)
    rng = np.random.default_rng(2)
    T, H, G, d, e = 11, 4, 2, 6, 5
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, G, d)), rng.normal(size=(T, G, e))
    assert np.allclose(plain.attend(q, k, np.ones_like(v), 0.5, 0), 1.0)
    s = math.exp(0.5 * (q[0, 0] @ k[0, 0]))
    ones = plain.attend(q, k, np.ones_like(v), 0.5, 1)
    assert (ones < 1.0).all() and np.isclose(ones[0, 0, 0], s / (1.0 + s))
    twice = lambda x: np.stack([x, x], axis=2)
    assert np.allclose(plain.differential(twice(q), twice(k), v, 0.5, 1.0), 0.0)
    assert np.allclose(plain.differential(twice(q), twice(k), v, 0.5, 0.25), 0.75 * plain.attend(q, k, v, 0.5, 0))
    u = rng.normal(size=(7, 3))
    assert np.allclose(plain.short_conv(u, np.ones((3, 1))), u)
    x = plain.rotate(u[:, None, :2].repeat(2, axis=1), 10.0, 2)
    assert np.allclose((x ** 2).sum(-1), (u[:, None, :2] ** 2).sum(-1)) and np.allclose(x[0], u[0, :2]) and not np.allclose(x[1], u[1, :2])
    # without the running maximum: S = sum of decayed e^i k v^T, the floor e^(-m) times e^m is one
    zi, zf = rng.normal(size=T) * 3, rng.normal(size=T) * 2 + 1
    got, (S, n, m) = plain.memory(q[:, 0], k[:, 0], v[:, 0], zi, zf, 4.0, den_eps=0.0)
    f = -np.log1p(np.exp(-4.0 * np.tanh(zf / 4.0)))
    i = 4.0 * np.tanh(zi / 4.0)
    for t in range(T):
        weight = np.array([math.exp(i[j] + f[j + 1:t + 1].sum()) for j in range(t + 1)])
        num, den = (weight * (k[:t + 1, 0] @ q[t, 0])) @ v[:t + 1, 0], (weight * (k[:t + 1, 0] @ q[t, 0])).sum()
        assert np.allclose(got[t], num / max(abs(den), 1.0))
    half, state = plain.memory(q[:4, 0], k[:4, 0], v[:4, 0], zi[:4], zf[:4], 4.0)
    rest, _ = plain.memory(q[4:, 0], k[4:, 0], v[4:, 0], zi[4:], zf[4:], 4.0, state=state)
    assert np.allclose(np.concatenate([half, rest]), plain.memory(q[:, 0], k[:, 0], v[:, 0], zi, zf, 4.0)[0])
    for name, t in w.items():
        moved = t + 0.1 * rng.normal(size=t.shape)
        assert np.abs(plain.forward(pcfg, dict(w, **{name: moved}), ids) - full).max() > 1e-3, name
