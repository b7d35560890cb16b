"""Paditar on a GPU against the plain implementation, in 32-bit and in bfloat16: each new mechanism's kernels alone,
whole prompts, single tokens through the cache, portions, unequal batches on reused slots and pages, far keys and every constant
under sharp softmaxes, long decoding, greedy generation, the trace replay and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import paditar_helpers as ph
import plain_paditar as plain
import tiny_paditar

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
NAMES = ["PA", "PB", "PC", "PD"]
DEV = "cuda:0"


def _t(a, dtype):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(DEV).to(getattr(torch, dtype))


def _back(t):
    return t.float().cpu().double().numpy()


def _close(got, want, dtype, what, bf16=2e-2, f32=2e-5):
    got = _back(got.detach()) if isinstance(got, torch.Tensor) else got
    tol = (f32 if dtype == "float32" else bf16) * max(1.0, float(np.abs(want).max()))
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert np.isfinite(got).all(), what
    assert np.abs(got - want).max() <= tol, f"{what}: {np.abs(got - want).max():.3e} > {tol:.3e}"


def _ti(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def _stored(cache, page, row, g, D):
    """The row of a cache page as values in order (stored rows have their 16-byte pieces swizzled by their place in the page)."""
    v = _back(cache[page, g, row])
    n = 16 // cache.element_size()
    if D % n:
        return v
    return np.concatenate([v[((c ^ (row & 7)) if (c | 7) < D // n else c) * n:][:n] for c in range(D // n)])


class Batch:
    """A step's description on the device: lens[i] new tokens of sequence i after past[i] earlier ones, then padding rows."""

    def __init__(self, lens, past, slots, padding=0):
        self.n_seqs, self.n_tokens = len(lens), sum(lens) + padding
        pos, start = [], [0]
        for n, p in zip(lens, past):
            pos += list(range(p, p + n))
            start.append(start[-1] + n)
        self.tok_pos, self.seq_start, self.slots = _ti(pos + [-1] * padding), _ti(start), _ti(slots)
        self.seq_end = _ti([n + p for n, p in zip(lens, past)])

    def kw(self, end=True):
        return dict(tok_pos=self.tok_pos, seq_start=self.seq_start, slots=self.slots, n_seqs=self.n_seqs, **({"seq_end": self.seq_end} if end else {}))


# ---- what lies between product and attention ----

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [
    # heads, key heads, maps, dim, vdim, laid-out size, taps, rotated values, norm, temperature, values from keys
    (3, 1, 1, 12, 12, 16, 3, 0, True, True, True), (6, 2, 1, 64, 64, 64, 4, 0, True, True, True), (2, 2, 1, 128, 128, 128, 4, 0, True, True, True),
    (4, 2, 2, 10, 14, 32, 0, 6, False, False, False), (6, 1, 2, 32, 64, 64, 0, 16, False, False, False), (2, 1, 2, 64, 128, 128, 0, 64, False, False, False),
    (3, 3, 2, 6, 30, 32, 0, 6, False, False, False), (5, 5, 1, 18, 18, 32, 2, 0, True, False, True), (3, 1, 1, 200, 72, 208, 6, 96, True, True, False),
    (4, 4, 2, 130, 20, 260, 5, 30, True, True, False), (2, 1, 1, 512, 300, 512, 8, 512, True, False, False), (40, 8, 1, 16, 16, 16, 1, 16, False, True, True),
    (9, 3, 2, 16, 200, 208, 7, 8, True, True, False)])
def test_heads_made_ready_for_attention(dtype, sizes):
    """The kernel between the q/k/v product and attention against the plain mechanisms, every one beside every other, over steps of
    unequal portions (0 to 21 tokens a sequence and step) on shuffled slots with a padding row: the convolution's state passes from
    step to step (a former owner's is not read), cache rows are read back through shuffled page lists; in 32-bit the same rows come
    out whatever the cut."""
    from rust_deeplearning_b200.kernels import ops
    from rust_deeplearning_b200.parts.head_attention import query_temperature
    H, G, M, d, e, D, taps, rot, norm, temp, shared = sizes
    rng = np.random.default_rng(sum(sizes))
    eps, page, T = 1e-3, 4, 45
    q8 = lambda a: _back(_t(a, dtype))
    C = (H + G) * M * d
    W = C + (0 if shared else G * e)
    bias = _back(_t(rng.normal(size=C) * 0.3, "float32"))
    conv = q8(rng.normal(size=(C, taps)) * 0.6) if taps else None
    wq, wk = _back(_t(rng.normal(size=d) + 1.0, "float32")), _back(_t(rng.normal(size=d) + 1.0, "float32"))
    coef, every, base = 0.6, 7, 60.0
    rows = [q8(rng.normal(size=(T, W))) for _ in range(3)]
    want = []
    for r in rows:
        c = r[:, :C] + bias
        if taps:
            c = plain.short_conv(c, conv)
        q, k = c[:, :H * M * d].reshape(T, H, M, d), c[:, H * M * d:].reshape(T, G, M, d)
        v = k.reshape(T, G, d) if shared else r[:, C:].reshape(T, G, e)
        if norm:
            q, k = plain.unit(q, eps) * wq, plain.unit(k, eps) * wk
        if rot:
            q, k = plain.rotate(q, base, rot), plain.rotate(k, base, rot)
        if temp:
            q = q * np.array([plain.temperature(p, coef, every) for p in range(T)])[:, None, None, None]
        lay = np.zeros((T, H * M + 2 * G, D))
        for h in range(H):
            for m in range(M):
                lay[:, h * M + m, m * d:(m + 1) * d] = q[:, h, m]
        lay[:, H * M:H * M + G, :M * d] = k.reshape(T, G, M * d)
        lay[:, H * M + G:, :v.shape[2]] = v
        want.append(lay.reshape(T, -1))
    freq = base ** (-2.0 * np.arange(rot // 2) / max(rot, 1))
    ang = np.arange(60)[:, None] * freq
    kw = dict(n_heads=H, n_kv_heads=G, maps=M, dim=d, vdim=d if shared else e, pad=D, q_col=0, k_col=H * M * d, v_col=None if shared else C,
              bias=_t(bias, "float32"), conv=_t(conv.T, dtype).contiguous() if taps else None, eps=eps)
    if norm:
        kw.update(wq=_t(wq, "float32"), wk=_t(wk, "float32"))
    if rot:
        kw.update(cos=_t(np.cos(ang), "float32"), sin=_t(np.sin(ang), "float32"))
    if temp:
        kw.update(q_factor=query_temperature(coef, every, 60).to(DEV))
    n_pages = -(-T // page)
    order = rng.permutation(3 * n_pages).reshape(3, n_pages)

    def run(cuts, slots):
        state = torch.full((7, taps - 1, C), 99.0, dtype=torch.float32, device=DEV) if taps > 1 else None      # what a former owner left
        k = torch.zeros((3 * n_pages, G, page, D), dtype=getattr(torch, dtype), device=DEV)
        v = torch.zeros_like(k)
        past, outs = [0, 0, 0], [[], [], []]
        for lens in cuts:
            live = [i for i in range(3) if lens[i]]
            b = Batch([lens[i] for i in live], [past[i] for i in live], [slots[i] for i in live], padding=1)
            x = _t(np.concatenate([rows[i][past[i]:past[i] + lens[i]] for i in live] + [np.full((1, W), 5.0)]), dtype)
            out = ops.head_prepare(x, state=state, pages=ops.KVPages(k, v, _ti(order[live]), page, n_pages), **kw, **b.kw())
            at = 0
            for i in live:
                outs[i].append(out[at:at + lens[i]].clone())
                at += lens[i]
                past[i] += lens[i]
        assert past == [T, T, T]
        return [torch.cat(o) for o in outs], k, v

    whole, k, v = run([(T, T, T)], [4, 0, 6])
    for i in range(3):
        _close(whole[i], want[i], dtype, f"sequence {i}", bf16=1e-2)
        got = _back(whole[i])
        for p in (0, 3, 4, 17, T - 1):
            for g in range(G):
                pg, r = order[i][p // page], p % page
                assert np.array_equal(_stored(k, pg, r, g, D), got[p, (H * M + g) * D:(H * M + g + 1) * D])
                assert np.array_equal(_stored(v, pg, r, g, D), got[p, (H * M + G + g) * D:(H * M + G + g + 1) * D])
    cuts = [(21, 2, 1), (1, 1, 1), (1, 7, 2), (0, 9, 3), (2, 0, 17), (20, 8, 0), (0, 18, 21)]
    same = (lambda a, b, what: torch.equal(a, b)) if dtype == "float32" else (lambda a, b, what: _close(b, _back(a), dtype, what, bf16=8e-3) or True)
    parts, k2, v2 = run(cuts, [1, 5, 2])
    assert all(same(a, b, "portions") for a, b in zip(whole, parts)) and same(k, k2, "keys") and same(v, v2, "values")
    singles, k2, v2 = run([(30, 3, 44)] + [(1, 1, 1)] + [(1, 1, 0)] * 14 + [(0, 1, 0)] * 27, [3, 2, 1])
    assert all(same(a, b, "single tokens") for a, b in zip(whole, singles)) and same(k, k2, "keys") and same(v, v2, "values")


@pytest.mark.parametrize("dtype", DTYPES)
def test_preparation_of_many_sequences(dtype):
    """Forty sequences of 1 to 30 new tokens, some with earlier ones, in one step and each in a step of its own."""
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(8)
    H, G, d, taps, n = 3, 1, 16, 4, 40
    C = (H + G) * d
    lens = [int(v) for v in rng.integers(1, 31, size=n)]
    lens[3:9] = [1] * 6
    past = [int(v) for v in rng.choice([0, 0, 1, 2, 5, 64], size=n)]
    slots = [int(v) for v in rng.permutation(n)]
    rows = _t(rng.normal(size=(sum(lens), C)), dtype)
    kw = dict(n_heads=H, n_kv_heads=G, maps=1, dim=d, vdim=d, pad=d, q_col=0, k_col=H * d, v_col=None, bias=_t(rng.normal(size=C), "float32"),
              conv=_t(rng.normal(size=(taps, C)), dtype), wq=_t(rng.normal(size=d), "float32"), wk=_t(rng.normal(size=d), "float32"), eps=1e-5)
    before = _t(rng.normal(size=(n, taps - 1, C)), "float32")
    together, alone = before.clone(), before.clone()
    got = ops.head_prepare(rows, state=together, **kw, **Batch(lens, past, slots).kw())
    at = 0
    for i in range(n):
        one = ops.head_prepare(rows[at:at + lens[i]], state=alone, **kw, **Batch([lens[i]], [past[i]], [slots[i]]).kw())
        if dtype == "float32":
            assert torch.equal(one, got[at:at + lens[i]]), f"sequence {i}: {lens[i]} tokens after {past[i]}"
        else:
            _close(one, _back(got[at:at + lens[i]]), dtype, f"sequence {i}", bf16=8e-3)
        at += lens[i]
    assert torch.equal(together, alone)


def test_preparation_in_a_ring():
    """In a ring only the last writer of a cache row writes."""
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(3)
    n, page, past, G, d = 19, 4, 6, 2, 16
    x = _t(rng.normal(size=(n, 3 * G * d)), "bfloat16")
    k, v = (torch.zeros((3, G, page, d), dtype=x.dtype, device=DEV) for _ in range(2))
    out = ops.head_prepare(x, n_heads=G, n_kv_heads=G, maps=1, dim=d, vdim=d, pad=d, q_col=0, k_col=G * d, v_col=2 * G * d,
                           pages=ops.KVPages(k, v, _ti([[2, 0, 1]]), page, 3), **Batch([n], [past], [0]).kw())
    assert torch.equal(out, x)
    for p in range(past + n - 12, past + n):
        for g in range(G):
            assert np.array_equal(_stored(k, [2, 0, 1][(p // page) % 3], p % page, g, d), _back(out[p - past, (G + g) * d:(G + g + 1) * d]))
            assert np.array_equal(_stored(v, [2, 0, 1][(p // page) % 3], p % page, g, d), _back(out[p - past, (2 * G + g) * d:(2 * G + g + 1) * d]))


# ---- attention ----

@pytest.mark.parametrize("heads", [(12, 1), (16, 1), (9, 1), (22, 2), (26, 2)])
def test_large_groups_of_query_heads_in_decode(heads):
    """More than eight query heads a key head: the group's parts go to blocks that read the same keys; one key's score stands out at
    each of several distances, and with one in the denominator."""
    from rust_deeplearning_b200.kernels import ops
    H, G = heads
    D, page = 64, 16
    rng = np.random.default_rng(H)
    lens = [1, 15, 16, 17, 90, 200]
    n_pages = 13
    order = rng.permutation(len(lens) * n_pages).reshape(len(lens), n_pages)
    k, v = (torch.zeros((len(lens) * n_pages, G, page, D), dtype=torch.bfloat16, device=DEV) for _ in range(2))
    q = _back(_t(rng.normal(size=(len(lens), H, D)) * 0.5, "bfloat16"))
    want0, want1 = np.zeros((len(lens), H, D)), np.zeros((len(lens), H, D))
    qkv = []
    for i, n in enumerate(lens):
        kk, vv = (_back(_t(rng.normal(size=(n, G, D)) * s, "bfloat16")) for s in (0.5, 1.0))
        for g in range(G):
            kk[(7 * i + 3) % n, g] = _back(_t(q[i, g * (H // G)] * 1.5, "bfloat16"))       # a key that stands out for the group's first head
        qq = np.zeros((n, H, D))
        qq[-1] = q[i]
        want0[i], want1[i] = plain.attend(qq, kk, vv, 0.3, 0)[-1], plain.attend(qq, kk, vv, 0.3, 1)[-1]
        qkv.append(np.concatenate([kk, vv], axis=1).reshape(n, -1))
    for i, n in enumerate(lens):      # written by the preparation kernel (queries are not part of it)
        x = _t(np.concatenate([np.zeros((n, G * D)), qkv[i]], axis=1), "bfloat16")
        ops.head_prepare(x, n_heads=G, n_kv_heads=G, maps=1, dim=D, vdim=D, pad=D, q_col=0, k_col=G * D, v_col=2 * G * D,
                         pages=ops.KVPages(k, v, _ti(order[i:i + 1]), page, n_pages), **Batch([n], [0], [0]).kw())
    b = ops.AttentionBatch(len(lens), len(lens), _ti(range(len(lens))), _ti([n - 1 for n in lens]), _ti(range(len(lens) + 1)),
                           _ti([n - 1 for n in lens]), _ti(lens), max_keys=max(lens))
    pages = ops.KVPages(k, v, _ti(order), page, n_pages)
    rows = _t(q.reshape(len(lens), -1), "bfloat16")
    common = dict(n_heads=H, n_kv_heads=G, head_dim=D, score_scale=0.3, softcap=None, window=None)
    for sinks, want in ((None, want0), (torch.zeros(H, device=DEV), want1)):
        for ks in (16, 64):
            got = ops.attention(rows, b, pages, kind="decode", sinks=sinks, keys_per_split=ks, **common)
            _close(got, want.reshape(len(lens), -1), "bfloat16", f"{heads}, {ks} keys a block", bf16=1.5e-2)


# ---- the memory ----

def _memory_case(rng, H, d, e, lens, dtype, cap, spread):
    rows = []
    for n in lens:
        x = rng.normal(size=(n, H * (2 * d + e + 2)))
        x[:, H * (2 * d + e):] *= spread
        rows.append(_back(_t(x, dtype)))
    return rows


@pytest.mark.parametrize("dtype,kind", [("float32", "scan"), ("bfloat16", "scan"), ("bfloat16", "chunked")])
@pytest.mark.parametrize("shape", [(2, 16, 16, 15.0, 1.0), (3, 48, 48, 4.0, 3.0), (1, 128, 96, 15.0, 6.0), (2, 32, 176, 30.0, 12.0), (2, 10, 22, 7.0, 2.0), (1, 200, 33, 15.0, 2.0)])
def test_matrix_memory(dtype, kind, shape):
    """The recurrence over sequences of 1 to 200 tokens, in one step, in portions and ending in single tokens, on shuffled slots
    (states of other slots stay), against the plain one: gates that nearly never forget, that forget at once, inputs of e^-15 to
    e^15, a denominator that its floor replaces and one that it does not."""
    from rust_deeplearning_b200.kernels import ops
    H, d, e, cap, spread = shape
    if kind == "chunked" and (d % 16 or e % 16 or d > 128):
        pytest.skip("sizes the chunked form leaves to the scan")
    rng = np.random.default_rng(d + e)
    lens = [1, 2, 63, 64, 65, 200, 130]
    rows = _memory_case(rng, H, d, e, lens, dtype, cap, spread)
    bi, bf = rng.normal(size=H), rng.normal(size=H) * 3 + 2
    bi, bf = _back(_t(bi, "float32")), _back(_t(bf, "float32"))
    scale = d ** -0.5
    q_col, k_col, v_col, i_col = 0, H * d, 2 * H * d, H * (2 * d + e)
    want, last = [], []
    for r in rows:
        o = np.zeros((len(r), H, e))
        st = []
        for h in range(H):
            o[:, h], s = plain.memory(r[:, h * d:(h + 1) * d] * scale, r[:, k_col + h * d:k_col + (h + 1) * d], r[:, v_col + h * e:v_col + (h + 1) * e],
                                      r[:, i_col + h] + bi[h], r[:, i_col + H + h] + bf[h], cap)
            st.append(s)
        want.append(o.reshape(len(r), H * e))
        last.append(st)
    copies = ops.matrix_memory_copies(e)
    slots_n = len(lens) + 3
    pad = -(-rows[0].shape[1] // 8) * 8
    kw = dict(q_col=q_col, k_col=k_col, v_col=v_col, i_col=i_col, f_col=i_col + H, n_heads=H, dim=d, vdim=e, i_bias=_t(bi, "float32"), f_bias=_t(bf, "float32"),
              cap=cap, q_scale=scale, den_eps=1e-6)

    def run(cuts, seed):
        slots = [int(v) for v in np.random.default_rng(seed).permutation(slots_n)[:len(lens)]]
        S, N = (torch.full((slots_n, H, *s), 3.0, dtype=torch.float32, device=DEV) for s in ((d, e), (copies, d + 1)))
        for s in slots:
            S[s], N[s] = 0.0, 0.0
        past, outs = [0] * len(lens), [[] for _ in lens]
        for cut in cuts:
            live = [i for i in range(len(lens)) if past[i] < lens[i]]
            if not live:
                break
            take = [min(cut[i % len(cut)], lens[i] - past[i]) for i in live]
            x = np.zeros((sum(take) + 1, pad))
            x[:-1, :rows[0].shape[1]] = np.concatenate([rows[i][past[i]:past[i] + n] for i, n in zip(live, take)])
            b = Batch(take, [past[i] for i in live], [slots[i] for i in live], padding=1)
            o = ops.matrix_memory(_t(x, dtype), state=S, norm=N, kind=kind if max(take) > 1 else "scan", **kw, **b.kw(end=False))
            at = 0
            for i, n in zip(live, take):
                outs[i].append(o[at:at + n].clone())
                at += n
                past[i] += n
        assert past == lens
        free = [s for s in range(slots_n) if s not in slots]
        assert float((S[free] - 3.0).abs().max()) == 0.0 and float((N[free] - 3.0).abs().max()) == 0.0
        for i, s in enumerate(slots):
            n = _back(N[s])
            assert all(np.array_equal(n[:, 0], n[:, c]) for c in range(copies))          # every copy alike
            for h in range(H):
                wS, wn, wm = last[i][h]
                tol = 1e-4 if dtype == "float32" or kind == "scan" else 2e-3
                assert np.abs(_back(S[s, h]) - wS).max() <= tol * max(1.0, np.abs(wS).max())
                assert np.abs(n[h, 0, :d] - wn).max() <= tol * max(1.0, np.abs(wn).max()) and abs(n[h, 0, d] * np.log(2.0) - wm) <= 1e-4 * max(1.0, abs(wm))
        return [torch.cat(o) for o in outs]

    # a quotient's error is that of its numerator over its denominator, which may be its floor: the outputs are compared with the
    # size of what was summed, the root mean square of the sequence's outputs
    def check(outs, what):
        for i, (o, w) in enumerate(zip(outs, want)):
            size = max(1.0, float(np.abs(w).max()))
            err = np.abs(_back(o) - w).max()
            tol = (1e-4 if kind == "scan" else 3e-3) * size
            assert err <= tol, f"{what}, sequence {i} of {lens[i]}: {err:.3e} > {tol:.3e}"

    whole = run([[200]], 1)
    check(whole, "whole")
    parts = run([[64, 3, 17], [2, 40, 64], [128, 70, 9], [200, 200, 200]], 2)
    check(parts, "portions")
    singles = run([[60, 1, 190]] + [[1]] * 139, 3)
    check(singles, "single tokens")
    if kind == "scan":
        assert all(torch.equal(a, b) and torch.equal(a, c) for a, b, c in zip(whole, parts, singles))


# ---- from results to the output product's rows ----

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 14, 16, 3, 22), (6, 64, 64, 2, 48), (2, 128, 128, 2, 128), (3, 30, 32, 1, 200), (1, 300, 304, 5, 8), (5, 8, 16, 2, 512)])
def test_results_become_the_products_rows(dtype, sizes):
    from rust_deeplearning_b200.kernels import ops
    H, e, D, H2, e2 = sizes
    rng = np.random.default_rng(sum(sizes))
    T, eps, lam = 37, 1e-3, 0.4
    q8 = lambda a: _back(_t(a, dtype))
    x, o = q8(rng.normal(size=(T, 2 * H * D))), _back(_t(rng.normal(size=(T, H2 * e2)) * 3, "float32"))
    wide = q8(rng.normal(size=(T, 8 + H * e + H2 * e2 + 16)))
    gate1, gate2, gate3 = wide[:, 8:8 + H * e], wide[:, 8 + H * e:8 + H * e + H2 * e2], wide[:, 3:3 + H]
    weight = _back(_t(rng.normal(size=H2 * e2), "float32"))
    maps = x.reshape(T, H, 2, D)[..., :e]
    diff = plain.unit(maps[:, :, 0] - lam * maps[:, :, 1], eps) * 0.6 * plain.sigmoid(gate1).reshape(T, H, e)
    mem = (plain.unit(o.reshape(T, H2, e2), eps).reshape(T, -1) * weight * plain.sigmoid(gate2)) * 1.7
    head = maps[:, :, 0] * plain.sigmoid(gate3)[:, :, None] * 0.9
    tw = _t(wide, dtype)
    s1 = ops.ContextSide(_t(x, dtype), H, e, D, 2, lam, eps, None, 0.6, tw[:, 8:8 + H * e], "value")
    s2 = ops.ContextSide(_t(o, "float32"), H2, e2, e2, norm_eps=eps, weight=_t(weight, "float32"), factor=1.7, gate=tw[:, 8 + H * e:8 + H * e + H2 * e2], gate_kind="value")
    s3 = ops.ContextSide(_t(x, dtype), H, e, 2 * D, factor=0.9, gate=tw[:, 3:3 + H], gate_kind="head")
    ones = lambda n, rest: [np.ones((T, n)), np.zeros((T, rest))]
    for sides, want, n_ones in (((s1,), [diff.reshape(T, -1)], 0), ((s2,), [mem], 1), ((s3, s2), [head.reshape(T, -1), mem], 2), ((s2, s1), [mem, diff.reshape(T, -1)], 2)):
        n = sum(w.shape[1] for w in want)
        width = -(-(n + n_ones) // 8) * 8
        got = ops.context_finish(list(sides), width, n_ones, getattr(torch, dtype))
        _close(got, np.concatenate(want + ones(n_ones, width - n - n_ones), axis=1), dtype, f"{len(sides)} sides", bf16=6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 7, 16, 60, 300])
def test_what_joins_the_stream(dtype, rows):
    """A branch, rows and a vector join the stream in one kernel with the norm that follows, and the ways without one of them; rows
    the stream was built on stay as they are."""
    from rust_deeplearning_b200.parts.norm import ResidualStream, RMSNorm
    rng = np.random.default_rng(rows)
    for W in (64, 76, 2048):
        f = lambda *s: _back(_t(rng.normal(size=s), "float32"))
        x, emb, vec, w1, w2 = f(rows, W), f(rows, W), f(W), f(W) * 0.1, f(W) * 0.1
        branch = _back(_t(rng.normal(size=(rows, W)), dtype))
        n1, n2 = (RMSNorm(_t(w, "float32"), 1e-4, 1.0) for w in (w1, w2))
        for with_branch in (False, True):
            for e, v in ((emb, vec), (None, vec), (emb, None)):
                want = x + (plain.rms_norm(branch, w1, 1e-4) if with_branch else 0.0) + (0.0 if e is None else e) + (0.0 if v is None else v)
                for asked in (True, False):
                    tx = _t(x, "float32")
                    stream = ResidualStream(tx)
                    if with_branch:
                        stream.add(_t(branch, dtype), n1)
                    stream.enter(None if e is None else _t(e, "float32"), None if v is None else _t(v, "float32"))
                    if asked:
                        _close(stream.normed(n2, getattr(torch, dtype)), plain.rms_norm(want, w2, 1e-4), dtype, "normed", bf16=6e-3)
                    _close(stream.value(), want, "float32", "stream")
                    if not with_branch:
                        assert np.array_equal(_back(tx), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 12, 40, 200])
def test_plain_feed_forward(dtype, rows):
    from rust_deeplearning_b200.parts.feed_forward import PlainMLP
    rng = np.random.default_rng(rows)
    for W, ff in ((64, 96), (36, 20), (128, 264)):
        up, down = _t(rng.normal(size=(ff, W)) * 0.3, dtype), _t(rng.normal(size=(W, ff)) * 0.1, dtype)
        x = _t(rng.normal(size=(rows, W)), dtype)
        want = plain.feed_forward(_back(x), {"up": _back(up), "down": _back(down)}, "")
        _close(PlainMLP(W, ff, "relu2", up, down).forward(x), want, dtype, f"width {W}")


# ---- the model ----

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_first_tokens(name, dtype):
    eng = ph.engine(name, dtype, page_size=16)
    for seed, n in ((1, 1), (2, 2), (3, 37), (4, 170)):
        ids = ph.prompt(name, seed, n)
        slot = eng.new_sequence()
        ph.assert_logits(eng.step([slot], [ids], "all"), ph.plain_logits(name, ids), dtype, f"{name} whole n={n}")
        eng.release(slot)
    ids = ph.prompt(name, 5, 6)
    slot = eng.new_sequence()
    for t in range(6):      # positions 0, 1, 2, ... each as a step of its own
        ph.assert_logits(eng.step([slot], [[ids[t]]], "all"), ph.plain_logits(name, ids)[t:t + 1], dtype, f"{name} position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_stream_after_every_layer_run(name, dtype):
    model = ph.loaded_model(name, dtype)
    eng = ph.engine(name, dtype, page_size=16)
    ids = ph.prompt(name, 8, 21)
    cfg, w = ph.plain_model(name)
    streams, seen = [], []
    plain.forward(cfg, w, ids, streams=streams)
    for block in model.layers:
        def spy(stream, batch, cache, run, inner=block.forward):
            inner(stream, batch, cache, run)
            seen.append(stream.value().clone())
        block.forward = spy
    try:
        eng.step([eng.new_sequence()], [ids], "last")
    finally:
        for block in model.layers:
            del block.forward
    assert len(seen) == len(streams) == len(model.schedule)
    for i, (got, want) in enumerate(zip(seen, streams)):
        _close(got, want, dtype, f"stream after run {i}", bf16=6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token(name, dtype):
    """The last 60 tokens one by one: pages of 16 are crossed, the temperature steps."""
    eng = ph.engine(name, dtype, page_size=16)
    ids = ph.prompt(name, 6, 130)
    want = ph.plain_logits(name, ids)
    other = eng.new_sequence()
    eng.step([other], [ids[:20]], [[]])          # shifts which pages the next sequence gets
    slot = eng.new_sequence()
    ph.assert_logits(eng.step([slot], [ids[:70]], "all"), want[:70], dtype, "prefix")
    for t in range(70, 130):
        ph.assert_logits(eng.step([slot], [[ids[t]]], "all"), want[t:t + 1], dtype, f"{name} position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_down_to_two_tokens(name, dtype):
    """A prompt cut into portions of 2 to 90 tokens on a cached prefix: the convolution and the memory look back over the cuts."""
    eng = ph.engine(name, dtype, page_size=16)
    ids = ph.prompt(name, 7, 166)
    want = ph.plain_logits(name, ids)
    slot = eng.new_sequence()
    at = 0
    for n in (5, 2, 19, 2, 3, 16, 11, 90, 2, 16):
        ph.assert_logits(eng.step([slot], [ids[at:at + n]], "all"), want[at:at + n], dtype, f"{name} portion at {at}")
        at += n
    assert at == 166


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_on_reused_slots_and_pages(name, dtype):
    """Batches one after another on a cache with 4 slots and few pages: prompts of unequal lengths in one step, then one
    token each; shorter requests end earlier; later batches land on what earlier ones gave back (keys, the convolution's state and
    the memory).  Each request's logits equal those it gives alone (the plain implementation runs it alone)."""
    eng = ph.engine(name, dtype, max_tokens=14 * 16, max_seqs=4, page_size=16)
    shapes = [([5, 11, 17], [8, 8, 8]), ([1, 9, 23, 30], [12, 3, 7, 1]), ([40, 2, 100], [2, 22, 5])]
    for b, (lens, extra) in enumerate(shapes):
        seqs = [ph.prompt(name, 100 + 10 * b + i, n + e) for i, (n, e) in enumerate(zip(lens, extra))]
        want = [ph.plain_logits(name, s) for s in seqs]
        slots = [eng.new_sequence() for _ in seqs]
        got = eng.step(slots, [s[:n] for s, n in zip(seqs, lens)], "all")
        ph.assert_logits(got, ph.cat([w[:n] for w, n in zip(want, lens)]), dtype, f"batch {b} prompts")
        pos, live = list(lens), list(range(len(seqs)))
        while live:
            got = eng.step([slots[i] for i in live], [[seqs[i][pos[i]]] for i in live], "last")
            ph.assert_logits(got, ph.cat([want[i][pos[i]:pos[i] + 1] for i in live]), dtype, f"batch {b} decode at {pos}")
            for i in live:
                pos[i] += 1
            for i in [i for i in live if pos[i] == len(seqs[i])]:
                eng.release(slots[i])
            live = [i for i in live if pos[i] < len(seqs[i])]
        assert eng.cache.n_free_slots == 4
    if dtype == "bfloat16":
        assert eng.graph_replays > 0


@pytest.mark.parametrize("name,factor", [("PA", 5.0), ("PB", 5.0)])
def test_far_keys_and_every_constant_show(name, factor):
    """With scores multiplied nearly all weight lies on one key per query and map, often a far one.  The oracle itself shows that
    every constant of the configuration moves the logits; the engine follows it in 32-bit, whole, in portions and token by token."""
    from rust_deeplearning_b200 import Engine, load_model, write_random_model
    cfg, seed = tiny_paditar.config(name)
    for layer in cfg["layers"]:
        m = layer["mixer"]
        (m["left"] if "left" in m else m)["scale"] *= factor
    folder = os.path.join(ph.mh.tmp_root(), f"tiny_{name}_sharp")
    write_random_model(folder, cfg, seed, "bfloat16")
    pcfg, w = plain.load_folder(folder)
    ids = ph.prompt(name, 9, 90)
    want = plain.forward(pcfg, w, ids)

    def moves(change):
        moved = json.loads(json.dumps(pcfg))
        change(moved)
        return np.abs(plain.forward(moved, w, ids) - want).max()

    for i, layer in enumerate(pcfg["layers"]):
        m = layer["mixer"]
        if "left" in m:
            for side, key in ((None, "left_scale"), (None, "right_scale"), ("left", "scale"), ("right", "gate_cap")):
                assert moves(lambda c: (lambda o: o.update({key: o[key] * 1.2}))(c["layers"][i]["mixer"] if side is None else c["layers"][i]["mixer"][side])) > 1e-3, (i, key)
            for key, value in (("coef", m["left"]["q_temp"]["coef"] * 1.2), ("every", m["left"]["q_temp"]["every"] + 1)):
                assert moves(lambda c: c["layers"][i]["mixer"]["left"]["q_temp"].update({key: value})) > 1e-3, (i, key)
        else:
            for key, value in (("scale", m["scale"] * 1.1), ("diff", m["diff"] + 0.05), ("rot", {"base": m["rot"]["base"] * 1.3, "dims": m["rot"]["dims"]}),
                               ("rot", {"base": m["rot"]["base"], "dims": m["rot"]["dims"] - 2})):
                assert moves(lambda c: c["layers"][i]["mixer"].update({key: value})) > 1e-3, (i, key)
    assert moves(lambda c: c["loop"].update(times=c["loop"]["times"] - 1)) > 1e-1
    eng = Engine(load_model(folder, "float32", DEV), max_tokens=1024, page_size=16)
    want = ph.plain_want(pcfg, w, ids)
    check = lambda got, rows, what: ph.assert_logits(got, rows, "float32", what)
    slot = eng.new_sequence()
    check(eng.step([slot], [ids], "all"), want, "whole")
    slot = eng.new_sequence()
    for a, b in ((0, 13), (13, 15), (15, 34), (34, 50)):
        check(eng.step([slot], [ids[a:b]], "all"), want[a:b], f"portion {a}")
    slot = eng.new_sequence()
    check(eng.step([slot], [ids[:20]], "all"), want[:20], "prefix")
    for t in range(20, 90):
        check(eng.step([slot], [[ids[t]]], "all"), want[t:t + 1], f"position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """400 single-token steps: crosses pages, the memory runs on."""
    name = "PC"
    eng = ph.engine(name, dtype)
    ids = ph.prompt(name, 11, 400)
    want = ph.plain_logits(name, ids)
    slot = eng.new_sequence()
    eng.step([slot], [ids[:3]], [[]])
    for t in range(3, 400):
        got = eng.step([slot], [[ids[t]]], "last")
        if t % 7 == 0 or t > 380:
            ph.assert_logits(got, want[t:t + 1], dtype, f"position {t}")


def test_steps_beyond_the_position_tables_are_refused():
    from rust_deeplearning_b200 import StepError
    name = "PA"
    eng = ph.engine(name, "float32", page_size=16)
    slot = eng.new_sequence()
    ids = ph.prompt(name, 1, 400)
    eng.step([slot], [ids[:399]], [[]])
    ph.assert_logits(eng.step([slot], [ids[399:]], "last"), ph.plain_logits(name, ids)[-1:], "float32", "last position")
    with pytest.raises(StepError, match="401 positions"):
        eng.step([slot], [[1]], "last")


def test_greedy_generation_through_the_entry_point():
    from rust_deeplearning_b200 import Generator
    name = "PB"
    cfg, w = ph.plain_model(name)
    prompts = [ph.prompt(name, 300 + i, n) for i, n in enumerate((1, 9, 23))]
    gen = Generator(ph.loaded_model(name, "float32"), max_batch=4, max_context=128).with_temperature(0.0)
    got = gen.generate_batch(prompts, 10)
    for p, g in zip(prompts, got):
        assert g[:len(p)] == p
        # the plain loop, as long as its own margin between the best and the second best token is not a close call
        ids = list(p)
        for tok in g[len(p):]:
            last = plain.forward(cfg, w, ids)[-1]
            row = np.sort(last)
            if row[-1] - row[-2] < 5e-3:
                break
            assert tok == int(np.argmax(last))
            ids.append(tok)
        assert gen.generate(p, 10) == g


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_process(dtype, tmp_path):
    """bin/trace_run on a Paditar folder: two requests as one batch, then one token each, the shorter one ending first."""
    name = "PA"
    a, b = ph.prompt(name, 40, 30), ph.prompt(name, 41, 21)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:26], "want": [0, 25]}, {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[26]], "want": [0]}, {"id": "b", "tokens": [b[19]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[27]], "want": [0]}, {"id": "b", "tokens": [b[20]], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[28]], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": [a[29]], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", ph.model_folder(name), "--dtype", dtype,
                        "--out", str(tmp_path), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and r.stdout.split() == [x for i in range(5) for x in ("done", str(i))], (r.stdout, r.stderr)
    wa, wb = ph.plain_logits(name, a), ph.plain_logits(name, b)
    V = ph.vocab(name)
    read = lambda n: torch.tensor(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, V))
    ph.assert_logits(read(0), ph.cat([wa[:1], wa[25:26], wb[18:19]]), dtype, "step 0")
    ph.assert_logits(read(1), wa[26:27], dtype, "step 1")
    ph.assert_logits(read(2), ph.cat([wa[27:28], wb[20:21]]), dtype, "step 2")
    ph.assert_logits(read(3), wa[28:29], dtype, "step 3")
    ph.assert_logits(read(4), wa[29:30], dtype, "step 4")


def test_command_line_generates_with_a_paditar_folder(capsys):
    """The command line picks the architecture by config.json; its greedy tokens are the entry point's."""
    import io
    from rust_deeplearning_b200 import Generator, cli
    name = "PB"
    p = ph.prompt(name, 50, 12)
    out = io.StringIO()
    code = cli.main([ph.model_folder(name), "--prompt-ids", " ".join(map(str, p)), "--max-tokens", "6", "--temperature", "0",
                     "--dtype", "float32", "--max-context", "64"], stdout=out)
    assert code == 0
    assert "arch=Paditar" in capsys.readouterr().err
    gen = Generator(ph.loaded_model(name, "float32"), max_batch=1, max_context=64).with_temperature(0.0)
    assert [int(t) for t in out.getvalue().split()] == gen.generate(p, 6)[len(p):]
