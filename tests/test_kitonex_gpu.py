"""Kitonex on a GPU against the plain implementation, in 32-bit and in bfloat16: each new mechanism's kernels alone,
whole prompts, single tokens through the cache, portions, unequal batches on reused slots and pages, chunk edges and far
keys under sharp softmaxes, long decoding, greedy generation, the trace replay and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kitonex_helpers as kh
import plain_kitonex as plain
import tiny_kitonex

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
NAMES = ["KA", "KB"]
DEV = "cuda:0"


def _t(a, dtype):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(DEV).to(getattr(torch, dtype))


def _back(t):
    return t.float().cpu().double().numpy()


def _close(got, want, dtype, what, bf16=2e-2):
    got = _back(got.detach())
    tol = (2e-5 if dtype == "float32" else bf16) * max(1.0, float(np.abs(want).max()))
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
        seq, pos, start = [], [], [0]
        for i, (n, p) in enumerate(zip(lens, past)):
            seq += [i] * n
            pos += list(range(p, p + n))
            start.append(start[-1] + n)
        self.pos = pos
        self.tok_seq, self.tok_pos = _ti(seq + [0] * padding), _ti(pos + [-1] * padding)
        self.seq_start, self.slots, self.past = _ti(start), _ti(slots), _ti(past)
        self.seq_end = _ti([n + p for n, p in zip(lens, past)])

    def kw(self):
        return dict(tok_seq=self.tok_seq, tok_pos=self.tok_pos, seq_start=self.seq_start, slots=self.slots, seq_end=self.seq_end, n_seqs=self.n_seqs)


# ---- each mechanism alone ----

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [
    # query heads, key heads, laid-out size, key size, value size, taps, blending
    (3, 1, 12, 12, 9, 3, True), (6, 2, 16, 16, 8, 4, True), (4, 4, 64, 64, 64, 2, False), (5, 1, 24, 20, 24, 8, True), (2, 1, 8, 8, 8, 1, True),
    (2, 2, 11, 7, 11, 5, False), (36, 6, 128, 128, 96, 4, True), (20, 6, 256, 256, 256, 4, True), (30, 10, 256, 256, 64, 6, True),
    (40, 8, 100, 100, 100, 4, True), (100, 10, 50, 50, 41, 3, False)])
def test_bias_convolution_norms_blending_and_cache_write(dtype, sizes):
    """The kernel between the q/k/v product and attention against the plain mechanisms, over steps of unequal portions (0 to 21
    tokens a sequence and step: one token, fewer than the taps, more than a block takes at once) on shuffled slots with a padding row:
    the convolution's state passes from step to step, cache rows are read back through shuffled page lists; in 32-bit the same
    rows come out whatever the cut."""
    from rust_deeplearning_b200.kernels import ops
    H, G, D, d, e, taps, mix = sizes
    rng = np.random.default_rng(sum(sizes))
    eps, page, lam = 1e-3, 4, 0.3
    C, T = (H + 2 * G) * D, 45
    heads = [(H, d), (G, d), (G, e)]
    pad = lambda parts: np.concatenate([np.concatenate([p.reshape(n, s, -1), np.zeros((n, D - s, p.size // (n * s)))], axis=1).reshape(n * D, -1)
                                        for p, (n, s) in zip(parts, heads)])
    bias = [rng.normal(size=n * s) * 0.3 for n, s in heads]
    conv = [rng.normal(size=(n * s, taps)) * 0.6 for n, s in heads]
    wq, wk = rng.normal(size=H * d) + 1.0, rng.normal(size=G * d) + 1.0
    q8 = lambda a: _back(_t(a, dtype))                 # the values the kernel sees
    conv = [q8(c) for c in conv]
    bias, wq, wk = [_back(_t(b, "float32")) for b in bias], _back(_t(wq, "float32")), _back(_t(wk, "float32"))
    lay = lambda a, n, s: np.concatenate([a.reshape(-1, n, s), np.zeros((a.size // (n * s), n, D - s))], axis=2).reshape(-1, n * D)
    seqs = []
    for i in range(3):
        rows = [q8(rng.normal(size=(T, n * s))) for n, s in heads]
        first = q8(rng.normal(size=(T, G * e)))
        u = [plain.short_conv(r + b, c) for r, b, c in zip(rows, bias, conv)]
        want = [plain.rms_norm(u[0], wq, eps), plain.rms_norm(u[1], wk, eps), (1 - lam) * u[2] + lam * first if mix else u[2]]
        seqs.append((np.concatenate([lay(r, n, s) for r, (n, s) in zip(rows, heads)], axis=1), lay(first, G, e),
                     np.concatenate([lay(r, n, s) for r, (n, s) in zip(want, heads)], axis=1)))
    tb, tc = _t(pad(bias)[:, 0], "float32"), _t(pad(conv).T, dtype).contiguous()
    twq, twk = _t(lay(wq[None], H, d)[0], "float32"), _t(lay(wk[None], G, d)[0], "float32")
    n_pages = -(-T // page)
    order = rng.permutation(3 * n_pages).reshape(3, n_pages)
    kw = dict(bias=tb, conv=tc, wq=twq, wk=twk, eps=eps, q_count=H * d, k_count=G * d)

    def run(cuts, slots):
        state = torch.full((7, taps - 1, C), 99.0, dtype=torch.float32, device=DEV) if taps > 1 else None      # what a former owner left
        k = torch.zeros((3 * n_pages, G, page, D), dtype=getattr(torch, dtype), device=DEV)
        v = torch.zeros_like(k)
        past, outs = [0, 0, 0], [[], [], []]
        for lens in cuts:
            live = [i for i in range(3) if lens[i]]
            b = Batch([lens[i] for i in live], [past[i] for i in live], [slots[i] for i in live], padding=1)
            rows = np.concatenate([seqs[i][0][past[i]:past[i] + lens[i]] for i in live] + [np.full((1, C), 5.0)])
            first = np.concatenate([seqs[i][1][past[i]:past[i] + lens[i]] for i in live] + [np.zeros((1, G * D))])
            x = _t(rows, dtype)
            pages = ops.KVPages(k, v, _ti(order[live]), page, n_pages)
            out = ops.qkv_prepare(x, H, G, D, state=state, v_first=_t(first, dtype) if mix else None, v_lambda=lam, pages=pages, **kw, **b.kw())
            assert np.array_equal(_back(x), rows.astype(np.float32) if dtype == "float32" else rows)
            at = 0
            for i in live:
                outs[i].append(out[at:at + lens[i]].clone())
                at += lens[i]
                past[i] += lens[i]
        assert past == [T, T, T]
        return [torch.cat(o) for o in outs], k, v

    whole, k, v = run([(T, T, T)], [4, 0, 6])
    for i in range(3):
        _close(whole[i], seqs[i][2], dtype, f"sequence {i}", bf16=1.5e-2)
        got = _back(whole[i])
        for p in (0, 3, 4, 17, T - 1):
            for g in range(G):
                pg, r = order[i][p // page], p % page
                assert np.array_equal(_stored(k, pg, r, g, D), got[p, (H + g) * D:(H + g + 1) * D])
                assert np.array_equal(_stored(v, pg, r, g, D), got[p, (H + G + g) * D:(H + G + g + 1) * D])
    cuts = [(21, 2, 1), (1, 1, 1), (1, 7, 2), (0, 9, 3), (2, 0, 17), (20, 8, 0), (0, 18, 21)]
    parts, k2, v2 = run(cuts, [1, 5, 2])
    for a, b in zip(whole, parts):
        if dtype == "float32":
            assert torch.equal(a, b)
        else:
            _close(b, _back(a), dtype, "portions", bf16=1e-2)
    singles, _, _ = run([(30, 3, 44)] + [(1, 1, 1)] + [(1, 1, 0)] * 14 + [(0, 1, 0)] * 27, [3, 2, 1])
    for a, b in zip(whole, singles):
        if dtype == "float32":
            assert torch.equal(a, b)
        else:
            _close(b, _back(a), dtype, "single tokens", bf16=1e-2)
    if dtype == "float32":
        assert torch.equal(k, k2) and torch.equal(v, v2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_preparation_of_many_sequences(dtype):
    """Forty sequences of 1 to 30 new tokens, some with earlier ones, in one step and each in a step of its own."""
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(8)
    H, G, D, taps, n = 3, 1, 16, 4, 40
    C = (H + 2 * G) * D
    lens = [int(v) for v in rng.integers(1, 31, size=n)]
    lens[3:9] = [1] * 6
    past = [int(v) for v in rng.choice([0, 0, 1, 2, 5, 64], size=n)]
    slots = [int(v) for v in rng.permutation(n)]
    rows = _t(rng.normal(size=(sum(lens), C)), dtype)
    kw = dict(bias=_t(rng.normal(size=C), "float32"), conv=_t(rng.normal(size=(taps, C)), dtype), wq=_t(rng.normal(size=H * D), "float32"),
              wk=_t(rng.normal(size=G * D), "float32"), eps=1e-5, q_count=H * D, k_count=G * D)
    before = _t(rng.normal(size=(n, taps - 1, C)), "float32")
    together, alone = before.clone(), before.clone()
    got = ops.qkv_prepare(rows, H, G, D, state=together, **kw, **Batch(lens, past, slots).kw())
    at = 0
    for i in range(n):
        one = ops.qkv_prepare(rows[at:at + lens[i]], H, G, D, state=alone, **kw, **Batch([lens[i]], [past[i]], [slots[i]]).kw())
        assert torch.equal(one, got[at:at + lens[i]]), f"sequence {i}: {lens[i]} tokens after {past[i]}"
        at += lens[i]
    assert torch.equal(together, alone)


@pytest.mark.parametrize("dtype", DTYPES)
def test_preparation_in_a_ring_and_without_its_mechanisms(dtype):
    """With nothing asked for the rows pass through unchanged; in a ring only the last writer of a cache row writes."""
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(3)
    for H, G, D in ((2, 1, 16), (3, 3, 7)):
        n, page, past = 19, 4, 6
        b = Batch([n], [past], [0])
        x = _t(rng.normal(size=(n, (H + 2 * G) * D)), dtype)
        k, v = (torch.zeros((3, G, page, D), dtype=x.dtype, device=DEV) for _ in range(2))
        out = ops.qkv_prepare(x, H, G, D, pages=ops.KVPages(k, v, _ti([[2, 0, 1]]), page, 3), **b.kw())
        assert torch.equal(out, x)
        for p in range(past + n - 12, past + n):
            pg, r = [2, 0, 1][(p // page) % 3], p % page
            for g in range(G):
                assert np.array_equal(_stored(k, pg, r, g, D), _back(x)[p - past, (H + g) * D:(H + g + 1) * D])
                assert np.array_equal(_stored(v, pg, r, g, D), _back(x)[p - past, (H + G + g) * D:(H + G + g + 1) * D])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [72, 75, 1000, 2304, 9000])
def test_copies_of_the_stream(dtype, width):
    """One step of a stream of several copies: from one row that stands for all and from copies (in place), one result and two with
    a gate per row, no result, chosen rows, no norm; in 32-bit a row does not depend on how many rows the step has."""
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(width)
    rows, eps = 6, 1e-4
    for S in ((1, 2, 3, 4, 6) if width < 3000 else (2, 5)):
        w = {"c.in": rng.normal(size=S), "c.out": rng.normal(size=S), "c.mix": rng.normal(size=(S, S)), "d.in": rng.normal(size=S)}
        w = {k: _back(_t(v, "float32")) for k, v in w.items()}
        tw = {k: _t(v, "float32") for k, v in w.items()}
        nw = _t(rng.normal(size=width) + 1.0, dtype)
        norm = ops.NormParams(nw, eps, 0.0)
        one = _t(rng.normal(size=(rows, width)), "float32")
        many = _t(rng.normal(size=(rows, S, width)), "float32")
        a, b = _t(rng.normal(size=(rows, width)), dtype), _t(rng.normal(size=(rows, width)), dtype)
        logits = _t(rng.normal(size=(rows, 3)), "float32")
        gate = logits[:, 2:]
        y2 = _back(a) + _back(b) * plain.sigmoid(_back(gate))
        idx = _ti([4, 0, 4])
        for start in (one, many):
            x = _back(start) if start is many else np.repeat(_back(start)[:, None], S, axis=1)
            xs = x.transpose(1, 0, 2)
            if width == 9000 and start is one and S > 4:
                continue
            # reading alone
            _, u = ops.hyper(start, S, read=tw["d.in"], norm=norm, out_dtype=getattr(torch, dtype))
            _close(u, plain.rms_norm(plain.read_copies(xs, w, "d."), _back(nw), eps), dtype, "read")
            for y, kw in ((_back(a), dict(a=a)), (y2, dict(a=a, b=b, b_gate=gate)), (_back(a) + _back(b) * plain.sigmoid(_back(gate)), dict(a=a, b=b, b_gate=gate.contiguous()))):
                kw = dict(kw, mix=tw["c.mix"], write=tw["c.out"])
                want = plain.write_copies(xs, y, w, "c.")
                got, u = ops.hyper(start, S, read=tw["d.in"], norm=norm, out_dtype=getattr(torch, dtype), row_index=idx, **kw)
                assert got is None
                wu = plain.rms_norm(plain.read_copies(want, w, "d."), _back(nw), eps)
                _close(u, wu[[4, 0, 4]], dtype, "chosen rows")
                inp = start.clone()
                got, u = ops.hyper(inp, S, read=tw["d.in"], norm=norm, out_dtype=getattr(torch, dtype), **kw)
                _close(got, want.transpose(1, 0, 2), "float32", f"copies {S}")
                _close(u, wu, dtype, "written and read")
                assert (got is inp) == (start is many)
                only, none = ops.hyper(start.clone(), S, **kw)
                assert none is None and torch.equal(only, got)
                _, plain_sum = ops.hyper(got, S, read=tw["d.in"])
                _close(plain_sum, plain.read_copies(want, w, "d."), "float32", "sum without a norm")
                if dtype == "float32":
                    few = {k: (v[3:4].contiguous() if k in ("a", "b", "b_gate") else v) for k, v in kw.items()}
                    g1, u1 = ops.hyper(start[3:4].clone(), S, read=tw["d.in"], norm=norm, out_dtype=torch.float32, **few)
                    assert torch.equal(g1, got[3:4]) and torch.equal(u1, u[3:4])


@pytest.mark.parametrize("case", [
    # heads, key heads, size, chunk, buckets, largest, window
    (6, 2, 64, 33, 16, 20, None), (3, 1, 64, 100, 32, 100, None), (4, 4, 128, 64, 8, 500, None), (8, 1, 16, 7, 6, 5, None), (2, 2, 64, None, 32, 70, None),
    (2, 1, 256, 130, 32, 64, None), (5, 1, 48, 40, 10, 39, None), (4, 2, 64, 128, 16, 90, 50), (12, 1, 32, 25, 16, 24, None)])
def test_attention_kernels_with_chunks_a_distance_bias_and_one_in_the_denominator(case):
    """Every attention kernel against the plain one: the float kernel in both dtypes, both prompt kernels (with the step's rows
    after cached ones: the one that reads both), the decode kernel over pages in random order.  For every query one key stands
    out by far: the first of its chunk, the last of the chunk before (which must not count), the query itself, a far one."""
    from rust_deeplearning_b200.kernels import ops
    H, G, D, chunk, buckets, largest, window = case
    rng = np.random.default_rng(sum(v or 0 for v in case))
    lens, page = [1, 150, 61, 290], 16
    scale = 2.0 / D ** 0.5
    rel = _back(_t(rng.normal(size=(buckets, H)) * 1.5, "float32"))
    longest = min(chunk or 400, 400)
    from rust_deeplearning_b200.parts.attention import distance_buckets
    bias = ops.DistanceBias.of(_t(rel[distance_buckets(buckets, largest, longest)].T, "float32"))
    sinks = torch.zeros(H, dtype=torch.float32, device=DEV)
    seqs = []
    for n in lens:
        q, k, v = rng.normal(size=(n, H, D)), rng.normal(size=(n, G, D)), rng.normal(size=(n, G, D))
        for i in range(n):
            c = chunk or 10 ** 9
            lo = i // c * c
            target = [lo, lo - 1, i, max(lo, i - 40), lo + (i - lo) // 2][i % 5]
            if target >= 0 and i % 2 == 0:
                q[i] = 3.0 * k[target].repeat(H // G, axis=0) / np.abs(k[target]).max()
        seqs.append(tuple(_back(_t(a, "bfloat16")) for a in (q, k, v)))

    def want(q, k, v):
        if window is None:
            return plain.attend(q, k, v, scale, rel, largest, chunk)
        out = np.zeros((len(q), H, D))
        for i in range(len(q)):           # a window inside the chunk: the plain one on the keys it leaves
            lo = max(0 if chunk is None else i // chunk * chunk, i - window + 1)
            for a in range(H):
                s = k[lo:i + 1, a // (H // G)] @ q[i, a] * scale + rel[[plain.bucket(i - j, buckets, largest) for j in range(lo, i + 1)], a]
                e = np.exp(s)
                out[i, a] = e @ v[lo:i + 1, a // (H // G)] / (1 + e.sum())
        return out

    expected = [want(*s).reshape(len(s[0]), H * D) for s in seqs]
    n_pages = [-(-n // page) for n in lens]
    order = rng.permutation(sum(n_pages))
    table = np.zeros((len(lens), max(n_pages)), dtype=np.int32)
    at = 0
    for i, n in enumerate(n_pages):
        table[i, :n] = order[at:at + n]
        at += n
    packed = [np.concatenate([a.reshape(len(a), -1) for a in s], axis=1) for s in seqs]
    common = dict(n_heads=H, n_kv_heads=G, head_dim=D, score_scale=scale, softcap=None, window=window, chunk=chunk, distance_bias=bias, sinks=sinks)

    def tiles(ls):
        t = [(i, q0) for i, n in enumerate(ls) for q0 in range(0, n, ops.PREFILL_QUERY_TILE)]
        return _ti([a for a, _ in t]), _ti([b for _, b in t]), len(t)

    def batch(ls, past, cached):
        b = Batch(ls, past, [0] * len(ls))
        ts, tq, nt = tiles(ls)
        return b, ops.AttentionBatch(sum(ls), len(ls), b.tok_seq, b.tok_pos, b.seq_start, b.past, _ti(cached), ts, tq, nt, max_keys=max(p + n for p, n in zip(past, ls)))

    for dtype in DTYPES:
        rows = _t(np.concatenate(packed), dtype)
        cols = (rows, H * D, (H + G) * D)
        k = torch.zeros((sum(n_pages), G, page, D), dtype=rows.dtype, device=DEV)
        v = torch.zeros_like(k)
        pages = ops.KVPages(k, v, _ti(table), page, table.shape[1])
        b, ab = batch(lens, [0] * 4, [0] * 4)
        ops.qkv_prepare(rows, H, G, D, pages=pages, **b.kw())
        kinds = ["plain"]
        if dtype == "bfloat16":
            kinds += ["prefill"] + (["prefill_tc"] if D % 64 == 0 else [])
        for kind in kinds:
            _close(ops.attention(rows, ab, pages, new_kv=cols, kind=kind, **common), np.concatenate(expected), dtype, f"{kind}, whole prompts")
        # the last 23 tokens of the longer prompts after cached ones
        tail = [(i, max(0, n - 23)) for i, n in enumerate(lens)]
        rows2 = _t(np.concatenate([packed[i][p:] for i, p in tail]), dtype)
        b2, ab2 = batch([lens[i] - p for i, p in tail], [p for _, p in tail], [p for _, p in tail])
        for kind in [x for x in kinds if x != "prefill_tc"]:
            _close(ops.attention(rows2, ab2, pages, new_kv=(rows2, H * D, (H + G) * D), kind=kind, **common),
                   np.concatenate([expected[i][p:] for i, p in tail]), dtype, f"{kind}, portions")
        # single tokens: for several positions of every sequence the query alone, all its keys in the cache
        for back in (0, 1, 2, 3, 17, 40):
            pos = [max(0, n - 1 - back) for n in lens]
            rows3 = _t(np.stack([packed[i][p] for i, p in enumerate(pos)]), dtype)
            b3, ab3 = batch([1] * 4, pos, [p + 1 for p in pos])
            ex = np.stack([expected[i][p] for i, p in enumerate(pos)])
            _close(ops.attention(rows3, ab3, pages, kind="plain", **common), ex, dtype, f"plain, single tokens {pos}")
            if dtype == "bfloat16" and H // G <= 8:
                for ks in (page, 4 * page):
                    _close(ops.attention(rows3, ab3, pages, kind="decode", keys_per_split=ks, **common), ex, dtype, f"decode, {ks} keys a block, {pos}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_positions(dtype):
    from rust_deeplearning_b200.kernels import ops
    rng = np.random.default_rng(0)
    E, P = _t(rng.normal(size=(9, 37)), dtype), _t(rng.normal(size=(5, 37)), dtype)
    ids, pos = [8, 0, 3, 3, 1], [4, 0, 2, -1, 3]
    status = torch.zeros(1, dtype=torch.int32).pin_memory()
    got = ops.embed_rows(E, _ti(ids), 2.0, status, P, _ti(pos))
    want = 2.0 * _back(E)[ids] + np.where(np.array(pos)[:, None] >= 0, _back(P)[pos], 0.0)
    _close(got, want, "float32", "embedding")
    torch.cuda.synchronize()
    assert int(status[0]) == 0
    got = ops.embed_rows(E, _ti(ids), 2.0, status, P, _ti([4, 5, 2, 1, 3]))         # position 5 has no vector: poisoned and reported
    torch.cuda.synchronize()
    assert int(status[0]) == 2 and torch.isnan(got[1]).all() and torch.isfinite(got[[0, 2, 3, 4]]).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 12, 40, 200])
def test_limited_feed_forward(dtype, rows):
    """The gated form with a limit in every product it rides in: few rows, some, many; limits that bind on both sides."""
    from rust_deeplearning_b200.parts.feed_forward import GatedMLP
    rng = np.random.default_rng(rows)
    for W, ff, limit in ((64, 96, 0.8), (36, 20, 2.0), (128, 264, 0.3)):
        w = {"gate": rng.normal(size=(ff, W)) * 0.3, "up": rng.normal(size=(ff, W)) * 0.3, "down": rng.normal(size=(W, ff)) * 0.3}
        wt = {k: _t(v, dtype) for k, v in w.items()}
        x = _t(rng.normal(size=(rows, W)), dtype)
        want = plain.limited(_back(x), {k: _back(v) for k, v in wt.items()}, "", limit)
        part = GatedMLP(W, ff, "swish_limit", wt["gate"], wt["up"], wt["down"], limit)
        _close(part.forward(x), want, dtype, f"width {W}, limit {limit}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 200])
@pytest.mark.parametrize("shape", [(8, 2, (4, 2), True), (6, 2, (3, 1), False), (6, 3, (6, 3), True), (40, 6, (5, 2), True), (64, 4, (1, 1), True), (3, 3, None, True), (70, 1, (35, 2), False)])
def test_router_in_groups_and_experts_with_a_gated_shared_one(dtype, rows, shape):
    from rust_deeplearning_b200.parts.routed_experts import RoutedExperts
    from rust_deeplearning_b200.kernels import ops
    n_exp, top, groups, shared = shape
    rng = np.random.default_rng(3 + n_exp + top)
    W, ff = 48, 24
    r = {"experts": n_exp, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r, **({"shared": {"ff": 16}} if shared else {})}
    w = {"router": rng.normal(size=(n_exp, W)) * 0.3, "shared.sg": rng.normal(size=(1, W)) * 0.3}
    for p in [f"e{e}." for e in range(n_exp)] + (["shared."] if shared else []):
        n = 16 if p == "shared." else ff
        w[p + "gate"], w[p + "up"], w[p + "down"] = (rng.normal(size=s) * 0.3 for s in ((n, W), (n, W), (W, n)))
    wt = {k: _t(v, dtype) for k, v in w.items()}
    w = {k: _back(v) for k, v in wt.items()}
    xt = _t(rng.normal(size=(rows, W)), dtype)
    x = _back(xt)
    chosen, weight, margin = plain.router(x, w, "", r)
    router = torch.cat([wt["router"].float(), wt["shared.sg"].float()])
    sel, sel_w, extra = ops.moe_route(xt, router, None, top, "sigmoid", groups=groups, norm_eps=1e-20, extra=1)
    safe = margin > 1e-5
    assert safe.any()
    assert np.array_equal(sel.cpu().numpy()[safe], chosen[safe])        # in the order of the scores
    _close(sel_w[torch.tensor(safe, device=DEV)], weight[safe], "float32", "weights")
    _close(extra, x @ w["shared.sg"].T, "float32", "the shared expert's gate")
    part = RoutedExperts(hidden_size=W, expert_size=ff, n_experts=n_exp, n_identity=0, top=top, form="silu", form_param=0.0,
                         w_router=wt["router"], correction=None, gates=[wt[f"e{e}.gate"] for e in range(n_exp)],
                         ups=[wt[f"e{e}.up"] for e in range(n_exp)], downs=[wt[f"e{e}.down"] for e in range(n_exp)], scoring="sigmoid",
                         groups=groups, normalise_eps=1e-20, shared_gate=wt["shared.sg"] if shared else None,
                         shared=(wt["shared.gate"], wt["shared.up"], wt["shared.down"]) if shared else None)
    want = plain.feed_forward(x, w, "", f)
    keep = torch.tensor(safe, device=DEV)
    _close(part.forward(xt)[keep], want[safe], dtype, "experts", bf16=3e-2)
    a, b, gate = part.forward_gated_parts(xt)
    got = _back(a) + (_back(b) * plain.sigmoid(_back(gate)) if shared else 0.0)
    _close(torch.tensor(got)[torch.tensor(safe)], want[safe], dtype, "experts in parts", bf16=3e-2)


# ---- the model ----

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_first_tokens(name, dtype):
    eng = kh.engine(name, dtype, page_size=16)
    for seed, n in ((1, 1), (2, 2), (3, 37), (4, 70)):
        ids = kh.prompt(name, seed, n, dtype)
        slot = eng.new_sequence()
        kh.assert_logits(eng.step([slot], [ids], "all"), kh.plain_logits(name, ids), dtype, f"{name} whole n={n}")
        eng.release(slot)
    ids = kh.prompt(name, 5, 6, dtype)
    slot = eng.new_sequence()
    for t in range(6):      # positions 0, 1, 2, ... each as a step of its own
        kh.assert_logits(eng.step([slot], [[ids[t]]], "all"), kh.plain_logits(name, ids)[t:t + 1], dtype, f"{name} position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_stream_after_every_layer(name, dtype):
    """The sum of the copies after each layer against the plain one."""
    model = kh.loaded_model(name, dtype)
    eng = kh.engine(name, dtype, page_size=16)
    ids = kh.prompt(name, 8, 21, dtype)
    cfg, w = kh.plain_model(name)
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
    assert len(seen) == len(streams)
    for i, (got, want) in enumerate(zip(seen, streams)):
        _close(got, want, dtype, f"stream after layer {i}", bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token(name, dtype):
    """The last 60 tokens one by one: chunks of 7, 11, 33 and 40 positions begin and end inside them, pages of 16 are crossed and
    the rings wrap."""
    eng = kh.engine(name, dtype, page_size=16)
    ids = kh.prompt(name, 6, 90, dtype)
    want = kh.plain_logits(name, ids)
    other = eng.new_sequence()
    eng.step([other], [ids[:20]], [[]])          # shifts which pages the next sequence gets
    slot = eng.new_sequence()
    kh.assert_logits(eng.step([slot], [ids[:30]], "all"), want[:30], dtype, "prefix")
    for t in range(30, 90):
        kh.assert_logits(eng.step([slot], [[ids[t]]], "all"), want[t:t + 1], dtype, f"{name} position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_down_to_two_tokens(name, dtype):
    """A prompt cut into portions of 2 to 19 tokens on a cached prefix (pages of 8: rings wrap inside a portion); chunks are
    counted from the sequence's start, the convolution looks back over the cuts."""
    eng = kh.engine(name, dtype, page_size=8)
    ids = kh.prompt(name, 7, 66, dtype)
    want = kh.plain_logits(name, ids)
    slot = eng.new_sequence()
    at = 0
    for n in (5, 2, 19, 2, 3, 16, 11, 8):
        kh.assert_logits(eng.step([slot], [ids[at:at + n]], "all"), want[at:at + n], dtype, f"{name} portion at {at}")
        at += n
    assert at == 66


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_on_reused_slots_and_pages(name, dtype):
    """Batches one after another on a cache with 4 slots and few pages: prompts of unequal lengths in one step, then one
    token each; shorter requests end earlier; later batches land on what earlier ones gave back (keys and the convolution's state).
    Each request's logits equal those it gives alone (the plain implementation runs it alone)."""
    eng = kh.engine(name, dtype, max_tokens=10 * 16, max_seqs=4, page_size=16)
    shapes = [([5, 11, 17], [8, 8, 8]), ([1, 9, 23, 30], [12, 3, 7, 1]), ([40, 2, 20], [2, 22, 5])]
    for b, (lens, extra) in enumerate(shapes):
        seqs = [kh.prompt(name, 100 + 10 * b + i, n + e, dtype) for i, (n, e) in enumerate(zip(lens, extra))]
        want = [kh.plain_logits(name, s) for s in seqs]
        slots = [eng.new_sequence() for _ in seqs]
        got = eng.step(slots, [s[:n] for s, n in zip(seqs, lens)], "all")
        kh.assert_logits(got, np.concatenate([w[:n] for w, n in zip(want, lens)]), dtype, f"batch {b} prompts")
        pos, live = list(lens), list(range(len(seqs)))
        while live:
            got = eng.step([slots[i] for i in live], [[seqs[i][pos[i]]] for i in live], "last")
            kh.assert_logits(got, np.stack([want[i][pos[i]] for i in live]), dtype, f"batch {b} decode at {pos}")
            for i in live:
                pos[i] += 1
            for i in [i for i in live if pos[i] == len(seqs[i])]:
                eng.release(slots[i])
            live = [i for i in live if pos[i] < len(seqs[i])]
        assert eng.cache.n_free_slots == 4
    if dtype == "bfloat16":
        assert eng.graph_replays > 0


@pytest.mark.parametrize("name,factor", [("KA", 6.0), ("KB", 8.0)])
def test_chunk_edges_far_keys_and_every_constant_show(name, factor):
    """With scores multiplied nearly all weight lies on one key per query and head: over 90 positions often the first of its
    chunk, the last of a chunk before (which must not count) or a far one.  The oracle itself shows that a chunk one longer, a
    bias that ends elsewhere, another share in the blend, a tap less or another limit moves the logits; the engine follows it in
    32-bit, whole, in portions and token by token."""
    from rust_deeplearning_b200 import Engine, load_model, write_random_model
    cfg, seed = tiny_kitonex.config(name)
    for layer in cfg["layers"]:
        layer["mixer"]["scale"] *= factor
    folder = os.path.join(kh.mh.tmp_root(), f"tiny_{name}_sharp")
    write_random_model(folder, cfg, seed, "bfloat16")
    pcfg, w = plain.load_folder(folder)
    ids = [int(v) for v in np.random.default_rng(9).integers(0, cfg["vocab"], size=90)]
    margins = []
    want = plain.forward(pcfg, w, ids, margins)
    safe = np.minimum.reduce(margins) > 2e-5
    n = int(np.argmin(safe)) if not safe.all() else len(ids)      # logits after a close call are another computation
    assert n > 50

    def moves(change=None, weights=None):
        moved = json.loads(json.dumps(pcfg))
        if change:
            change(moved["layers"])
        return np.abs(plain.forward(moved, dict(w, **(weights or {})), ids)[:n] - want[:n]).max()

    for i, layer in enumerate(pcfg["layers"]):
        m = layer["mixer"]
        if m.get("mask"):
            for by in (1, -1):
                assert moves(lambda ls: ls[i]["mixer"]["mask"].update(size=m["mask"]["size"] + by)) > 1e-2, i
        assert moves(lambda ls: ls[i]["mixer"].update(bias_max=m["bias_max"] * 1.7)) > 1e-3, i
        if m["v_mix"] and i:
            assert moves(weights={f"l{i}.mix.vmix": w[f"l{i}.mix.vmix"] + 0.05}) > 1e-3, i
        if m.get("conv", 1) > 1:
            c = w[f"l{i}.mix.k.conv"].copy()
            c[:, 0] = 0.0
            assert moves(weights={f"l{i}.mix.k.conv": c}) > 1e-2, i
        if (layer.get("mlp") or {}).get("limit"):
            assert moves(lambda ls: ls[i]["mlp"].update(limit=layer["mlp"]["limit"] * 1.1)) > 1e-3, i
    assert moves(weights={"pos": w["pos"] * 0.9}) > 1e-2
    eng = Engine(load_model(folder, "float32", DEV), max_tokens=1024, page_size=16)
    slot = eng.new_sequence()
    kh.assert_logits(eng.step([slot], [ids[:n]], "all"), want[:n], "float32", "whole")
    slot = eng.new_sequence()
    for a, b in ((0, 13), (13, 15), (15, 34), (34, 50)):
        kh.assert_logits(eng.step([slot], [ids[a:b]], "all"), want[a:b], "float32", f"portion {a}")
    slot = eng.new_sequence()
    kh.assert_logits(eng.step([slot], [ids[:20]], "all"), want[:20], "float32", "prefix")
    for t in range(20, n):
        kh.assert_logits(eng.step([slot], [[ids[t]]], "all"), want[t:t + 1], "float32", f"position {t}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """300 single-token steps with every expert chosen: crosses pages, wraps the rings many times, chunks begin and end."""
    name = "KC"
    eng = kh.engine(name, dtype)
    ids = kh.mh.prompt(11, 300, kh.vocab(name))
    want = kh.plain_logits(name, ids)
    slot = eng.new_sequence()
    eng.step([slot], [ids[:3]], [[]])
    for t in range(3, 300):
        got = eng.step([slot], [[ids[t]]], "last")
        if t % 7 == 0 or t > 280:
            kh.assert_logits(got, want[t:t + 1], dtype, f"position {t}")


def test_steps_beyond_the_position_table_are_refused():
    from rust_deeplearning_b200 import StepError
    name = "KA"
    eng = kh.engine(name, "float32", page_size=16)
    slot = eng.new_sequence()
    ids = kh.mh.prompt(1, 400, kh.vocab(name))
    eng.step([slot], [ids[:399]], [[]])
    kh.assert_logits(eng.step([slot], [ids[399:]], "last"), kh.plain_logits(name, ids)[-1:], "float32", "last position")
    with pytest.raises(StepError, match="401 positions"):
        eng.step([slot], [[1]], "last")


def test_greedy_generation_through_the_entry_point():
    from rust_deeplearning_b200 import Generator
    name = "KB"
    cfg, w = kh.plain_model(name)
    prompts = [kh.prompt(name, 300 + i, n, "float32") for i, n in enumerate((1, 9, 23))]
    gen = Generator(kh.loaded_model(name, "float32"), max_batch=4, max_context=128).with_temperature(0.0)
    got = gen.generate_batch(prompts, 10)
    for p, g in zip(prompts, got):
        assert g[:len(p)] == p
        # the plain loop, as long as its own margin between the best and the second best token is not a close call
        ids = list(p)
        for tok in g[len(p):]:
            last = plain.forward(cfg, w, ids)[-1]
            row = np.sort(last)
            if row[-1] - row[-2] < 1e-3 or plain.min_margin(cfg, w, ids) < 2e-5:
                break
            assert tok == int(np.argmax(last))
            ids.append(tok)
        assert gen.generate(p, 10) == g


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_process(dtype, tmp_path):
    """bin/trace_run on a Kitonex folder: two requests as one batch, then one token each, the shorter one ending first."""
    name = "KA"
    a, b = kh.prompt(name, 40, 30, dtype), kh.prompt(name, 41, 21, dtype)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:26], "want": [0, 25]}, {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[26]], "want": [0]}, {"id": "b", "tokens": [b[19]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[27]], "want": [0]}, {"id": "b", "tokens": [b[20]], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[28]], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": [a[29]], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", kh.model_folder(name), "--dtype", dtype,
                        "--out", str(tmp_path), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and r.stdout.split() == [x for i in range(5) for x in ("done", str(i))], (r.stdout, r.stderr)
    wa, wb = kh.plain_logits(name, a), kh.plain_logits(name, b)
    V = kh.vocab(name)
    read = lambda n: torch.tensor(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, V))
    kh.assert_logits(read(0), np.stack([wa[0], wa[25], wb[18]]), dtype, "step 0")
    kh.assert_logits(read(1), wa[26:27], dtype, "step 1")
    kh.assert_logits(read(2), np.stack([wa[27], wb[20]]), dtype, "step 2")
    kh.assert_logits(read(3), wa[28:29], dtype, "step 3")
    kh.assert_logits(read(4), wa[29:30], dtype, "step 4")


def test_command_line_generates_with_a_kitonex_folder(capsys):
    """The command line picks the architecture by config.json; its greedy tokens are the entry point's."""
    import io
    from rust_deeplearning_b200 import Generator, cli
    name = "KB"
    p = kh.prompt(name, 50, 12, "float32")
    out = io.StringIO()
    code = cli.main([kh.model_folder(name), "--prompt-ids", " ".join(map(str, p)), "--max-tokens", "6", "--temperature", "0",
                     "--dtype", "float32", "--max-context", "64"], stdout=out)
    assert code == 0
    assert "arch=Kitonex" in capsys.readouterr().err
    gen = Generator(kh.loaded_model(name, "float32"), max_batch=1, max_context=64).with_temperature(0.0)
    assert [int(t) for t in out.getvalue().split()] == gen.generate(p, 6)[len(p):]
