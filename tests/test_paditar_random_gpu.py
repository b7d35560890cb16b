"""Paditar configurations drawn at random (seeded): one to four layers in any order, any stretch of them run one to three times or no
loop at all, head sizes that are and are not multiples of 8 and 16, one to three key heads with one to nine query heads each, values
narrower and wider than keys, one to eight taps, memories of one to three heads with caps from 2 to 20, with and without a
feed-forward, any constants, pages of 16, 32 and 64 rows.  Each case runs one to four sequences of unequal length through the engine
in both dtypes - whole, as a prefix with single tokens after it, and as portions of 1 to 29 tokens a step that mix with one another - and
compares the logits with the plain implementation (within what rounding alone does at each position); in float32 the three ways of cutting also have to give the same bits."""
import tempfile

import numpy as np
import pytest
import torch

import model_helpers as mh
import paditar_helpers as ph
import plain_paditar as plain

pytestmark = pytest.mark.gpu


def draw(case: int):
    rng = np.random.default_rng(900 + case)
    pick = lambda *v: v[int(rng.integers(0, len(v)))]
    layers = []
    for _ in range(int(rng.integers(1, 5))):
        kv = pick(1, 2, 3)
        heads = kv * pick(1, 2, 3, 5, 9)
        if rng.integers(0, 3) == 0:
            dim = pick(8, 16, 24, 32, 64, 10, 40)
            m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": pick(16, 20, 48, 64, 128, 2 * dim), "scale": pick(dim ** -0.5, 0.3), "diff": pick(0.2, 0.5, 0.7),
                 "rot": {"base": pick(100.0, 10000.0), "dims": 2 * int(rng.integers(1, dim // 2 + 1))}}
            kind = "attention"
        else:
            dim, rd = pick(16, 24, 32, 64, 40, 128, 10, 96), pick(16, 32, 48, 64, 10, 128)
            m = {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": pick(dim ** -0.5, 0.2), "conv": int(rng.integers(1, 9)),
                          "q_temp": {"coef": pick(0.1, 0.5), "every": pick(3, 16, 64)}},
                 "right": {"heads": pick(1, 2, 3), "dim": rd, "vdim": pick(rd, 16, 40, 64), "gate_cap": pick(2.0, 8.0, 20.0)},
                 "left_scale": pick(0.5, 1.0, 1.3), "right_scale": pick(0.6, 1.0, 1.5)}
            kind = "parallel"
        layers.append({"type": kind, "mixer": m, "mlp": pick(None, {"kind": "dense", "ff": pick(40, 64, 96, 52)}, {"kind": "dense", "ff": 80})})
    cfg = {"architecture": "Paditar", "width": pick(48, 64, 72, 88, 136, 50), "vocab": int(rng.integers(90, 400)), "norm": {"eps": pick(1e-6, 1e-5, 1e-3)},
           "max_positions": 128, "layers": layers}
    if rng.integers(0, 4):
        start = int(rng.integers(0, len(layers)))
        cfg["loop"] = {"start": start, "stop": int(rng.integers(start + 1, len(layers) + 1)), "times": pick(1, 2, 2, 3)}
    return rng, cfg, pick(16, 32, 64), [int(v) for v in rng.integers(1, 100, size=int(rng.integers(1, 5)))]


@pytest.mark.parametrize("case", range(24))
def test_a_configuration_drawn_at_random(case):
    from rust_deeplearning_b200 import Engine, load_model, write_random_model
    rng, cfg, page, lengths = draw(case)
    what = f"case {case}: width {cfg['width']}, loop {cfg.get('loop')}, " + "; ".join(f"{l['mixer']} mlp {l['mlp']}" for l in cfg["layers"]) + f", page {page}, lengths {lengths}"
    with tempfile.TemporaryDirectory(prefix="rdl_random_") as folder:
        write_random_model(folder, cfg, case, "bfloat16")
        pcfg, pw = plain.load_folder(folder)
        seqs = [mh.prompt(3000 + 10 * case + i, n, cfg["vocab"]) for i, n in enumerate(lengths)]
        want = [ph.plain_want(pcfg, pw, s) for s in seqs]
        largest = max(float(np.abs(w.logits).max()) for w in want)
        for dtype in ("float32", "bfloat16"):
            eng = Engine(load_model(folder, dtype, "cuda:0"), max_tokens=2048, max_seqs=8, page_size=page)
            # the least tolerance is one for the whole case, from the largest logit of all its sequences (a step's few rows may hold small
            # logits only, while the rounding of a bfloat16 model is that of its largest values)
            exact = dtype == "float32"
            floor = 3e-5 * max(1.0, largest) if exact else 0.035 * largest + 1e-3

            def compare(got, rows, label):
                """rows: (sequence, position) of each row of got"""
                g = got.float().cpu().double().numpy()
                w, limit = np.stack([want[i].logits[p] for i, p in rows]), np.array([max(floor, want[i].limits[dtype][p]) for i, p in rows])
                assert np.isfinite(g).all(), f"{dtype}, {label}: non-finite logits; {what}"
                err = np.abs(g - w).max(axis=1)
                r = int((err / limit).argmax())
                # three samples of rounding do not show its rarest effect (a read-out that nearly cancels may change its sign): in
                # bfloat16 a row in fifty may lie up to four times as far
                over = err > limit
                ok = not over.any() if exact else err[r] <= 4.0 * limit[r] and over.sum() <= max(1, len(rows) // 50)
                assert ok, f"{dtype}, {label}: error {err[r]:.3e} > {limit[r]:.3e} (row {r} of {len(rows)}, {rows[r]}); {what}"

            slots = [eng.new_sequence() for _ in seqs]
            whole = eng.step(slots, seqs, "all").clone()
            compare(whole, [(i, p) for i, s in enumerate(seqs) for p in range(len(s))], "whole")
            first_row = np.concatenate([[0], np.cumsum(lengths)])
            for s in slots:
                eng.release(s)
            k = int(rng.integers(1, 12))
            cut = [max(1, len(s) - k) for s in seqs]
            slots = [eng.new_sequence() for _ in seqs]
            eng.step(slots, [s[:c] for s, c in zip(seqs, cut)], [[] for _ in seqs])
            for j in range(k):
                live = [i for i, (s, c) in enumerate(zip(seqs, cut)) if c + j < len(s)]
                if not live:
                    break
                got = eng.step([slots[i] for i in live], [[seqs[i][cut[i] + j]] for i in live], "last")
                compare(got, [(i, cut[i] + j) for i in live], f"single tokens, step {j}")
                for r, i in enumerate(live):
                    assert not exact or torch.equal(got[r], whole[first_row[i] + cut[i] + j]), \
                        f"float32 bits of position {cut[i] + j} of sequence {i} differ between a single-token step and the whole prompt; {what}"
            for s in slots:
                eng.release(s)
            slots = [eng.new_sequence() for _ in seqs]
            pos = [0] * len(seqs)
            while any(p < len(s) for p, s in zip(pos, seqs)):
                live = [i for i in range(len(seqs)) if pos[i] < len(seqs[i])]
                toks = [seqs[i][pos[i]:pos[i] + int(rng.integers(1, 30))] for i in live]
                got = eng.step([slots[i] for i in live], toks, "all")
                compare(got, [(i, pos[i] + p) for i, t in zip(live, toks) for p in range(len(t))], f"portions from {pos}")
                r = 0
                for i, t in zip(live, toks):
                    at = first_row[i] + pos[i]
                    assert not exact or torch.equal(got[r:r + len(t)], whole[at:at + len(t)]), \
                        f"float32 bits of a portion of {len(t)} at position {pos[i]} of sequence {i} differ from the whole prompt; {what}"
                    r += len(t)
                    pos[i] += len(t)
            for s in slots:
                eng.release(s)
            eng.check_status()
