#!/usr/bin/env python3
"""Decode and prefill throughput of the Gemma-2-2B-shaped model with random weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl reference]

Prints ONE JSON line.  `value` is decoded tokens per second at batch 8 (device-timed with CUDA
events around exactly K single-token steps after W warm-up steps, from 2,048-token prompts, cache
sized for the context length of 8,192).  `e2e` is the same through the Python entry point
(`Generator.generate_batch`): host token lists in, host token lists out, every step copying its
batch description from pinned host memory and reading the sampled tokens back.  `prefill` is one
2,048-token prompt in one step; `points` holds decode at batch 1 and 64; `roofline` compares the
bytes a decode step must read (every weight once, the cache of the live requests) with its time.
A decode step reads 5.2 GB of weights, far more than the 126 MB L2, so nothing stays cached
between timed iterations.
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# the Gemma 2 2B shape
GEMMA2_2B = {
    "architectures": ["Gemma2ForCausalLM"], "model_type": "gemma2",
    "num_hidden_layers": 26, "hidden_size": 2304, "num_attention_heads": 8, "num_key_value_heads": 4,
    "head_dim": 256, "intermediate_size": 9216, "vocab_size": 256000, "rms_norm_eps": 1e-6,
    "rope_theta": 10000.0, "sliding_window": 4096, "query_pre_attn_scalar": 256,
    "attn_logit_softcapping": 50.0, "final_logit_softcapping": 30.0, "max_position_embeddings": 8192,
    "hidden_activation": "gelu_pytorch_tanh", "tie_word_embeddings": True, "bos_token_id": 2, "eos_token_id": 1,
}
# BASELINE.json configs[3] and [4]: the 9B and 27B shapes
GEMMA2_9B = dict(GEMMA2_2B, num_hidden_layers=42, hidden_size=3584, num_attention_heads=16, num_key_value_heads=8,
                 head_dim=256, intermediate_size=14336, query_pre_attn_scalar=256)
GEMMA2_27B = dict(GEMMA2_2B, num_hidden_layers=46, hidden_size=4608, num_attention_heads=32, num_key_value_heads=16,
                  head_dim=128, intermediate_size=36864, query_pre_attn_scalar=144)
CONTEXT = 8192
PROMPT = 2048
NEW_TOKENS = 128
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                d = json.load(f)
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
        except (ValueError, KeyError, TypeError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """nvidia-smi clocks and throttle reasons every 200 ms while the timed regions run."""
    FIELDS = ["clocks.sm", "clocks.max.sm", "power.draw", "clocks_event_reasons.hw_slowdown",
              "clocks_event_reasons.hw_thermal_slowdown", "clocks_event_reasons.sw_thermal_slowdown",
              "clocks_event_reasons.sw_power_cap"]

    def __init__(self):
        self.proc, self.lines = None, []

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", "--query-gpu=" + ",".join(self.FIELDS),
                                          "--format=csv,noheader,nounits", "-lms", "200"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, mx, reasons = [], [], set()
        for line in self.lines:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) != len(self.FIELDS):
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for name, val in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), parts[3:]):
                if val == "Active":
                    reasons.add(name)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm)}


def weight_bytes(spec, element_size=2):
    total = 0
    for t in spec.tensor_specs().values():
        n = 1
        for s in t.shape:
            n *= s
        total += n * element_size
    return total


def cache_bytes_read(cfg, layers, lengths, element_size=2):
    """Bytes of keys and values a decode step reads for sequences of the given lengths."""
    per_key = 2 * cfg["num_key_value_heads"] * cfg["head_dim"] * element_size
    total = 0
    for i in range(layers):
        local = cfg["sliding_window"] is not None and i % 2 == 0
        for n in lengths:
            total += per_key * (min(n, cfg["sliding_window"]) if local else n)
    return total


def prefill_flops(cfg, layers, T):
    H, nh, nkv, hd, I, V = (cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"],
                            cfg["head_dim"], cfg["intermediate_size"], cfg["vocab_size"])
    linear = 2 * T * (H * (nh + 2 * nkv) * hd + nh * hd * H + 3 * H * I) * layers
    attn = 0
    for i in range(layers):
        local = cfg["sliding_window"] is not None and i % 2 == 0
        keys = sum(min(p + 1, cfg["sliding_window"]) if local else p + 1 for p in range(T))
        attn += 4 * nh * hd * keys
    return linear + attn + 2 * V * H      # logits at the last row only


def decode_run(engine, batch, steps, warmup, vocab, torch, rng, prompt_len=PROMPT):
    """Prefill `batch` prompts of `prompt_len` tokens, then time `steps` single-token steps on the device."""
    slots = [engine.new_sequence() for _ in range(batch)]
    prompts = [[int(v) for v in rng.integers(0, vocab, size=prompt_len)] for _ in range(batch)]
    engine.step(slots, prompts, [[] for _ in slots])
    feed = [[[int(v)] for v in rng.integers(0, vocab, size=batch)] for _ in range(steps + warmup)]
    from rust_deeplearning_b200.kernels import library
    for k in range(warmup):
        engine.step(slots, feed[k], "last")
    torch.cuda.synchronize()
    launches0 = library.launch_count
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for k in range(warmup, warmup + steps):
        engine.step(slots, feed[k], "last")
    stop.record()
    torch.cuda.synchronize()
    ms = start.elapsed_time(stop) / steps
    launches = library.launch_count - launches0
    lengths = [engine.length(s) for s in slots]
    for s in slots:
        engine.release(s)
    mid = [n - steps // 2 for n in lengths]
    return ms, launches, mid


def spread(lo, hi, n):
    """n prompt lengths from lo to hi in equal steps."""
    return [lo + (hi - lo) * i // (n - 1) for i in range(n)]


def workload(cfg, prompt_lens, new_tokens, pk, torch, rng, seed=0):
    """One of the larger shapes end to end on the engine: all prompts in one step (device-timed), then
    `new_tokens` single-token steps; the steps around the middle of the run are timed on the device.
    Returns a flat dict of figures."""
    import gc
    from rust_deeplearning_b200 import Engine, random_model
    from rust_deeplearning_b200.config.base import architecture_for
    torch.cuda.empty_cache()
    torch.cuda.reset_peak_memory_stats()
    model = random_model(cfg, seed=seed, dtype="bfloat16", device="cuda:0")
    torch.cuda.synchronize()
    load_peak = torch.cuda.max_memory_allocated()
    arch = architecture_for(cfg)
    wbytes = weight_bytes(arch.build_spec(arch.parse_config(cfg)))
    V, L = cfg["vocab_size"], cfg["num_hidden_layers"]
    longest = max(prompt_lens) + new_tokens
    per_seq = [-(-(n + new_tokens) // 64) * 64 for n in prompt_lens]
    engine = Engine(model, max_tokens=sum(per_seq), max_seqs=len(prompt_lens), max_context=-(-longest // 64) * 64)
    prompts = [[int(v) for v in rng.integers(0, V, size=n)] for n in prompt_lens]
    slots = [engine.new_sequence() for _ in prompts]
    ev = lambda: torch.cuda.Event(enable_timing=True)
    p0, p1 = ev(), ev()
    torch.cuda.synchronize()
    p0.record()
    engine.step(slots, prompts, "last")
    p1.record()
    torch.cuda.synchronize()
    prefill_ms = p0.elapsed_time(p1)
    first = max(3, new_tokens // 2 - 10)             # the timed steps lie around the middle of the run
    timed = min(20, new_tokens - 1 - first)
    feed = rng.integers(0, V, size=(new_tokens - 1, len(prompts)))
    t0, t1 = ev(), ev()
    for k in range(new_tokens - 1):
        if k == first:
            t0.record()
        if k == first + timed:
            t1.record()
        engine.step(slots, [[int(v)] for v in feed[k]], "last")
    if first + timed >= new_tokens - 1:
        t1.record()
    torch.cuda.synchronize()
    engine.check_status()
    ms = t0.elapsed_time(t1) / timed
    mid = [n + first + timed // 2 for n in prompt_lens]
    step_bytes = wbytes + cache_bytes_read(cfg, L, mid)
    out = {"layers": L, "prompts": f"{len(prompt_lens)} of {min(prompt_lens)}..{max(prompt_lens)} tokens", "new_tokens": new_tokens,
           "decode_tok_s": round(len(prompts) / (ms * 1e-3), 1), "decode_ms_per_step": round(ms, 3),
           "decode_step_gb": round(step_bytes / 1e9, 2),
           "decode_hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4),
           "prefill_tokens": sum(prompt_lens), "prefill_ms": round(prefill_ms, 1),
           "prefill_tok_s": round(sum(prompt_lens) / (prefill_ms * 1e-3), 1),
           "weights_gb": round(wbytes / 1e9, 2), "load_peak_gb": round(load_peak / 1e9, 2),
           "cache_gb": round(engine.cache.nbytes() / 1e9, 2)}
    for s in slots:
        engine.release(s)
    del engine, model
    gc.collect()
    torch.cuda.empty_cache()
    return out


# ---- a second design beside its closest registered model, at equal layer sizes (--design ligirax) ----

def ligirax_shape(width, heads, dim, rot_dim, vdim, kv_rank, window, experts, identity, top, ff, layers, vocab, shared_from=None):
    """A Ligirax configuration of `layers` equal layers (the later half reading the rows of layer `shared_from` if given)."""
    rot = {"base": 10000.0, "dims": rot_dim, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    out = []
    for i in range(layers):
        m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": (dim + rot_dim) ** -0.5,
             "rot": rot, "mask": {"size": window}}
        if shared_from is not None and i > shared_from:
            m["kv_from"] = shared_from
        out.append({"type": "latent_attention", "mixer": m,
                    "mlp": {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "router": {"experts": experts, "identity": identity, "top": top}}})
    return {"architecture": "Ligirax", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "logit_scale": 1.0,
            "max_positions": CONTEXT, "layers": out}


def gemma_like(width, heads, head_dim, intermediate, window, layers, vocab, kv_heads=None):
    """The Gemma 2 configuration with the same width, head count and window, whose feed-forward is as wide as the
    experts a Ligirax token uses (as wide as Dokulorn's dense feed-forward)."""
    return dict(GEMMA2_2B, num_hidden_layers=layers, hidden_size=width, num_attention_heads=heads,
                num_key_value_heads=kv_heads or heads, head_dim=head_dim, intermediate_size=intermediate, vocab_size=vocab,
                sliding_window=window, query_pre_attn_scalar=head_dim, max_position_embeddings=CONTEXT)


def dokulorn_shape(width, heads, kv_heads, dim, ff, layers, vocab):
    """A Dokulorn configuration of `layers` layers, each with a dense feed-forward: retention layers, and every fourth
    layer a pair (softmax attention with grouped key/value heads beside lightning attention)."""
    decay = [1.0 - 2.0 ** (-5 - 5 * h / max(heads - 1, 1)) for h in range(heads)]
    ret = {"heads": heads, "dim": dim, "vdim": dim, "decay": decay, "rot": {"base": 1e6, "dims": dim}}
    par = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"base": 1e4, "dims": dim // 2},
                    "scale": 1.0, "softcap": 20.0},
           "right": {"heads": heads, "dim": dim, "vdim": dim, "decay": decay}}
    out = [{"type": "parallel" if i % 4 == 3 else "retention", "mixer": par if i % 4 == 3 else ret, "mlp": {"kind": "dense", "ff": ff}}
           for i in range(layers)]
    return {"architecture": "Dokulorn", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "postln_alpha": 2.0,
            "embedding": {"scale": 10.0}, "max_positions": CONTEXT, "layers": out}


def revepel_shape(width, ssm_heads, state, heads, kv_heads, dim, window, experts, top, ff, shared_ff, layers, vocab, rank=64):
    """A Revepel configuration of `layers` layers in the order state space, delta rule, attention, attention on the keys of
    the layer before it; every layer with routed two-matrix experts and a shared one."""
    rot = {"base": 10000.0, "dims": dim, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared_ff}}
    out = []
    for i in range(layers):
        kind = i % 4
        if kind == 0:
            layer = {"type": "mamba2", "mixer": {"heads": ssm_heads, "vdim": width // ssm_heads, "state": state, "groups": 1, "norm_groups": 1, "conv": 4}}
        elif kind == 1:
            layer = {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": heads, "dim": dim, "vdim": dim, "conv": 4,
                                                        "decay_rank": rank, "gate_rank": rank}}
        else:
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window}, "rot": rot}
            if kind == 3:
                m["kv_from"] = i - 1
            layer = {"type": "attention", "mixer": m}
        out.append(dict(layer, mlp=mlp))
    return {"architecture": "Revepel", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": 10.0}, "logit_scale": 1.0,
            "max_positions": CONTEXT, "layers": out}


def gasetar_shape(width, heads, kv_heads, dim, window, latent_heads, latent_dim, rot_dim, vdim, kv_rank, experts, top, ff, shared_ff,
                  dense_ff, vocab, layers=4):
    """A Gasetar configuration of four layers: window attention with a dense feed-forward, latent attention with routed
    experts, and two window-attention layers with routed experts (each with a shared expert)."""
    rot = {"base": 100000.0, "dims": dim * 3 // 4, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": 50.0, "mask": {"size": window}, "rot": rot}
    latent = {"heads": latent_heads, "dim": latent_dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
              "scale": (latent_dim + rot_dim) ** -0.5, "rot": {"base": 10000.0, "dims": rot_dim}}
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared_ff}}
    order = [("attention", attn, {"kind": "dense", "ff": dense_ff}), ("latent_attention", latent, moe), ("attention", attn, moe), ("attention", attn, moe)]
    return {"architecture": "Gasetar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
            "residual_mult": 0.5, "logit_scale": 1.0, "logit_softcap": 30.0, "max_positions": CONTEXT,
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in order[:layers]]}


def kitonex_shape(width, heads, kv_heads, dim, chunk, bias_max, streams, experts, top, groups, keep, ff, shared_ff, dense_ff, vocab, layers=4):
    """A Kitonex configuration of four layers, chunked attention with a dense feed-forward and with routed experts in turn (in
    groups, with a gated shared expert), four taps, 32 distance buckets."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "conv": 4, "mask": {"size": chunk},
            "bias_max": bias_max, "bias_buckets": 32, "v_mix": True}
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}},
           "shared": {"ff": shared_ff}}
    return {"architecture": "Kitonex", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "streams": streams, "max_positions": CONTEXT,
            "layers": [{"type": "attention", "mixer": attn, "mlp": moe if i % 2 else {"kind": "dense", "ff": dense_ff, "limit": 7.0}} for i in range(layers)]}


def gasetar_window_shape(width, heads, kv_heads, dim, window, experts, top, ff, shared_ff, dense_ff, vocab, layers=4):
    """A Gasetar configuration of window-attention layers alone, with a dense feed-forward and with routed experts in turn."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window},
            "rot": {"base": 100000.0, "dims": dim}}
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared_ff}}
    return {"architecture": "Gasetar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
            "residual_mult": 0.5, "max_positions": CONTEXT,
            "layers": [{"type": "attention", "mixer": attn, "mlp": moe if i % 2 else {"kind": "dense", "ff": dense_ff}} for i in range(layers)]}


def paditar_shape(width, heads, kv_heads, dim, ff, vocab, times=2):
    """A Paditar configuration of four layers - two pairs (attention beside a matrix memory) that run `times` times, differential
    attention (two maps of half a head each), a pair - each with a dense feed-forward."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "conv": 4, "q_temp": {"coef": 0.1, "every": 4096}}
    pair = {"type": "parallel", "mixer": {"left": left, "right": {"heads": heads, "dim": dim, "vdim": dim, "gate_cap": 15.0}, "left_scale": 0.7, "right_scale": 0.7}}
    diff = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim // 2, "vdim": dim, "scale": (dim // 2) ** -0.5,
                                           "diff": 0.3, "rot": {"base": 1e4, "dims": dim // 2}}}
    return {"architecture": "Paditar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": times},
            "max_positions": CONTEXT, "layers": [dict(l, mlp={"kind": "dense", "ff": ff}) for l in (pair, pair, diff, pair)]}


def dokulorn_pairs_shape(width, heads, kv_heads, dim, ff, vocab, times=2):
    """The Dokulorn configuration with as many layers as a Paditar one runs: pairs (softmax attention beside lightning attention)
    where that one has pairs, a retention layer where it has differential attention."""
    cfg = dokulorn_shape(width, heads, kv_heads, dim, ff, 4, vocab)
    ret, pair = cfg["layers"][0], cfg["layers"][3]
    cfg["layers"] = [pair] * (2 * times) + [ret, pair]
    return cfg


DESIGN_SIZES = {
    # name: (the design's arguments, the Gemma 2 arguments of equal width / heads / active feed-forward width)
    "w1024": (dict(width=1024, heads=8, dim=64, rot_dim=64, vdim=128, kv_rank=192, window=1024, experts=16, identity=2, top=2, ff=1024,
                   layers=4, vocab=32000, shared_from=1),
              dict(width=1024, heads=8, head_dim=128, intermediate=2048, window=1024, layers=4, vocab=32000)),
    "w2048": (dict(width=2048, heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=4096, experts=64, identity=2, top=6, ff=1408,
                   layers=4, vocab=32000),
              dict(width=2048, heads=16, head_dim=128, intermediate=8448, window=4096, layers=4, vocab=32000)),
}
DOKULORN_SIZES = {
    # four layers each: three retention layers and a pair, all with a dense feed-forward; Gemma 2 with the same width,
    # heads, head size and feed-forward width (its windows as long as the context: all keys are read)
    "w1024": (dict(width=1024, heads=8, kv_heads=4, dim=128, ff=4096, layers=4, vocab=32000),
              dict(width=1024, heads=8, kv_heads=4, head_dim=128, intermediate=4096, window=CONTEXT, layers=4, vocab=32000)),
    "w2048": (dict(width=2048, heads=16, kv_heads=8, dim=128, ff=8192, layers=4, vocab=32000),
              dict(width=2048, heads=16, kv_heads=8, head_dim=128, intermediate=8192, window=CONTEXT, layers=4, vocab=32000)),
}
REVEPEL_SIZES = {
    # four layers each (state space, delta rule, attention, attention on shared keys), every layer with routed experts whose
    # active width (top x ff + shared) is Dokulorn's dense width; Dokulorn, the closest registered design (state of fixed size
    # beside keys and values), with the same width, heads, head size and feed-forward width
    "w1024": (dict(width=1024, ssm_heads=16, state=128, heads=8, kv_heads=4, dim=128, window=1024, experts=16, top=2, ff=1024,
                   shared_ff=2048, layers=4, vocab=32000),
              dict(width=1024, heads=8, kv_heads=4, dim=128, ff=4096, layers=4, vocab=32000)),
    "w2048": (dict(width=2048, ssm_heads=32, state=128, heads=16, kv_heads=8, dim=128, window=4096, experts=32, top=4, ff=1024,
                   shared_ff=4096, layers=4, vocab=32000),
              dict(width=2048, heads=16, kv_heads=8, dim=128, ff=8192, layers=4, vocab=32000)),
}
GASETAR_SIZES = {
    # four layers each (window attention + dense, latent attention + experts, two of window attention + experts); Gemma 2 with
    # the same width, heads, key heads, head size and window, and a feed-forward as wide as the experts a token uses (top x ff + shared)
    "w1024": (dict(width=1024, heads=8, kv_heads=2, dim=128, window=1024, latent_heads=8, latent_dim=64, rot_dim=64, vdim=128, kv_rank=192,
                   experts=32, top=4, ff=384, shared_ff=512, dense_ff=2048, vocab=32000),
              dict(width=1024, heads=8, kv_heads=2, head_dim=128, intermediate=2048, window=1024, layers=4, vocab=32000)),
    "w2048": (dict(width=2048, heads=16, kv_heads=8, dim=128, window=4096, latent_heads=16, latent_dim=128, rot_dim=64, vdim=128, kv_rank=512,
                   experts=64, top=6, ff=1024, shared_ff=2304, dense_ff=8448, vocab=32000),
              dict(width=2048, heads=16, kv_heads=8, head_dim=128, intermediate=8448, window=4096, layers=4, vocab=32000)),
}
KITONEX_SIZES = {
    # four layers each, attention with a dense feed-forward and with routed experts in turn; Gasetar, the closest registered
    # design (norms over the whole projections, routed experts beside a shared one), with window attention in every layer and the
    # same width, heads, key heads, head size, experts and feed-forward widths, its window as long as Kitonex's chunk
    "w1024": (dict(width=1024, heads=8, kv_heads=2, dim=128, chunk=1024, bias_max=1024, streams=2, experts=32, top=4, groups=8, keep=4, ff=384,
                   shared_ff=512, dense_ff=2048, vocab=32000),
              dict(width=1024, heads=8, kv_heads=2, dim=128, window=1024, experts=32, top=4, ff=384, shared_ff=512, dense_ff=2048, vocab=32000)),
    "w2048": (dict(width=2048, heads=16, kv_heads=8, dim=128, chunk=4096, bias_max=128, streams=4, experts=64, top=6, groups=8, keep=4, ff=1024,
                   shared_ff=2304, dense_ff=8448, vocab=32000),
              dict(width=2048, heads=16, kv_heads=8, dim=128, window=4096, experts=64, top=6, ff=1024, shared_ff=2304, dense_ff=8448, vocab=32000)),
}
PADITAR_SIZES = {
    # four layers, six runs; Dokulorn, the closest registered design (softmax attention beside a recurrence with a state of fixed
    # size in one layer), with six layers, the same width, heads, key heads and head size, and feed-forwards of equal size
    # (three matrices of two thirds the width)
    "w1024": (dict(width=1024, heads=8, kv_heads=4, dim=128, ff=4608, vocab=32000),
              dict(width=1024, heads=8, kv_heads=4, dim=128, ff=3072, vocab=32000)),
    "w2048": (dict(width=2048, heads=16, kv_heads=8, dim=128, ff=9216, vocab=32000),
              dict(width=2048, heads=16, kv_heads=8, dim=128, ff=6144, vocab=32000)),
}
# design -> (its shape, its sizes, the title, the registered design it stands beside and that design's shape)
DESIGNS = {"ligirax": (ligirax_shape, DESIGN_SIZES, "ligirax beside gemma2 at equal width, heads and active feed-forward width", "gemma2", gemma_like),
           "dokulorn": (dokulorn_shape, DOKULORN_SIZES, "dokulorn beside gemma2 at equal width, heads, head size and feed-forward width", "gemma2",
                        gemma_like),
           "gasetar": (gasetar_shape, GASETAR_SIZES, "gasetar beside gemma2 at equal width, heads, key heads, head size, window and active feed-forward width",
                       "gemma2", gemma_like),
           "kitonex": (kitonex_shape, KITONEX_SIZES, "kitonex beside gasetar at equal width, heads, key heads, head size, window (chunk), experts and feed-forward widths",
                       "gasetar", gasetar_window_shape),
           "paditar": (paditar_shape, PADITAR_SIZES, "paditar beside dokulorn at equal runs, width, heads, key heads, head size and feed-forward size",
                       "dokulorn", dokulorn_pairs_shape),
           "revepel": (revepel_shape, REVEPEL_SIZES, "revepel beside dokulorn at equal width, heads, head size and active feed-forward width",
                       "dokulorn", dokulorn_shape)}


def design_point(cfg, vocab, torch, rng, steps, warmup, prompt_len, batches, long_prompt=CONTEXT):
    """Prefill tokens/s (one prompt in one step, median of 5 after 3; and one long prompt, median of 3 after 1) and decode
    tokens/s at each batch."""
    import gc
    from rust_deeplearning_b200 import Engine, random_model
    from rust_deeplearning_b200.kernels import library
    model = random_model(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    engine = Engine(model, max_tokens=max(batches) * (prompt_len + 256), max_seqs=max(batches), max_context=max(prompt_len + 256, long_prompt))
    prompt = [int(v) for v in rng.integers(0, vocab, size=prompt_len)]
    times = []
    launches = 0
    for k in range(8):
        slot = engine.new_sequence()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        before = library.launch_count
        start.record()
        engine.step([slot], [prompt], "last")
        stop.record()
        torch.cuda.synchronize()
        launches = library.launch_count - before
        engine.release(slot)
        if k >= 3:
            times.append(start.elapsed_time(stop))
    out = {"prefill_tokens": prompt_len, "prefill_ms": round(statistics.median(times), 3),
           "prefill_tok_s": round(prompt_len / (statistics.median(times) * 1e-3), 1), "prefill_launches": launches}
    long_ids = [int(v) for v in rng.integers(0, vocab, size=long_prompt)]
    times = []
    for k in range(4):
        slot = engine.new_sequence()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        engine.step([slot], [long_ids], "last")
        stop.record()
        torch.cuda.synchronize()
        engine.release(slot)
        if k >= 1:
            times.append(start.elapsed_time(stop))
    out["prefill_long_tokens"] = long_prompt
    out["prefill_long_ms"] = round(statistics.median(times), 3)
    out["prefill_long_tok_s"] = round(long_prompt / (statistics.median(times) * 1e-3), 1)
    for b in batches:
        ms, n_launch, _ = decode_run(engine, b, steps, warmup, vocab, torch, rng, prompt_len)
        out[f"decode_b{b}_ms"] = round(ms, 4)
        out[f"decode_b{b}_tok_s"] = round(b / (ms * 1e-3), 1)
        out[f"decode_b{b}_launches_per_step"] = n_launch // steps
    engine.check_status()
    del engine, model
    gc.collect()
    torch.cuda.empty_cache()
    return out


def design_comparison(args):
    import numpy as np
    import torch
    torch.cuda.set_device(0)
    rng = np.random.default_rng(0)
    clocks = ClockSampler()
    clocks.start()
    sizes = {}
    shape_of, table, title, beside, beside_shape = DESIGNS[args.design]
    for name, (lig, gem) in table.items():
        if args.size and name != args.size:
            continue
        sizes[name] = {
            args.design: design_point(shape_of(**lig), lig["vocab"], torch, rng, min(args.steps, 50), args.warmup, PROMPT, (1, 8, 64)),
            beside: design_point(beside_shape(**gem), gem["vocab"], torch, rng, min(args.steps, 50), args.warmup, PROMPT, (1, 8, 64)),
            "shapes": {args.design: lig, beside: gem}}
    print(json.dumps({"design": title, "dtype": "bf16",
                      "data": "synthetic: random weights, seeded uniform-random token ids", "prompt_len": PROMPT,
                      "sizes": sizes, "clocks": clocks.stop(), "peaks": peaks()}))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=100)
    ap.add_argument("--warmup", type=int, default=10)
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the configuration has")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--only", choices=["decode", "prefill"], default=None,
                    help="run one small case (for profiling) and print a short line instead of the full record")
    ap.add_argument("--batch", type=int, default=8, help="batch of the --only decode case")
    ap.add_argument("--context", type=int, default=PROMPT, help="prompt length of the --only decode case")
    ap.add_argument("--no-large", action="store_true", help="leave out the 9B and 27B shapes and the long contexts")
    ap.add_argument("--design", choices=["ligirax", "dokulorn", "revepel", "gasetar", "kitonex", "paditar"], default=None,
                    help="instead of the default workload: prefill and decode of this design beside its closest registered design "
                         "(Gemma 2; for revepel, Dokulorn; for kitonex, Gasetar) at equal layer sizes")
    ap.add_argument("--size", default=None, help="with --design: one of the sizes only")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference is a Rust workspace (no Python package, no GPU code); no cargo/rustc in this image, "
                          "pip install of the reference tree fails: neither setup.py nor pyproject.toml"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this library is single-GPU by design (got --gpus {args.gpus})")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.design is not None:
        return design_comparison(args)
    if args.steps + args.warmup > NEW_TOKENS - 1:
        args.steps = NEW_TOKENS - 1 - args.warmup

    import numpy as np
    import torch
    from rust_deeplearning_b200 import Engine, Generator, random_model
    from rust_deeplearning_b200.config.base import architecture_for
    from rust_deeplearning_b200.kernels import library

    cfg = dict(GEMMA2_2B)
    full_layers = cfg["num_hidden_layers"]
    layers = args.layers or full_layers
    cfg["num_hidden_layers"] = layers
    pk = peaks()
    rng = np.random.default_rng(0)
    torch.cuda.set_device(0)
    model = random_model(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    arch = architecture_for(cfg)
    spec = arch.build_spec(arch.parse_config(cfg))
    wbytes = weight_bytes(spec)
    V = cfg["vocab_size"]

    if args.only is not None:
        # one case, few steps: what a profiler is pointed at
        engine = Engine(model, max_tokens=args.batch * CONTEXT, max_seqs=args.batch, max_context=CONTEXT)
        if args.only == "decode":
            ms, launches, _ = decode_run(engine, args.batch, args.steps, args.warmup, V, torch, rng, args.context)
            print(json.dumps({"case": "decode", "batch": args.batch, "context": args.context, "layers": layers, "ms_per_step": round(ms, 4),
                              "tokens_per_s": round(args.batch / (ms * 1e-3), 1), "launches": launches}))
        else:
            prompt = [int(v) for v in rng.integers(0, V, size=PROMPT)]
            for _ in range(args.warmup + args.steps):
                slot = engine.new_sequence()
                start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                t0 = time.perf_counter()
                start.record()
                engine.step([slot], [prompt], "last")
                stop.record()
                host_ms = (time.perf_counter() - t0) * 1e3     # the host's share: validation, batch description, launches
                torch.cuda.synchronize()
                engine.release(slot)
            print(json.dumps({"case": "prefill", "tokens": PROMPT, "layers": layers, "ms": round(start.elapsed_time(stop), 3),
                              "host_ms": round(host_ms, 3)}))
        return 0

    clocks = ClockSampler()
    clocks.start()

    # ---- decode, device-timed: batch 8 (the headline), 1 and 64 ----
    engine = Engine(model, max_tokens=64 * CONTEXT, max_seqs=64, max_context=CONTEXT)
    ms8, launches, mid8 = decode_run(engine, 8, args.steps, args.warmup, V, torch, rng)
    # ---- end to end through the Python entry point: host tokens in and out ----
    # (right after the device-timed run of the same batch, so that both see the same clocks)
    gen = Generator(model, max_cache_tokens=8 * CONTEXT, max_batch=8, max_context=CONTEXT).with_temperature(0.0)
    gen.with_stop_tokens([])
    prompts = [[int(v) for v in rng.integers(0, V, size=PROMPT)] for _ in range(8)]
    marks = {}
    count = [0]
    first, last = 8 * args.warmup, 8 * (args.warmup + args.steps)

    def on_token(_req, _tok):
        count[0] += 1
        if count[0] == first:
            marks["t0"] = time.perf_counter()
        elif count[0] == last:
            marks["t1"] = time.perf_counter()

    gen.generate_batch_results(prompts, args.warmup + args.steps + 1, stream=on_token)
    e2e_tps = 8 * args.steps / (marks["t1"] - marks["t0"])
    h2d = next(iter(gen.engine._graphs.values())).layout.size * 4 if gen.engine._graphs else 0
    del gen
    torch.cuda.empty_cache()

    side = min(args.steps, 50)
    ms1, _, _ = decode_run(engine, 1, side, args.warmup, V, torch, rng)
    ms64, _, mid64 = decode_run(engine, 64, side, args.warmup, V, torch, rng)

    # ---- prefill: one prompt of 2,048 tokens in one step ----
    prompt = [int(v) for v in rng.integers(0, V, size=PROMPT)]
    times = []
    for k in range(3 + 5):
        slot = engine.new_sequence()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        engine.step([slot], [prompt], "last")
        stop.record()
        torch.cuda.synchronize()
        engine.release(slot)
        if k >= 3:
            times.append(start.elapsed_time(stop))
    prefill_ms = statistics.median(times)
    pflops = prefill_flops(cfg, layers, PROMPT)

    # ---- long contexts on the same model: decode above the window (the windowed layers' ring is in use), a long prompt ----
    long_points = {}
    if not args.no_large:
        LONG = 6000
        for b in (1, 8):
            ms, _, mid = decode_run(engine, b, 20, 3, V, torch, rng, LONG)
            long_points[f"decode_b{b}_ctx{LONG}"] = round(b / (ms * 1e-3), 1)
            long_points[f"decode_b{b}_ctx{LONG}_hbm_frac"] = round((wbytes + cache_bytes_read(cfg, layers, mid)) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
        long_prompt = [int(v) for v in rng.integers(0, V, size=CONTEXT)]
        times8k = []
        for k in range(3):
            slot = engine.new_sequence()
            start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            start.record()
            engine.step([slot], [long_prompt], "last")
            stop.record()
            torch.cuda.synchronize()
            engine.release(slot)
            if k >= 1:
                times8k.append(start.elapsed_time(stop))
        ms8k = statistics.median(times8k)
        long_points[f"prefill_{CONTEXT}_tok_s"] = round(CONTEXT / (ms8k * 1e-3), 1)
        long_points[f"prefill_{CONTEXT}_frac"] = round(prefill_flops(cfg, layers, CONTEXT) / (ms8k * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)

    # ---- the larger shapes of the reference's list: 9B (8 unequal prompts, 256 new) and 27B (16 prompts, 128 new) ----
    large = {}
    if not args.no_large and args.layers is None:
        del engine, model
        import gc
        gc.collect()
        torch.cuda.empty_cache()
        for name, shape, lens, new in (("gemma2_9b", GEMMA2_9B, spread(64, 6000, 8), 256),
                                       ("gemma2_27b", GEMMA2_27B, spread(1024, 4096, 16), 128)):
            try:
                large[name] = workload(shape, lens, new, pk, torch, rng)
            except Exception as e:      # the headline above stands whatever becomes of the larger shapes
                large[name] = {"error": f"{type(e).__name__}: {e}"[:200]}
                gc.collect()
                torch.cuda.empty_cache()
    clock_info = clocks.stop()

    step_bytes = wbytes + cache_bytes_read(cfg, layers, mid8)
    achieved = step_bytes / (ms8 * 1e-3) / 1e9
    value = 8 / (ms8 * 1e-3)
    out = {
        "metric": "Gemma2-2B decode tok/s @ batch 8 (prefill tok/s @ 2,048 tokens and batch 1/64 alongside)",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms8, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: random weights N(0, 0.02), seeded uniform-random token ids",
        "config": {
            "model": "Gemma 2 2B shape", "layers": layers, "layers_in_configuration": full_layers,
            "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
            "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"], "vocab": V,
            "sliding_window": cfg["sliding_window"], "global_batch": 8, "seq_len": CONTEXT, "prompt_len": PROMPT,
            "new_tokens": NEW_TOKENS, "parallelism": "single GPU", "cache": "paged, 64 positions a page, sized for 8192 a sequence",
            "l2": "inputs larger than L2: 5.2 GB of weights read per step",
            "points_long": "2B shape: decode at batch 1 and 8 from 6000-token prompts, one prompt of 8192 tokens",
            "points_9b": "42 layers, hidden 3584, 16/8 heads, head 256, intermediate 14336; 8 prompts 64..6000, 256 new",
            "points_27b": "46 layers, hidden 4608, 32/16 heads, head 128, intermediate 36864; 16 prompts 1024..4096, 128 new",
        },
        "clocks": clock_info,
        "e2e": {"value": round(e2e_tps, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 8 * 4},
        "gpu_launches": launches,
        "prefill": {"value": round(PROMPT / (prefill_ms * 1e-3), 1), "tokens": PROMPT, "ms": round(prefill_ms, 3),
                    "frac": round(pflops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peaks": pk["source"]},
        "points": {"decode_b1": round(1 / (ms1 * 1e-3), 1), "decode_b64": round(64 / (ms64 * 1e-3), 1),
                   "decode_b64_hbm_frac": round((wbytes + cache_bytes_read(cfg, layers, mid64)) / (ms64 * 1e-3) / 1e9
                                                / pk["hbm_gbs"], 4),
                   "decode_b1_hbm_frac": round((wbytes + cache_bytes_read(cfg, layers, [PROMPT + NEW_TOKENS // 2])) / (ms1 * 1e-3) / 1e9
                                               / pk["hbm_gbs"], 4)},
    }
    out["points"].update(long_points)
    for name, figures in large.items():
        for k, v in figures.items():
            out["points"][f"{name}_{k}"] = v
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
