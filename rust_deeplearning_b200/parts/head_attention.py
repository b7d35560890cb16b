"""Attention whose projections are treated head by head, with optionally several softmaxes per head.

Grouped-query attention over the paged cache (every earlier position is seen), with what lies between the q/k/v product and the
attention kernel done in one pass (`ops.head_prepare`) and what lies between attention and the output product in another
(`ops.context_finish`).  Parameters and tensor roles, all optional beyond the sizes:

  (biases)       tensor roles "q_bias", "k_bias": added to the projections; "o_bias": added to the output product
  (convolution)  a causal convolution over time on every channel of q and k, directly after the projections (tensor roles
                 "q_conv", "k_conv", [channels, taps]); the last taps - 1 projected values are state per sequence
  values_from_keys   there is no W_v: the values are the keys as they leave the convolution (before any norm)
  head_norm_eps  every query and key head is divided by its root mean square and multiplied by a weight of the head's size that
                 all heads share (tensor roles "q_norm", "k_norm" [head_dim]), in float
  position       rotary positions on q and k (half-split pairs)
  q_temperature  {"coef", "every"}: q is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at position p
  off_by_one     one joins the softmax's denominator: a sink whose logit is 0, for every head
  differential   {"diff", "eps"}: differential attention ("Differential Transformer", Ye et al.).  Every query and key head has
                 two maps of head_dim values: two softmaxes that weight one set of values;
                 o = a_1 - lambda a_2, lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff (tensor roles "lq1", "lk1", "lq2", "lk2"
                 [head_dim], all heads share it); every head of o is normed to a root mean square of 1 - diff
  gate           "value": the concatenated heads are multiplied element by element by sigmoid(W_g x) before W_o;
                 "head": every head by one number, sigmoid(W_g x)_h
  value_dim      values of another size than keys

The two maps of a key head lie side by side in one cache row and a query map is laid out with zeros under the other one
(`csrc/head_prepare.cu`), so that the attention kernels see twice the query heads on the same key heads and read keys and values
once.  All heads are laid out with one size (the largest of maps * head_dim and value_dim, rounded up to 16), zeros after their own
values.
"""
from __future__ import annotations

import math

import torch

from ..cache.cache import KVRequirement, RunCache, StateRequirement
from ..kernels import ops
from .joint import ContextMixer, stacked
from .registry import BuildContext, build_part, register_part
from .spec import PartSpec


def query_temperature(coef: float, every: float, positions: int) -> torch.Tensor:
    """float32 [positions]: 1 + coef ln(floor((p + 1) / every) + 1)."""
    p = torch.arange(1, positions + 1, dtype=torch.float64)
    return (1.0 + float(coef) * torch.log(torch.floor(p / float(every)) + 1.0)).to(torch.float32)


def differential_lambda(lq1, lk1, lq2, lk2, diff: float) -> float:
    dot = lambda a, b: float((a.to(torch.float64) * b.to(torch.float64)).sum())
    return math.exp(dot(lq1, lk1)) - math.exp(dot(lq2, lk2)) + float(diff)


class HeadAttention(ContextMixer):
    # the step's batch description lists its prompts cut into tiles of this many query rows (the prefill kernels' tiling)
    query_tile_rows = ops.PREFILL_QUERY_TILE

    def __init__(self, *, hidden_size, n_heads, n_kv_heads, head_dim, value_dim, score_scale, wq, wk, wv, wo, position=None, biases=None,
                 out_bias=None, convs=None, norms=None, head_norm_eps=None, q_factor=None, off_by_one=False, differential=None, lam=0.0,
                 gate=None, wg=None):
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads cannot share {n_kv_heads} key/value heads")
        if (gate is None) != (wg is None) or gate not in (None, "head", "value"):
            raise ValueError("head_attention: gate is None, 'head' or 'value' and comes with its matrix")
        if (norms is None) != (head_norm_eps is None):
            raise ValueError("head_attention: the heads' norm comes with its eps and both weights")
        self.maps = 2 if differential is not None else 1
        self.values_from_keys = wv is None
        if self.values_from_keys and (self.maps != 1 or value_dim != head_dim):
            raise ValueError("head_attention: keys can serve as values with one map and one size only")
        if position is not None and not (hasattr(position, "tables") and getattr(position, "pairing", "half") == "half"):
            raise ValueError("head_attention: the position part must offer tables() of half-split pairs")
        self.hidden_size, self.n_heads, self.n_kv_heads, self.dim, self.vdim = hidden_size, n_heads, n_kv_heads, head_dim, value_dim
        self.score_scale, self.position, self.q_factor = float(score_scale), position, q_factor
        self.D = -(-max(self.maps * head_dim, value_dim) // 16) * 16       # the size all heads are laid out with
        self.q_heads = n_heads * self.maps                                # as the attention kernels see them
        nq, nk = self.q_heads * head_dim, n_kv_heads * self.maps * head_dim
        self.q_col, self.k_col = 0, nq
        self.v_col = None if self.values_from_keys else nq + nk
        at = nq + nk + (0 if self.values_from_keys else n_kv_heads * value_dim)
        self.gate, self.gate_cols = gate, (at, at + (wg.shape[0] if wg is not None else 0))
        self.in_matrix = stacked(*(w for w in (wq, wk, wv, wg) if w is not None))
        self.out_matrix, self.out_bias = wo, out_bias
        self.bias = torch.cat([b.to(torch.float32).reshape(-1) for b in biases]).contiguous() if biases is not None else None
        self.conv, self.conv_state = None, None
        if convs is not None:
            taps = convs[0].shape[1]
            if convs[1].shape[1] != taps or not 1 <= taps <= ops.SHORT_CONV_MAX_TAPS:
                raise ValueError(f"head_attention: both convolutions must have the same 1 to {ops.SHORT_CONV_MAX_TAPS} taps")
            self.conv = torch.cat(list(convs), dim=0).to(wq.dtype).t().contiguous()       # [taps, channels]
            if taps > 1:
                self.conv_state = StateRequirement((taps - 1, nq + nk), "float32")
        self.norm_eps = float(head_norm_eps) if head_norm_eps is not None else 0.0
        self.norms = tuple(w.to(torch.float32).contiguous() for w in norms) if norms is not None else (None, None)
        self.sinks = torch.zeros(self.q_heads, dtype=torch.float32, device=wq.device) if off_by_one else None
        self.differential, self.lam = differential, float(lam)

    def needs(self):
        return KVRequirement(self.n_kv_heads, self.D, None), self.conv_state

    def context(self, rows, batch, cache: RunCache, run: int) -> ops.ContextSide:
        if not cache.owns_kv:
            raise ValueError("head_attention: a run keeps keys and values of its own")
        nh, nkv, D = self.q_heads, self.n_kv_heads, self.D
        pages = ops.KVPages(cache.k, cache.v, batch.tables[cache.kv_group], cache.page_size, cache.ring_pages) if cache.k is not None else None
        fast = rows.dtype is torch.bfloat16 and D <= 256
        fast_decode = fast and cache.page_size % 16 == 0 and cache.page_size <= 64
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        prep = dict(n_heads=self.n_heads, n_kv_heads=nkv, maps=self.maps, dim=self.dim, vdim=self.vdim, pad=D, q_col=self.q_col, k_col=self.k_col,
                    v_col=self.v_col, tok_pos=batch.tok_pos, seq_start=batch.seq_start, slots=batch.slots, seq_end=batch.seq_end,
                    n_seqs=batch.n_seqs, bias=self.bias, conv=self.conv, state=cache.state if self.conv_state is not None else None,
                    wq=self.norms[0], wk=self.norms[1], eps=self.norm_eps, cos=cos, sin=sin, q_factor=self.q_factor, pages=pages)
        common = dict(n_heads=nh, n_kv_heads=nkv, head_dim=D, score_scale=self.score_scale, softcap=None, window=None, sinks=self.sinks,
                      status=batch.status)
        qkv = ops.head_prepare(rows, write_kv=not batch.is_decode, **prep)      # every key is kept: the write never overwrites one that is read
        if batch.is_decode:
            ctx = ops.attention(qkv, batch.attention_batch("all"), pages, kind="decode" if fast_decode else "plain",
                                scratch=lambda n: batch.scratch_buffer("decode", n), **common)
        else:
            kind = "plain"
            if fast and batch.n_tiles:
                kind = "prefill_tc" if (D % 64 == 0 and not batch.has_past) else "prefill"
            ctx = ops.attention(qkv, batch.attention_batch("past"), pages, new_kv=(qkv, nh * D, (nh + nkv) * D), kind=kind, **common)
        d = self.differential
        return ops.ContextSide(ctx, self.n_heads, self.vdim, D, self.maps, self.lam, d["eps"] if d is not None else None, None,
                               1.0 - d["diff"] if d is not None else 1.0,
                               rows[:, self.gate_cols[0]:self.gate_cols[1]] if self.gate is not None else None, self.gate)


def _build_head_attention(spec: PartSpec, ctx: BuildContext) -> HeadAttention:
    p, t = spec.params, spec.tensors
    get = lambda *names: tuple(ctx.tensor(t[n]) for n in names)
    factor = None
    if p.get("q_temperature") is not None:
        q = p["q_temperature"]
        key = ("query_temperature", q["coef"], q["every"], p["max_positions"])
        if key not in ctx.shared:     # one table for all layers that share the constants
            ctx.shared[key] = query_temperature(q["coef"], q["every"], p["max_positions"]).to(ctx.device)
        factor = ctx.shared[key]
    d = p.get("differential")
    return HeadAttention(
        hidden_size=p["hidden_size"], n_heads=p["n_heads"], n_kv_heads=p["n_kv_heads"], head_dim=p["head_dim"],
        value_dim=p.get("value_dim", p["head_dim"]), score_scale=p["score_scale"],
        wq=ctx.tensor(t["q"]), wk=ctx.tensor(t["k"]), wv=None if p.get("values_from_keys") else ctx.tensor(t["v"]), wo=ctx.tensor(t["o"]),
        position=build_part("position", p["position"], ctx) if p.get("position") is not None else None,
        biases=get("q_bias", "k_bias") if "q_bias" in t else None, out_bias=ctx.tensor(t["o_bias"]) if "o_bias" in t else None,
        convs=get("q_conv", "k_conv") if "q_conv" in t else None, norms=get("q_norm", "k_norm") if "q_norm" in t else None,
        head_norm_eps=p.get("head_norm_eps"), q_factor=factor, off_by_one=p.get("off_by_one", False), differential=d,
        lam=differential_lambda(*get("lq1", "lk1", "lq2", "lk2"), d["diff"]) if d is not None else 0.0,
        gate=p.get("gate"), wg=ctx.tensor(t["g"]) if "g" in t else None)


register_part("mixer", "head_attention", _build_head_attention, replace=True)
