"""The matrix-memory mixer: the mLSTM of xLSTM ("xLSTM: Extended Long Short-Term Memory", Beck et al.) with capped gates.

Per head, over a sequence's tokens (S [dim, vdim], n [dim] and m start at zero):
    i = cap tanh((W_i x + b_i) / cap),   f = log sigmoid(cap tanh((W_f x + b_f) / cap))
    m_t = max(f + m_(t-1), i)
    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,      n_t by the same rule with k for k v^T
    o_t = S_t^T (q_scale q) / (max(|n_t . q_scale q|, e^(-m_t)) + den_eps)
Every head's o is divided by its root mean square; the concatenated heads are multiplied by the weight `norm` and by
sigmoid(W_g x), element by element, before W_o.  The cap, q's scale, den_eps and the norm's eps are parameters.

One product makes q, k, v and all gates' logits; the recurrence runs in float from those rows (`ops.matrix_memory`).  Per
sequence the cache keeps S, and n with m (in as many copies as the recurrence kernel has blocks a head), in float.
"""
from __future__ import annotations

import torch

from ..cache.cache import RunCache, StateRequirement
from ..kernels import ops
from .joint import ContextMixer, stacked
from .registry import BuildContext, register_part
from .spec import PartSpec


class MatrixMemory(ContextMixer):
    def __init__(self, *, hidden_size, n_heads, dim, vdim, gate_cap, q_scale, den_eps, eps, wq, wk, wv, wg, wi, wf, i_bias, f_bias, norm_weight, wo):
        self.hidden_size, self.n_heads, self.dim, self.vdim = hidden_size, n_heads, dim, vdim
        self.cap, self.q_scale, self.den_eps, self.eps = float(gate_cap), float(q_scale), float(den_eps), float(eps)
        if not self.cap > 0.0:
            raise ValueError(f"matrix_memory: the gates' cap must be positive, got {self.cap}")
        H = n_heads
        self.k_col, self.v_col = H * dim, 2 * H * dim
        self.g_col = self.v_col + H * vdim
        self.i_col = self.g_col + H * vdim
        self.in_matrix = stacked(wq, wk, wv, wg, wi, wf)
        self.out_matrix = wo
        f32 = lambda t: t.to(torch.float32).contiguous()
        self.i_bias, self.f_bias, self.norm_weight = f32(i_bias), f32(f_bias), f32(norm_weight)

    def needs(self):
        return None, (StateRequirement((self.n_heads, self.dim, self.vdim), "float32"),
                      StateRequirement((self.n_heads, ops.matrix_memory_copies(self.vdim), self.dim + 1), "float32"))

    def context(self, rows, batch, cache: RunCache, run: int) -> ops.ContextSide:
        H = self.n_heads
        o = ops.matrix_memory(rows, q_col=0, k_col=self.k_col, v_col=self.v_col, i_col=self.i_col, f_col=self.i_col + H, n_heads=H,
                              dim=self.dim, vdim=self.vdim, i_bias=self.i_bias, f_bias=self.f_bias, cap=self.cap, q_scale=self.q_scale,
                              den_eps=self.den_eps, state=cache.state[0], norm=cache.state[1], tok_pos=batch.tok_pos,
                              seq_start=batch.seq_start, slots=batch.slots, n_seqs=batch.n_seqs)
        return ops.ContextSide(o, H, self.vdim, self.vdim, norm_eps=self.eps, weight=self.norm_weight,
                               gate=rows[:, self.g_col:self.g_col + H * self.vdim], gate_kind="value")


def _build_matrix_memory(spec: PartSpec, ctx: BuildContext) -> MatrixMemory:
    p, t = spec.params, spec.tensors
    w = {f"w{n}": ctx.tensor(t[n]) for n in ("q", "k", "v", "g", "i", "f", "o")}
    return MatrixMemory(hidden_size=p["hidden_size"], n_heads=p["n_heads"], dim=p["dim"], vdim=p["vdim"], gate_cap=p["gate_cap"],
                        q_scale=p.get("q_scale", 1.0), den_eps=p.get("den_eps", 1e-6), eps=p["eps"], i_bias=ctx.tensor(t["i_bias"]),
                        f_bias=ctx.tensor(t["f_bias"]), norm_weight=ctx.tensor(t["norm"]), **w)


register_part("mixer", "matrix_memory", _build_matrix_memory, replace=True)
