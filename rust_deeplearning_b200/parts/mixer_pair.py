"""Two mixers side by side: both read the same input and their results are added up.  Two forms:

  norms       each result is normed over the model width with a plain weight of its own (tensor roles "left_out",
              "right_out"), and the mixer's result is `factor` times their sum:
                  y = factor * (rms_norm(left(x); w_left) + rms_norm(right(x); w_right)).
              The sum is formed in float32 (one kernel for both norms and the sum).
  scales      a constant on each result, no norms (parameters "left_scale", "right_scale"):
                  y = left_scale * left(x) + right_scale * right(x).
              Both mixers are `ContextMixer`s (`parts/joint.py`) and share one input product and one output product.

The two are built through the mixer registry from their own descriptions (`params["left"]`, `params["right"]`:
`PartSpec`s of any registered kinds), so any pair can stand side by side as long as at most one of them keeps
keys and values: a layer run has one key/value store.  State of both is kept side by side.
"""
from __future__ import annotations

from ..cache.cache import RunCache
from ..kernels import ops
from .joint import ContextMixer, JointProducts
from .registry import BuildContext, build_part, register_part
from .spec import PartSpec


def _states(state):
    return () if state is None else (tuple(state) if isinstance(state, (tuple, list)) else (state,))


class MixerPair:
    def __init__(self, left, right, w_left=None, w_right=None, eps: float = 0.0, factor: float = 0.5, scales=None):
        if (scales is None) == (w_left is None or w_right is None):
            raise ValueError("mixer_pair: either both results are normed or both have a constant")
        self.left, self.right = left, right
        self.w_left, self.w_right, self.eps, self.factor = w_left, w_right, float(eps), float(factor)
        (lk, ls), (rk, rs) = left.needs(), right.needs()
        if lk is not None and rk is not None:
            raise ValueError("mixer_pair: both mixers keep keys and values; a layer run has one store")
        self._left_state, self._right_state = ls, rs
        # one side's state as that side declared it; of two sides, all tensors in order
        state = _states(ls) + _states(rs) if (ls is not None and rs is not None) else (ls if ls is not None else rs)
        self._needs = (lk if lk is not None else rk, state)
        # the step's batch description is cut into query tiles for whichever of the two asks
        self.query_tile_rows = max(getattr(left, "query_tile_rows", 0) or 0, getattr(right, "query_tile_rows", 0) or 0)
        self.products = None
        if scales is not None:
            if not (isinstance(left, ContextMixer) and isinstance(right, ContextMixer)):
                raise ValueError("mixer_pair: a pair with constants takes two mixers whose products can be shared")
            self.products = JointProducts((left, right), scales)
            self.takes_deferred_rows = self.delivers_branch = True

    def needs(self):
        return self._needs

    def _caches(self, cache: RunCache):
        """The run's cache as each side declared it."""
        if self._left_state is None or self._right_state is None:
            return cache, cache
        n = len(_states(self._left_state))

        def own(declared, tensors):
            return cache._replace(state=tensors if isinstance(declared, (tuple, list)) else tensors[0])
        return own(self._left_state, cache.state[:n]), own(self._right_state, cache.state[n:])

    def forward(self, x, batch, cache: RunCache, run: int, sink=None):
        lc, rc = self._caches(cache)
        if self.products is not None:
            return self.products.forward(x, batch, (lc, rc), run, sink)
        a = self.left.forward(x, batch, lc, run)
        b = self.right.forward(x, batch, rc, run)
        return ops.norm_pair(a, b, self.w_left, self.w_right, self.eps, self.factor)


def _build_mixer_pair(spec: PartSpec, ctx: BuildContext) -> MixerPair:
    p, t = spec.params, spec.tensors
    left = build_part("mixer", p["left"], ctx)
    right = build_part("mixer", p["right"], ctx)
    if "left_scale" in p:
        return MixerPair(left, right, scales=(p["left_scale"], p["right_scale"]))
    return MixerPair(left, right, ctx.tensor(t["left_out"]), ctx.tensor(t["right_out"]), p["eps"], p.get("factor", 0.5))


register_part("mixer", "mixer_pair", _build_mixer_pair, replace=True)
