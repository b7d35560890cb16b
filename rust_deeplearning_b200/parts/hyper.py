"""Hyper-connections: a residual stream of several copies per token, and the block that reads and writes it.

Instead of one x there are S copies x_1 .. x_S, all equal at the start.  Every sublayer has its own small matrices:
    u = sum_s read[s] x_s;    y = sublayer(norm(u));    x_t <- sum_s mix[s, t] x_s + write[t] y     (all t at once)
and the model's output is formed from the sum of the copies.  The copies are float32 and so is all arithmetic on them.

`HyperStream` is the stream (`ModelSpec.stream` kind "hyper"); like `ResidualStream` it lets a result wait until the next
part asks for its input, so that "write the result into the copies, read the weighted sum, norm it" is ONE kernel
(`ops.hyper`).  `HyperBlock` is the arrangement (block kind "hyper"): norm -> mixer -> back into the copies; norm ->
feed-forward -> back into the copies; a layer without a feed-forward ends after the mixer.  Its tensors, by role: "read1",
"mix1", "write1" for the mixer's connection and "read2", "mix2", "write2" for the feed-forward's.

A feed-forward that keeps parts of its result apart (`forward_parts`, or `forward_gated_parts` with a gate per token on the
second part) has them added up in the stream's kernel.
"""
from __future__ import annotations

from typing import Dict, NamedTuple, Optional

import torch

from ..kernels import ops
from .registry import BuildContext, build_part, register_part
from .spec import LayerSpec, PartSpec


class Connection(NamedTuple):
    """A sublayer's connection to the copies, float32."""
    read: torch.Tensor       # [S]
    mix: torch.Tensor        # [S from, S to]
    write: torch.Tensor      # [S]


class HyperStream:
    """S copies of the stream (float32 [rows, S, width]; while they are all equal, the one row [rows, width]) with at most
    one result waiting to be written into them."""

    def __init__(self, x: torch.Tensor, n_copies: int, ones: torch.Tensor):
        if x.dtype is not torch.float32:
            raise ValueError("the residual stream is float32")
        self.x, self.n_copies, self._ones = x, n_copies, ones        # ones: float32 [S], the weights of the plain sum
        self._pending = None                 # ((a, b, gate), Connection)
        self.norm_after_block = None         # the model's hint; this stream has no use for it

    def _result(self):
        if self._pending is None:
            return {}
        (a, b, gate), c = self._pending
        return dict(a=a, b=b, b_gate=gate, mix=c.mix, write=c.write)

    def add(self, result, connection: Connection):
        """The sublayer's result goes back into the copies; result: (a, b or None, gate or None), y = a + b sigmoid(gate)."""
        self._flush()
        self._pending = (result, connection)

    def _flush(self):
        if self._pending is not None:
            copies, _ = ops.hyper(self.x, self.n_copies, **self._result())
            self.x, self._pending = copies, None

    def normed(self, norm, read: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
        """norm(sum_s read[s] x_s) after any waiting result has been written into the copies."""
        copies, y = ops.hyper(self.x, self.n_copies, read=read, norm=norm.fused_params(), out_dtype=out_dtype, **self._result())
        if copies is not None:
            self.x = copies
        self._pending = None
        return y

    def normed_rows(self, norm, rows: torch.Tensor, out_dtype: torch.dtype, deferred_ok: bool = False) -> torch.Tensor:
        """norm(sum of the copies) for an int32 list of rows (a waiting result stays waiting)."""
        return ops.hyper(self.x, self.n_copies, read=self._ones, norm=norm.fused_params(), out_dtype=out_dtype, row_index=rows,
                         **self._result())[1]

    def value(self) -> torch.Tensor:
        """The sum of the copies, float32 [rows, width]."""
        self._flush()
        return ops.hyper(self.x, self.n_copies, read=self._ones)[1]


def _build_stream(spec: PartSpec, ctx: BuildContext):
    n = int(spec.params["copies"])
    ones = torch.ones(n, dtype=torch.float32, device=ctx.device)
    return lambda x: HyperStream(x, n, ones)


register_part("stream", "hyper", _build_stream, replace=True)


class HyperBlock:
    def __init__(self, mixer, feed_forward, norms: Dict[str, object], act_dtype: torch.dtype, first: Connection, second: Optional[Connection]):
        for n in norms.values():
            if not callable(getattr(n, "fused_params", None)):
                raise ValueError("hyper block: the norms must be scale-only root-mean-square norms (fused_params)")
        self.mixer, self.feed_forward, self.act_dtype = mixer, feed_forward, act_dtype
        self.pre_mixer, self.pre_ff = norms["pre_mixer"], norms.get("pre_feed_forward")
        self.first, self.second = first, second

    first_norm = None       # it reads a weighted sum of copies

    def _feed_forward(self, x):
        ff = self.feed_forward
        if hasattr(ff, "forward_gated_parts"):
            return ff.forward_gated_parts(x)
        if hasattr(ff, "forward_parts"):
            return (*ff.forward_parts(x), None)
        return ff.forward(x), None, None

    def forward(self, stream: HyperStream, batch, cache, run: int):
        x = stream.normed(self.pre_mixer, self.first.read, self.act_dtype)
        stream.add((self.mixer.forward(x, batch, cache, run), None, None), self.first)
        if self.feed_forward is not None:
            x = stream.normed(self.pre_ff, self.second.read, self.act_dtype)
            stream.add(self._feed_forward(x), self.second)


def _build_hyper(layer: LayerSpec, ctx: BuildContext) -> HyperBlock:
    mixer = build_part("mixer", layer.mixer, ctx)
    ff = build_part("feed_forward", layer.feed_forward, ctx) if layer.feed_forward is not None else None
    norms = {role: build_part("norm", s, ctx) for role, s in layer.norms.items()}
    t = layer.tensors

    def connection(q):
        return Connection(*(ctx.tensor(t[f"{role}{q}"]).to(torch.float32).contiguous() for role in ("read", "mix", "write")))

    return HyperBlock(mixer, ff, norms, ctx.dtype, connection(1), connection(2) if ff is not None else None)


register_part("block", "hyper", _build_hyper, replace=True)
