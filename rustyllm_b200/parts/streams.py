"""A residual of several streams (hyper-connections): S copies of the embedding's output run through the model side by
side.  A sublayer reads one weighted sum of a token's streams and its output is mixed back into all of them at once:

    u    = sum_s in[s] X[s]
    y    = channel_scale * sublayer(norm(u))               (channel_scale: a learned value a channel, where the design has one)
    X[t] = sum_s mix[s, t] X[s] + out[t] y                 (every t from the old streams)

The streams are float32 [M, S, d]; a model says how many it has (``ModelSpec.streams``), the decoder opens them behind the
embedding and reads their plain sum in front of the head.  Between two sublayers one kernel (csrc/streams.cu) does the join
of the first and the normed read of the second, across layers too: what a block's first read needs is its
``first_norm_request``, and the block in front hands the normed rows over as ``pending``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from .. import kernels as K
from ..config.spec import ParamSource, ParamSpec
from .base import Block, FeedForward, Mixer, Norm, Runtime
from .registry import register_block


@dataclass(frozen=True)
class StreamRead:
    """What a join needs to make the next sublayer's input on the way: y = rms_norm(sum_s coef[s] X[s]) * weight."""
    coef: Optional[torch.Tensor]          # [S] float32; None: the plain sum
    weight: torch.Tensor                  # [d] float32
    eps: float


def open_streams(x0: torch.Tensor, streams: int, dtype: torch.dtype, read: Optional[StreamRead]):
    """x0 [M, d] -> (X [M, S, d] with x0 in every stream, the first sublayer's normed input or None)."""
    M, d = x0.shape
    X = torch.empty((M, streams, d), dtype=torch.float32, device=x0.device)
    if read is None:
        K.streams_open(x0, X)
        return X, None
    out = torch.empty((M, d), dtype=dtype, device=x0.device)
    K.streams_open(x0, X, read.coef, read.weight, read.eps, out)
    return X, out


def read_streams(X: torch.Tensor, read: StreamRead, dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    n = X.shape[0] if rows is None else rows.numel()
    out = torch.empty((n, X.shape[2]), dtype=dtype, device=X.device)
    K.streams_read(X, read.coef, read.weight, read.eps, out, rows)
    return out


@register_block("hyper_connected")
class HyperConnectedBlock(Block):
    """A pre-norm layer over several streams.  ``names``: "mixer" and "feed_forward", the prefixes of the connections'
    tensors (+ "in" [S], "out" [S], "mix" [S, S] indexed [from, to]); optionally "mixer_scale" and "feed_forward_scale",
    tensors of a value a channel on what the sublayer returns.  A layer without a feed-forward has the first half only.
    """

    def __init__(self, runtime: Runtime, mixer: Mixer, mixer_norm: Norm, feed_forward: FeedForward, feed_forward_norm: Norm,
                 hidden_size: int, streams: int, names: Dict[str, str]):
        if streams < 1:
            raise ValueError(f"streams must be >= 1, got {streams}")
        self.runtime = runtime
        self.mixer, self.mixer_norm = mixer, mixer_norm
        self.feed_forward, self.feed_forward_norm = feed_forward, feed_forward_norm
        self.d, self.streams, self.names = hidden_size, int(streams), names
        self.has_ff = not getattr(feed_forward, "absent", False)
        for part, what in ((mixer, "mixer"), (feed_forward, "feed-forward"))[:2 if self.has_ff else 1]:
            if not hasattr(part, "forward_out"):
                raise ValueError(f"a hyper_connected block needs a {what} that returns its output (forward_out)")
        for norm in (mixer_norm, feed_forward_norm)[:2 if self.has_ff else 1]:
            if not hasattr(norm, "eps") or not hasattr(norm, "request"):
                raise ValueError("a hyper_connected block needs RMS norms (a weight and an eps)")
        self.in1 = self.out1 = self.mix1 = self.scale1 = self.in2 = self.out2 = self.mix2 = self.scale2 = None

    def sub_parts(self):
        return {"mixer": self.mixer, "mixer_norm": self.mixer_norm,
                "feed_forward": self.feed_forward, "feed_forward_norm": self.feed_forward_norm}

    def param_specs(self) -> Dict[str, ParamSpec]:
        S, specs = self.streams, {}
        for q, key in ((1, "mixer"), (2, "feed_forward"))[:2 if self.has_ff else 1]:
            p = self.names[key]
            specs[f"in{q}"] = ParamSpec((ParamSource(p + "in", (S,)),), role="vector", init="ones")
            specs[f"out{q}"] = ParamSpec((ParamSource(p + "out", (S,)),), role="vector", init="ones")
            specs[f"mix{q}"] = ParamSpec((ParamSource(p + "mix", (S, S)),), role="vector", init="normal")
            if key + "_scale" in self.names:
                specs[f"scale{q}"] = ParamSpec((ParamSource(self.names[key + "_scale"], (self.d,)),), role="vector", init="ones")
        return specs

    folds_norms = True
    norm_requests = (StreamRead,)

    def _read(self, q: int) -> Optional[StreamRead]:
        norm = self.mixer_norm if q == 1 else self.feed_forward_norm
        return StreamRead(self.in1 if q == 1 else self.in2, norm.weight, norm.eps)

    def first_norm_request(self, num_tokens: int) -> StreamRead:
        return self._read(1)

    def _join(self, X, terms, q: int, read: Optional[StreamRead]):
        """The streams take a sublayer's output; returns the normed input of the next sublayer where one is asked for."""
        mix, to, scale = (self.mix1, self.out1, self.scale1) if q == 1 else (self.mix2, self.out2, self.scale2)
        y, factor = terms[0]
        if len(terms) > 1:                               # mixers side by side
            acc = torch.zeros((X.shape[0], self.d), dtype=torch.float32, device=X.device)
            for yt, f in terms:
                K.scaled_add(acc, yt, f)
            y, factor = acc, 1.0
        kw = {}
        if not torch.is_tensor(y):                       # experts' rows, still unweighted (parts/moe.py, ExpertRows)
            if y.weights is None:
                raise K.KernelError("experts' rows that were weighed on their input: not built into the join of several streams")
            kw.update(row=y.row, weights=y.weights)
            y = y.rows
        else:
            kw.update(y_factor=factor)
        out = None
        if read is not None:
            out = torch.empty((X.shape[0], self.d), dtype=self.runtime.compute_dtype, device=X.device)
            kw.update(coef=read.coef, norm_weight=read.weight, eps=read.eps, out=out)
        K.streams_join(X, y, mix, to, scale, **kw)
        return out

    def forward(self, X: torch.Tensor, step, cache, pending=None, next_norm=None):
        if X.dim() != 3 or X.shape[1] != self.streams:
            raise K.KernelError(f"a block of {self.streams} streams was given a residual of shape {tuple(X.shape)}")
        h = pending if pending is not None else read_streams(X, self._read(1), self.runtime.compute_dtype)
        terms = self.mixer.forward_out(h, step, cache)
        if not self.has_ff:
            return self._join(X, terms, 1, next_norm)
        h = self._join(X, terms, 1, self._read(2))
        if getattr(self.feed_forward, "offers_rows", False):
            terms = self.feed_forward.forward_out(h, step, rows_ok=True)
        else:
            terms = self.feed_forward.forward_out(h, step)
        return self._join(X, terms, 2, next_norm)
