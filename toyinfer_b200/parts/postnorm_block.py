"""A layer that norms its sublayers' outputs only.

h <- h + n1(mixer(h));  h <- h + n2(ffn(h)), over a float32 stream h that the sublayers read as it is (rounded to the engine's
type for their products); the feed-forward, with its norm, may be absent.  A sublayer's output stays pending with the norm it
has yet to pass, and the next reader of the stream applies that norm, adds in 32-bit and rounds the sum for its first product
in one kernel (kernels/wide.py: ``post_norm_add_norm``), so the stream is read and written once per sublayer.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Block, BuildContext, ParamSpec, PartSpec, build_part, register_part


class PostNormBlock(Block):
    def __init__(self, ctx: BuildContext, prefix: str, norm: PartSpec, mixer: PartSpec,
                 feed_forward: Optional[PartSpec] = None, names: Optional[Dict[str, str]] = None):
        n = {"norm_mixer": "norm1", "norm_ff": "norm2", "mixer": "mix.", "feed_forward": "mlp."}
        n.update(names or {})
        named = lambda key: build_part("norm", PartSpec(norm.kind, dict(norm.params, name=n[key])), ctx, prefix)
        self.norm_mixer, self.norm_ff, self.feed_forward = named("norm_mixer"), None, None
        if not hasattr(self.norm_mixer, "pending"):
            raise ValueError(f"a block that norms outputs needs a norm that can stay pending on one; {norm.kind!r} cannot")
        self.mixer = build_part("mixer", mixer, ctx, prefix + n["mixer"])
        if feed_forward is not None:
            self.norm_ff = named("norm_ff")
            self.feed_forward = build_part("feed_forward", feed_forward, ctx, prefix + n["feed_forward"])
        self._children = tuple(c for c in (self.norm_mixer, self.mixer, self.norm_ff, self.feed_forward) if c is not None)

    def param_specs(self) -> Dict[str, ParamSpec]:
        out: Dict[str, ParamSpec] = {}
        for c in self._children:
            out.update(c.param_specs())
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for c in self._children:
            c.bind(tensors)

    def check_kernels(self, dtype) -> None:
        for c in self._children:
            c.check_kernels(dtype)

    @property
    def captures_start(self) -> bool:
        return bool(self.mixer.captures_start and (self.feed_forward is None or self.feed_forward.captures_start))

    def _mix(self, h, delta, batch, mem, shared):
        x = self.norm_mixer.read_forward(h, delta)                   # h takes what was pending; x = h rounded
        return self.norm_mixer.pending(self.mixer.forward(x, batch, mem, shared))

    def _feed(self, h, a, batch):
        x = self.norm_ff.read_forward(h, a)
        return self.norm_ff.pending(self.feed_forward.forward(x, batch))

    def forward(self, h, delta, batch, mem, shared):
        trace = getattr(batch, "trace", None)
        if trace is not None and trace.active:
            with trace.range("layer.attn_block"):
                a = self._mix(h, delta, batch, mem, shared)
            if self.feed_forward is None:
                return h, a
            with trace.range("layer.mlp_block"):
                return h, self._feed(h, a, batch)
        a = self._mix(h, delta, batch, mem, shared)
        if self.feed_forward is None:
            return h, a
        return h, self._feed(h, a, batch)


register_part("block", "postnorm", PostNormBlock)
