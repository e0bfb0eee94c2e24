"""A parallel layer over a float32 stream that is averaged over depth, whose mixer may read a token-shifted input.

With X_0 the embedding's rows and y the stream that the layer is given (y = X_0 before the first layer):

    z = norm(y);   z'_t = z_t + (z_{t-1} - z_t) * shift          (z before a sequence's first token: zeros)
    X_{i+1} = y + mult * (mixer(z') + feed_forward(z));          y <- sum_{j <= i+1} dwa[j] X_j

for the layer with i results before it (``depth``); the averaging follows Pagliardini, Mohtashami, Fleuret and Jaggi,
"DenseFormer".  ``shift=False``: the mixer reads z; ``average=False``: y <- X_{i+1}; the feed-forward may be absent.  Weights
beside the sublayers': the norm's, ``shift`` [width], ``dwa`` [depth + 2].

The layer's two outputs stay pending (kernels.depth.DepthUpdate); the norm that reads the stream next (the next layer's, the
head's) forms the result, the average, the normed row and the shifted one in one kernel.  ``h`` is X_0 throughout; the later
results travel with the pending update.

The last z of every sequence is part of what a layer carries from token to token: the block asks the cache for its mixer's
memory and, beside it, a float32 row [width] per slot.

In a step of single tokens the feed-forward, which does not wait for the mixer, runs on a stream of its own beside it.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels.depth import DepthUpdate, MAX_RESULTS, ShiftedRead
from ..tracing import ranged
from .base import Block, BuildContext, ParamSpec, PartSpec, StateRequest, build_part, register_part


class AveragedParallelBlock(Block):
    two_streams = True          # single-token steps run the feed-forward beside the mixer (tests clear it to compare)

    def __init__(self, ctx: BuildContext, prefix: str, norm: PartSpec, mixer: PartSpec, feed_forward: Optional[PartSpec] = None,
                 depth: int = 0, mult: float = 1.0, shift: bool = True, average: bool = True, names: Optional[Dict[str, str]] = None):
        n = {"norm": "", "mixer": "mix.", "feed_forward": "mlp.", "shift": "shift", "average": "dwa"}
        n.update(names or {})
        self.hidden, self.prefix, self.n = ctx.hidden_size, prefix, n
        self.depth, self.mult = int(depth), float(mult)
        self.norm = build_part("norm", norm, ctx, prefix + n["norm"])
        self.mixer = build_part("mixer", mixer, ctx, prefix + n["mixer"])
        self.feed_forward = build_part("feed_forward", feed_forward, ctx, prefix + n["feed_forward"]) if feed_forward is not None else None
        self._children = tuple(c for c in (self.norm, self.mixer, self.feed_forward) if c is not None)
        self.has_shift, self.has_average = bool(shift), bool(average)
        self.shift: Optional[torch.Tensor] = None
        self.average: Optional[torch.Tensor] = None
        self._side = None           # the feed-forward's stream, made when first needed

    def param_specs(self) -> Dict[str, ParamSpec]:
        out: Dict[str, ParamSpec] = {}
        for c in self._children:
            out.update(c.param_specs())
        if self.has_shift:
            out[self.prefix + self.n["shift"]] = ParamSpec((self.hidden,), role="norm", init="normal", mean=0.5, std=0.2)
        if self.has_average:
            n = self.depth + 2
            out[self.prefix + self.n["average"]] = ParamSpec((n,), role="norm", init="normal", mean=1.0 / n, std=0.3 / n)
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for c in self._children:
            c.bind(tensors)
        f32 = lambda name: tensors.pop(self.prefix + self.n[name]).to(torch.float32).contiguous()
        if self.has_shift:
            self.shift = f32("shift")
        if self.has_average:
            self.average = f32("average")

    def check_kernels(self, dtype) -> None:
        from .. import kernels as K
        if self.depth + 1 > MAX_RESULTS:
            raise K.KernelError(f"a layer with {self.depth} results before it is not supported (up to {MAX_RESULTS - 1})")
        for c in self._children:
            c.check_kernels(dtype)

    @property
    def captures_start(self) -> bool:
        return bool(self.mixer.captures_start and (self.feed_forward is None or self.feed_forward.captures_start))

    # -- memory: the mixer's, and the last normed row ---------------------------
    def memory_request(self):
        own = self.mixer.memory_request()
        if not self.has_shift:
            return own
        members = () if own is None else tuple(own) if isinstance(own, (tuple, list)) else (own,)
        return members + (StateRequest((self.hidden,), torch.float32),)

    def _memories(self, mem):
        """(the mixer's memory as the mixer expects it, the shift's state or None)."""
        if not self.has_shift:
            return mem, None
        if not isinstance(mem, tuple) or not hasattr(mem[-1], "state"):
            raise RuntimeError("a layer with a token shift needs a state beside its mixer's memory; the schedule gave it none")
        own = self.mixer.memory_request()
        if own is None:
            return None, mem[-1]
        return (mem[:-1] if isinstance(own, (tuple, list)) else mem[0]), mem[-1]

    def forward(self, h, delta, batch, mem, shared):
        trace = getattr(batch, "trace", None)
        mix_mem, before = self._memories(mem)
        read = ShiftedRead(self.shift, before.state, batch) if self.has_shift else None
        z, zs, results = self.norm.read_forward(h, delta, read)
        if zs is None:
            zs = z
        ff, f = self.feed_forward, None
        beside = ff is not None and self.two_streams and batch.mode == "extend" and z.is_cuda and not (trace is not None and trace.timing)
        if beside:
            # (memory: what the side stream made is used again on the side stream only, after a fork that follows its last reader)
            if self._side is None:
                self._side = torch.cuda.Stream(device=z.device)
            main = torch.cuda.current_stream(z.device)
            forked, joined = torch.cuda.Event(), torch.cuda.Event()
            forked.record(main)
            self._side.wait_event(forked)
            with torch.cuda.stream(self._side):
                f = ff.forward(z, batch)
                joined.record(self._side)
        with ranged(batch, "layer.attn_block"):
            a = self.mixer.forward(zs, batch, mix_mem, shared)
        if beside:
            main.wait_event(joined)
        elif ff is not None:
            with ranged(batch, "layer.mlp_block"):
                f = ff.forward(z, batch)
        # how the pending layer's y was formed is how this layer's input was formed
        c_in = delta.average_out if delta is not None else None
        return h, DepthUpdate(results, a, f, self.mult, c_in, self.average)


register_part("block", "averaged_parallel", AveragedParallelBlock)
