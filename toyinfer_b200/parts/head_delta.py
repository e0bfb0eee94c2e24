"""Linear attention by the gated delta rule with one decay per head, short convolutions and a silu-gated output.

Per token x: q = silu(conv(Wq x)), k = silu(conv(Wk x)) [qk_heads, dim], v = silu(conv(Wv x)) [heads, vdim], each through a
causal convolution over time per channel (no bias); q and k are made unit vectors per head, q also times dim^-1/2;
beta = sigmoid(Wb x) and g = exp(-exp(A_h) softplus(Wa x + dt)), one of each per head.  Per head, with a state S [dim, vdim]
carried from token to token in float32 (zero when the sequence starts), in this order:

    S <- g S;   e = beta (v - S^T k);   S <- S + k e^T;   o = S^T q

(value head h with query/key head h // (heads / qk_heads)); then o / rms(o) per head times a weight [vdim] shared by the
heads, times silu(Wg x), and Wo (Yang, Kautz and Hatamizadeh, "Gated Delta Networks").

What a sequence carries, one float32 row per slot (``StateRequest``): the convolutions' last ``conv - 1`` inputs over all
of q, k and v's channels, then S [heads, dim, vdim].  All six projections of the input are one product.  The mixer with a
decay per key channel (channel_delta.py) runs on the same kernels.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels as K
from ..kernels import recurrent as KR
from ..tracing import ranged
from .base import BuildContext, Mixer, ParamSpec, StateRequest, register_part


class HeadDeltaAttention(Mixer):
    captures_start = True

    def __init__(self, ctx: BuildContext, prefix: str, n_heads: int, n_qk_heads: int, dim: int, vdim: int, conv: int, eps: float,
                 names: Optional[Dict[str, str]] = None):
        if n_qk_heads < 1 or n_heads % n_qk_heads:
            raise ValueError(f"{n_heads} value heads cannot share {n_qk_heads} query/key heads evenly")
        self.ctx, self.hidden = ctx, ctx.hidden_size
        self.n_heads, self.n_qk, self.dim, self.vdim, self.taps = int(n_heads), int(n_qk_heads), int(dim), int(vdim), int(conv)
        self.eps = float(eps)
        n = {"q": "q", "k": "k", "v": "v", "conv": ".conv", "beta": "b", "rate": "A_log", "norm": "norm", "decay": "a",
             "decay_bias": "dt_bias", "gate": "g", "o": "o"}
        n.update(names or {})
        self.n, self.prefix = n, prefix
        self.channels = 2 * self.n_qk * self.dim + self.n_heads * self.vdim
        self.state_conv = 0
        self.state_s = (self.taps - 1) * self.channels
        self.w_in = self.w_o = self.conv_w = self.dt_bias = self.rate = self.norm_w = None

    def _name(self, k: str) -> str:
        return self.prefix + self.n[k]

    def param_specs(self) -> Dict[str, ParamSpec]:
        H, G, d, vd, hid = self.n_heads, self.n_qk, self.dim, self.vdim, self.hidden
        small = lambda shape, **kw: ParamSpec(shape, role="norm", init="normal", **kw)
        conv = self.n["conv"]
        return {
            self._name("q"): ParamSpec((G * d, hid), std=0.1), self._name("q") + conv: small((G * d, self.taps), std=0.5),
            self._name("k"): ParamSpec((G * d, hid), std=0.1), self._name("k") + conv: small((G * d, self.taps), std=0.5),
            self._name("v"): ParamSpec((H * vd, hid), std=0.1), self._name("v") + conv: small((H * vd, self.taps), std=0.5),
            self._name("beta"): ParamSpec((H, hid), std=0.1), self._name("rate"): small((H,), std=0.5),
            self._name("norm"): ParamSpec((vd,), role="norm", init="one_plus_normal", std=0.1),
            self._name("decay"): ParamSpec((H, hid), std=0.1), self._name("decay_bias"): small((H,), std=1.0, mean=-2.0),
            self._name("gate"): ParamSpec((H * vd, hid), std=0.1),
            self._name("o"): ParamSpec((hid, H * vd), std=0.05),
        }

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        t = lambda k: tensors.pop(self._name(k))
        f32 = lambda name: tensors.pop(name).to(torch.float32).contiguous()
        conv = self.n["conv"]
        self.conv_w = torch.cat([f32(self._name(k) + conv) for k in ("q", "k", "v")], dim=0).contiguous()
        # rows of zeros bring a token's row of results to a multiple of 16 bytes, which the tensor-core kernel's loads need
        parts = [t(k) for k in ("q", "k", "v", "gate", "beta", "decay")]
        spare = -sum(p.shape[0] for p in parts) % 8
        if spare:
            parts.append(torch.zeros((spare, self.hidden), dtype=parts[0].dtype, device=parts[0].device))
        self.w_in = torch.cat(parts, dim=0).contiguous()
        self.dt_bias = f32(self._name("decay_bias"))
        self.rate = torch.exp(f32(self._name("rate"))).contiguous()
        self.norm_w = f32(self._name("norm"))
        self.w_o = t("o").contiguous()

    def check_kernels(self, dtype) -> None:
        if self.dim > 256:
            raise K.KernelError(f"delta rule: heads of {self.dim} query/key elements are not supported (up to 256)")
        if not 1 <= self.taps <= 8:
            raise K.KernelError(f"short convolution: {self.taps} taps are not supported (1 to 8)")

    def memory_request(self):
        return StateRequest((self.state_s + self.n_heads * self.dim * self.vdim,), torch.float32)

    def launch_plan(self, n_seq: int, plan_len: int, dtype, device, n_live=None):
        return ("delta",)

    def forward(self, x, batch, mem, shared) -> torch.Tensor:
        if mem is None or not hasattr(mem, "state"):
            raise RuntimeError("a delta-rule mixer needs a state; the schedule gave it none")
        H, G, d, vd, C = self.n_heads, self.n_qk, self.dim, self.vdim, self.channels
        with ranged(batch, "mixer.qkv"):
            y = K.linear(x, self.w_in)
            M = y.shape[0]
            u = KR.short_conv(y[:, :C], self.conv_w, mem.state, self.state_conv, batch, act="silu")
        gate, beta, decay = y[:, C:C + H * vd], y[:, C + H * vd:C + H * vd + H], y[:, C + H * vd + H:C + H * vd + 2 * H]
        q = u[:, :G * d].view(M, G, d)
        k = u[:, G * d:2 * G * d].view(M, G, d)
        v = u[:, 2 * G * d:].view(M, H, vd)
        with ranged(batch, "mixer.attention"):
            o = KR.delta_rule(q, k, v, decay, self.dt_bias, self.rate, beta, mem.state, self.state_s, batch, head_decay=True)
            a = KR.head_gated_rmsnorm(o, gate, self.norm_w, H, self.eps, gate_act="silu")
        with ranged(batch, "mixer.out"):
            return K.linear(a, self.w_o)


register_part("mixer", "head_delta", HeadDeltaAttention)
