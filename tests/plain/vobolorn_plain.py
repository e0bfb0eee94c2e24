"""Plain, slow Vobolorn: whole sequences, no cache, one function per mechanism.

The oracle of the Vobolorn tests.  It shares no code with toyinfer_b200: the configuration is a dict as config.json holds
it, the weights a dict of tensors by checkpoint name, and every mechanism is written with elementary torch operations in
float64.

The design in this file's notation (one row per token; W applies as W x; weights [out, in]):

* embedding:   X = E[token]
* norm:        n(u; w) = u / sqrt(mean(u^2) + eps) * w
* layer:       X <- X + n(mixer(X); norm1);  X <- X + n(feed_forward(X); norm2)      (the sublayers read X as it is)
* attention, attention_2:  q = Wq X [H, d], k = Wk X [G, d], v = Wv X [G, dv], the first kind with a bias on each;
               every head of q and of k normed over its own d elements with one weight per side; in the second kind
               q_p <- q_p (1 + coef ln(floor((p + 1) / every) + 1)) at position p;
               layers that mix values: v <- (1 - lam) v + lam v0, v0 the values of the same token in the first of them;
               s_ij = (q_i . k_j) * scale, softmax over j <= i, head h reads kv head h // (H / G); in the first kind the
               heads side by side times sigmoid(Wg X), element by element; Wo
* latent_attention:  q = Wuq n(Wdq X; dq.norm), head by head [d plain | r rotated]; Wdkv X = [c' | b'];
               c = n(c'; dkv.norm); key of head h [Wuk_h c | turn(b')], value Wuv_h c; turning neighbours (2e, 2e + 1) by
               p base^(-2e/r); s and softmax as above; head h times sigmoid(Wg X)_h; Wo
* feed-forward: Wdown (silu(Wgate X) * (Wup X))
* output:      z = W_head n(X; final.norm);  logits = cap * tanh(z / cap)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence, Tuple

import torch

F64 = torch.float64


def rms_norm(u: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    u = u.to(F64)
    return u / torch.sqrt((u * u).mean(dim=-1, keepdim=True) + eps) * w.to(F64)


def sigmoid(a: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-a))


def project(x: torch.Tensor, p: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    y = x.to(F64) @ p[name].to(F64).T
    return y + p[name + ".b"].to(F64) if name + ".b" in p else y


def query_temperature(positions: int, coef: float, every: int) -> torch.Tensor:
    """What the query at each of the positions 0 .. positions - 1 is multiplied by."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(positions)], dtype=F64)


def mixed_values(v: torch.Tensor, v0: torch.Tensor, lam: float) -> torch.Tensor:
    return (1.0 - lam) * v + lam * v0


def neighbours_turned(x: torch.Tensor, base: float) -> torch.Tensor:
    """x [T, heads, r]: elements (2e, 2e + 1) of every head turned by position * base^(-2e/r)."""
    T, r = x.shape[0], x.shape[-1]
    out = x.clone()
    for e in range(r // 2):
        a = torch.arange(T, dtype=F64) * base ** (-2.0 * e / r)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, w = x[..., 2 * e], x[..., 2 * e + 1]
        out[..., 2 * e], out[..., 2 * e + 1] = u * c - w * s, w * c + u * s
    return out


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    T = s.shape[-1]
    s = torch.where(torch.arange(T)[None, :] <= torch.arange(T)[:, None], s, torch.full_like(s, -math.inf))
    w = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return w / w.sum(dim=-1, keepdim=True)


def grouped_attention(x: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float,
                      v0: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """(the mixer's output [T, width], its own unmixed values [T, G, dv]); ``v0``: the values to mix in, or None.  A bias
    counts where ``p`` holds one, the query temperature where ``m`` gives one, the gate where ``p`` holds its rows."""
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = project(x, p, "q").view(T, H, d), project(x, p, "k").view(T, G, d)
    own = project(x, p, "v").view(T, G, dv)
    q, k = rms_norm(q, p["q.norm"], eps), rms_norm(k, p["k.norm"], eps)
    if m.get("q_temp"):
        q = q * query_temperature(T, float(m["q_temp"]["coef"]), int(m["q_temp"]["every"]))[:, None, None]
    v = own if v0 is None else mixed_values(own, v0, float(p["vmix"]))
    o = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        o[:, h] = causal_softmax((q[:, h] @ k[:, g].T) * float(m["scale"])) @ v[:, g]
    o = o.reshape(T, H * dv)
    if "g" in p:
        o = o * sigmoid(project(x, p, "g"))
    return project(o, p, "o"), own


def latent_attention(x: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = x.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = project(rms_norm(project(x, p, "dq"), p["dq.norm"], eps), p, "uq").view(T, H, d + r)
    down = project(x, p, "dkv")
    c = rms_norm(down[:, :rank], p["dkv.norm"], eps)
    key_rot, q_rot = down[:, None, rank:], q[:, :, d:]
    if r:
        key_rot, q_rot = neighbours_turned(key_rot, float(m["rot"]["base"])), neighbours_turned(q_rot, float(m["rot"]["base"]))
    key, val = project(c, p, "uk").view(T, H, d), project(c, p, "uv").view(T, H, dv)
    o = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        s = (q[:, h, :d] @ key[:, h].T + q_rot[:, h] @ key_rot[:, 0].T) * float(m["scale"])
        o[:, h] = causal_softmax(s) @ val[:, h]
    o = o * sigmoid(project(x, p, "g"))[:, :, None]
    return project(o.reshape(T, H * dv), p, "o")


def feed_forward(x: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    a = project(x, p, "gate")
    return project(a * sigmoid(a) * project(x, p, "up"), p, "down")


def layer_tensors(weights: Dict[str, torch.Tensor], layer: int, part: str) -> Dict[str, torch.Tensor]:
    pre = f"l{layer}.{part}."
    return {k[len(pre):]: v.to(F64) for k, v in weights.items() if k.startswith(pre)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int]) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """Returns (logits [T, vocab], the residual stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    x = weights["embed"].to(F64)[list(tokens)]
    v0, after = None, []
    for i, L in enumerate(cfg["layers"]):
        p, m = layer_tensors(weights, i, "mix"), L["mixer"]
        if L["type"] == "latent_attention":
            y = latent_attention(x, p, m, eps)
        else:
            y, own = grouped_attention(x, p, m, eps, v0 if m.get("v_mix") else None)
            if m.get("v_mix") and v0 is None:
                v0 = own
        x = x + rms_norm(y, weights[f"l{i}.norm1"], eps)
        if L.get("mlp") is not None:
            x = x + rms_norm(feed_forward(x, layer_tensors(weights, i, "mlp")), weights[f"l{i}.norm2"], eps)
        after.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["head"].to(F64).T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = float(cap) * torch.tanh(logits / float(cap))
    return logits, after
