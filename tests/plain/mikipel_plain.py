"""Plain, slow Mikipel: whole sequences, no cache, one function per mechanism.

The oracle of the Mikipel tests.  It shares no code with toyinfer_b200: the configuration is a dict as config.json holds
it, the weights a dict of tensors by checkpoint name, and every mechanism is written with elementary torch operations in
float64, token by token where the mechanism is a recurrence.

The design in this file's notation (one row per token; W applies as W x; weights [out, in]):

* embedding:   X_0 = E[token] * embedding.scale;  y_0 = X_0
* norm:        n(v; w) = v / sqrt(mean(v^2) + eps) * w
* layer i:     z = n(y_i; norm1);  z'_t = z_t + (z_{t-1} - z_t) * shift  (z_{-1} = 0);
               X_{i+1} = y_i + residual_mult * (mixer(z') + feed_forward(z));  y_{i+1} = sum_{j <= i+1} dwa_i[j] X_j
* attention:   q = Wq z' [H, d], k = Wk z' [G, d], v = Wv z' [G, dv]; the first R = rot.dims elements of every head of q and
               k turned in pairs (e, e + R/2) by p f_e, f_e = base^(-2e/R) / factor; every head of q and k over its own
               root mean square; s_ij = (q_i . k_j) * scale; softmax over j <= i; head h reads kv head h // (H / G); Wo
* latent_attention: q = Wq z', head by head [d plain | r rotated]; Wdkv z' = [c' | b']; c = n(c'; dkv.norm); key of head h
               [Wuk_h c | turn(b')], value Wuv_h c; turning pairs (2e, 2e + 1); the scores and the softmax as above; Wo
* delta:       q, k [G, d] and v [H, dv] each through a causal convolution over time per channel and silu; q and k over
               sqrt(sum of squares + 1e-6) per head, q also times d^(-1/2); beta = sigmoid(Wb z');
               g = exp(-exp(A_log) * softplus(Wa z' + dt_bias)); per head S [d, dv] from zero:
               S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;
               n(o; norm) per head times silu(Wg z'); Wo.  Head h uses query/key head h // (H / G)
* dense:       Wdown gelu(Wup z), gelu(a) = a (1 + erf(a / sqrt(2))) / 2
* experts:     t = Wr z + b; the ``top`` largest t; weights softmax over those t; expert e Wdown_e (silu(Wgate_e z) * (Wup_e z))
* output:      r = E n(y_last; final.norm);  logits = cap * tanh(r / cap)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence, Tuple

import torch

F64 = torch.float64


def rms_norm(v: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    v = v.to(F64)
    out = v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)
    return out if w is None else out * w.to(F64)


def sigmoid(a: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-a))


def silu(a: torch.Tensor) -> torch.Tensor:
    return a * sigmoid(a)


def softplus(a: torch.Tensor) -> torch.Tensor:
    return torch.clamp(a, min=0.0) + torch.log1p(torch.exp(-a.abs()))


def gelu(a: torch.Tensor) -> torch.Tensor:
    return 0.5 * a * (1.0 + torch.erf(a / math.sqrt(2.0)))


def token_shift(z: torch.Tensor, mix: torch.Tensor) -> torch.Tensor:
    before = torch.cat([torch.zeros_like(z[:1]), z[:-1]], dim=0)
    return z + (before - z) * mix.to(F64)


def depth_average(results: Sequence[torch.Tensor], w: torch.Tensor) -> torch.Tensor:
    """sum_j w[j] * results[j] over the embedding and every layer's result so far."""
    assert len(results) == w.numel()
    return sum(float(w[j]) * r for j, r in enumerate(results))


def frequencies(rot: dict) -> torch.Tensor:
    R = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * torch.arange(R // 2, dtype=F64) / R)
    if rot.get("scaling"):
        f = f / float(rot["scaling"]["factor"])
    return f


def turn(x: torch.Tensor, rot: Optional[dict], pairs: str) -> torch.Tensor:
    """x [T, heads, n]: the first rot.dims elements of every head turn by position * frequency; ``pairs`` "half" or "neighbours"."""
    if not rot:
        return x
    R = int(rot["dims"])
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    out = x.clone()
    if pairs == "half":
        u, v = x[..., : R // 2], x[..., R // 2: R]
        out[..., : R // 2], out[..., R // 2: R] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., 0:R:2], x[..., 1:R:2]
        out[..., 0:R:2], out[..., 1:R:2] = u * c - v * s, v * c + u * s
    return out


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    T = s.shape[-1]
    s = torch.where(torch.arange(T)[None, :] <= torch.arange(T)[:, None], s, torch.full_like(s, -math.inf))
    w = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return w / w.sum(dim=-1, keepdim=True)


def attention(z: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = z.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (z @ p["q"].T).view(T, H, d), (z @ p["k"].T).view(T, G, d), (z @ p["v"].T).view(T, G, dv)
    q, k = turn(q, m.get("rot"), "half"), turn(k, m.get("rot"), "half")
    q, k = rms_norm(q, None, eps), rms_norm(k, None, eps)
    o = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        o[:, h] = causal_softmax((q[:, h] @ k[:, g].T) * float(m["scale"])) @ v[:, g]
    return o.reshape(T, H * dv) @ p["o"].T


def latent_attention(z: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = z.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (z @ p["q"].T).view(T, H, d + r)
    down = z @ p["dkv"].T
    c = rms_norm(down[:, :rank], p["dkv.norm"], eps)
    rot = m.get("rot") if r else None
    key_rot = turn(down[:, None, rank:], rot, "neighbours")[:, 0]
    q_rot = turn(q[:, :, d:], rot, "neighbours")
    key, val = (c @ p["uk"].T).view(T, H, d), (c @ p["uv"].T).view(T, H, dv)
    o = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        s = (q[:, h, :d] @ key[:, h].T + q_rot[:, h] @ key_rot.T) * float(m["scale"])
        o[:, h] = causal_softmax(s) @ val[:, h]
    return o.reshape(T, H * dv) @ p["o"].T


def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n]: the last column weighs the current token; zeros before the start; then silu."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1 - j)
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return silu(out)


def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               S: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """q, k [T, G, d] unit vectors (q scaled), v [T, H, dv], g, beta [T, H]; S [H, d, dv] or None -> (o [T, H, dv], S)."""
    T, H, dv = v.shape
    G, d = q.shape[1], q.shape[2]
    S = torch.zeros(H, d, dv, dtype=F64) if S is None else S.clone()
    o = torch.zeros(T, H, dv, dtype=F64)
    own = torch.arange(H) // (H // G)                   # the query/key head of every value head
    for t in range(T):
        kk, qq = k[t, own], q[t, own]
        M = g[t, :, None, None] * S
        u = beta[t, :, None] * (v[t] - torch.einsum("hdv,hd->hv", M, kk))
        S = M + kk[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, qq)
    return o, S


def delta_unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta(z: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = z.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(z @ p["q"].T, p["q.conv"]).view(T, G, d)
    k = short_conv(z @ p["k"].T, p["k.conv"]).view(T, G, d)
    v = short_conv(z @ p["v"].T, p["v.conv"]).view(T, H, dv)
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(z @ p["a"].T + p["dt_bias"]))
    beta = sigmoid(z @ p["b"].T)
    o, _ = delta_scan(delta_unit(q) * d ** -0.5, delta_unit(k), v, g, beta)
    o = rms_norm(o, p["norm"], eps).reshape(T, H * dv) * silu(z @ p["g"].T)
    return o @ p["o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "delta": delta}


def dense_ff(z: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    return gelu(z @ p["up"].T) @ p["down"].T


def route(t: torch.Tensor, top: int) -> Tuple[List[int], torch.Tensor]:
    """One token's router logits (the bias added) -> (the chosen experts, their weights)."""
    chosen = sorted(range(t.numel()), key=lambda e: (-float(t[e]), e))[:top]
    w = torch.exp(t[chosen] - t[chosen].max())
    return chosen, w / w.sum()


def experts_ff(z: torch.Tensor, p: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    logits = z @ p["router"].T + p["router.b"]
    out = torch.zeros(z.shape[0], p["e0.down"].shape[0], dtype=F64)
    weight = torch.zeros_like(logits)                   # [T, experts], zero where an expert is not chosen
    for t in range(z.shape[0]):
        chosen, w = route(logits[t], int(f["router"]["top"]))
        weight[t, chosen] = w.to(F64)
    for e in range(logits.shape[1]):
        who = weight[:, e].nonzero()[:, 0]
        zz = z[who]
        out[who] += weight[who, e, None] * ((silu(zz @ p[f"e{e}.gate"].T) * (zz @ p[f"e{e}.up"].T)) @ p[f"e{e}.down"].T)
    return out


def feed_forward(z: torch.Tensor, p: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    return dense_ff(z, p) if f["kind"] == "dense" else experts_ff(z, p, f)


def layer_tensors(weights: Dict[str, torch.Tensor], layer: int, part: str) -> Dict[str, torch.Tensor]:
    pre = f"l{layer}.{part}."
    return {k[len(pre):]: v.to(F64) for k, v in weights.items() if k.startswith(pre)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int]) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """Returns (logits [T, vocab], the averaged stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    E = weights["embed"].to(F64)
    mult = float(cfg.get("residual_mult", 1.0))
    y = E[list(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    results, after = [y], []
    for i, L in enumerate(cfg["layers"]):
        w = lambda name: weights[f"l{i}.{name}"].to(F64)
        z = rms_norm(y, w("norm1"), eps)
        out = MIXERS[L["type"]](token_shift(z, w("shift")), layer_tensors(weights, i, "mix"), L["mixer"], eps)
        if L.get("mlp") is not None:
            out = out + feed_forward(z, layer_tensors(weights, i, "mlp"), L["mlp"])
        results.append(y + mult * out)
        y = depth_average(results, w("dwa"))
        after.append(y)
    logits = rms_norm(y, weights["final.norm"], eps) @ E.T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = float(cap) * torch.tanh(logits / float(cap))
    return logits, after
