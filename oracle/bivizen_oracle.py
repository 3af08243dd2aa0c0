"""Plain, slow restatement of the Bivizen architecture in float64 PyTorch (test infrastructure only; the
product never imports it).  One function per mechanism; whole sequences only: no cache, no pages, no
state slots, no batching, no fused forms, so every schedule of the engine can be compared against it.

Notation: x residual [T, width]; W[name] checkpoint tensors (linear weights [out, in]); t a position
(0-based inside its sequence); rms(v) = v / sqrt(mean(v^2) + eps)."""
from __future__ import annotations

from typing import Dict, List

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)


def silu(v: torch.Tensor) -> torch.Tensor:
    return v * torch.sigmoid(v)


def softplus(v: torch.Tensor) -> torch.Tensor:
    return torch.clamp_min(v, 0.0) + torch.log1p(torch.exp(-v.abs()))


def rotate_halves(u: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """u [T, heads, d]: column i < dims / 2 turns with column i + dims / 2 by t * base^(-2i / dims)"""
    out, half = u.clone(), dims // 2
    t = torch.arange(u.shape[0], dtype=u.dtype)
    for i in range(half):
        ang = t * (base ** (-2.0 * i / dims))
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = u[:, :, i], u[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = a * c - b * s, b * c + a * s
    return out


def softcap(s: torch.Tensor, cap) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def attention_mixer(h, W, p, m, v_first):
    """rotary grouped-query attention with capped scores, values mixed with the first mixing layer's, a
    sigmoid gate per head.  -> (output [T, width], the layer's own values)"""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, d)
    own = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, dv)
    q = rotate_halves(q, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves(k, m["rot"]["dims"], m["rot"]["base"])
    v = own
    if m.get("v_mix") and v_first is not None:
        lam = W[p + "vmix"]
        v = (1.0 - lam) * own + lam * v_first
    gate = torch.sigmoid(h @ W[p + "g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    hidden = torch.triu(torch.ones(T, T, dtype=torch.bool), 1)
    for a in range(H):
        g = a // (H // G)
        s = softcap(q[:, a] @ k[:, g].T * m["scale"], m["softcap"]).masked_fill(hidden, float("-inf"))
        out[:, a] = torch.softmax(s, -1) @ v[:, g] * gate[:, a:a + 1]
    return out.reshape(T, H * dv) @ W[p + "o"].T, own


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps] (the last tap meets the newest input), nothing before position 0"""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * u[:T - back]
    return out


def delta_rule(q, k, v, beta, g):
    """one head: q, k [T, d], v [T, dv], beta, g [T] -> read-outs [T, dv], final state [d, dv]"""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def delta_mixer(h, W, p, m, eps):
    """gated delta rule: short convolutions + SiLU on q, k, v, unit q and k, one decay and one step size per head"""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def conved(name, heads, n):
        return silu(causal_conv(h @ W[p + name].T, W[p + name + ".conv"])).view(T, heads, n)

    def unit(u):
        return u / torch.sqrt(u.pow(2).sum(-1, keepdim=True) + 1e-6)
    q, k, v = unit(conved("q", G, d)) * d ** -0.5, unit(conved("k", G, d)), conved("v", H, dv)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = torch.stack([delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], g[:, a])[0]
                     for a in range(H)], 1)
    o = rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).view(T, H, dv)
    return o.reshape(T, H * dv) @ W[p + "o"].T


def gated_linear_rule(q, k, v, alpha):
    """one head: q, k, alpha [T, d], v [T, dv] -> read-outs [T, dv], final state [d, dv]"""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def gla_mixer(h, W, p, m, eps):
    """gated linear attention: a decay per key channel from a low-rank projection"""
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ W[p + "k"].T).view(T, H, d), (h @ W[p + "v"].T).view(T, H, dv)
    z = h @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = torch.sigmoid(z).pow(1.0 / m["tau"]).view(T, H, d)
    o = torch.stack([gated_linear_rule(q[:, a], k[:, a], v[:, a], alpha[:, a])[0] for a in range(H)], 1)
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, H * dv) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def feed_forward(h, W, p, limit):
    g = torch.clamp_max(h @ W[p + "gate"].T, limit)
    u = torch.clamp(h @ W[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def layer(x, W, i, spec, config, v_first):
    """both sublayers read the one norm's output; -> (x, the values later mixing layers mix in)"""
    eps, p, m = config["norm"]["eps"], f"l{i}.", spec["mixer"]
    h = rms(x, eps) * W[p + "norm1"]
    if spec["type"] == "attention":
        y, own = attention_mixer(h, W, p + "mix.", m, v_first)
        if m.get("v_mix") and v_first is None:
            v_first = own
    elif spec["type"] == "delta":
        y = delta_mixer(h, W, p + "mix.", m, eps)
    elif spec["type"] == "gla":
        y = gla_mixer(h, W, p + "mix.", m, eps)
    else:
        raise ValueError(spec["type"])
    y = y * W[p + "ls1"]
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, W, p + "mlp.", spec["mlp"]["limit"]) * W[p + "ls2"]
    return x + y, v_first


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, layer_outputs: List[torch.Tensor] = None):
    """-> logits [T, vocab] (float64) of one whole sequence"""
    W = {k: v.to(F64) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    v_first = None
    for i, spec in enumerate(config["layers"]):
        x, v_first = layer(x, W, i, spec, config, v_first)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return (rms(x, config["norm"]["eps"]) * W["final.norm"]) @ W["head"].T


def greedy(config, weights, prompt, n_new: int):
    """-> (new ids, top-2 logit margin of every choice)"""
    ids, out, margins = list(prompt), [], []
    for _ in range(n_new):
        last = forward(config, weights, ids)[-1]
        top = torch.topk(last, 2).values
        tok = int(last.argmax())
        out.append(tok)
        margins.append(float(top[0] - top[1]))
        ids.append(tok)
    return out, margins
