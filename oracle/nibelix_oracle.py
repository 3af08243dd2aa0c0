"""Plain, slow restatement of the Nibelix architecture in float64 PyTorch (test infrastructure only; the
product never imports it).  One function per mechanism; whole sequences only: no cache, no pages, no
state slots, no batching, no fused forms, so every schedule of the engine can be compared against it.

Notation: x residual [T, width]; W[name] checkpoint tensors (linear weights [out, in]); t a position
(0-based inside its sequence); rms(v) = v / sqrt(mean(v^2) + eps)."""
from __future__ import annotations

import math
from typing import Dict, List

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)


def silu(v: torch.Tensor) -> torch.Tensor:
    return v * torch.sigmoid(v)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def dynamic_tanh(x, W, name):
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


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


def lightning_rule(q, k, v, decay):
    """one head: q, k [T, d], v [T, dv], one number `decay` -> read-outs [T, dv], final state [d, dv]"""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def lightning_mixer(h, W, p, m, eps):
    """linear attention with a fixed decay per head; one norm over all heads, sigmoid gate per channel"""
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ W[p + n].T).view(T, H, s) for n, s in (("q", d), ("k", d), ("v", dv)))
    o = torch.stack([lightning_rule(q[:, a], k[:, a], v[:, a], m["decay"][a])[0] for a in range(H)], 1)
    o = rms(o.reshape(T, H * dv), eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def windowed_map(q, k, v, scale, window):
    """one softmax map: q, k [T, d], v [T, dv]; a query sees itself and the window - 1 keys before it (0: all)"""
    T = q.shape[0]
    t = torch.arange(T)
    back = t[:, None] - t[None, :]
    hidden = back < 0
    if window:
        hidden = hidden | (back >= window)
    return torch.softmax((q @ k.T * scale).masked_fill(hidden, float("-inf")), -1) @ v


def diff_lambda(W, p, diff):
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, W, p, m, eps):
    """differential attention: two maps per head over the same values, sliding window, sigmoid gate per head"""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (h @ W[p + "q"].T).view(T, 2 * H, d), (h @ W[p + "k"].T).view(T, 2 * G, d)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    q, k = (rotate_halves(u, m["rot"]["dims"], m["rot"]["base"]) for u in (q, k))
    gate, lam = torch.sigmoid(h @ W[p + "g"].T), diff_lambda(W, p, m["diff"])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        a1, a2 = (windowed_map(q[:, 2 * a + j], k[:, 2 * g + j], v[:, g], m["scale"], m["mask"]["size"]) for j in (0, 1))
        out[:, a] = combine_maps(a1, a2, lam, m["diff"], eps) * gate[:, a:a + 1]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def dense_ff(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert_ff(h, W, p):
    return gelu_erf(h @ W[p + "up"].T) @ W[p + "down"].T


def route(h, w_router, correction, r):
    """-> chosen outputs [T, top] (indices), their weights [T, top]"""
    s = torch.softmax(h @ w_router.T, -1)
    choice = s + correction
    T, E = choice.shape
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = E // g["count"]
    best = choice.view(T, g["count"], size).amax(-1).topk(g["keep"], -1).indices
    barred = torch.ones(T, g["count"], dtype=torch.bool)
    barred.scatter_(1, best, False)
    choice = choice.masked_fill(barred.repeat_interleave(size, 1), float("-inf"))
    idx = choice.topk(r["top"], -1).indices
    return idx, s.gather(1, idx) * r["scale"]


def moe_ff(h, W, p, mlp):
    r = mlp["router"]
    idx, wt = route(h, W[p + "router"], W[p + "correction"], r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(idx[t].tolist(), wt[t]):
            out[t] += w * (h[t] if e >= r["experts"] else expert_ff(h[t], W, p + f"e{e}."))
    if mlp.get("shared"):
        out += torch.sigmoid(h @ W[p + "shared.sg"].T) * expert_ff(h, W, p + "shared.")
    return out


def layer(x, W, i, spec, config):
    """both sublayers read the same x through a norm of their own"""
    eps, p, m = config["norm"]["eps"], f"l{i}.", spec["mixer"]
    mixer = {"lightning": lightning_mixer, "attention": attention_mixer}[spec["type"]]
    y = mixer(dynamic_tanh(x, W, p + "norm1"), W, p + "mix.", m, eps) * W[p + "ls1"]
    mlp = spec.get("mlp")
    if mlp is not None:
        h = dynamic_tanh(x, W, p + "norm2")
        y = y + (dense_ff(h, W, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp)) * W[p + "ls2"]
    return x + config["residual_mult"] * y


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, layer_outputs: List[torch.Tensor] = None):
    """-> logits [T, vocab] (float64) of one whole sequence"""
    W = {k: v.to(F64) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(config["layers"]):
        x = layer(x, W, i, spec, config)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    z = dynamic_tanh(x, W, "final.norm") @ W["head"].T
    cap = config.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


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
