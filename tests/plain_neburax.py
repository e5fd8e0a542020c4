"""Neburax, written down plainly: one slow function per mechanism, in the precision of the tensors it is given (the tests
pass float64), token by token where the design has a recurrence.  Shares no code with the package.

Notation: W width, T tokens of ONE sequence (positions 0..T-1), H query or state heads, G key/value heads or groups.
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp_min(z, 0.0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K], bias [C]: y_t = bias + sum_j taps[:, K-1-j] * x_{t-j}, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = bias.expand_as(x).clone()
    for j in range(min(K, T)):
        y[j:] += taps[:, K - 1 - j] * x[:T - j]
    return y


# ---- attention inside chunks, queries and keys normed as whole rows -----------------------------------------------------
def chunked_attention(q, k, v, scale: float, chunk: int):
    """q [T, H, d], k [S, G, d], v [S, G, dv] with the queries the last T of S positions: softmax over the earlier keys of
    the query's own chunk, chunks counted from position 0."""
    T, H, _ = q.shape
    S, G, dv = v.shape
    i, j = torch.arange(S - T, S)[:, None], torch.arange(S)[None, :]
    hidden = (j > i) | (j // chunk != i // chunk)
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, g]
    return out


def left_mixer(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w["q"].T, eps) * w["q.norm"]).view(T, H, d)
    k = (rms(h @ w["k"].T, eps) * w["k.norm"]).view(T, G, d)
    v = (h @ w["v"].T).view(T, G, dv)
    return chunked_attention(q, k, v, float(m["scale"]), int(m["mask"]["size"])).reshape(T, H * dv) @ w["o"].T


# ---- recurrences --------------------------------------------------------------------------------------------------------------
def block_products(u, mats, bias):
    """u [T, n * b], mats [n, b, b], bias [n, b]: every block of u through its own matrix."""
    n, b = bias.shape
    parts = [u[:, i * b:(i + 1) * b] @ mats[i].T + bias[i] for i in range(n)]
    return torch.cat(parts, 1)


def gated_linear_recurrence(u, r, i, lam, state=None):
    """All [T, C], lam [C]: S <- a S + sqrt(1 - a^2) i u with a = exp(-8 r softplus(lam)); returns (S of every token, the
    last)."""
    S = torch.zeros(u.shape[1], dtype=u.dtype) if state is None else state.clone()
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def right_mixer(h, w):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    r = torch.sigmoid(block_products(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(block_products(u, w["ri"], w["ri.b"]))
    s, _ = gated_linear_recurrence(u, r, i, w["lam"])
    return (s * y) @ w["o"].T


def parallel_mixer(h, w, m, eps):
    return (float(m["left_scale"]) * left_mixer(h, _sub(w, "left."), m["left"], eps)
            + float(m["right_scale"]) * right_mixer(h, _sub(w, "right.")))


def state_space_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, P], B and C [T, G, N], dt [T, H]: S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; returns
    (y [T, H, P], the state after them [H, N, P])."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return out, S


def gated_group_norm(y, z, gain, groups: int, eps):
    """The gate first, then every one of ``groups`` equal parts over its own root mean square, then the gain."""
    T, n = y.shape
    return rms((y * silu(z)).view(T, groups, n // groups), eps).reshape(T, n) * gain


def state_space_mixer(h, w, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    y, _ = state_space_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_group_norm(y.reshape(T, inner), z, w["norm"], int(m["norm_groups"]), eps) @ w["o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------------------------
def squared_relu_ff(h, w):
    return torch.relu(h @ w["up"].T + w["up.b"]) ** 2 @ w["down"].T + w["down.b"]


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(z, correction, top):
    """z [E] -> (chosen, weights): the choice by softmax score plus correction, the weights by the score alone, over
    their sum."""
    s = torch.softmax(z, -1)
    order = sorted(range(len(z)), key=lambda e: (-float(s[e] + correction[e]), e))[:top]
    return order, s[order] / (s[order].sum() + 1e-20)


def moe_ff(h, w, f: dict, routers=None):
    E, top = int(f["router"]["experts"]), int(f["router"]["top"])
    z = h @ w["router"].T
    if routers is not None:
        routers.append((top, torch.softmax(z, -1) + w["correction"]))
    out = gated_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"]) if f.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weights = choose_experts(z[t], w["correction"], top)
        for e, s in zip(chosen, weights):
            x = h[t:t + 1]
            out[t] += s * (gated_ff(x, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]) if e < E else x)[0]
    return out


# ---- the model ------------------------------------------------------------------------------------------------------------------
def _sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def owner(config: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    j = config["layers"][i].get("weights_of")
    return i if j is None else owner(config, j)


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, tap=None, routers=None):
    """Logits [T, vocab] of one sequence; ``tap(i, x)`` sees the stream after every layer; ``routers``, a list, collects
    ``(top, choice scores)`` of every routed feed-forward."""
    eps = float(config["norm"]["eps"])
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{owner(config, i)}."
        mw = _sub(weights, p + "mix.")
        y = parallel_mixer(x, mw, layer["mixer"], eps) if layer["type"] == "parallel" else state_space_mixer(x, mw, layer["mixer"], eps)
        x = x + rms(y, eps) * weights[p + "norm1"]
        f = layer.get("mlp")
        if f:
            fw = _sub(weights, p + "mlp.")
            y = squared_relu_ff(x, fw) if f["kind"] == "dense" else moe_ff(x, fw, f, routers)
            x = x + rms(y, eps) * weights[p + "norm2"]
        if tap is not None:
            tap(i, x)
    return (rms(x, eps) * weights["final.norm"]) @ weights["embed"].T


def greedy(config: dict, weights: Dict[str, torch.Tensor], prompt, steps: int) -> List[int]:
    """Greedy continuation, recomputing the whole sequence every step (the lower id wins a tie)."""
    toks = list(prompt)
    out = []
    for _ in range(steps):
        nxt = int(torch.argmax(forward(config, weights, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
