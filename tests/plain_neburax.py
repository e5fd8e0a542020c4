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


# ---- how safe the routers' choices are ------------------------------------------------------------------------------------
def choice_margins(scores, top: int):
    """For rows of choice scores [N, E]: how far the last chosen lies above the first rejected, per row."""
    if top >= scores.shape[1]:
        return torch.full((scores.shape[0],), math.inf, dtype=scores.dtype)
    ranked = scores.sort(-1, descending=True).values
    return ranked[:, top - 1] - ranked[:, top]


# ---- random weights for the tests -------------------------------------------------------------------------------------------
def random_model(config: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    """Weights whose values are bfloat16 numbers.  The routers are made robust against rounding, so that a bfloat16
    engine and this implementation choose the same experts: the first columns of the embedding carry, per token id, the
    router's logits (a router's row e reads column e, plus a little of everything else), drawn again until every layer's
    choice has a safe margin; the norms' gains are zero in those columns, so nothing is ever added there."""
    g = torch.Generator().manual_seed(seed)
    W, V = config["width"], config["vocab"]
    own = [(i, L) for i, L in enumerate(config["layers"]) if L.get("weights_of") is None]
    mixtures = [(i, L["mlp"]) for i, L in own if L.get("mlp") and L["mlp"]["kind"] == "moe"]
    routes = {i: f["router"]["experts"] + int(f["router"].get("identity") or 0) for i, f in mixtures}
    E_max = max(list(routes.values()) + [0])
    assert E_max <= W // 2

    def mat(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16().to(dtype)

    def vec(n, around=0.0, spread=0.1):
        return (around + spread * torch.randn(n, generator=g)).bfloat16().to(dtype)

    def taps(n, K):
        return (torch.randn(n, K, generator=g) * 0.6).bfloat16().to(dtype)

    def out_gain():
        v = vec(W, 0.5)
        v[:E_max] = 0.0
        return v

    t: Dict[str, torch.Tensor] = {"final.norm": vec(W, 1.0)}
    corrections = {}
    for i, f in mixtures:
        corrections[i] = (0.1 * torch.randn(routes[i], generator=g)).bfloat16().double()
        t[f"l{i}.mlp.correction"] = corrections[i].to(dtype)
    embed = torch.randn(V, W, generator=g)
    if E_max:
        accepted = torch.zeros(0, E_max, dtype=torch.float64)
        for _ in range(400):
            if len(accepted) >= V:
                break
            cand = ((torch.rand(4096, E_max, generator=g) * 2 - 1) * 1.5).bfloat16().double()
            for i, f in mixtures:
                cand = cand[choice_margins(torch.softmax(2.0 * cand[:, :routes[i]], -1) + corrections[i], f["router"]["top"]) > 0.02]
            accepted = torch.cat([accepted, cand])
        assert len(accepted) >= V, "no safe logits found for some token ids"
        embed[:, :E_max] = accepted[:V].float()
    t["embed"] = embed.bfloat16().to(dtype)
    for i, L in own:
        p, m = f"l{i}.", L["mixer"]
        t[p + "norm1"] = out_gain()
        q = p + "mix."
        if L["type"] == "mamba2":
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner = H * P
            C = inner + 2 * G * N
            t[q + "in"] = mat(inner + C + H, W, 1.5)
            t[q + "conv"], t[q + "conv.b"] = taps(C, m["conv"]), vec(C, 0.0, 0.3)
            t[q + "dt_bias"], t[q + "A_log"], t[q + "D"] = vec(H, -2.0, 1.0), vec(H, -1.0, 1.5), vec(H, 0.7, 0.4)
            t[q + "norm"], t[q + "o"] = vec(inner, 1.0), mat(W, inner)
        else:
            a, b = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            t[q + "left.q"], t[q + "left.k"], t[q + "left.v"] = mat(H * d, W), mat(G * d, W), mat(G * dv, W)
            t[q + "left.q.norm"], t[q + "left.k.norm"], t[q + "left.o"] = vec(H * d, 1.3, 0.3), vec(G * d, 1.3, 0.3), mat(W, H * dv)
            n, K, blocks = b["width"], b["conv"], b["blocks"]
            q += "right."
            t[q + "y"], t[q + "y.b"], t[q + "x"], t[q + "x.b"] = mat(n, W), vec(n, 0.0, 0.5), mat(n, W), vec(n, 0.0, 0.5)
            t[q + "conv"], t[q + "conv.b"], t[q + "lam"], t[q + "o"] = taps(n, K), vec(n, 0.0, 0.3), vec(n, -2.0, 2.0), mat(W, n)
            size = n // blocks
            for r in ("ra", "ri"):
                t[q + r] = (torch.randn(blocks, size, size, generator=g) * 1.5 / math.sqrt(size)).bfloat16().to(dtype)
                t[q + r + ".b"] = vec(n, 0.0, 0.7).view(blocks, size)
        f = L.get("mlp")
        if not f:
            continue
        t[p + "norm2"] = out_gain()
        q = p + "mlp."
        if f["kind"] == "dense":
            t[q + "up"], t[q + "up.b"], t[q + "down"], t[q + "down.b"] = mat(f["ff"], W), vec(f["ff"], 0.0, 0.3), mat(W, f["ff"]), vec(W, 0.0, 0.5)
            continue
        sizes = {f"e{e}": f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f.get("shared"):
            sizes["shared"] = f["shared"]["ff"]
        for name, ff in sizes.items():
            t[f"{q}{name}.gate"], t[f"{q}{name}.up"], t[f"{q}{name}.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
        router = torch.randn(routes[i], W, generator=g) * 0.004 / math.sqrt(W)
        router[:, :E_max] = 0.0
        for e in range(routes[i]):
            router[e, e] = 2.0
        t[q + "router"] = router.bfloat16().to(dtype)
    return t
