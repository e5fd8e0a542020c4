"""Nugolorn, written down plainly: one slow function per mechanism, in the precision of the tensors it is given
(the tests pass float64), token by token where the design has a recurrence.  Shares no code with the package.

Notation: W width, T tokens of ONE sequence (positions 0..T-1), H query or value heads, G key/value heads.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def silu(z):
    return z * torch.sigmoid(z)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_rms_norm(x, w, eps, groups):
    """Every one of ``groups`` equal parts of the row over its own root mean square, the row times ``w``."""
    T, W = x.shape
    return rms(x.reshape(T, groups, W // groups), eps).reshape(T, W) * w


# ---- what happens before the scores ------------------------------------------------------------------------------------
def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, K-1-j] * x_{t-j}, zeros before the start."""
    T = x.shape[0]
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(K):
        if j < T:
            y[j:] += taps[:, K - 1 - j] * x[:T - j]
    return y


def rotary_frequencies(base: float, dims: int) -> List[float]:
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def rotate_halves(x, positions, freqs):
    """x [T, heads, d]; dimension i pairs with i + len(freqs), for i < len(freqs); the rest passes."""
    half = len(freqs)
    out = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(x.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def query_temperature(positions, coef: float, every: int, dtype):
    return torch.tensor([1.0 + coef * math.log((int(p) + 1) // every + 1) for p in positions], dtype=dtype)


# ---- the two kinds of attention ------------------------------------------------------------------------------------------
def sigmoid_attention(q, k, v, scale: float, bias):
    """q [T, H, d], k [S, G, d], v [S, G, dv] with the queries the last T of S positions: weights sigmoid(score + bias_h),
    not normalised."""
    T, H, _ = q.shape
    S, G, dv = v.shape
    seen = torch.arange(S)[None, :] <= torch.arange(S - T, S)[:, None]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        w = torch.sigmoid((q[:, h] @ k[:, g].T) * scale + bias[h]) * seen
        out[:, h] = w @ v[:, g]
    return out


def log_bias_attention(q, k, v, scale: float, r1, r2):
    """Softmax attention whose scores lose r1_h * ln(1 + r2_h * distance)."""
    T, H, _ = q.shape
    S, G, dv = v.shape
    i, j = torch.arange(S - T, S)[:, None], torch.arange(S)[None, :]
    distance = (i - j).clamp_min(0).to(q.dtype)
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale - r1[h] * torch.log(1.0 + r2[h] * distance)
        out[:, h] = torch.softmax(s.masked_fill(j > i, -math.inf), -1) @ v[:, g]
    return out


def attention_mixer(h, w: Dict[str, torch.Tensor], m: dict, shared=None):
    """Returns (output, (keys, values) as a later layer may read them)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freqs = rotary_frequencies(m["rot"]["base"], m["rot"]["dims"]) if m.get("rot") and m["rot"]["dims"] else []
    pos = torch.arange(T)
    q = causal_conv(h @ w["q"].T + w["q.b"], w["q.conv"]).view(T, H, d)
    q = rotate_halves(q, pos, freqs)
    if m.get("kv_from") is None:
        k = causal_conv(h @ w["k"].T + w["k.b"], w["k.conv"]).view(T, G, d)
        v = causal_conv(h @ w["v"].T + w["v.b"], w["v.conv"]).view(T, G, dv)
        shared = (rotate_halves(k, pos, freqs), v)
    o = sigmoid_attention(q, shared[0], shared[1], float(m["scale"]), w["pb"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T, shared


def left_mixer(h, w, m):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(range(T), float(m["q_temp"]["coef"]), int(m["q_temp"]["every"]), h.dtype)[:, None, None]
    o = log_bias_attention(q, k, v, float(m["scale"]), w["r1"], w["r2"]).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- recurrences --------------------------------------------------------------------------------------------------------------
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta_rule(q, k, v, beta, decay, state=None):
    """q, k [T, G, d], v [T, H, dv], beta [T, H], decay [T, H, d]; returns (o [T, H, dv], the state after them)."""
    T, H, dv = v.shape
    G, d = k.shape[1:]
    S = torch.zeros(H, d, dv, dtype=v.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, dv, dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = decay[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, g])
            S[h] = S[h] + torch.outer(k[t, g], u)
            out[t, h] = S[h].T @ q[t, g]
    return out, S


def right_mixer(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).view(T, G, d)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).view(T, G, d)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).view(T, H, dv)
    beta = torch.sigmoid(h @ w["b"].T)
    step = torch.nn.functional.softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(T, H, d)
    decay = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
    o, _ = channel_delta_rule(unit(q) * d ** -0.5, unit(k), v, beta, decay)
    gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T).view(T, H, dv)
    return (rms(o, eps) * w["norm"] * gate).reshape(T, H * dv) @ w["o"].T


def side_by_side_mixer(h, w, m, eps):
    left = left_mixer(h, _sub(w, "left."), m["left"])
    right = right_mixer(h, _sub(w, "right."), m["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


def wkv_rule(r, k, v, decay, u, state=None):
    """r, k, v, decay [T, H, d], u [H, d]: the current token's write enters the read-out with the weight u only."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return out, S


def wkv_mixer(h, w, m, eps):
    T, W = h.shape
    H, d = m["heads"], m["dim"]
    before = torch.cat([torch.zeros(1, W, dtype=h.dtype), h[:-1]])
    mix = {s: h + (before - h) * w[f"mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(T, H, d)
    o, _ = wkv_rule(r, k, v, decay, w["u"])
    return (rms(o, eps).reshape(T, H * d) * w["norm"] * gate) @ w["o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------------------------
def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(z, correction, top):
    """z [E] -> (chosen, their softmax scores, not renormalised); the choice goes by score plus correction."""
    s = torch.softmax(z, -1)
    order = sorted(range(len(z)), key=lambda e: (-float(s[e] + correction[e]), e))[:top]
    return order, s[order]


def moe_ff(h, w, f: dict, routers=None):
    E, top = int(f["router"]["experts"]), int(f["router"]["top"])
    z = h @ w["router"].T
    if routers is not None:
        routers.append((top, torch.softmax(z, -1) + w["correction"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, scores = choose_experts(z[t], w["correction"], top)
        for e, s in zip(chosen, scores):
            x = h[t:t + 1]
            out[t] += s * (gated_ff(x, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]) if e < E else x)[0]
    return out


# ---- the model ------------------------------------------------------------------------------------------------------------------
def _sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, tap=None, routers=None):
    """Logits [T, vocab] of one sequence; ``tap(i, x)`` sees the stream after every layer; ``routers``, a list, collects
    ``(top, choice scores)`` of every routed feed-forward."""
    eps, groups = float(config["norm"]["eps"]), int(config["norm"].get("groups", 1))
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    mult = float(config["residual_mult"])
    published: Dict[int, tuple] = {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        mw = _sub(weights, p + "mix.")
        h = group_rms_norm(x, weights[p + "norm1"], eps, groups)
        kind, m = layer["type"], layer["mixer"]
        if kind == "attention":
            y, published[i] = attention_mixer(h, mw, m, published.get(m.get("kv_from")))
        elif kind == "parallel":
            y = side_by_side_mixer(h, mw, m, eps)
        elif kind == "wkv":
            y = wkv_mixer(h, mw, m, eps)
        else:
            raise ValueError(kind)
        f = layer.get("mlp")
        if f:
            fw = _sub(weights, p + "mlp.")
            y = y + (gated_ff(h, fw["gate"], fw["up"], fw["down"]) if f["kind"] == "dense" else moe_ff(h, fw, f, routers))
        x = x + mult * y
        if tap is not None:
            tap(i, x)
    return group_rms_norm(x, weights["final.norm"], eps, groups) @ weights["head"].T * float(config["logit_scale"])


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


def router_margin(config: dict, weights: Dict[str, torch.Tensor], tokens) -> float:
    """The smallest margin over the sequence's tokens and layers; the tests assert that their weights leave a safe one, so
    that an engine that rounds differently still chooses the same experts."""
    seen: list = []
    forward(config, weights, tokens, routers=seen)
    return min([float(choice_margins(scores, top).min()) for top, scores in seen] + [math.inf])


# ---- random weights for the tests -------------------------------------------------------------------------------------------
def random_model(config: dict, seed: int, dtype=torch.float32, rank: Optional[int] = None) -> Dict[str, torch.Tensor]:
    """Weights whose values are bfloat16 numbers.  The routers are made robust against rounding, so that a bfloat16
    engine and this implementation choose the same experts: the first columns of the embedding carry, per token id, the
    router's logits (a router's row e reads column e, plus a little of everything else), drawn again until every layer's
    choice has a safe margin at every size the stream's norm may have; every tensor that writes into the stream is small
    in those columns.  ``rank``: the inner size of the low-rank products (else one per product, all different)."""
    g = torch.Generator().manual_seed(seed)
    W, V = config["width"], config["vocab"]
    groups = int(config["norm"].get("groups", 1))
    mixtures = [(i, L["mlp"]) for i, L in enumerate(config["layers"]) if L.get("mlp") and L["mlp"]["kind"] == "moe"]
    routes = {i: f["router"]["experts"] + int(f["router"].get("identity") or 0) for i, f in mixtures}
    E_max = max(list(routes.values()) + [0])
    assert E_max <= W // groups, "the router's columns lie in the first group of the norm"
    ranks = iter(range(3, 1000, 2))

    def low_rank():
        return rank or next(ranks)

    def mat(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16().to(dtype)

    def vec(n, around=0.0, spread=0.1):
        return (around + spread * torch.randn(n, generator=g)).bfloat16().to(dtype)

    def taps(n, K):
        return (torch.randn(n, K, generator=g) * 0.6).bfloat16().to(dtype)

    def writer(i, gain=0.4):                         # [W, i]: output rows of the router's columns are small
        m = torch.randn(W, i, generator=g) * gain / math.sqrt(i)
        m[:E_max] *= 0.001
        return m.bfloat16().to(dtype)

    t: Dict[str, torch.Tensor] = {"head": mat(V, W, 2.0), "final.norm": vec(W, 1.0)}
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
            cand = ((torch.rand(8192, E_max, generator=g) * 2 - 1) * 1.5).bfloat16().double()
            for stride in (12, 1):                                # a coarse look first, then the whole range
                for i, f in mixtures:
                    for step in range(0, 72, stride):             # logits = 2 * column / rms(stream): 0.15 to 3.2
                        z = cand[:, :routes[i]] * 0.15 * 2.0 ** (step / 16)
                        cand = cand[choice_margins(torch.softmax(z, -1) + corrections[i], f["router"]["top"]) > 0.011]
            accepted = torch.cat([accepted, cand])
        assert len(accepted) >= V, "no safe logits found for some token ids"
        embed[:, :E_max] = accepted[:V].float()
    t["embed"] = embed.bfloat16().to(dtype)
    for i, L in enumerate(config["layers"]):
        p = f"l{i}."
        m = L["mixer"]
        t[p + "norm1"] = vec(W, 1.0)
        t[p + "norm1"][:E_max] = 1.0
        if L["type"] == "attention":
            H, G, d, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            rows = [("q", H * d, 2.0)] + ([("k", G * d, 2.0), ("v", G * dv, 1.0)] if m.get("kv_from") is None else [])
            for n, size, gain in rows:
                t[p + f"mix.{n}"], t[p + f"mix.{n}.b"], t[p + f"mix.{n}.conv"] = mat(size, W, gain), vec(size, 0.0, 0.5), taps(size, K)
            t[p + "mix.pb"], t[p + "mix.g"], t[p + "mix.o"] = vec(H, -4.0, 0.7), mat(H, W, 2.0), writer(H * dv)
        elif L["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            t[q + "q"], t[q + "k"], t[q + "v"], t[q + "g"] = mat(H * d, W, 2.0), mat(G * d, W, 2.0), mat(G * dv, W), mat(H * dv, W, 2.0)
            t[q + "r1"], t[q + "r2"], t[q + "o"] = vec(H, 0.6, 0.3), vec(H, 0.5, 0.1).abs(), writer(H * dv)
            H, G, d, dv, K = b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"]
            q = p + "mix.right."
            for n, size in (("q", G * d), ("k", G * d), ("v", H * dv)):
                t[q + n], t[q + n + ".conv"] = mat(size, W, 2.0), taps(size, K)
            ra, rg = low_rank(), low_rank()
            t[q + "b"], t[q + "A_log"], t[q + "dt_bias"] = mat(H, W, 2.0), vec(H, -1.0, 0.7), vec(H * d, 0.0, 1.0)
            t[q + "a1"], t[q + "a2"], t[q + "g1"], t[q + "g2"] = mat(ra, W, 2.0), mat(H * d, ra), mat(rg, W, 2.0), mat(H * dv, rg)
            t[q + "norm"], t[q + "o"] = vec(dv, 1.0), writer(H * dv)
            for side in ("left", "right"):
                out = vec(W, 0.6)
                out[:E_max] = 0.001
                t[p + f"mix.{side}.out"] = out
        else:
            H, d = m["heads"], m["dim"]
            q = p + "mix."
            for s in "rkvgw":
                t[q + f"mu.{s}"] = torch.rand(W, generator=g).bfloat16().to(dtype)
            for s in "rkvg":
                t[q + s] = mat(H * d, W, 1.0)
            r = low_rank()
            t[q + "w1"], t[q + "w2"], t[q + "w0"] = mat(r, W, 2.0), mat(H * d, r), vec(H * d, -1.5, 1.0)
            t[q + "u"], t[q + "norm"], t[q + "o"] = vec(H * d, 0.0, 0.7).view(H, d), vec(H * d, 1.0), writer(H * d)
        f = L.get("mlp")
        if f and f["kind"] == "dense":
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(f["ff"], W, 1.5), mat(f["ff"], W, 1.5), writer(f["ff"])
        elif f:
            ff = f["expert"]["ff"]
            for e in range(f["router"]["experts"]):
                t[f"{p}mlp.e{e}.gate"], t[f"{p}mlp.e{e}.up"], t[f"{p}mlp.e{e}.down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), writer(ff)
            router = torch.randn(routes[i], W, generator=g) * 0.008 / math.sqrt(W)
            router[:, :E_max] = 0.0
            for e in range(routes[i]):
                router[e, e] = 2.0
            t[p + "mlp.router"] = router.bfloat16().to(dtype)
    return t
