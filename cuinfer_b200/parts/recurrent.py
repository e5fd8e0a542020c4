"""Mixers that carry a state (a matrix per head, or a number per channel) from token to token instead of a cache of keys,
and a pair of mixers side by side.

The recurrent ones keep their state in 32 bits in the request's state slot (zero when the request is admitted), read it at the start
of a step and write it back at the end, so a prompt may be cut anywhere.  What enters the recurrence besides the
projections — gates, decays, their logarithms and exponentials, unit norms, the read-out, the norm after it — is 32-bit.

``mlstm`` — a matrix memory with exponential gates.  For the input h, H heads, key size d, value size dv:
``q = Wq h / sqrt(d)``, ``k = Wk h``, ``v = Wv h``; per head a log input gate ``i = c tanh((Wi h + bi) / c)`` and a log
forget gate ``f = logsigmoid(c tanh((Wf h + bf) / c))`` (c = ``gate_cap``); with a running maximum m that starts at 0::

    m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' = exp(f + m - m') n + exp(i - m') k
    o  = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6)

then each head's o divided by its root mean square, times a gain over all heads, times ``sigmoid(Wg h)``, then ``Wo``.
Spec: ``PartSpec("mlstm", num_heads, dim, vdim, gate_cap, eps, names={...})``.

``gated_delta`` — the gated delta rule.  G query/key heads of size d, H value heads of size dv (head i uses q/k head
``i // (H / G)``): q, k, v go through a short causal convolution per channel (``taps`` columns, the last one the current
token's; the last ``taps - 1`` inputs are state too) and SiLU; q and k become unit vectors (``x / sqrt(sum x^2 + 1e-6)``),
q also times ``1 / sqrt(d)``; ``beta = sigmoid(Wb h)`` and ``g = exp(-exp(A_log) * softplus(Wa h + dt_bias))`` per head::

    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q

then each head's o divided by its root mean square over dv, times a gain of dv values shared by the heads, times
``silu(Wg h)``, then ``Wo``.  Spec: ``PartSpec("gated_delta", num_heads, num_kv_heads, dim, vdim, taps, eps, names={...})``.

``channel_delta`` — the gated delta rule with a decay per head and key channel and low-rank gates.  As above, except that the
decay is a vector over the key channels, ``g = exp(-exp(A_log_h) * softplus(A2 (A1 h) + dt_bias))`` laid out [H, d], which
multiplies the rows of S, and the output gate is ``sigmoid(G2 (G1 h))``.  The inner sizes of the two low-rank products are
the checkpoint's.  Spec: ``PartSpec("channel_delta", num_heads, num_kv_heads, dim, vdim, taps, eps, rank, names={...})``
(``rank``: what the random-weights mode draws).

``wkv`` — RWKV-style time mixing.  The five inputs of r, k, v, g and w are interpolations ``h + (h' - h) * mu_s`` between the
row h and the row h' of the token before (zeros before a sequence's first), mix_s below; ``r = Wr mix_r``, ``k = Wk mix_k``, ``v = Wv mix_v`` (H heads of d),
``gate = silu(Wg mix_g)``, decay ``w = exp(-exp(W2 tanh(W1 mix_w) + w0))`` per head and channel::

    o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T

then each head's o divided by its root mean square, times a gain over all heads, times the gate, then ``Wo``.  The previous
h is state too.  Spec: ``PartSpec("wkv", num_heads, dim, eps, rank, names={...})``.

``state_space`` — the state-space recurrence with a scalar decay per head (Mamba-2).  One projection ``W_in h`` gives
``[z (H P) | x (H P) | B (G N) | C (G N) | dt (H)]``; x, B and C pass a short causal convolution per channel (with a bias;
its last ``taps - 1`` inputs are state too) and SiLU; ``dt = softplus(dt + dt_bias)``; head i uses B and C of group
``i // (H / G)``::

    S <- exp(-exp(A_log) dt) S + dt x B^T;  y = S C + D x

then ``y * silu(z)``, each of ``norm_groups`` equal parts over its own root mean square, times a gain, then ``Wo``.  Spec:
``PartSpec("state_space", num_heads, vdim, state_size, groups, taps, norm_groups, eps, names={...})``.

``gated_linear`` — a linear recurrence with one number of state per channel (Griffin's block with the RG-LRU).  Two branches
of ``width`` channels with biases: ``y = gelu_tanh(Wy h + by)`` and ``u = conv(Wx h + bx)``, a short causal convolution per
channel with a bias; u in ``blocks`` equal parts, each with two square matrices: ``r = sigmoid(Ra u + ra)``,
``i = sigmoid(Ri u + ri)``::

    a = exp(-8 r softplus(lam));  S <- a S + sqrt(1 - a^2) i u

then ``Wo (out_scale * S * y)``.  Spec: ``PartSpec("gated_linear", width, blocks, taps, out_scale=1.0, names={...})``.

``side_by_side`` — two mixers on the same input.  Without ``scales``: ``(rms(left) * left.out + rms(right) * right.out) / 2``,
norms of whole rows; with ``scales = (a, b)``: ``a * left + b * right``.
Spec: ``PartSpec("side_by_side", left=PartSpec(...), right=PartSpec(...), eps, scales=None, names={"left": "left", "right": "right",
"out": "out"})``: the mixers' tensors lie under ``left`` and ``right``, the norms' gains are ``left.out`` and ``right.out``.  One of
the two may keep a paged cache; both may keep state.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, List, Optional

import torch

from .. import kernels
from .base import Mixer
from .context import StepContext
from .linear import Linear, dense_operand, padded_rows, per_head_products
from .registry import MIXERS
from .spec import PartSpec, StateNeed, TensorSpec

MLSTM_FLOOR = 1e-6          # added to the read-out's denominator
DELTA_UNIT_EPS = 1e-6       # inside the root of the unit norm of queries and keys
FEW_ROWS = 16               # rows up to which the state-space mixer's projections are one product in 32 bits
LRU_DECODE_MAX_ROWS = 64    # rows up to which a step of single tokens takes the gated linear recurrence in one launch


def _names(spec: PartSpec, defaults: Dict[str, str]) -> Dict[str, str]:
    names = dict(defaults)
    names.update(spec.get("names") or {})
    return names


@MIXERS.register("mlstm")
class MatrixMemory(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.num_heads, self.dim, self.vdim = int(spec.num_heads), int(spec.dim), int(spec.vdim)
        self.gate_cap = float(spec.gate_cap)
        self.eps = float(spec.get("eps", 1e-6))
        if min(self.num_heads, self.dim, self.vdim) <= 0 or not self.gate_cap > 0:
            raise ValueError("mlstm: sizes and gate_cap must be positive")
        if self.dim > 256:
            raise ValueError(f"mlstm: key size {self.dim} is beyond what the scan kernel keeps in registers (256)")
        n = _names(spec, {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "i": "i", "f": "f",
                          "i_bias": "i.b", "f_bias": "f.b"})
        p, H, d, dv = prefix, self.num_heads, self.dim, self.vdim
        self.main = Linear([f"{p}.{n['q']}", f"{p}.{n['k']}", f"{p}.{n['v']}", f"{p}.{n['g']}"], [H * d, H * d, H * dv, H * dv],
                           hidden_size, dtype)
        self.gates = Linear([f"{p}.{n['i']}", f"{p}.{n['f']}"], [H, H], hidden_size, dtype)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], H * dv, dtype)
        self._vec_specs = [TensorSpec(f"{p}.{n['norm']}", (H * dv,), keep_stored_precision=True, init="ones"),
                           TensorSpec(f"{p}.{n['i_bias']}", (H,), keep_stored_precision=True, init="zeros"),
                           TensorSpec(f"{p}.{n['f_bias']}", (H,), keep_stored_precision=True, init="zeros")]
        self.gain = self.i_bias = self.f_bias = None

    def tensors(self) -> List[TensorSpec]:
        return self.main.tensors() + self.gates.tensors() + self.o.tensors() + self._vec_specs

    def load(self, store) -> None:
        for lin in (self.main, self.gates, self.o):
            lin.load(store)
        self.gain, self.i_bias, self.f_bias = (store.get(s) for s in self._vec_specs)
        if self.i_bias.dtype != self.f_bias.dtype:
            self.i_bias, self.f_bias = self.i_bias.float(), self.f_bias.float()

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.main.weight

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return StateNeed((self.num_heads, self.dim * self.vdim + self.dim + 1), "float32")

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return (self.main.workspace_bytes(tokens) + tokens * 2 * self.num_heads * 4 + tokens * self.num_heads * self.vdim * (4 + width)
                + self.o.workspace_bytes(tokens))

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        H, d, dv = self.num_heads, self.dim, self.vdim
        rows = self.main.forward(x)
        gates = self.gates.forward(x, out_dtype=torch.float32)
        q, k, v, g = rows[:, :H * d], rows[:, H * d:2 * H * d], rows[:, 2 * H * d:2 * H * d + H * dv], rows[:, 2 * H * d + H * dv:]
        o = torch.empty((rows.shape[0], H * dv), dtype=torch.float32, device=rows.device)
        kernels.mlstm_scan(q, k, v, gates, self.i_bias, self.f_bias, self.gate_cap, d ** -0.5, ctx.run_state(run),
                           ctx.query_start_loc, ctx.state_slots, o, H, d, dv, floor=MLSTM_FLOOR)
        out = torch.empty((rows.shape[0], H * dv), dtype=rows.dtype, device=rows.device)
        kernels.head_rms_gate(o, g, self.gain, self.eps, False, out, H, dv)
        return self.o.forward(out)


@MIXERS.register("gated_delta")
class GatedDelta(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.num_heads, self.num_kv_heads = int(spec.num_heads), int(spec.num_kv_heads)
        self.dim, self.vdim, self.taps = int(spec.dim), int(spec.vdim), int(spec.taps)
        self.eps = float(spec.get("eps", 1e-6))
        if min(self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.taps) <= 0 or self.num_heads % self.num_kv_heads:
            raise ValueError("gated_delta: sizes must be positive and num_heads a multiple of num_kv_heads")
        if self.dim > 256:
            raise ValueError(f"gated_delta: key size {self.dim} is beyond what the scan kernel keeps in registers (256)")
        n = _names(spec, {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "b": "b", "a": "a",
                          "A_log": "A_log", "dt_bias": "dt_bias", "conv": "{}.conv"})
        p, H, G, d, dv = prefix, self.num_heads, self.num_kv_heads, self.dim, self.vdim
        self.channels = 2 * G * d + H * dv
        self.main = Linear([f"{p}.{n['q']}", f"{p}.{n['k']}", f"{p}.{n['v']}", f"{p}.{n['g']}"], [G * d, G * d, H * dv, H * dv],
                           hidden_size, dtype)
        self.gates = Linear([f"{p}.{n['b']}", f"{p}.{n['a']}"], [H, H], hidden_size, dtype)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], H * dv, dtype)
        self._tap_specs = [TensorSpec(f"{p}.{n['conv'].format(n[role])}", (size, self.taps))
                           for role, size in (("q", G * d), ("k", G * d), ("v", H * dv))]
        self._vec_specs = [TensorSpec(f"{p}.{n['norm']}", (dv,), keep_stored_precision=True, init="ones"),
                           TensorSpec(f"{p}.{n['A_log']}", (H,), keep_stored_precision=True, init="zeros"),
                           TensorSpec(f"{p}.{n['dt_bias']}", (H,), keep_stored_precision=True, init="zeros")]
        self.conv_taps = self.gain = self.a_log = self.dt_bias = None

    def tensors(self) -> List[TensorSpec]:
        return self.main.tensors() + self.gates.tensors() + self.o.tensors() + self._tap_specs + self._vec_specs

    def load(self, store) -> None:
        for lin in (self.main, self.gates, self.o):
            lin.load(store)
        self.conv_taps = store.get_stacked(self._tap_specs).to(self.dtype).contiguous()
        self.gain, self.a_log, self.dt_bias = (store.get(s) for s in self._vec_specs)
        if self.a_log.dtype != self.dt_bias.dtype:
            self.a_log, self.dt_bias = self.a_log.float(), self.dt_bias.float()

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.main.weight

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return (StateNeed((self.num_heads, self.dim * self.vdim), "float32", name="memory"),
                StateNeed((max(self.taps - 1, 1), self.channels), "float32", name="conv"))

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return (self.main.workspace_bytes(tokens) + tokens * (2 * self.num_heads + self.channels) * 4
                + tokens * self.num_heads * self.vdim * (4 + width) + self.o.workspace_bytes(tokens))

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        H, G, d, dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        state = ctx.run_state(run)
        rows = self.main.forward(x)
        gates = self.gates.forward(x, out_dtype=torch.float32)
        qkv = torch.empty((rows.shape[0], self.channels), dtype=torch.float32, device=rows.device)
        kernels.delta_prep(rows, self.conv_taps, state["conv"], ctx.query_start_loc, ctx.token_request, ctx.state_slots, G, H, d, dv,
                           DELTA_UNIT_EPS, d ** -0.5, qkv, one_token_each=ctx.decode_only)
        o = torch.empty((rows.shape[0], H * dv), dtype=torch.float32, device=rows.device)
        kernels.delta_scan(qkv, gates, self.a_log, self.dt_bias, state["memory"], ctx.query_start_loc, ctx.state_slots, o, G, H, d, dv)
        out = torch.empty((rows.shape[0], H * dv), dtype=rows.dtype, device=rows.device)
        kernels.head_rms_gate(o, rows[:, self.channels:], self.gain, self.eps, True, out, H, dv)
        return self.o.forward(out)


@MIXERS.register("channel_delta")
class ChannelDelta(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.num_heads, self.num_kv_heads = int(spec.num_heads), int(spec.num_kv_heads)
        self.dim, self.vdim, self.taps = int(spec.dim), int(spec.vdim), int(spec.taps)
        self.eps = float(spec.get("eps", 1e-6))
        if min(self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.taps) <= 0 or self.num_heads % self.num_kv_heads:
            raise ValueError("channel_delta: sizes must be positive and num_heads a multiple of num_kv_heads")
        if self.dim > 256:
            raise ValueError(f"channel_delta: key size {self.dim} is beyond what the scan kernel keeps in registers (256)")
        n = _names(spec, {"q": "q", "k": "k", "v": "v", "o": "o", "norm": "norm", "b": "b", "a1": "a1", "a2": "a2", "g1": "g1", "g2": "g2",
                          "A_log": "A_log", "dt_bias": "dt_bias", "conv": "{}.conv"})
        p, H, G, d, dv = prefix, self.num_heads, self.num_kv_heads, self.dim, self.vdim
        rank = int(spec.get("rank", 64))
        self.channels = 2 * G * d + H * dv
        # one projection of h: queries, keys, values and the inner values of the two low-rank products
        self.main = Linear([f"{p}.{n[r]}" for r in ("q", "k", "v", "a1", "g1")], [G * d, G * d, H * dv, rank, rank], hidden_size, dtype,
                           pad=True, free_out=(3, 4))
        self.beta = Linear([f"{p}.{n['b']}"], [H], hidden_size, dtype, pad=True)
        self.decay = Linear([f"{p}.{n['a2']}"], [H * d], rank, dtype, pad=True, free_in=True)
        self.gate = Linear([f"{p}.{n['g2']}"], [H * dv], rank, dtype, pad=True, free_in=True)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], H * dv, dtype)
        self._tap_specs = [TensorSpec(f"{p}.{n['conv'].format(n[role])}", (size, self.taps))
                           for role, size in (("q", G * d), ("k", G * d), ("v", H * dv))]
        self._vec_specs = [TensorSpec(f"{p}.{n['norm']}", (dv,), keep_stored_precision=True, init="ones"),
                           TensorSpec(f"{p}.{n['A_log']}", (H,), keep_stored_precision=True, init="zeros"),
                           TensorSpec(f"{p}.{n['dt_bias']}", (H * d,), keep_stored_precision=True, init="zeros")]
        self.conv_taps = self.gain = self.a_log = self.dt_bias = None

    def _linears(self) -> List[Linear]:
        return [self.main, self.beta, self.decay, self.gate, self.o]

    def tensors(self) -> List[TensorSpec]:
        return [t for lin in self._linears() for t in lin.tensors()] + self._tap_specs + self._vec_specs

    def load(self, store) -> None:
        for lin in self._linears():
            lin.load(store)
        if (self.decay.in_features, self.gate.in_features) != tuple(self.main.out_features[3:]):
            raise ValueError(f"{self.prefix}: the two halves of a low-rank product have different inner sizes")
        self.conv_taps = store.get_stacked(self._tap_specs).to(self.dtype).contiguous()
        self.gain, self.a_log, self.dt_bias = (store.get(s) for s in self._vec_specs)
        if self.a_log.dtype != self.dt_bias.dtype:
            self.a_log, self.dt_bias = self.a_log.float(), self.dt_bias.float()

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.main.weight

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return (StateNeed((self.num_heads, self.dim * self.vdim), "float32", name="memory"),
                StateNeed((max(self.taps - 1, 1), self.channels), "float32", name="conv"))

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return (sum(lin.workspace_bytes(tokens) for lin in (self.main, self.gate, self.o))
                + tokens * (self.num_heads * (3 + 3 * self.dim) + self.channels) * 4 + tokens * self.num_heads * self.vdim * (4 + width))

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        H, G, d, dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        state = ctx.run_state(run)
        rows = self.main.forward(x)
        beta = self.beta.forward(x, out_dtype=torch.float32)
        at, ra, rg = self.channels, self.main.out_features[3], self.main.out_features[4]
        decay = self.decay.forward(dense_operand(rows[:, at:at + ra]), out_dtype=torch.float32)
        gate = self.gate.forward(dense_operand(rows[:, at + ra:at + ra + rg]))
        qkv = torch.empty((rows.shape[0], self.channels), dtype=torch.float32, device=rows.device)
        kernels.delta_prep(rows, self.conv_taps, state["conv"], ctx.query_start_loc, ctx.token_request, ctx.state_slots, G, H, d, dv,
                           DELTA_UNIT_EPS, d ** -0.5, qkv, one_token_each=ctx.decode_only)
        o = torch.empty((rows.shape[0], H * dv), dtype=torch.float32, device=rows.device)
        kernels.channel_delta_scan(qkv, beta, decay, self.a_log, self.dt_bias, state["memory"], ctx.query_start_loc, ctx.state_slots,
                                   o, G, H, d, dv, one_token_each=ctx.decode_only)
        out = torch.empty((rows.shape[0], H * dv), dtype=rows.dtype, device=rows.device)
        kernels.head_rms_gate(o, gate[:, :H * dv], self.gain, self.eps, False, out, H, dv)
        return self.o.forward(out)


WKV_STREAMS = ("r", "k", "v", "g", "w")       # what reads a mix of the token and the one before it, the decay last


@MIXERS.register("wkv")
class TimeMixing(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.num_heads, self.dim = int(spec.num_heads), int(spec.dim)
        self.eps = float(spec.get("eps", 1e-6))
        if min(self.num_heads, self.dim) <= 0:
            raise ValueError("wkv: sizes must be positive")
        if self.dim > 256:
            raise ValueError(f"wkv: head size {self.dim} is beyond what the scan kernel keeps in registers (256)")
        n = _names(spec, {"r": "r", "k": "k", "v": "v", "g": "g", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u", "mu": "mu.{}", "norm": "norm",
                          "o": "o"})
        p, H, d = prefix, self.num_heads, self.dim
        rank = int(spec.get("rank", 64))
        self._product_specs = [TensorSpec(f"{p}.{n[s]}", (H * d, hidden_size)) for s in WKV_STREAMS[:4]]
        self.w1 = Linear([f"{p}.{n['w1']}"], [rank], hidden_size, dtype, pad=True, free_out=(0,))
        self.w2 = Linear([f"{p}.{n['w2']}"], [H * d], rank, dtype, pad=True, free_in=True)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], H * d, dtype)
        self._mu_specs = [TensorSpec(f"{p}.{n['mu'].format(s)}", (hidden_size,), keep_stored_precision=True, init="zeros") for s in WKV_STREAMS]
        self._vec_specs = [TensorSpec(f"{p}.{n['norm']}", (H * d,), keep_stored_precision=True, init="ones"),
                           TensorSpec(f"{p}.{n['w0']}", (H * d,), keep_stored_precision=True, init="zeros"),
                           TensorSpec(f"{p}.{n['u']}", (H, d), keep_stored_precision=True, init="zeros")]
        self.products: Optional[torch.Tensor] = None          # [4, H d, W]
        self.mu: Optional[torch.Tensor] = None                # 32-bit [5, W]
        self.gain = self.w0 = self.bonus = None

    def tensors(self) -> List[TensorSpec]:
        return self._product_specs + self.w1.tensors() + self.w2.tensors() + self.o.tensors() + self._mu_specs + self._vec_specs

    def load(self, store) -> None:
        self.products = store.get_stacked(self._product_specs).to(self.dtype).view(4, self.num_heads * self.dim, self.hidden_size)
        for lin in (self.w1, self.w2, self.o):
            lin.load(store)
        if self.w2.in_features != self.w1.out_features[0]:
            raise ValueError(f"{self.prefix}: the two halves of a low-rank product have different inner sizes")
        self.mu = torch.stack([store.get(s).float() for s in self._mu_specs]).contiguous()
        self.gain, self.w0, self.bonus = (store.get(s) for s in self._vec_specs)
        if self.w0.dtype != self.bonus.dtype:
            self.w0, self.bonus = self.w0.float(), self.bonus.float()

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.products

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return (StateNeed((self.num_heads, self.dim * self.dim), "float32", name="memory"),
                StateNeed((self.hidden_size,), "float32", name="shift"))

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        hd = self.num_heads * self.dim
        return tokens * (5 * self.hidden_size * width + 4 * hd * width + hd * (24 + width) + self.num_heads * 8) + 3 * self.w1.workspace_bytes(tokens) + self.o.workspace_bytes(tokens)

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        H, d, T = self.num_heads, self.dim, x.shape[0]
        state = ctx.run_state(run)
        mixes = torch.empty((5, T, self.hidden_size), dtype=x.dtype, device=x.device)
        kernels.token_shift(x, self.mu, state["shift"], ctx.query_start_loc, ctx.token_request, ctx.state_slots, mixes)
        rkvg = torch.empty((4, T, H * d), dtype=x.dtype, device=x.device)
        per_head_products(mixes[:4], self.products, rkvg)
        low = self.w1.forward(mixes[4], out_dtype=torch.float32)
        inner = torch.empty((T, self.w1.out_features[0]), dtype=x.dtype, device=x.device)
        kernels.tanh_rows(low, inner)
        decay = self.w2.forward(dense_operand(inner), out_dtype=torch.float32)
        o = torch.empty((T, H * d), dtype=torch.float32, device=x.device)
        kernels.wkv_scan(rkvg[0], rkvg[1], rkvg[2], decay, self.w0, self.bonus, state["memory"], ctx.query_start_loc, ctx.state_slots,
                         o, H, d, d, one_token_each=ctx.decode_only)
        out = torch.empty((T, H * d), dtype=x.dtype, device=x.device)
        kernels.head_rms_gate(o, rkvg[3], self.gain, self.eps, True, out, H, d)
        return self.o.forward(out)


@MIXERS.register("state_space")
class StateSpace(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.num_heads, self.vdim, self.state_size = int(spec.num_heads), int(spec.vdim), int(spec.state_size)
        self.groups, self.taps, self.norm_groups = int(spec.groups), int(spec.taps), int(spec.get("norm_groups", 1))
        self.eps = float(spec.get("eps", 1e-6))
        if min(self.num_heads, self.vdim, self.state_size, self.groups, self.taps, self.norm_groups) <= 0 or self.num_heads % self.groups:
            raise ValueError("state_space: sizes must be positive and num_heads a multiple of groups")
        if self.state_size > 256:
            raise ValueError(f"state_space: state size {self.state_size} is beyond what the scan kernels keep in registers (256)")
        self.inner = self.num_heads * self.vdim
        if self.inner % self.norm_groups:
            raise ValueError(f"state_space: {self.inner} values do not split into {self.norm_groups} groups")
        n = _names(spec, {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm",
                          "o": "o"})
        p, H = prefix, self.num_heads
        self.channels = self.inner + 2 * self.groups * self.state_size
        # one matrix [z | x | B | C | dt].  Steps of many rows multiply its two parts apart, so that the step sizes come out in
        # 32 bits beside rows in the engine's dtype; steps of few rows take all of it in 32 bits at once
        self.all = Linear([f"{p}.{n['in']}"], [self.inner + self.channels + H], hidden_size, dtype, pad=True)
        self.main = Linear([f"{p}.{n['in']}"], [self.inner + self.channels], hidden_size, dtype)
        self.steps = Linear([f"{p}.{n['in']}"], [H], hidden_size, dtype)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], self.inner, dtype)
        self._tap_spec = TensorSpec(f"{p}.{n['conv']}", (self.channels, self.taps))
        self._conv_bias_spec = TensorSpec(f"{p}.{n['conv_bias']}", (self.channels,), keep_stored_precision=True, init="zeros")
        self._vec_specs = [TensorSpec(f"{p}.{n[v]}", (H,), keep_stored_precision=True, init="ones" if v == "D" else "zeros")
                           for v in ("dt_bias", "A_log", "D")]
        self._gain_spec = TensorSpec(f"{p}.{n['norm']}", (self.inner,), keep_stored_precision=True, init="ones")
        self.conv_taps = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.gain = None

    def tensors(self) -> List[TensorSpec]:
        return self.all.tensors() + self.o.tensors() + [self._tap_spec, self._conv_bias_spec, *self._vec_specs, self._gain_spec]

    def load(self, store) -> None:
        self.all.load(store)
        self.o.load(store)
        rows = self.inner + self.channels
        self.main.weight = self.all.weight[:rows]
        self.steps.weight = padded_rows(self.all.weight[rows:rows + self.num_heads].clone())
        self.conv_taps = store.get(self._tap_spec).float().t().contiguous()
        self.conv_bias = store.get(self._conv_bias_spec).float().contiguous()
        self.dt_bias, self.a_log, self.skip = (store.get(s).float().contiguous() for s in self._vec_specs)
        self.gain = store.get(self._gain_spec)

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.all.weight

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return (StateNeed((self.num_heads, self.vdim * self.state_size), "float32", name="memory"),
                StateNeed((max(self.taps - 1, 1), self.channels), "float32", name="conv"))

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return (self.main.workspace_bytes(tokens) + tokens * (self.num_heads + 8) * 4 + tokens * self.channels * width
                + tokens * self.inner * (4 + width) + self.o.workspace_bytes(tokens))

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        H, G, P, N, T = self.num_heads, self.groups, self.vdim, self.state_size, x.shape[0]
        state = ctx.run_state(run)
        if T <= FEW_ROWS or self.dtype == torch.float32:
            rows = self.all.forward(x, out_dtype=torch.float32)
            dt = rows[:, self.inner + self.channels:]
        else:
            rows = self.main.forward(x)
            dt = self.steps.forward(x, out_dtype=torch.float32)
        xbc = torch.empty((T, self.channels), dtype=self.dtype, device=x.device)
        conv = kernels.ShortConv(self.conv_taps, state["conv"], ctx.query_start_loc, ctx.token_request, ctx.state_slots,
                                 one_token_each=ctx.decode_only)
        kernels.short_conv(rows[:, self.inner:], conv, xbc, bias=self.conv_bias, silu=True)
        y = torch.empty((T, self.inner), dtype=torch.float32, device=x.device)
        kernels.ssm_scan(xbc, dt, self.dt_bias, self.a_log, self.skip, state["memory"], ctx.query_start_loc, ctx.state_slots, y, H, G, P, N,
                         chunks=not ctx.decode_only and kernels.ssm_chunk_supports(xbc, H, G, P, N))
        out = torch.empty((T, self.inner), dtype=self.dtype, device=x.device)
        kernels.gated_group_rms(y, rows[:, :self.inner], self.gain, self.eps, self.norm_groups, out)
        return self.o.forward(out)


@MIXERS.register("gated_linear")
class GatedLinear(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.width, self.blocks, self.taps = int(spec.width), int(spec.blocks), int(spec.taps)
        self.out_scale = float(spec.get("out_scale", 1.0))
        if min(self.width, self.blocks, self.taps) <= 0 or self.width % self.blocks:
            raise ValueError("gated_linear: sizes must be positive and width a multiple of blocks")
        self.block = self.width // self.blocks
        n = _names(spec, {"y": "y", "x": "x", "y_bias": "y.b", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "ra": "ra", "ri": "ri",
                          "ra_bias": "ra.b", "ri_bias": "ri.b", "lam": "lam", "o": "o"})
        p, C, b = prefix, self.width, self.block
        self.main = Linear([f"{p}.{n['y']}", f"{p}.{n['x']}"], [C, C], hidden_size, dtype)
        self.o = Linear([f"{p}.{n['o']}"], [hidden_size], C, dtype)
        self._gate_specs = [TensorSpec(f"{p}.{n[r]}", (self.blocks, b, b)) for r in ("ra", "ri")]
        self._gate_bias_specs = [TensorSpec(f"{p}.{n[r]}", (self.blocks, b), keep_stored_precision=True, init="zeros")
                                 for r in ("ra_bias", "ri_bias")]
        self._tap_spec = TensorSpec(f"{p}.{n['conv']}", (C, self.taps))
        self._vec_specs = [TensorSpec(f"{p}.{n[v]}", (C,), keep_stored_precision=True, init="zeros")
                           for v in ("y_bias", "x_bias", "conv_bias", "lam")]
        self.gates: Optional[torch.Tensor] = None             # [blocks, 2 b, b]: a block's Ra, then its Ri
        self.gate_bias: Optional[torch.Tensor] = None         # 32-bit [2 C]
        self.conv_taps = self.y_bias = self.x_bias = self.conv_bias = None
        self.rate: Optional[torch.Tensor] = None              # softplus(lam), 32-bit [C]

    def tensors(self) -> List[TensorSpec]:
        return self.main.tensors() + self.o.tensors() + self._gate_specs + self._gate_bias_specs + [self._tap_spec] + self._vec_specs

    def load(self, store) -> None:
        self.main.load(store)
        self.o.load(store)
        self.gates = torch.cat([store.get(s) for s in self._gate_specs], dim=1).to(self.dtype).contiguous()
        self.gate_bias = torch.cat([store.get(s).float().reshape(-1) for s in self._gate_bias_specs]).contiguous()
        self.conv_taps = store.get(self._tap_spec).float().t().contiguous()
        self.y_bias, self.x_bias, self.conv_bias, lam = (store.get(s).float().contiguous() for s in self._vec_specs)
        self.rate = torch.nn.functional.softplus(lam.double()).float().contiguous()

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.main.weight

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.o.warm_next = weight

    def state_need(self):
        return (StateNeed((self.width,), "float32", name="memory"),
                StateNeed((max(self.taps - 1, 1), self.width), "float32", name="conv"))

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return (self.main.workspace_bytes(tokens) + tokens * self.width * (2 * width + 8) + tokens * self.width * 8
                + self.o.workspace_bytes(tokens))

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        C, b, T = self.width, self.block, x.shape[0]
        state = ctx.run_state(run)
        rows = self.main.forward(x)
        u = torch.empty((T, C), dtype=self.dtype, device=x.device)
        conv = kernels.ShortConv(self.conv_taps, state["conv"], ctx.query_start_loc, ctx.token_request, ctx.state_slots,
                                 one_token_each=ctx.decode_only)
        kernels.short_conv(rows[:, C:], conv, u, in_bias=self.x_bias, bias=self.conv_bias)
        out = torch.empty((T, C), dtype=self.dtype, device=x.device)
        if ctx.decode_only and T <= LRU_DECODE_MAX_ROWS and b <= kernels.LRU_DECODE_MAX_BLOCK:
            kernels.lru_decode(u, self.gates, self.gate_bias, self.rate, rows, self.y_bias, self.out_scale, state["memory"], ctx.state_slots, out)
            return self.o.forward(out)
        pairs = torch.empty((T, C, 2), dtype=torch.float32, device=x.device)
        if kernels.lru_mma_supports(u, b):
            kernels.lru_gates(u, self.gates, self.gate_bias, self.rate, pairs)
        else:
            logits = torch.empty((T, 2 * C), dtype=torch.float32, device=x.device)
            per_head_products(u.view(T, self.blocks, b).transpose(0, 1), self.gates, logits.view(T, self.blocks, 2 * b).transpose(0, 1))
            kernels.lru_gates(u, self.gates, self.gate_bias, self.rate, pairs, logits=logits)
        kernels.lru_scan(pairs, rows, self.y_bias, self.out_scale, state["memory"], ctx.query_start_loc, ctx.state_slots, ctx.max_query_len, out)
        return self.o.forward(out)


@MIXERS.register("side_by_side")
class SideBySide(Mixer):
    def __init__(self, spec: PartSpec, *, hidden_size: int, prefix: str, dtype: torch.dtype) -> None:
        super().__init__(spec, hidden_size=hidden_size, prefix=prefix, dtype=dtype)
        self.eps = float(spec.get("eps", 1e-6))
        scales = spec.get("scales")
        self.scales = (float(scales[0]), float(scales[1])) if scales is not None else None
        n = _names(spec, {"left": "left", "right": "right", "out": "out"})
        self.sides: Dict[str, Mixer] = {}
        for side in ("left", "right"):
            sub: PartSpec = spec.get(side)
            self.sides[side] = MIXERS.get(sub.kind)(sub, hidden_size=hidden_size, prefix=f"{prefix}.{n[side]}", dtype=dtype)
        if all(m.cache_need() is not None for m in self.sides.values()):
            raise ValueError("side_by_side: one of the two mixers may keep a paged cache")
        self.capturable = all(m.capturable for m in self.sides.values())
        self._gain_specs = [TensorSpec(f"{prefix}.{n[side]}.{n['out']}", (hidden_size,), keep_stored_precision=True, init="ones")
                            for side in ("left", "right")] if self.scales is None else []
        self.gains: Optional[List[torch.Tensor]] = None

    def tensors(self) -> List[TensorSpec]:
        return [t for m in self.sides.values() for t in m.tensors()] + self._gain_specs

    def load(self, store) -> None:
        for m in self.sides.values():
            m.load(store)
        self.gains = [store.get(s) for s in self._gain_specs]
        if self.gains and self.gains[0].dtype != self.gains[1].dtype:
            self.gains = [g.float() for g in self.gains]

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.sides["left"].first_weight()

    def warm_after(self, weight: Optional[torch.Tensor]) -> None:
        self.sides["left"].warm_after(self.sides["right"].first_weight())
        self.sides["right"].warm_after(weight)

    def cache_need(self):
        needs = [m.cache_need() for m in self.sides.values()]
        return needs[0] if needs[0] is not None else needs[1]

    def _state_needs(self, side: str) -> tuple:
        need = self.sides[side].state_need()
        return () if need is None else tuple(need) if isinstance(need, (tuple, list)) else (need,)

    def state_need(self):
        """Both mixers' tensors under names of their own."""
        out = tuple(replace(need, name=f"{side}.{need.name}") for side in self.sides for need in self._state_needs(side))
        return out or None

    def _context(self, side: str, ctx: StepContext, run: int) -> StepContext:
        """The step as one of the mixers sees it: its own state tensors under the names it gave them."""
        needs = self._state_needs(side)
        if not needs:
            return ctx
        have = ctx.run_state(run)
        own = {need.name: have[f"{side}.{need.name}"] for need in needs}
        return replace(ctx, state={run: own if needs[0].name else own[""]})

    def workspace_bytes(self, tokens: int) -> int:
        width = 2 if self.dtype == torch.bfloat16 else 4
        return max(m.workspace_bytes(tokens) for m in self.sides.values()) + 2 * tokens * self.hidden_size * width

    def forward(self, x: torch.Tensor, ctx: StepContext, run: int) -> torch.Tensor:
        left, right = (self.sides[side].forward(x, self._context(side, ctx, run), run) for side in ("left", "right"))
        out = torch.empty_like(left)
        if self.scales is not None:
            kernels.pair_sum(left, right, self.scales[0], self.scales[1], out)
            return out
        kernels.pair_rms_mean(left, right, self.gains[0], self.gains[1], self.eps, out)
        return out
