"""Neburax without a GPU: configuration, tensor names, caches and states of the layers, layers that run with another's tensors,
and the plain implementation against itself and against cases worked by hand."""
from __future__ import annotations

import json
import math
import os

import pytest
import torch

import plain_neburax as plain
from cuinfer_b200.cache import CacheManager, CacheStorage, group_runs
from cuinfer_b200.config import ConfigError
from cuinfer_b200.config.registry import architecture_of
from cuinfer_b200.parts import DecoderModel
from cuinfer_b200.weights import open_weight_store
from cuinfer_b200.weights.safetensors_io import WeightError, write_safetensors

_SSM = {"type": "mamba2", "mixer": {"heads": 6, "vdim": 10, "state": 13, "groups": 3, "conv": 3, "norm_groups": 4},
        "mlp": {"kind": "moe", "router": {"experts": 6, "top": 3, "identity": 2}, "expert": {"ff": 20}, "shared": {"ff": 12}}}
_PAIR = {"type": "parallel",
         "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 11, "vdim": 9, "scale": 0.3, "mask": {"size": 13}},
                   "right": {"width": 42, "blocks": 3, "conv": 2}, "left_scale": 0.7, "right_scale": 1.3},
         "mlp": {"kind": "dense", "ff": 36}}
CONFIG = {"architecture": "Neburax", "vocab": 97, "width": 72, "norm": {"eps": 1e-5},
          "layers": [_SSM, _PAIR, dict(_SSM, mlp=None), dict(_PAIR, weights_of=1), dict(_SSM, weights_of=0), dict(_PAIR, weights_of=3)]}


def _build(cfg):
    arch = architecture_of(cfg)
    typed = arch.parse(cfg)
    return typed, DecoderModel(arch.spec(typed), torch.float32)


def test_every_tensor_is_expected_under_its_name_and_shape():
    typed, model = _build(CONFIG)
    tensors = plain.random_model(CONFIG, 1)
    expected = {t.name: t for t in model.tensors()}
    assert set(expected) == set(tensors)
    for name, spec in expected.items():
        assert spec.accepts(tensors[name].shape), f"{name}: {spec.shape} / {tuple(tensors[name].shape)}"
    assert typed.to_dict() == CONFIG
    assert not any(n.startswith(("l3.", "l4.", "l5.")) for n in expected), "layers that run with another's tensors have none"
    assert "l2.norm2" not in expected and "l2.norm1" in expected and "head" not in expected


def test_layers_with_anothers_tensors_have_caches_and_states_of_their_own():
    _, model = _build(CONFIG)
    assert model.order == (0, 1, 2, 1, 0, 1) and not model.cache_source
    needs = model.cache_needs()
    assert sorted(needs) == [1, 3, 5]
    for need in needs.values():
        assert (need.num_kv_heads, need.head_dim, need.window, need.chunked) == (2, 20, 13, True)
    states = model.state_needs()
    assert sorted(states) == [0, 1, 2, 3, 4, 5]
    assert {n.name: n.shape for n in states[0]} == {"memory": (6, 130), "conv": (2, 60 + 2 * 39)}
    assert {n.name: n.shape for n in states[1]} == {"right.memory": (42,), "right.conv": (1, 42)}
    groups = group_runs(needs)
    storage = CacheStorage(groups, 16, [4] * len(groups), states, 3, torch.float32, "cpu")
    pointers = [t.data_ptr() for t in storage.state_tensors()]
    assert len(set(pointers)) == len(pointers) == 12
    for t in storage.state_tensors():
        t.fill_(1.0)
    storage.zero_slots([1])
    for t in storage.state_tensors():
        assert not t[1].any() and t[0].all() and t[2].all()


def test_pages_before_the_chunk_are_given_back():
    _, model = _build(CONFIG)
    manager = CacheManager(group_runs(model.cache_needs()), 4, 8, 2)
    assert manager.admit("a") is not None and manager.allocate("a", 12)
    manager.commit("a", 12)
    assert [p >= 0 for p in manager.block_table("a")] == [True] * 3             # the next token is still of the first chunk
    assert manager.allocate("a", 18)
    manager.commit("a", 18)
    assert [p >= 0 for p in manager.block_table("a")] == [False] * 6 + [True] * 2      # token 30: its chunk starts at 26, in page 6
    manager.release("a")
    for turn in range(5):
        assert manager.admit(turn) is not None and manager.allocate(turn, 30)
        manager.commit(turn, 30)
        manager.release(turn)
    manager.check()


def test_loading_and_a_wrong_shape(tmp_path):
    def folder(name, tensors):
        os.makedirs(tmp_path / name)
        write_safetensors(str(tmp_path / name / "model.safetensors"), tensors)
        return str(tmp_path / name)

    tensors = plain.random_model(CONFIG, 1)
    _, model = _build(CONFIG)
    model.load(open_weight_store(folder("good", tensors), torch.float32, "cpu"))
    mixer = model.blocks[0].mixer
    whole = tensors["l0.mix.in"]
    assert torch.equal(mixer.main.weight, whole[:-6]) and torch.equal(mixer.steps.weight[:6], whole[-6:]) and mixer.steps.weight.shape[0] == 8
    right = model.blocks[1].mixer.sides["right"]
    assert torch.equal(right.gates[:, :14], tensors["l1.mix.right.ra"]) and torch.equal(right.gates[:, 14:], tensors["l1.mix.right.ri"])
    assert torch.allclose(right.rate.double(), plain.softplus(tensors["l1.mix.right.lam"].double()))
    assert model.lm_head.weight is model.embedding
    for name, shape in (("l0.mix.in", (205, 72)), ("l1.mix.left.q.norm", (11,)), ("l1.mix.right.ra", (3, 13, 14))):
        with pytest.raises(WeightError, match=name):
            _build(CONFIG)[1].load(open_weight_store(folder(name, dict(tensors, **{name: torch.zeros(shape)})), torch.float32, "cpu"))
    with pytest.raises(WeightError, match="l3.norm1"):
        _build(CONFIG)[1].load(open_weight_store(folder("extra", dict(tensors, **{"l3.norm1": torch.zeros(72)})), torch.float32, "cpu"))


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][2]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][2]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][2]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(rot={"base": 1e4, "dims": 4}), "rot"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(blocks=4), "blocks"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][3].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=True), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=0), "differs"),
    (lambda c: c["layers"][3]["mixer"].update(left_scale=0.8), "differs"),
    (lambda c: c["layers"][4].update(mlp=None), "differs"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "ff"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
])
def test_refusals(change, message):
    cfg = json.loads(json.dumps(CONFIG))          # entries share nothing
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        _build(cfg)


def test_absent_options_mean_none():
    cfg = json.loads(json.dumps(CONFIG))          # entries share nothing
    cfg["layers"] = cfg["layers"][:3]
    cfg["layers"][0]["mlp"]["router"].pop("identity")
    cfg["layers"][0]["mlp"].pop("shared")
    cfg["layers"][1]["mixer"]["left"].pop("mask")
    typed, model = _build(cfg)
    assert (typed.layers[0].mlp.identity, typed.layers[0].mlp.shared) == (0, 0)
    assert model.cache_needs()[1].window is None and not model.cache_needs()[1].chunked
    names = {t.name: t.shape for t in model.tensors()}
    assert names["l0.mlp.router"] == (6, 72) and "l0.mlp.shared.up" not in names


# ---- the plain implementation against itself -------------------------------------------------------------------------------
def test_plain_portions_of_the_recurrences_agree():
    g = torch.Generator().manual_seed(4)
    T, H, G, P, N = 11, 4, 2, 5, 6
    x, B, C = torch.randn(T, H, P, generator=g).double(), torch.randn(T, G, N, generator=g).double(), torch.randn(T, G, N, generator=g).double()
    dt, a_log, D = torch.rand(T, H, generator=g).double(), torch.randn(H, generator=g).double(), torch.randn(H, generator=g).double()
    whole, S = plain.state_space_scan(x, B, C, dt, a_log, D)
    a, s = plain.state_space_scan(x[:4], B[:4], C[:4], dt[:4], a_log, D)
    b, s = plain.state_space_scan(x[4:], B[4:], C[4:], dt[4:], a_log, D, s)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(s, S)
    for h in range(H):                                                # the masked-product form of the same sums
        L = torch.cumsum(-torch.exp(a_log[h]) * dt[:, h], 0)
        M = torch.tril(torch.exp(L[:, None] - L[None, :])) * (C[:, h // 2] @ B[:, h // 2].T) * dt[None, :, h]
        assert torch.allclose(whole[:, h], M @ x[:, h] + D[h] * x[:, h])
    u, r, i, lam = torch.randn(T, 7, generator=g).double(), torch.rand(T, 7, generator=g).double(), torch.rand(T, 7, generator=g).double(), torch.randn(7, generator=g).double()
    whole, last = plain.gated_linear_recurrence(u, r, i, lam)
    a, s = plain.gated_linear_recurrence(u[:3], r[:3], i[:3], lam)
    b, s = plain.gated_linear_recurrence(u[3:], r[3:], i[3:], lam, s)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(s, last)
    decay = torch.exp(-8.0 * r[0] * torch.log1p(torch.exp(lam)))
    assert torch.allclose(whole[0], torch.sqrt(1 - decay ** 2) * i[0] * u[0])       # the first token has no case of its own


def test_plain_chunks_and_router_by_hand():
    q = torch.zeros(6, 2, 3).double()
    k, v = torch.randn(6, 1, 3).double(), torch.arange(6.0).view(6, 1, 1).double()
    out = plain.chunked_attention(q, k, v, 1.0, 4)[:, 0, 0]
    assert torch.allclose(out, torch.tensor([0.0, 0.5, 1.0, 1.5, 4.0, 4.5]).double())
    chosen, w = plain.choose_experts(torch.log(torch.tensor([0.1, 0.5, 0.15, 0.25])).double(), torch.tensor([1.0, 0.0, 0.0, 0.9]).double(), 2)
    assert chosen == [3, 0] and torch.allclose(w, torch.tensor([0.25, 0.1]).double() / 0.35)
    assert math.isclose(float(plain.gelu_tanh(torch.tensor(1.0).double())), 0.841192, rel_tol=1e-6)


def test_plain_model_is_causal_and_runs_layers_again():
    tensors = {k: v.double() for k, v in plain.random_model(CONFIG, 3).items()}
    toks = torch.randint(0, 97, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = plain.forward(CONFIG, tensors, toks)
    assert torch.allclose(plain.forward(CONFIG, tensors, toks[:17]), whole[:17])
    copied = dict(tensors)
    for i in (3, 4, 5):
        copied.update({f"l{i}." + k.split(".", 1)[1]: v for k, v in tensors.items() if k.startswith(f"l{plain.owner(CONFIG, i)}.")})
    spelled = dict(CONFIG, layers=[{k: v for k, v in L.items() if k != "weights_of"} for L in CONFIG["layers"]])
    assert torch.allclose(plain.forward(spelled, copied, toks), whole)
