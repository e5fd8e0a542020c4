"""Nugolorn without a GPU: configuration, tensor names, sizes that the checkpoint decides, which cache and state each layer
keeps or reads, refusals, and the plain implementation against itself."""
from __future__ import annotations

import copy
import json
import math
import os

import pytest
import torch

import plain_nugolorn as plain
from cuinfer_b200.cache.manager import CacheManager, group_runs
from cuinfer_b200.cache.storage import CacheStorage
from cuinfer_b200.config import ConfigError
from cuinfer_b200.config.registry import get_architecture
from cuinfer_b200.parts.model import DecoderModel
from cuinfer_b200.weights import open_weight_store
from cuinfer_b200.weights.safetensors_io import WeightError, write_safetensors


def _moe(experts, top, ff, identity=0):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff}}


CONFIG = {"architecture": "Nugolorn", "vocab": 97, "width": 72, "norm": {"eps": 1e-5, "groups": 3}, "residual_mult": 0.7,
          "logit_scale": 1.3, "layers": [
    {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 10, "scale": 0.3, "conv": 3,
                                    "rot": {"base": 100.0, "dims": 8}}, "mlp": _moe(6, 3, 20, 2)},
    {"type": "wkv", "mixer": {"heads": 3, "dim": 20}, "mlp": None},
    {"type": "parallel", "mixer": {
        "left": {"heads": 3, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.25, "q_temp": {"coef": 0.25, "every": 7}},
        "right": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 6, "conv": 2}}, "mlp": {"kind": "dense", "ff": 36}},
    {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 10, "scale": 0.35, "conv": 5,
                                    "rot": {"base": 100.0, "dims": 8}, "kv_from": 0}, "mlp": _moe(4, 4, 28)},
]}


def _build(cfg):
    arch = get_architecture("Nugolorn")
    typed = arch.parse(cfg)
    return typed, DecoderModel(arch.spec(typed), torch.float32)


def _folder(path, cfg, tensors):
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    return str(path)


def test_tensor_names_and_shapes_are_the_plain_models():
    typed, model = _build(CONFIG)
    tensors = plain.random_model(CONFIG, 0)
    expected = {t.name: t for t in model.tensors()}
    assert set(expected) == set(tensors)
    for name, spec in expected.items():
        assert spec.accepts(tensors[name].shape), f"{name}: {spec.shape} / {tuple(tensors[name].shape)}"
    assert {n for n, s in expected.items() if s.free_axes} == {"l1.mix.w1", "l1.mix.w2", "l2.mix.right.a1", "l2.mix.right.a2",
                                                               "l2.mix.right.g1", "l2.mix.right.g2"}
    assert "l3.mix.k" not in expected and "l3.mix.v.conv" not in expected and "l3.mix.q.conv" in expected
    assert typed.to_dict() == CONFIG


def test_the_checkpoint_decides_the_inner_sizes(tmp_path):
    tensors = plain.random_model(CONFIG, 1)
    _, model = _build(CONFIG)
    store = open_weight_store(_folder(tmp_path / "a", CONFIG, tensors), torch.float32, "cpu")
    model.load(store)
    right = model.blocks[2].mixer.sides["right"]
    assert right.main.out_features[3:] == [tensors["l2.mix.right.a1"].shape[0], tensors["l2.mix.right.g1"].shape[0]]
    assert right.decay.in_features != right.gate.in_features, "the two low-rank products have inner sizes of their own"
    assert model.blocks[1].mixer.w2.in_features == tensors["l1.mix.w1"].shape[0]
    # every other axis is checked, and the two halves of a product must agree
    for name, shape in (("l1.mix.w2", (61, 5)), ("l2.mix.right.a1", (5, 71)), ("l0.mix.q.conv", (48, 4))):
        bad = dict(tensors, **{name: torch.zeros(shape)})
        with pytest.raises(WeightError, match=name):
            _build(CONFIG)[1].load(open_weight_store(_folder(tmp_path / name, CONFIG, bad), torch.float32, "cpu"))
    bad = dict(tensors, **{"l1.mix.w2": torch.zeros(60, tensors["l1.mix.w1"].shape[0] + 1)})
    with pytest.raises(ValueError, match="inner sizes"):
        _build(CONFIG)[1].load(open_weight_store(_folder(tmp_path / "halves", CONFIG, bad), torch.float32, "cpu"))


def test_rows_of_stacked_projections_are_padded_to_eight():
    from cuinfer_b200.parts.linear import padded_rows
    w = torch.randn(13, 5)
    p = padded_rows(w)
    assert p.shape == (16, 5) and torch.equal(p[:13], w) and not p[13:].any()
    assert padded_rows(p) is p


def test_caches_and_states_of_the_layers():
    _, model = _build(CONFIG)
    needs = model.cache_needs()
    assert sorted(needs) == [0, 2] and model.cache_source == {3: 0}
    assert (needs[0].num_kv_heads, needs[0].head_dim, needs[0].window) == (2, 22, None)
    assert (needs[2].num_kv_heads, needs[2].head_dim) == (3, 24)
    states = model.state_needs()
    assert states[0].shape == (2, 4 * 12 + 2 * 12 + 2 * 10) and states[3].shape == (4, 48)      # the reader convolves its queries only
    assert {n.name: n.shape for n in states[1]} == {"memory": (3, 400), "shift": (72,)}
    assert {n.name: n.shape for n in states[2]} == {"right.memory": (4, 72), "right.conv": (1, 2 * 24 + 24)}
    groups = group_runs(needs)
    storage = CacheStorage(groups, 16, [4] * len(groups), states, 3, torch.float32, "cpu")
    for t in storage.state_tensors():
        t.fill_(1.0)
    storage.zero_slots([1])
    for t in storage.state_tensors():
        assert not t[1].any() and t[0].all() and t[2].all()


def test_a_pool_of_the_live_tokens_is_used_again():
    _, model = _build(CONFIG)
    manager = CacheManager(group_runs(model.cache_needs()), 16, 8, 2)
    for turn in range(5):
        rid = f"r{turn}"
        assert manager.admit(rid) is not None and manager.allocate(rid, 100)
        manager.commit(rid, 100)
        manager.release(rid)
    manager.check()


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(mask={"size": 4}), "mask"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=True), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=12), "vdim"),
    (lambda c: c["layers"][2]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][2]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][2]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["norm"].update(groups=5), "groups"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
])
def test_refusals(change, message):
    cfg = copy.deepcopy(CONFIG)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        _build(cfg)


def test_absent_options_mean_none_or_one():
    cfg = copy.deepcopy(CONFIG)
    cfg["layers"][0]["mixer"].pop("rot"), cfg["layers"][3]["mixer"].pop("rot")
    cfg["layers"][2]["mixer"]["left"].pop("q_temp")
    cfg["layers"][0]["mlp"]["router"].pop("identity")
    cfg["norm"].pop("groups")
    typed, model = _build(cfg)
    assert typed.norm_groups == 1 and typed.layers[0].mlp.identity == 0
    assert model.blocks[0].mixer.position.rotary_dim == 0 and model.blocks[2].mixer.sides["left"].q_temp is None
    assert {t.name: t.shape for t in model.tensors()}["l0.mlp.router"] == (6, 72)


# ---- the plain implementation against itself -------------------------------------------------------------------------------
def test_plain_chunks_of_the_recurrences_agree():
    g = torch.Generator().manual_seed(4)
    T, H, G, d, dv = 11, 4, 2, 6, 5
    q, k, v = torch.randn(T, G, d, generator=g).double(), torch.randn(T, G, d, generator=g).double(), torch.randn(T, H, dv, generator=g).double()
    beta, decay = torch.rand(T, H, generator=g).double(), torch.rand(T, H, d, generator=g).double()
    whole, S = plain.channel_delta_rule(q, k, v, beta, decay)
    a, s = plain.channel_delta_rule(q[:4], k[:4], v[:4], beta[:4], decay[:4])
    b, s = plain.channel_delta_rule(q[4:], k[4:], v[4:], beta[4:], decay[4:], s)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(s, S)
    # a decay that is one number per head and no memory of other tokens: the closed form of one step
    one, _ = plain.channel_delta_rule(q[:1], k[:1], v[:1], beta[:1], decay[:1])
    for h in range(H):
        assert torch.allclose(one[0, h], beta[0, h] * v[0, h] * (k[0, h // 2] @ q[0, h // 2]))
    r, kk, u = torch.randn(T, H, d, generator=g).double(), torch.randn(T, H, d, generator=g).double(), torch.randn(H, d, generator=g).double()
    vv = torch.randn(T, H, d, generator=g).double()
    whole, S = plain.wkv_rule(r, kk, vv, decay, u)
    a, s = plain.wkv_rule(r[:7], kk[:7], vv[:7], decay[:7], u)
    b, s = plain.wkv_rule(r[7:], kk[7:], vv[7:], decay[7:], u, s)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(s, S)
    # with a bonus of ones and a decay of ones the read-out is causal linear attention
    lin, _ = plain.wkv_rule(r, kk, vv, torch.ones_like(decay), torch.ones_like(u))
    for h in range(H):
        w = torch.tril(r[:, h] @ kk[:, h].T)
        assert torch.allclose(lin[:, h], w @ vv[:, h])


def test_plain_model_is_causal_and_its_layers_read_one_norm():
    tensors = {k: v.double() for k, v in plain.random_model(CONFIG, 3).items()}
    toks = torch.randint(0, 97, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = plain.forward(CONFIG, tensors, toks)
    assert torch.allclose(plain.forward(CONFIG, tensors, toks[:17]), whole[:17])
    assert plain.router_margin(CONFIG, tensors, toks) > 0
    scaled = plain.forward(dict(CONFIG, logit_scale=2.6), tensors, toks)
    assert torch.allclose(scaled, 2.0 * whole)
    still = plain.forward(dict(CONFIG, residual_mult=0.0), tensors, toks)
    assert torch.allclose(still[3], still[[i for i in range(30) if toks[i] == toks[3]][0]])


def test_plain_log_bias_and_temperature_by_hand():
    q = torch.tensor([[[1.0, 0.0]]]).double()
    k = torch.zeros(4, 1, 2).double()
    v = torch.arange(4.0).view(4, 1, 1).double()
    out = plain.log_bias_attention(q, k, v, 1.0, torch.tensor([2.0]).double(), torch.tensor([0.5]).double())
    w = [(1 + 0.5 * (3 - j)) ** -2.0 for j in range(4)]
    assert math.isclose(float(out), sum(j * x for j, x in enumerate(w)) / sum(w), rel_tol=1e-12)
    temp = plain.query_temperature([0, 5, 6, 13, 20], 0.5, 7, torch.float64)
    assert torch.allclose(temp, 1.0 + 0.5 * torch.log(torch.tensor([1.0, 1.0, 2.0, 3.0, 4.0]).double()))
