"""Mumopel without a device: its configuration, its spec (parts, cache slots, tensor names, the order of runs) and what the
plain implementation itself must do (the streams, the sink, the chunks, the norm over all heads, the router)."""
import copy

import pytest
import torch

import plain_mumopel as P
from firefly_b200.cache.spec import PagedKVSpec
from firefly_b200.config.base import ConfigError, LayerSpec, PartSpec
from firefly_b200.models import config_from_dict, expected_weights, spec_for
from firefly_b200.models.decoder import DecoderModel
from firefly_b200.parts import Runtime, build_part
from firefly_b200.parts.base import declared
from firefly_b200.parts.streams import HyperConnectionBlock

ATT = {"heads": 4, "kv_heads": 2, "dim": 20, "vdim": 12, "scale": 0.3, "mask": {"size": 9}, "rot": {"base": 300.0, "dims": 12}}
FULL = {"heads": 3, "kv_heads": 1, "dim": 16, "vdim": 24, "scale": 0.2}
MOE = {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 16, "limit": 1.0}, "shared": {"ff": 24, "limit": 0.5}}
CFG = {"architecture": "Mumopel", "vocab": 60, "width": 32, "streams": 3, "logit_softcap": 8.0, "norm": {"eps": 1e-5},
       "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [
           {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 40}},
           {"type": "attention", "mixer": FULL, "mlp": MOE},
           {"type": "attention", "mixer": ATT, "mlp": None},
           {"type": "attention", "mixer": ATT, "mlp": {k: v for k, v in MOE.items() if k != "shared"}},
       ]}
CPU = Runtime(torch.device("cpu"), torch.float32)


def test_the_spec_names_every_tensor_and_every_run_has_pages_of_its_own():
    w = P.random_weights(CFG, 0)
    spec = spec_for(config_from_dict(CFG))
    names = {x.name: tuple(x.shape) for x in expected_weights(spec) if not x.optional}
    assert names == {k: tuple(v.shape) for k, v in w.items()}
    assert {x.name for x in expected_weights(spec) if x.optional} == {"head", "l2.norm2", "l2.norm2.b", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"}
    model = DecoderModel(spec, CPU)
    assert [layer for layer, _, _ in model.schedule] == P.layer_order(CFG) == [0, 1, 2, 1, 2, 3]
    slots = model.cache_slot_specs()
    assert sorted(slots) == list(range(6)) and all(isinstance(s, PagedKVSpec) for s in slots.values())
    # a chunk's keys are kept like all others: a page holds heads of the longer kind
    assert [(s.num_kv_heads, s.head_dim, s.window) for s in slots.values()] == [(2, 20, None), (1, 24, None), (2, 20, None)] * 1 + \
        [(1, 24, None), (2, 20, None), (2, 20, None)]
    assert not model.host_synchronous and model.head.tied_to == "embed" and model.head.softcap == 8.0


def test_constants_reach_the_parts():
    spec = spec_for(config_from_dict(CFG))
    a, b = spec.layers[0].mixer.params, spec.layers[1].mixer.params
    assert (a["chunk"], a["scale"], a["qk_norm_over"], a["sink_leaf"]) == (9, 0.3, "all", "sink") and b["chunk"] is None
    assert spec.layers[0].position.params["pairing"] == "interleaved" and spec.layers[1].position is None
    m = spec.layers[1].feed_forward.params
    assert (m["limit"], m["shared_limit"], m["score"], m["router_bias"]) == (1.0, 0.5, "chosen_softmax", "router.b")
    assert spec.layers[3].feed_forward.params["shared_ff"] == 0
    rot = build_part("position", spec.layers[0].position, CPU)
    assert torch.allclose(rot.frequencies(), torch.tensor([300.0 ** (-2 * i / 12) for i in range(6)], dtype=torch.float64))


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0].update(type="attention_2"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c.pop("norm"), "eps"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(logit_softcap=-1.0), "softcap"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
])
def test_a_wrong_configuration_is_told_by_name(edit, word):
    raw = copy.deepcopy(CFG)
    edit(raw)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(raw)


def test_optional_entries_may_be_absent():
    raw = copy.deepcopy(CFG)
    for key in ("loop", "logit_softcap"):
        raw.pop(key)
    raw["layers"][0]["mixer"]["rot"]["dims"] = 0
    spec = spec_for(config_from_dict(raw))
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3] and spec.head.params["softcap"] == 0.0
    assert spec.layers[0].position is None
    assert config_from_dict(config_from_dict(raw).to_dict()) == config_from_dict(raw)
    assert config_from_dict(config_from_dict(CFG).to_dict()) == config_from_dict(CFG)


def test_options_that_exclude_each_other_are_told():
    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=16)
    with pytest.raises(ValueError, match="qk_norm_over"):
        build_part("mixer", PartSpec("gqa_attention", dict(base, qk_norm_over="all")), CPU)
    att, norm = PartSpec("gqa_attention", base, prefix="a"), PartSpec("rms_norm", dict(size=32, eps=1e-5, tensor="n"))
    one = HyperConnectionBlock(LayerSpec("hyper_connections", att, None, (norm,), params=dict(streams=2, connections=("c",))), CPU)
    assert {w.name for w in one.weight_specs()} >= {"c.in", "c.out", "c.mix", "n"}
    with pytest.raises(ValueError, match="connections"):
        HyperConnectionBlock(LayerSpec("hyper_connections", att, None, (norm,), params=dict(streams=2, connections=())), CPU)
    with pytest.raises(ConfigError, match="streams"):
        HyperConnectionBlock(LayerSpec("hyper_connections", att, None, (norm,), params=dict(streams=33, connections=("c",))), CPU)
    moe = build_part("feed_forward", spec_for(config_from_dict(CFG)).layers[1].feed_forward, CPU)
    assert declared(moe, "hands_on_rows")


# ------------------------------------------------------------------ the plain implementation --
def test_equal_streams_with_a_plain_mix_are_a_plain_residual():
    """in = 1/S each, mix the identity, out = 1 everywhere: every stream is the plain residual, and the sum S times it."""
    w = P.random_weights(CFG, 1)
    S = CFG["streams"]
    for k in list(w):
        if ".hc" in k:
            w[k] = torch.eye(S, dtype=torch.float64) if k.endswith("mix") else torch.full((S,), 1.0 if k.endswith("out") else 1.0 / S, dtype=torch.float64)
    toks = [3, 14, 15, 9, 2, 6, 5, 35, 8, 9, 7, 9, 3]
    sums = []
    P.forward(CFG, w, toks, sums)
    x = w["embed"][torch.tensor(toks)]
    for i, got in zip(P.layer_order(CFG), sums):
        L, p = CFG["layers"][i], f"l{i}"
        x = x + P.attention(P.layer_norm(x, w[p + ".norm1"], w[p + ".norm1.b"], 1e-5), w, p + ".mix", L["mixer"], 1e-5)
        if L["mlp"]:
            h = P.layer_norm(x, w[p + ".norm2"], w[p + ".norm2.b"], 1e-5)
            x = x + (P.dense_ff(h, w, p + ".mlp") if L["mlp"]["kind"] == "dense" else P.moe_ff(h, w, p + ".mlp", L["mlp"]))
        assert torch.allclose(got, S * x, rtol=1e-9, atol=1e-9)


def test_the_write_takes_all_streams_from_the_old_ones():
    X = torch.tensor([[[1.0]], [[10.0]]])
    mix, out, y = torch.tensor([[0.0, 1.0], [2.0, 3.0]]), torch.tensor([5.0, 7.0]), torch.tensor([[100.0]])
    assert P.streams_write(X, mix, out, y).flatten().tolist() == [2 * 10 + 500.0, 1 + 30 + 700.0]
    assert P.streams_read(X, torch.tensor([3.0, -1.0])).item() == -7.0


def test_a_sink_takes_its_share_of_the_softmax():
    q, k, v = torch.zeros(3, 2, 4), torch.zeros(3, 1, 4), torch.ones(3, 1, 5)
    sink = torch.tensor([0.0, float(torch.log(torch.tensor(3.0)))])
    o = P.sink_softmax_attention(q, k, v, 1.0, P.chunk_mask(3, None), sink)
    for i in range(3):
        assert torch.allclose(o[i, 0], torch.full((5,), (i + 1) / (i + 2.0))) and torch.allclose(o[i, 1], torch.full((5,), (i + 1) / (i + 4.0)))
    scaled = P.sink_softmax_attention(q, k, v, 9.0, P.chunk_mask(3, None), sink)
    assert torch.equal(scaled, o)                                            # the scale is on the scores, not on the sink


def test_chunks_count_from_the_start_of_the_sequence():
    see = P.chunk_mask(7, 3)
    assert [see[i].nonzero().flatten().tolist() for i in range(7)] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_the_rotation_turns_neighbours_and_leaves_the_rest():
    v = torch.randn(5, 2, 8, dtype=torch.float64)
    out = P.rotate_pairs(v, torch.arange(5), {"base": 10.0, "dims": 4})
    assert torch.equal(out[..., 4:], v[..., 4:]) and torch.equal(out[0], v[0])
    c, s = torch.cos(torch.tensor(3 * 10.0 ** -0.5, dtype=torch.float64)), torch.sin(torch.tensor(3 * 10.0 ** -0.5, dtype=torch.float64))
    assert torch.allclose(out[3, 1, 2:4], torch.stack([v[3, 1, 2] * c - v[3, 1, 3] * s, v[3, 1, 3] * c + v[3, 1, 2] * s]))


def test_the_router_s_weights_are_the_softmax_over_the_chosen():
    w = P.random_weights(CFG, 2)
    h = torch.randn(9, 32, dtype=torch.float64)
    ids, wts = P.route(h, w, "l1.mlp", MOE["router"])
    z = h @ w["l1.mlp.router"].T + w["l1.mlp.router.b"]
    assert torch.allclose(wts.sum(dim=1), torch.ones(9, dtype=torch.float64))
    assert torch.allclose(wts[:, 0] / wts[:, 1], torch.exp(torch.gather(z, 1, ids[:, :1]) - torch.gather(z, 1, ids[:, 1:2])).flatten())
