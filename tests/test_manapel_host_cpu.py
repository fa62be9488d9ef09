"""Host side of the Manapel path without a GPU: configuration reading and validation, the registry and the mixer and
feed-forward tables, and the restatement itself (tanh norm, unit heads, causality, shared keys, router)."""
import json

import pytest
import torch

import manapel_oracle as mo

F64 = torch.float64


def _cfg():
    att = {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 4, "scale": 0.5, "rot": {"base": 100.0, "dims": 4}}
    moe = {"kind": "moe", "expert": {"ff": 5}, "router": {"experts": 3, "top": 2}, "shared": {"ff": 7}}
    return {"architecture": "Manapel", "vocab": 11, "width": 12, "norm": {"eps": 1e-5}, "logit_scale": 0.5,
            "layers": [{"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": 10}},
                       {"type": "attention", "mixer": dict(att, kv_from=0, scale=0.7), "mlp": moe},
                       {"type": "attention", "mixer": dict(att, heads=1, kv_heads=1, dim=4), "mlp": None}]}


def test_config_round_trip():
    from llark_b200.models.manapel import ManapelConfig

    c = ManapelConfig.from_dict(_cfg())
    assert (c.vocab, c.width, c.eps, c.logit_scale) == (11, 12, 1e-5, 0.5)
    assert [l.mixer.get("kv_from") for l in c.layers] == [None, 0, None] and c.layers[2].mlp is None
    assert ManapelConfig.from_dict(json.loads(json.dumps(c.to_dict()))).to_dict() == c.to_dict()
    d = _cfg()
    del d["logit_scale"]
    assert ManapelConfig.from_dict(d).logit_scale == 1.0


@pytest.mark.parametrize("bad", [
    lambda d: d.update(architecture="Other"),
    lambda d: d["layers"][0].update(type="hgrn2"),
    lambda d: d["layers"][0]["mlp"].update(kind="clamped_glu"),
    lambda d: d.update(layers=[]),
    lambda d: d["layers"][1]["mixer"].update(kv_from=1),             # itself
    lambda d: d["layers"][0]["mixer"].update(kv_from=2),             # a later layer
    lambda d: d["layers"][2]["mixer"].update(kv_from=0),             # other sizes
    lambda d: d["layers"][2].update(mixer=dict(d["layers"][1]["mixer"], kv_from=1)),   # one that has none of its own
    lambda d: d["layers"][1]["mixer"].update(rot={"base": 50.0, "dims": 4}),
])
def test_config_validation(bad):
    from llark_b200.models.manapel import ManapelConfig

    d = json.loads(json.dumps(_cfg()))
    bad(d)
    with pytest.raises(ValueError):
        ManapelConfig.from_dict(d)


def test_registry_and_tables():
    from llark_b200.mixers import FEED_FORWARDS, MIXERS
    from llark_b200.models.manapel import FEED_FORWARD_KINDS, MIXER_TYPES
    from llark_b200.models.registry import model_class_for

    assert model_class_for({"architecture": "Manapel"}).__name__ == "ManapelForCausalLM"
    assert set(MIXER_TYPES.values()) <= set(MIXERS) and set(FEED_FORWARD_KINDS.values()) <= set(FEED_FORWARDS)
    unit = MIXERS[MIXER_TYPES["attention"]].Weights
    assert unit.biases and unit.unit_heads and not (unit.gated or unit.whole_norm or unit.interleaved or unit.plus_one)
    plain = MIXERS["rotary_attention"].Weights
    assert plain.gated and not plain.unit_heads
    moe = FEED_FORWARDS[FEED_FORWARD_KINDS["moe"]].Weights
    assert moe.top_softmax and not moe.gated
    assert FEED_FORWARDS["moe"].Weights.gated and not FEED_FORWARDS["moe"].Weights.top_softmax


def test_the_mixers_projection_holds_the_parts_the_layer_has():
    """q | k | v of one product for a layer with keys and values of its own, q alone for one that reads another's; biases
    follow, offsets close up, widths are padded to 16-byte rows."""
    from llark_b200.mixers import UnitRotaryAttentionWeights

    cfg = _cfg()
    W = mo.random_weights(cfg, seed=0, dtype=torch.float32)
    own, reads = (UnitRotaryAttentionWeights(W, f"l{i}.mix.", cfg["layers"][i]["mixer"], 12, "cpu", torch.float32) for i in (0, 1))
    assert (own.q_off, own.k_off, own.v_off, own.n_in) == (0, 12, 18, 22) and tuple(own.w_in.shape) == (24, 12)
    assert torch.equal(own.w_in[12:18], W["l0.mix.k"]) and torch.equal(own.b_in[18:22], W["l0.mix.v.b"]) and not own.b_in[22:].any()
    assert (reads.q_off, reads.n_in, reads.kv_from) == (0, 12, 0) and torch.equal(reads.w_in[:12], W["l1.mix.q"])
    assert torch.equal(reads.b_in[:12], W["l1.mix.q.b"])


def test_gate_and_up_rows_alternate():
    from llark_b200.mixers import ReluGluFFWeights

    W = mo.random_weights(_cfg(), seed=0, dtype=torch.float32)
    ff = ReluGluFFWeights(W, "l0.mlp.", {"ff": 10}, 12, "cpu", torch.float32)
    assert torch.equal(ff.w_gu[0::2], W["l0.mlp.gate"]) and torch.equal(ff.w_gu[1::2], W["l0.mlp.up"])


def test_restated_norm_heads_and_router():
    x = torch.tensor([[0.0, 1.0, -50.0]], dtype=F64)
    w, b = torch.tensor([2.0, 3.0, 4.0], dtype=F64), torch.tensor([0.5, 0.0, 1.0], dtype=F64)
    y = mo.tanh_norm(x, torch.tensor(0.5, dtype=F64), w, b)
    assert torch.allclose(y, torch.tensor([[0.5, 3.0 * 0.46211715726000975, -3.0]], dtype=F64))
    g = torch.Generator().manual_seed(0)
    m = {"rot": {"base": 10.0, "dims": 4}}
    h = torch.randn(7, 2, 6, generator=g, dtype=F64)
    u = mo.turned_unit(h, m, 1e-12)
    assert torch.allclose(u.pow(2).mean(-1), torch.ones(7, 2, dtype=F64))
    assert torch.allclose(u[0], mo.rms(h[0], 1e-12)) and torch.allclose(u[..., 4:], mo.rms(h, 1e-12)[..., 4:])
    assert not torch.allclose(u[3, :, :4], mo.rms(h, 1e-12)[3, :, :4])
    same = h[:1].expand(7, 2, 6)
    v = mo.turned_unit(same, m, 1e-12)
    assert torch.allclose((v[5] * v[3]).sum(-1), (v[4] * v[2]).sum(-1))  # the distance alone counts
    W = {"router": torch.eye(4, dtype=F64), "router.b": torch.tensor([0.0, 5.0, 0.0, -9.0], dtype=F64)}
    ids, wts = mo.route(torch.tensor([[1.0, -4.5, 3.0, 2.0]], dtype=F64), W, "", {"router": {"top": 2}})
    assert ids.tolist() == [[2, 0]] and torch.allclose(wts, torch.softmax(torch.tensor([[3.0, 1.0]], dtype=F64), -1))


def test_restated_model_is_causal_and_shares_keys():
    cfg = _cfg()
    W = mo.random_weights(cfg, seed=0)
    toks = [1, 5, 3, 9, 0, 2, 7, 7, 4]
    full, res = mo.forward(cfg, W, toks, return_residuals=True)
    assert full.shape == (9, 11) and len(res) == 3
    assert torch.allclose(mo.forward(cfg, W, toks[:5]), full[:5], atol=1e-12)
    assert "l1.mix.k" not in W and "l1.mix.q.b" in W and "l2.norm2" not in W
    moved = dict(W)
    moved["l0.mix.v"] = W["l0.mix.v"] * 2.0
    _, other = mo.forward(cfg, moved, toks, return_residuals=True)
    assert not torch.allclose(other[1] - other[0], res[1] - res[0])
    doubled = json.loads(json.dumps(cfg))
    doubled["logit_scale"] = 1.0
    assert torch.allclose(mo.forward(doubled, W, toks), 2.0 * full)
