"""Host side of the Buvesun path without a GPU: configuration reading and validation, the order of layer runs, the registry and
the mixer and feed-forward tables, packing, and the restatement itself (norm, rotation, decaying memory, window, router,
inputs that carry the weights, loop)."""
import json

import pytest
import torch

import buvesun_oracle as bo

F64 = torch.float64


def _cfg():
    moe = {"kind": "moe", "expert": {"ff": 5, "limit": 1.5}, "router": {"experts": 3, "top": 2}, "shared": {"ff": 7, "limit": 0.5}}
    left = {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 5, "scale": 0.5, "mask": {"size": 3}, "rot": {"base": 100.0, "dims": 4}}
    right = {"heads": 3, "dim": 4, "vdim": 2, "decay": [0.5, 0.9, 1.0]}
    return {"architecture": "Buvesun", "vocab": 11, "width": 12, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
            "residual_mult": 0.4, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "retention", "mlp": moe, "mixer": {"heads": 2, "dim": 6, "vdim": 3, "decay": [0.0, 0.7],
                                                                   "rot": {"base": 50.0, "dims": 6}}},
                       {"type": "parallel", "mlp": None, "mixer": {"left": left, "right": right, "left_scale": 0.8, "right_scale": -0.3}},
                       {"type": "retention", "mlp": dict(moe, shared=None), "mixer": {"heads": 1, "dim": 4, "vdim": 4, "decay": [0.99],
                                                                                      "rot": {"base": 50.0, "dims": 2}}}]}


def test_config_round_trip_and_layer_runs():
    from llark_b200.models.buvesun import BuvesunConfig

    c = BuvesunConfig.from_dict(_cfg())
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.residual_mult) == (11, 12, 1e-5, 2.0, 0.4)
    assert c.layers[1].mlp is None and c.loop == {"start": 1, "stop": 3, "times": 2}
    assert BuvesunConfig.from_dict(json.loads(json.dumps(c.to_dict()))).to_dict() == c.to_dict()
    assert [(i, f) for i, _, f in c.layer_runs()] == [(0, False), (1, True), (2, False), (1, True), (2, False)] == bo.layer_runs(_cfg())
    assert [t for _, t, _ in c.layer_runs()] == [None, 0, 0, 1, 1]
    for loop, runs in ((None, [(0, False), (1, False), (2, False)]),
                       ({"start": 0, "stop": 1, "times": 3}, [(0, True), (0, True), (0, True), (1, False), (2, False)]),
                       ({"start": 2, "stop": 3, "times": 1}, [(0, False), (1, False), (2, True)])):
        d = dict(_cfg(), loop=loop)
        assert [(i, f) for i, _, f in BuvesunConfig.from_dict(d).layer_runs()] == runs == bo.layer_runs(d)


@pytest.mark.parametrize("bad", [
    lambda d: d.update(architecture="Other"),
    lambda d: d["layers"][0].update(type="hgrn2"),
    lambda d: d["layers"][0]["mlp"].update(kind="dense"),
    lambda d: d.update(layers=[]),
    lambda d: d["layers"][0]["mixer"].update(decay=[0.5]),              # one per head
    lambda d: d["layers"][1]["mixer"]["right"].update(decay=[0.5, 1.5, 0.1]),
    lambda d: d["loop"].update(stop=4),
    lambda d: d["loop"].update(start=-1),
    lambda d: d["loop"].update(times=0),
])
def test_config_validation(bad):
    from llark_b200.models.buvesun import BuvesunConfig

    d = json.loads(json.dumps(_cfg()))
    bad(d)
    with pytest.raises(ValueError):
        BuvesunConfig.from_dict(d)


def test_registry_and_tables():
    from llark_b200.mixers import FEED_FORWARDS, MIXERS
    from llark_b200.models.buvesun import FEED_FORWARD_KINDS, MIXER_TYPES
    from llark_b200.models.registry import model_class_for

    assert model_class_for({"architecture": "Buvesun"}).__name__ == "BuvesunForCausalLM"
    assert set(MIXER_TYPES.values()) <= set(MIXERS) and set(FEED_FORWARD_KINDS.values()) <= set(FEED_FORWARDS)
    ret, light = MIXERS["retention"].Weights, MIXERS["lightning"].Weights
    assert (ret.rotates, ret.head_norm, ret.gate_silu) == (True, True, True)
    assert (light.rotates, light.head_norm, light.gate_silu) == (False, False, False)
    window = MIXERS["rotary_attention_window"].Weights
    assert window.interleaved and window.mask_kind == "window" and not (window.gated or window.biases or window.unit_heads)
    moe = FEED_FORWARDS[FEED_FORWARD_KINDS["moe"]].Weights
    assert moe.clamped and moe.sigmoid_input and not moe.top_softmax
    assert not FEED_FORWARDS["moe"].Weights.clamped and not FEED_FORWARDS["moe_top_softmax"].Weights.sigmoid_input


def test_packing_of_mixers_and_units():
    """One projection in per mixer (both sides of a parallel one together), one out over both sides' heads with the right
    side on a 16-byte boundary and its number in its norm; gate and up rows alternate."""
    from llark_b200.mixers import ClampedGluFFWeights, RetentionWeights, WeightedParallelMixersWeights

    cfg = _cfg()
    W = bo.random_weights(cfg, seed=0, dtype=torch.float32)
    r = RetentionWeights(W, "l0.mix.", cfg["layers"][0]["mixer"], 12, "cpu", torch.float32)
    assert (r.k_off, r.v_off, r.g_off, r.n_in) == (12, 24, 30, 36) and tuple(r.w_in.shape) == (40, 12)
    assert torch.equal(r.w_in[12:24], W["l0.mix.k"]) and torch.equal(r.w_in[30:36], W["l0.mix.g"]) and r.norm is None
    assert r.k_scale == 6 ** -0.5 and torch.allclose(r.powers[1, :4], torch.tensor([1.0, 0.7, 0.49, 0.343]))
    p = WeightedParallelMixersWeights(W, "l1.mix.", cfg["layers"][1]["mixer"], 12, "cpu", torch.float32)
    assert p.n_left == 24 and tuple(p.w_in.shape) == (24 + 40, 12) and torch.equal(p.w_in[24 + 12:24 + 24], W["l1.mix.right.k"])
    assert (p.o_left, p.o_right, p.n_out) == (10, 16, 22) and not p.w_o[:, 10:16].any()
    assert torch.equal(p.w_o[:, :10], W["l1.mix.left.o"]) and torch.equal(p.w_o[:, 16:], W["l1.mix.right.o"])
    assert torch.allclose(p.right_norm, -0.3 * W["l1.mix.right.norm"]) and p.left_scale == 0.8
    u = ClampedGluFFWeights(W, "l0.mlp.shared.", cfg["layers"][0]["mlp"]["shared"], 12, "cpu", torch.float32)
    assert torch.equal(u.w_gu[0::2], W["l0.mlp.shared.gate"]) and torch.equal(u.w_gu[1::2], W["l0.mlp.shared.up"]) and u.limit == 0.5


def test_equal_rotations_share_their_frequencies():
    from llark_b200.mixers import RetentionWeights

    W = bo.random_weights(_cfg(), seed=0, dtype=torch.float32)
    spec = _cfg()["layers"][0]["mixer"]
    a, b = (RetentionWeights(W, "l0.mix.", spec, 12, "cpu", torch.float32) for _ in range(2))
    c = RetentionWeights(W, "l0.mix.", dict(spec, rot={"base": 50.0, "dims": 4}), 12, "cpu", torch.float32)
    assert a.freq is b.freq and c.freq is not a.freq and c.freq.numel() == 2
    with pytest.raises(ValueError):
        RetentionWeights(W, "l0.mix.", dict(spec, rot={"base": 50.0, "dims": 8}), 12, "cpu", torch.float32)


def test_chunks_of_a_step_name_their_inner_ones():
    from llark_b200.state_cache import StepLayout

    c = StepLayout([70, 32, 5], [0, 0, 0], [4, 2, 9], "cpu").chunks(32)
    assert c.n.tolist() == [32, 32, 6, 32, 5] and c.index.tolist() == [0, 1, 2, 3, 4]
    assert c.inner.tolist() == [0, 1, -1, -1, -1] and c.last_slot.tolist() == [-1, -1, 4, 2, 9]


def test_restated_norms_rotations_and_units():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(4, 9, generator=g, dtype=F64) + 3.0
    assert torch.allclose(bo.layer_norm(x, torch.full((9,), 2.0, dtype=F64), 1e-5), 2.0 * torch.nn.functional.layer_norm(x, (9,), eps=1e-5))
    h = torch.randn(7, 2, 6, generator=g, dtype=F64)
    f = bo.frequencies(4, 10.0)
    p = torch.arange(7)
    halves, near = bo.turn(h, p, f, False), bo.turn(h, p, f, True)
    assert torch.equal(halves[..., 4:], h[..., 4:]) and torch.equal(near[0], h[0])
    assert torch.allclose(bo.turn(h[..., [0, 2, 1, 3, 4, 5]], p, f, False)[..., [0, 2, 1, 3, 4, 5]], near)
    z = torch.complex(h[..., 0], h[..., 1]) * torch.exp(1j * p.double() * f[0])[:, None]
    assert torch.allclose(near[..., 0], z.real) and torch.allclose(near[..., 1], z.imag)
    one = torch.eye(3, dtype=F64)
    W = {"gate": one, "up": one, "down": one}
    y = bo.clamped_unit(torch.tensor([[5.0, -9.0, 0.5]], dtype=F64), W, "", 2.0)
    want = [2.0 / (1 + torch.exp(torch.tensor(-3.404, dtype=F64))) * 3.0, -9.0 / (1 + torch.exp(torch.tensor(15.318, dtype=F64))) * -1.0,
            0.5 / (1 + torch.exp(torch.tensor(-0.851, dtype=F64))) * 1.5]
    assert torch.allclose(y[0], torch.stack(want))


def test_restated_memory_window_and_router():
    g = torch.Generator().manual_seed(1)
    q, k = (torch.randn(9, 2, 3, generator=g, dtype=F64) for _ in range(2))
    v = torch.randn(9, 2, 4, generator=g, dtype=F64)
    o, S = bo.decayed_memory(q, k, v, [0.5, 1.0])
    for t in (0, 3, 8):  # the closed form: a sum over everything before, weighed by the powers of the decay
        for h, d in enumerate((0.5, 1.0)):
            want = sum(d ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)
    first, S1 = bo.decayed_memory(q[:4], k[:4], v[:4], [0.5, 1.0])
    rest, S2 = bo.decayed_memory(q[4:], k[4:], v[4:], [0.5, 1.0], S1)
    assert torch.allclose(torch.cat([first, rest]), o) and torch.allclose(S2, S)
    y = bo.windowed_attention(q, k, v, 0.7, 3)
    moved = v.clone()
    moved[4] += 100.0
    changed = (bo.windowed_attention(q, k, moved, 0.7, 3) - y).abs().amax(dim=(1, 2)) > 0
    assert changed.nonzero().flatten().tolist() == [4, 5, 6]
    assert torch.allclose(bo.windowed_attention(q, k, v, 0.7, 1), v)
    W = {"router": torch.eye(4, dtype=F64)}
    ids, wts = bo.route(torch.tensor([[1.0, -4.5, 3.0, 2.0]], dtype=F64), W, "", {"router": {"top": 2}})
    assert ids.tolist() == [[2, 3]] and torch.allclose(wts, torch.sigmoid(torch.tensor([[3.0, 2.0]], dtype=F64)))


def test_restated_model_is_causal_and_loops():
    cfg = _cfg()
    W = bo.random_weights(cfg, seed=0)
    toks = [1, 5, 3, 9, 0, 2, 7, 7, 4]
    full, res = bo.forward(cfg, W, toks, return_residuals=True)
    assert full.shape == (9, 11) and len(res) == 5
    assert torch.allclose(bo.forward(cfg, W, toks[:5]), full[:5], atol=1e-12)
    assert "l1.norm2" not in W and "l2.mlp.shared.up" not in W and tuple(W["loop.in"].shape) == (12, 24)
    cut = json.loads(json.dumps(cfg))
    cut["loop"]["times"] = 1
    _, once = bo.forward(cfg | {"loop": cut["loop"]}, W, toks, return_residuals=True)
    assert len(once) == 3 and all(torch.equal(a, b) for a, b in zip(once, res[:3])) and not torch.allclose(res[4], res[2])
    blind = dict(W)
    blind["loop.in"] = torch.cat([W["loop.in"][:, :12], torch.zeros(12, 12, dtype=F64)], dim=1)
    assert not torch.allclose(bo.forward(cfg, blind, toks), full)  # the embedding joins in front of every pass
