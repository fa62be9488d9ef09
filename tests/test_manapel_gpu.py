"""Manapel on the GPU against the plain restatement in tests/manapel_oracle.py (float64 on the CPU): every mechanism alone
through its op or its class, then the whole model through the engine's step function, the slot cache, the scheduler,
generate() and the command-line tools. Configurations are small and deliberately unlike each other: key heads shared by all,
by two or by none, key and value sizes that differ (scalar attention route) or agree at a multiple of 16 (tensor-core route),
rotation over a part of the head and over all of it, layers that read the keys and values of the layer before, of one further
back and of one that two others read as well, one expert of one, mixtures with and without a shared expert, layers without a
feed-forward."""
import math

import pytest
import torch

import manapel_oracle as mo

pytestmark = pytest.mark.gpu
F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16


def _dev():
    return torch.device("cuda:0")


def _layout(lens, pos0, slots):
    from llark_b200.state_cache import StepLayout

    return StepLayout(lens, pos0, slots, _dev())


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm() / (b.norm() + 1e-30)).item()


def _errors(got, want):
    """Per position: rms of the difference of the logits with the mean over the vocabulary taken off, relative to the rms of
    the expected ones over all positions."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(dim=-1, keepdim=True)
    w = want.double().cpu()
    w = w - w.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def _agree(got, want, dtype):
    """fp32: every position. bf16: a router decides between two almost equal logits now and then, and rounding may turn the
    choice; so one position in twenty (at least one) may lie above the bound, none far above."""
    e = _errors(got, want)
    assert torch.isfinite(e).all()
    if dtype == F32:
        assert e.max() < 1e-4, e.max()
    else:
        assert (e > 6e-2).sum() <= max(1, e.numel() // 20) and e.max() < 0.6, (e.max(), (e > 6e-2).sum(), e.numel())


# ------------------------------------------------------------------------------------------------ configurations
def _att(heads, kv, dim, vdim, rot, kv_from=None, scale=None, mlp=None, base=100.0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
         "scale": scale or 1.0 / math.sqrt(dim)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _cfg(layers, vocab=97, width=72, eps=1e-6, logit_scale=1.5):
    return {"architecture": "Manapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": layers}


CONFIGS = {
    # every size differs from every other; the layer that reads another's keys sits right behind it or two further on, has a
    # mixture or a dense feed-forward, and one layer has no feed-forward at all
    "mixed": _cfg([_att(4, 2, 16, 12, 8, mlp=_dense(40)), _att(4, 2, 16, 12, 8, kv_from=0, scale=0.4, mlp=_moe(6, 2, 20, 33)),
                   _att(3, 3, 10, 6, 10, base=30.0, mlp=_moe(7, 3, 12)), _att(2, 1, 6, 8, 2, base=7.0),
                   _att(3, 3, 10, 6, 10, kv_from=2, base=30.0, mlp=_dense(31))]),
    # nothing a multiple of 4 but the rotated parts, an eps that counts beside the squares, a mixture of one expert first, a
    # layer whose keys and values two others read, a mixture that uses all of its experts, logits scaled down
    "odd_sizes": _cfg([_att(3, 1, 6, 5, 6, mlp=_moe(1, 1, 9, 7)), _att(3, 1, 6, 5, 6, kv_from=0, mlp=_moe(3, 3, 11)),
                       _att(3, 1, 6, 5, 6, kv_from=0, scale=1.3), _att(2, 2, 9, 9, 2, base=1000.0, mlp=_dense(17))],
                      vocab=33, width=51, eps=0.3, logit_scale=0.25),
    # sizes of the tensor-core routes: heads of 32 and 16, products at least 64 wide, a head rotated in part
    "tiles": _cfg([_att(4, 2, 32, 32, 16, base=1e4, mlp=_moe(5, 3, 64, 72)), _att(4, 2, 32, 32, 16, kv_from=0, base=1e4, mlp=_dense(96)),
                   _att(4, 4, 16, 16, 16, mlp=_moe(9, 4, 72, 64)), _att(4, 4, 16, 16, 16, kv_from=2, mlp=_moe(4, 2, 80))],
                  vocab=120, width=128, logit_scale=3.0),
}


def _model(cfg, W, dtype):
    from llark_b200.models.manapel import ManapelConfig, ManapelForCausalLM

    return ManapelForCausalLM(ManapelConfig.from_dict(cfg), W, device="cuda:0", dtype=dtype)


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class _Stores:
    """Stand-in cache for mixers used alone: slot stores filled with garbage."""

    def __init__(self, n_slots=4, positions=512):
        self.t, self.n, self.positions = [], n_slots, positions

    def add_store(self, shape, dtype, zero_on_alloc, per_position=False):
        lead = (self.positions,) if per_position else ()
        self.t.append(torch.full((self.n,) + lead + tuple(shape), float("nan"), device=_dev(), dtype=dtype))
        return len(self.t) - 1

    def view(self, h):
        return self.t[h]


def _run_mixers(W, specs, width, hs, portions, act, eps=1e-5, slot=2):
    """Mixers 'm0.', 'm1.', ... on one stand-in cache, one request in `slot` cut into `portions`: specs[i] may name an earlier
    one in kv_from; hs[i] [T, width] is mixer i's input. Returns their outputs."""
    from llark_b200.mixers import MIXERS
    from llark_b200.models.manapel import MIXER_TYPES

    cls = MIXERS[MIXER_TYPES["attention"]]
    Wf = {k: v.to(F32) for k, v in W.items()}
    stores, mixers = _Stores(), []
    for i, spec in enumerate(specs):
        j = spec.get("kv_from")
        mixers.append(cls(cls.Weights(Wf, f"m{i}.", spec, width, _dev(), act), stores, eps, act, None,
                          lender=mixers[j] if j is not None else None))
    outs, at = [[] for _ in specs], 0
    for n in portions:
        st = _layout([n], [at], [slot])
        for i, m in enumerate(mixers):
            outs[i].append(m.forward(hs[i][at:at + n].to(_dev(), act).contiguous(), st, stores).cpu())
        for m in mixers:
            m.end_step()
            assert m.step_kv is None
        at += n
    assert at == hs[0].shape[0]
    return [torch.cat(o) for o in outs]


def _oracle_mixers(W, specs, hs, eps=1e-5):
    outs, kept = [], {}
    for i, spec in enumerate(specs):
        y, kept[i] = mo.attention_mixer(hs[i], W, f"m{i}.", spec, eps, kept.get(spec.get("kv_from")))
        outs.append(y)
    return outs


def _mixer_weights(specs, width, seed):
    W = mo.random_weights(_cfg([{"type": "attention", "mixer": s, "mlp": None} for s in specs], width=width), seed=seed)
    return {"m" + k[1:].replace(".mix", "", 1): v for k, v in W.items() if ".mix." in k}


def _inputs(n, T, width, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(T, width, generator=g, dtype=F64).to(BF16).to(F64) for _ in range(n)]


PORTIONS = ([150], [1] * 150, [100] + [1] * 50, [31, 2, 2, 65, 1, 1, 30, 18])


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("C", [8, 51, 72, 1024, 1028, 2048, 4100])
def test_tanh_norm_and_the_sum_with_the_next_input_norm(C):
    from llark_b200 import ops

    g = torch.Generator().manual_seed(C)
    n, d = 13, _dev()

    def norm():
        return 0.2 + torch.rand((), generator=g, dtype=F64), torch.randn(C, generator=g, dtype=F64), torch.randn(C, generator=g, dtype=F64)

    def to_dev(p):
        return float(p[0]), p[1].to(d, F32), p[2].to(d, F32)

    x, y = 2.0 * torch.randn(n, C, generator=g, dtype=F64), 3.0 * torch.randn(n, C, generator=g, dtype=F64)
    x[0] *= 100.0   # saturated
    x[1] *= 1e-4    # all but linear
    a, b = norm(), norm()
    rows = torch.tensor([5, 0, 12, 1], dtype=torch.int32, device=d)
    for act, tol in ((F32, 2e-6), (BF16, 4e-3)):
        got = ops.seq_tanh_norm(x.to(d, F32), to_dev(a), act)
        assert got.dtype == act and _rel(got, mo.tanh_norm(x, *a)) < tol
        assert _rel(ops.seq_tanh_norm(x.to(d, F32), to_dev(a), act, rows=rows), mo.tanh_norm(x, *a)[rows.cpu().long()]) < tol
    for top in (0, 1, 3, 6):
        for with_y in (True, False):
            if not with_y and not top:
                continue
            z = torch.randn(n * max(top, 1), C, generator=g, dtype=F64)
            pos = torch.randperm(n * top, generator=g).to(torch.int32) if top else None
            wts = torch.rand(n, top, generator=g, dtype=F64)
            f = y.clone() if with_y else torch.zeros_like(x)
            for t in range(n):
                for k in range(top):
                    f[t] += wts[t, k] * z[int(pos[t * top + k])]
            want = x + mo.tanh_norm(f, *a)
            kw = {"y": y.to(d, F32) if with_y else None}
            if top:
                kw.update(z=z.to(d, F32), pos_of=pos.to(d), wts=wts.to(d, F32))
            assert _rel(ops.seq_tanh_norm_add(x.to(d, F32), to_dev(a), **kw), want) < 2e-6
            for act, tol in ((F32, 2e-6), (BF16, 4e-3)):
                got, nxt = ops.seq_tanh_norm_add(x.to(d, F32), to_dev(a), next_norm=to_dev(b), act=act, **kw)
                assert _rel(got, want) < 2e-6 and nxt.dtype == act and _rel(nxt, mo.tanh_norm(want, *b)) < tol


@pytest.mark.parametrize("M", [1, 2, 7, 8, 9, 70, 300])
@pytest.mark.parametrize("N,K", [(6, 10), (64, 64), (136, 72), (264, 512), (5000, 64), (5010, 48)])
def test_activations_in_the_products(M, N, K):
    """Squared ReLU and the gated ReLU on alternating rows, through the weight-streaming kernel (up to 8 rows), the tcgen05
    core and the tiled kernel, with and without a bias, on a column slice."""
    from llark_b200 import ops

    g = torch.Generator().manual_seed(M + N)
    x = torch.randn(M, K + 8, generator=g, dtype=F64).to(BF16).to(F64)
    w = (torch.randn(N, K, generator=g, dtype=F64) / math.sqrt(K)).to(BF16).to(F64)
    bias = torch.randn(N, generator=g, dtype=F64).to(F32).to(F64)
    d = _dev()
    for bb in (None, bias):
        z = x[:, :K] @ w.T + (bb if bb is not None else 0.0)
        want = {"relu2": torch.relu(z) ** 2, "relu_glu": torch.relu(z[:, 0::2]) * z[:, 1::2]}
        for act, y in want.items():
            for dt, out, tol in ((F32, F32, 1e-5), (BF16, F32, 1e-5), (BF16, BF16, 4e-3)):
                got = ops.linear(x.to(d, dt)[:, :K], w.to(d, dt), bias=bb.to(d, F32) if bb is not None else None, out_dtype=out,
                                 act=act)
                assert got.shape == y.shape and got.dtype == out and _rel(got, y) < tol, (act, dt, out)


@pytest.mark.parametrize("H,G,D,E,n_rot,interleaved", [
    (4, 2, 16, 12, 8, False), (3, 3, 10, 6, 10, False), (2, 1, 6, 8, 0, False), (3, 1, 32, 32, 32, False), (5, 5, 7, 4, 6, False),
    (2, 2, 24, 16, 16, True), (7, 1, 128, 64, 128, False), (3, 1, 128, 128, 32, False), (2, 1, 64, 256, 64, False),
    (1, 1, 256, 256, 128, False), (40, 8, 128, 128, 128, False), (2, 1, 320, 16, 64, False), (2, 1, 12, 8, 4, True)])
def test_rotated_heads_divided_by_their_root_mean_square(H, G, D, E, n_rot, interleaved):
    from llark_b200 import ops

    g = torch.Generator().manual_seed(H * D + E)
    T, pos0, eps = 9, 37, 1e-2
    n = H * D + G * D + G * E
    f = mo.frequencies(n_rot, 50.0)
    pos = torch.arange(pos0, pos0 + T)
    perm = torch.arange(D)  # the restatement rotates halves: bring interleaved pairs into that order and back
    if interleaved:
        perm = torch.cat([torch.arange(0, n_rot, 2), torch.arange(1, n_rot, 2), torch.arange(n_rot, D)])
    d = _dev()
    st = _layout([T], [pos0], [0])
    for off in (3, 4):  # columns in front of q: an odd offset takes the scalar kernel, a multiple of four the 16-byte one
        src = torch.randn(T, n + off + (-(n + off)) % 4, generator=g, dtype=F64)
        src[2] *= 0.01  # squares that eps counts beside
        q, k, v = src[:, off:off + H * D], src[:, off + H * D:off + (H + G) * D], src[:, off + (H + G) * D:off + n]

        def unit(x, heads):
            y = mo.turn(x.reshape(T, heads, D)[..., perm], pos, f)
            return mo.rms(y, eps)[..., torch.argsort(perm)].reshape(T, -1)

        for act in (F32, BF16):
            tol = 2e-6 if act == F32 else 4e-3
            kw = dict(qk_freq=f.to(d, F32) if n_rot else None, qk_interleaved=interleaved, unit=True)
            gq, gk, gv = ops.seq_qkv_rotary(src.to(d, F32), off, off + H * D, off + (H + G) * D, H, G, D, E, eps, act, st, **kw)
            assert _rel(gq, unit(q, H)) < tol and _rel(gk, unit(k, G)) < tol and _rel(gv, v) < tol
            assert _rel(gq[2], unit(q, H)[2]) < tol
            oq, ok, ov = ops.seq_qkv_rotary(src.to(d, F32), off, 0, 0, H, 0, D, E, eps, act, st, **kw)  # queries alone
            assert ok is None and ov is None and _rel(oq, gq) < tol


@pytest.mark.parametrize("n_exp,top", [(1, 1), (3, 3), (8, 4), (40, 6), (64, 32), (200, 8)])
def test_router_takes_the_largest_logits_and_weighs_them_among_themselves(n_exp, top):
    from llark_b200 import ops

    g = torch.Generator().manual_seed(n_exp)
    z = 4.0 * torch.randn(37, n_exp + 5, generator=g, dtype=F64)
    z[3, :n_exp] = torch.linspace(-900.0, 0.0, n_exp, dtype=F64)[torch.randperm(n_exp, generator=g)]  # far apart: exp() of most is 0
    z[4] -= 1e4
    z = z.to(F32).to(F64)
    ids, wts = ops.seq_moe_route_top(z.to(_dev(), F32)[:, :n_exp], top)
    best = torch.topk(z[:, :n_exp], top, dim=-1)
    assert torch.equal(ids.cpu().long(), best.indices)
    assert (wts.cpu().double() - torch.softmax(best.values, dim=-1)).abs().max() < 1e-6
    tied = torch.zeros(2, n_exp, device=_dev())
    ids, wts = ops.seq_moe_route_top(tied, top)  # ties go to the lower number
    assert ids.tolist() == [list(range(top))] * 2 and (wts - 1.0 / top).abs().max() < 1e-6


@pytest.mark.parametrize("T", [1, 5, 60, 300, 800])
@pytest.mark.parametrize("width,m", [(40, _moe(6, 2, 20, 33)), (51, _moe(3, 3, 11)), (96, _moe(9, 3, 64, 72)), (30, _moe(1, 1, 5, 3)),
                                     (64, _moe(33, 1, 67))])
def test_mixture_of_experts_alone(T, width, m):
    """Few tokens (weight-streaming kernels), some hundreds (grouped kernels) and, in bf16 with sizes for it, the tcgen05
    core's runs of rows; every position in fp32, the right experts in bf16 (the router's logits are the same)."""
    from llark_b200 import ops
    from llark_b200.mixers import FEED_FORWARDS
    from llark_b200.models.manapel import FEED_FORWARD_KINDS

    W = mo.random_weights(_cfg([_att(1, 1, 2, 2, 2, mlp=m)], width=width), seed=T)
    W = {k[len("l0.mlp."):]: v for k, v in W.items() if k.startswith("l0.mlp.")}
    h = _inputs(1, T, width, T)[0]
    want = mo.expert_mixture(h, W, "", m)
    cls = FEED_FORWARDS[FEED_FORWARD_KINDS["moe"]]
    d = _dev()
    one = (1.0, torch.ones(width, device=d), torch.zeros(width, device=d))
    for act, tol in ((F32, 1e-5), (BF16, 2e-2)):
        ff = cls(cls.Weights({k: v.to(F32) for k, v in W.items()}, "", m, width, d, act), act)
        t = ff.terms(h.to(d, act))
        got = torch.zeros(T, width, dtype=F64) if t["y"] is None else t["y"].double().cpu()
        wts, z, pos = t["wts"].double().cpu(), t["z"].double().cpu(), t["pos_of"].cpu().long()
        for k in range(m["router"]["top"]):
            got += wts[:, k:k + 1] * z[pos[k::m["router"]["top"]]]
        assert _rel(got, want) < tol
        x = torch.zeros(T, width, device=d)
        assert _rel(ops.seq_tanh_norm_add(x, one, **t), torch.tanh(got)) < 1e-5
        if not m.get("shared"):
            assert t["y"] is None


@pytest.mark.parametrize("ff", [3, 20, 33, 64, 200])
def test_dense_feed_forward_alone(ff):
    from llark_b200.mixers import FEED_FORWARDS
    from llark_b200.models.manapel import FEED_FORWARD_KINDS

    width = 72
    W = mo.random_weights(_cfg([_att(1, 1, 2, 2, 2, mlp=_dense(ff))], width=width), seed=ff)
    W = {k[len("l0.mlp."):]: v for k, v in W.items() if k.startswith("l0.mlp.")}
    cls = FEED_FORWARDS[FEED_FORWARD_KINDS["dense"]]
    for T in (1, 6, 90):
        h = _inputs(1, T, width, T)[0]
        for act, tol in ((F32, 1e-5), (BF16, 1e-2)):
            unit = cls(cls.Weights({k: v.to(F32) for k, v in W.items()}, "", _dense(ff), width, _dev(), act), act)
            assert _rel(unit.terms(h.to(_dev(), act))["y"], mo.relu_gated_ff(h, W, "")) < tol


SPECS = {
    "one": [_att(4, 2, 16, 12, 8)], "odd": [_att(3, 1, 7, 5, 6, scale=0.9)], "tile": [_att(2, 2, 32, 32, 16)],
    "wide": [_att(2, 1, 128, 128, 128, base=5e4)],
    "pair": [_att(4, 2, 16, 12, 8), _att(4, 2, 16, 12, 8, kv_from=0, scale=0.7)],
    "pair_tile": [_att(4, 2, 32, 32, 32), _att(4, 2, 32, 32, 32, kv_from=0)],
    "two_readers": [_att(3, 1, 16, 16, 4), _att(3, 1, 16, 16, 4, kv_from=0), _att(2, 2, 6, 6, 2), _att(3, 1, 16, 16, 4, kv_from=0)],
}


@pytest.mark.parametrize("name", sorted(SPECS))
def test_mixers_in_one_step_in_portions_and_token_by_token(name):
    """A mixer alone, and mixers that read the keys and values of another: each has an input of its own, so that keys made
    from the wrong input would show."""
    specs = [s["mixer"] for s in SPECS[name]]
    C = 40
    W = _mixer_weights(specs, C, seed=5)
    hs = _inputs(len(specs), 150, C, 4)
    want = _oracle_mixers(W, specs, hs)
    for portions in PORTIONS:
        for g, w in zip(_run_mixers(W, specs, C, hs, portions, F32), want):
            assert _rel(g, w) < 2e-5, portions
    for portions in ([150], [31, 2, 2, 65, 1, 1, 30, 18], [20] + [1] * 130):
        for g, w in zip(_run_mixers(W, specs, C, hs, portions, BF16), want):
            assert _rel(g, w) < 2e-2, portions


# ------------------------------------------------------------------------------------------------ keys at edges and far away
def _needle(T, H, G, D, E, n_rot, at, far, seed):
    """Projections that ARE the input (identity weights): queries and keys are random directions except that the query at
    position `at` points, in every head, along the key at position `far` in the entries that are not rotated (its rotated
    ones are zero); that key's value stands out. Two inputs: one for the layer that makes keys and values, one for queries."""
    g = torch.Generator().manual_seed(seed)
    C = H * D + G * D + G * E
    h = torch.randn(T, C, generator=g, dtype=F64)
    k_off, v_off = H * D, (H + G) * D
    for hd in range(H):
        kv = hd // (H // G)
        h[at, hd * D:(hd + 1) * D] = h[far, k_off + kv * D:k_off + (kv + 1) * D]
        h[at, hd * D:hd * D + n_rot] = 0.0
    h[far, v_off:] = 50.0 + torch.arange(G * E, dtype=F64)
    eye = torch.eye(C, dtype=F64)
    W = {}
    for p in ("m0.", "m1."):
        W.update({p + "q": eye[:k_off], p + "o": eye[:, :H * E].clone(), p + "q.b": torch.zeros(k_off, dtype=F64)})
    W.update({"m0.k": eye[k_off:v_off], "m0.v": eye[v_off:], "m0.k.b": torch.zeros(G * D, dtype=F64),
              "m0.v.b": torch.zeros(G * E, dtype=F64)})
    h = h.to(BF16).to(F64)
    other = torch.randn(T, C, generator=g, dtype=F64).to(BF16).to(F64)  # the second mixer's own "keys" say nothing
    other[:, :k_off] = h[:, :k_off]
    spec = _att(H, G, D, E, n_rot, scale=3.0)["mixer"]
    return [h, other], W, [spec, dict(spec, kv_from=0)], C


@pytest.mark.parametrize("at,far", [(383, 0), (383, 1), (383, 31), (383, 63), (383, 64), (383, 127), (383, 255), (383, 256),
                                    (383, 320), (383, 382), (383, 383), (200, 200), (200, 201), (200, 199), (63, 63), (63, 64),
                                    (64, 63), (128, 129), (255, 256), (256, 0), (1, 0), (0, 0), (0, 1)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_key_that_one_query_asks_for(at, far, dtype):
    """384 tokens. The key sits far back, at a key tile's edge (32 for the scalar kernel, 64 for the tensor-core one), at the
    edge of the first 256 entries of a store, at the query's own position, right before it, or right behind it (not seen)."""
    T, H, G, D, E = 384, 2, 1, 32, 32
    hs, W, specs, C = _needle(T, H, G, D, E, 4, at, far, seed=far)
    want = _oracle_mixers(W, specs, hs)
    for w in want:  # the read-out is the needle's value, or nothing like it
        assert (w[at, :H * E].abs().max() > 40.0) == (far <= at)
    tails = ([384], [383, 1], [256, 100, 27, 1], [200] + [1] * 184, [300, 2, 2] + [1] * 80)
    for portions in tails if dtype == F32 or at == 383 else tails[:4]:
        for g, w in zip(_run_mixers(W, specs, C, hs, portions, dtype), want):
            # a query that asks for a key it does not see has an ordinary sharp softmax, where bf16 rounding shows more
            assert _rel(g[at], w[at]) < (1e-4 if dtype == F32 else (2e-2 if far <= at else 0.1)), portions
            assert _rel(g, w) < (1e-4 if dtype == F32 else 3e-2), portions


def test_scores_depend_on_the_distance_only():
    """The outputs for the last tokens do not change when all positions move by the same amount: the same 40 inputs behind
    24 tokens whose keys point away from every query (they get no weight)."""
    H, D = 2, 16
    C = 3 * H * D
    eye = torch.eye(C, dtype=F64)
    zero = torch.zeros(H * D, dtype=F64)
    W = {"m0.q": eye[:H * D], "m0.k": eye[H * D:2 * H * D], "m0.v": eye[2 * H * D:], "m0.o": eye[:, :H * D].clone(),
         "m0.q.b": zero, "m0.k.b": zero, "m0.v.b": zero}
    h = _inputs(1, 64, C, 3)[0]
    d = torch.ones(D - 4, dtype=F64)
    for hd in range(H):
        h[:, hd * D + 4:(hd + 1) * D] = 1.0                                   # queries share a direction (unrotated part)
        h[:24, H * D + hd * D:H * D + (hd + 1) * D] = torch.cat([torch.zeros(4, dtype=F64), -d])
        h[24:, H * D + hd * D + 4:H * D + (hd + 1) * D] = d * 0.2
    spec = _att(H, H, D, D, 4, scale=8.0, base=30.0)["mixer"]
    a = _run_mixers(W, [spec], C, [h], [64], F32)[0][24:]
    b = _run_mixers(W, [spec], C, [h[24:]], [40], F32)[0]
    assert _rel(a, b) < 2e-5
    assert _rel(a, _oracle_mixers(W, [spec], [h])[0][24:]) < 2e-5


# ------------------------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_layer(name):
    cfg = CONFIGS[name]
    W = mo.random_weights(cfg, seed=1)
    toks = _tokens(75, cfg["vocab"], 1)
    want, want_layers = mo.forward(cfg, W, toks, return_residuals=True)
    m = _model(cfg, W, F32)
    cache = m.new_cache()
    logits, res = m.engine.step(cache, [cache.alloc()], [toks], want=[list(range(75))], return_residuals=True)
    assert len(res) == len(want_layers)
    for i, r in enumerate(res):
        assert _rel(r, want_layers[i]) < 2e-5, f"residual after layer {i}"
    _agree(logits, want, F32)
    assert _rel(logits, want) < 1e-4  # the scale of the logits too
    m16 = _model(cfg, W, BF16)
    c16 = m16.new_cache()
    _agree(m16.engine.step(c16, [c16.alloc()], [toks], want=[list(range(75))]), want, BF16)


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prefill_portions_and_decoding_agree(name, dtype):
    """The same 90 tokens: in one step; as a prompt and then token by token; token by token from the start; in portions."""
    cfg = CONFIGS[name]
    W = mo.random_weights(cfg, seed=3)
    toks = _tokens(90, cfg["vocab"], 2)
    m = _model(cfg, W, dtype)
    want = mo.forward(cfg, W, toks)
    for portions in ([90], [30] + [1] * 60, [1] * 90, [2] * 45, [7, 2, 2, 30, 1, 1, 2, 3, 2, 40]):
        cache = m.new_cache()
        s = cache.alloc()
        out, at = [], 0
        for n in portions:
            out.append(m.engine.step(cache, [s], [toks[at:at + n]], want=[list(range(n))]))
            at += n
        assert at == 90 and cache.length[s] == 90
        _agree(torch.cat(out), want, dtype)


def test_layers_that_read_anothers_keys_keep_none():
    cfg = CONFIGS["odd_sizes"]
    m = _model(cfg, mo.random_weights(cfg, seed=1), F32)
    cache = m.new_cache(n_slots=2)
    cache.alloc()
    one = 4 * cache.positions * (1 * (6 + 5) + 2 * (9 + 9))  # fp32: layer 0 (read by 1 and 2) and layer 3
    assert cache.bytes_per_slot() == one
    own = [e["mixer"] for e in cache.layers]
    assert own[1].h_k == own[0].h_k and own[2].h_v == own[0].h_v and own[3].h_k != own[0].h_k


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_unequal_batch_equals_each_request_alone_and_slots_are_reused(name, dtype):
    cfg = CONFIGS[name]
    W = mo.random_weights(cfg, seed=4)
    m = _model(cfg, W, dtype)
    prompts = [_tokens(n, cfg["vocab"], 10 + n) for n in (1, 33, 5, 70, 12)]
    tails = [_tokens(6, cfg["vocab"], 50 + i) for i in range(5)]
    stop_after = [2, 6, 1, 4, 6]  # decode steps each request takes part in
    want = [mo.forward(cfg, W, p + t[:k]) for p, t, k in zip(prompts, tails, stop_after)]

    def alone(cache, i):
        s = cache.alloc()
        out = [m.engine.step(cache, [s], [prompts[i]], want=[list(range(len(prompts[i])))])]
        for k in range(stop_after[i]):
            out.append(m.engine.step(cache, [s], [[tails[i][k]]]))
        cache.release(s)
        return torch.cat(out)

    cache = m.new_cache(n_slots=2)  # five requests: the stores have to grow while two are live
    for i in range(5):  # one after the other: the same slot again and again
        _agree(alone(cache, i), want[i], dtype)
    assert cache.allocs == 5 and cache.n_slots == 2 and not cache.in_use()
    slots = [cache.alloc() for _ in range(5)]  # together, in slots that hold the leftovers of the runs above
    assert cache.n_slots >= 5
    got = [[] for _ in range(5)]
    lg = m.engine.step(cache, slots, prompts, want=[list(range(len(p))) for p in prompts])
    r = 0
    for i, p in enumerate(prompts):
        got[i].append(lg[r:r + len(p)])
        r += len(p)
    live = list(range(5))
    for k in range(6):
        live = [i for i in live if stop_after[i] > k]
        lg = m.engine.step(cache, [slots[i] for i in live], [[tails[i][k]] for i in live])
        for j, i in enumerate(live):
            got[i].append(lg[j:j + 1])
        for i in list(live):
            if stop_after[i] == k + 1:
                cache.release(slots[i])
    for i in range(5):
        _agree(torch.cat(got[i]), want[i], dtype)
    assert not cache.in_use()


def test_mixed_steps_of_prompts_portions_and_single_tokens():
    """One step in which a request decodes a token, another goes on by a portion of its prompt and a third starts."""
    cfg = CONFIGS["mixed"]
    W = mo.random_weights(cfg, seed=11)
    m = _model(cfg, W, F32)
    a, b, c = (_tokens(n, cfg["vocab"], n) for n in (41, 60, 17))
    la, lb, lc = (mo.forward(cfg, W, q) for q in (a, b, c))
    cache = m.new_cache(n_slots=1)
    sa, sb = cache.alloc(), cache.alloc()
    m.engine.step(cache, [sa, sb], [a[:40], b[:20]], want=[[], []])
    sc = cache.alloc()
    lg = m.engine.step(cache, [sb, sa, sc], [b[20:50], [a[40]], c], want=[list(range(30)), [0], list(range(17))])
    _agree(lg, torch.cat([lb[20:50], la[40:], lc]), F32)
    _agree(m.engine.step(cache, [sb], [b[50:]], want=[list(range(10))]), lb[50:], F32)


def test_per_position_stores_grow_and_slots_are_reused():
    """A cache that starts with room for 8 positions and 1 slot: requests of 100 and 37 tokens in portions, two at a time."""
    cfg = CONFIGS["mixed"]
    W = mo.random_weights(cfg, seed=2)
    m = _model(cfg, W, F32)
    a, b = _tokens(100, cfg["vocab"], 1), _tokens(37, cfg["vocab"], 2)
    want_a, want_b = mo.forward(cfg, W, a), mo.forward(cfg, W, b)
    cache = m.new_cache(n_slots=1)
    assert cache.has_per_position
    cache.positions = 8  # before the first alloc: the stores are built this small
    sa = cache.alloc()
    got_a = [m.engine.step(cache, [sa], [a[:5]], want=[list(range(5))])]
    assert cache.positions == 8
    sb = cache.alloc()
    lg = m.engine.step(cache, [sa, sb], [a[5:30], b[:20]], want=[list(range(25)), list(range(20))])
    got_a.append(lg[:25])
    got_b = [lg[25:]]
    assert cache.positions == 32 and cache.n_slots == 2
    for t in range(20, 37):
        lg = m.engine.step(cache, [sb, sa], [[b[t]], [a[30 + t - 20]]])
        got_b.append(lg[:1])
        got_a.append(lg[1:])
    cache.release(sb)
    got_a.append(m.engine.step(cache, [sa], [a[47:]], want=[list(range(53))]))
    assert cache.positions == 128
    _agree(torch.cat(got_a), want_a, F32)
    _agree(torch.cat(got_b), want_b, F32)
    sc = cache.alloc()  # the slot b left, with b's keys still in it
    assert sc == sb
    _agree(m.engine.step(cache, [sc], [b], want=[list(range(37))]), want_b, F32)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_of_a_sequence(name):
    """Position 0 alone, and every prompt length up to a dozen."""
    cfg = CONFIGS[name]
    W = mo.random_weights(cfg, seed=6)
    m = _model(cfg, W, F32)
    toks = _tokens(12, cfg["vocab"], 6)
    want = mo.forward(cfg, W, toks)
    cache = m.new_cache()
    for n in range(1, 13):
        s = cache.alloc()
        _agree(m.engine.step(cache, [s], [toks[:n]], want=[list(range(n))]), want[:n], F32)
        cache.release(s)


def test_long_prompt_and_long_decoding():
    """520 tokens, the last 140 decoded one by one; the tiled kernels see prompts longer than their tiles, the per-position
    stores grow twice."""
    cfg = CONFIGS["tiles"]
    W = mo.random_weights(cfg, seed=7)
    toks = _tokens(520, cfg["vocab"], 7)
    want = mo.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = _model(cfg, W, dtype)
        cache = m.new_cache()
        s = cache.alloc()
        idx = [0, 1, 31, 32, 62, 63, 64, 65, 99, 127, 128, 255, 256, 299, 300, 379]
        out = [m.engine.step(cache, [s], [toks[:380]], want=[idx])]
        for t in range(380, 520):
            out.append(m.engine.step(cache, [s], [[toks[t]]]))
        assert cache.positions >= 520
        _agree(torch.cat(out), want[idx + list(range(380, 520))], dtype)


def test_a_large_step_takes_the_tensor_core_route_of_the_experts():
    """700 tokens at once: tokens x choices passes the bound from which the experts' rows run through the tcgen05 core."""
    from llark_b200 import ops

    cfg = _cfg([_att(2, 2, 16, 16, 16, mlp=_moe(6, 3, 64, 64)), _att(2, 2, 16, 16, 16, kv_from=0, mlp=_moe(4, 4, 80))], vocab=64, width=64)
    assert 700 * 3 >= ops.MOE_DENSE_MIN_ENTRIES
    W = mo.random_weights(cfg, seed=5)
    toks = _tokens(700, 64, 5)
    want = mo.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = _model(cfg, W, dtype)
        cache = m.new_cache()
        _agree(m.engine.step(cache, [cache.alloc()], [toks], want=[list(range(700))]), want, dtype)


def _random_config(seed):
    """A configuration drawn at random: 2 to 6 layers, widths and head sizes on and off the 16-byte and tensor-core routes, key
    heads that divide the heads, rotation over the whole head or a part, a layer that reads another's keys wherever one of
    equal sizes exists and a coin says so, any feed-forward or none."""
    import random

    r = random.Random(seed)
    layers = []
    for i in range(r.randint(2, 6)):
        owners = [j for j, l in enumerate(layers) if "kv_from" not in l["mixer"]]
        kind = r.random()
        mlp = None if kind < 0.15 else (_dense(r.choice([7, 40, 64, 100])) if kind < 0.5 else None)
        if kind >= 0.5:
            n = r.choice([1, 2, 5, 8, 16])
            mlp = _moe(n, r.randint(1, min(n, 4)), r.choice([9, 24, 64]), r.choice([None, 13, 64, 80]))
        if owners and r.random() < 0.5:
            j = r.choice(owners)
            layers.append({"type": "attention", "mlp": mlp, "mixer": dict(layers[j]["mixer"], kv_from=j, scale=r.choice([0.1, 0.3, 0.5]))})
            continue
        H = r.choice([1, 2, 4, 6, 8])
        G = r.choice([g for g in (1, 2, 3, 4, 6, 8) if H % g == 0])
        D = r.choice([8, 12, 16, 32, 64, 80])
        layers.append(_att(H, G, D, r.choice([D, D, 16, 24, 64]), r.choice([D, D // 4 * 2, 4]), scale=r.choice([None, 0.1, 0.3]),
                           mlp=mlp, base=r.choice([100.0, 1e4, 3e5])))
    return _cfg(layers, vocab=r.choice([37, 100, 256]), width=r.choice([48, 51, 64, 100, 136]), eps=r.choice([1e-5, 1e-6, 0.1]),
                logit_scale=r.choice([1.0, 0.3, 4.0]))


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed):
    """Each request alone in one step, as a prompt with its last tokens decoded, and three unequal requests together."""
    cfg = _random_config(seed)
    W = mo.random_weights(cfg, seed=seed)
    reqs = [_tokens(n, cfg["vocab"], seed + n) for n in (5, 70, 150)]
    want = [mo.forward(cfg, W, q) for q in reqs]
    for dtype in (F32, BF16):
        m = _model(cfg, W, dtype)
        if seed % 2:
            m.engine.max_positions = 200
        cache = m.new_cache(n_slots=2)
        for q, w in zip(reqs, want):
            s = cache.alloc()
            _agree(m.engine.step(cache, [s], [q], want=[list(range(len(q)))]), w, dtype)
            cache.release(s)
            cut = max(1, len(q) - 30)
            s = cache.alloc()
            out = [m.engine.step(cache, [s], [q[:cut]], want=[list(range(cut))])]
            out += [m.engine.step(cache, [s], [[t]]) for t in q[cut:]]
            cache.release(s)
            _agree(torch.cat(out), w, dtype)
        slots = [cache.alloc() for _ in reqs]
        cuts = [max(1, len(q) - 4) for q in reqs]
        lg = m.engine.step(cache, slots, [q[:c] for q, c in zip(reqs, cuts)], want=[list(range(c)) for c in cuts])
        outs, at = [], 0
        for c in cuts:
            outs.append([lg[at:at + c]])
            at += c
        for k in range(4):
            lg = m.engine.step(cache, slots, [[q[c + k]] for q, c in zip(reqs, cuts)])
            for i in range(3):
                outs[i].append(lg[i:i + 1])
        for i in range(3):
            _agree(torch.cat(outs[i]), want[i], dtype)


# ------------------------------------------------------------------------------------------------ entry points
def _checkpoint(folder, cfg, seed):
    import json

    from llark_b200.safetensors_io import save_file

    W = mo.random_weights(cfg, seed=seed)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(BF16) for k, v in W.items()}, str(folder / "model.safetensors"))
    return W


def _oracle_greedy(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(mo.forward(cfg, W, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_checkpoint_folder_registry_and_greedy_generation(tmp_path):
    """config.json + model.safetensors -> the registry picks the class; generate() and the scheduler reproduce the
    restatement's greedy continuation (fp32, so that the argmax is the restatement's)."""
    from llark_b200.models.registry import load_model
    from llark_b200.scheduler import BatchScheduler, Request

    cfg = CONFIGS["mixed"]
    W = _checkpoint(tmp_path, cfg, 8)
    m = load_model(str(tmp_path), dtype=F32)
    assert type(m).__name__ == "ManapelForCausalLM"
    prompts = [_tokens(9, cfg["vocab"], 1), _tokens(9, cfg["vocab"], 2)]
    want = [_oracle_greedy(cfg, W, p, 12) for p in prompts]
    out = m.generate(input_ids=torch.tensor(prompts, device="cuda:0"), max_new_tokens=12)
    assert out.tolist() == [p + w for p, w in zip(prompts, want)]
    reqs = [Request(prompt=prompts[0], max_new_tokens=12), Request(prompt=prompts[1][:4], max_new_tokens=5),
            Request(prompt=prompts[1], max_new_tokens=12, eos_token_id=[want[1][3]])]
    sched = BatchScheduler(m.engine, max_batch=2)
    for r in reqs:
        sched.submit(r)
    sched.run()
    assert reqs[0].output == want[0]
    assert reqs[1].output == _oracle_greedy(cfg, W, prompts[1][:4], 5)
    assert reqs[2].output == want[1][:want[1].index(want[1][3]) + 1]
    assert all(r.finished for r in reqs) and not sched.cache.in_use()


def test_command_line_and_trace_runner(tmp_path, monkeypatch, capsys):
    """generate_cli (scheduler, greedy) and the trace runner (given tokens step by step: two requests start together with
    unequal prompts, decode together, one ends earlier, a third starts later in the slot that was given back)."""
    import io
    import json

    import numpy as np

    from llark_b200 import generate_cli, trace_runner

    cfg = CONFIGS["odd_sizes"]
    W = _checkpoint(tmp_path, cfg, 9)
    V = cfg["vocab"]
    a, b, c = _tokens(40, V, 1), _tokens(9, V, 2), _tokens(21, V, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]},
                                     {"id": "b", "tokens": b[:5], "want": []}], "end": []}]
    for k in range(4):
        steps.append({"step": 1 + k, "entries": [{"id": "a", "tokens": [a[30 + k]], "want": [0]},
                                                 {"id": "b", "tokens": [b[5 + k]], "want": [0]}],
                      "end": ["b"] if k == 3 else []})
    steps.append({"step": 5, "entries": [{"id": "c", "tokens": c, "want": [20]}], "end": ["c"]})
    steps.append({"step": 6, "entries": [{"id": "a", "tokens": a[34:], "want": [5]}], "end": ["a"]})
    out = tmp_path / "out"
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace_runner.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "80"]) == 0
    printed = capsys.readouterr().out.split("\n")
    assert [l for l in printed if l.startswith("done")] == ["done %d" % i for i in range(7)]
    la, lb, lc = mo.forward(cfg, W, a), mo.forward(cfg, W, b), mo.forward(cfg, W, c)

    def rows(i):
        return torch.from_numpy(np.fromfile(out / ("%d.f32" % i), dtype="<f4").reshape(-1, V).copy())

    _agree(rows(0), la[[0, 29]], F32)
    for k in range(4):
        _agree(rows(1 + k), torch.stack([la[30 + k], lb[5 + k]]), F32)
    _agree(rows(5), lc[[20]], F32)
    _agree(rows(6), la[[39]], F32)

    prompts = tmp_path / "p.jsonl"
    prompts.write_text(json.dumps({"id": "x", "tokens": a[:7], "max_new_tokens": 6}) + "\n" +
                       json.dumps({"tokens": b[:3]}) + "\n")
    assert generate_cli.main(["--model", str(tmp_path), "--prompts", str(prompts), "--dtype", "float32",
                              "--max-new-tokens", "4"]) == 0
    lines = [json.loads(l) for l in capsys.readouterr().out.strip().split("\n")]
    assert lines == [{"id": "x", "tokens": _oracle_greedy(cfg, W, a[:7], 6)}, {"id": "1", "tokens": _oracle_greedy(cfg, W, b[:3], 4)}]
