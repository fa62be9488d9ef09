"""Buvesun on the GPU against the plain restatement in tests/buvesun_oracle.py (float64 on the CPU): every mechanism alone
through its op or its class, then the whole model through the engine's step function, the slot cache, the scheduler,
generate() and the command-line tools. Configurations are small and deliberately unlike each other: sizes on and off the
16-byte and tensor-core routes, key and value sizes that differ or agree, rotation over a part of the head and over all of
it, windows shorter and longer than the prompts, decays from 0 to 1, loops over the first, the last or all layers, over two
kinds of layers, once and several times, and no loop, mixtures with and without a shared expert, layers without a
feed-forward."""
import math

import pytest
import torch

import buvesun_oracle as bo

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
    """fp32: every position. bf16: a router decides between two almost equal scores now and then, and rounding may turn the
    choice; so one position in twenty (at least one) may lie above the bound, none far above."""
    e = _errors(got, want)
    assert torch.isfinite(e).all()
    if dtype == F32:
        assert e.max() < 1e-4, e.max()
    else:
        assert (e > 8e-2).sum() <= max(1, e.numel() // 20) and e.max() < 0.7, (e.max(), (e > 8e-2).sum(), e.numel())


# ------------------------------------------------------------------------------------------------ configurations
def _moe(experts, top, ff, shared=None, limit=1.5, shared_limit=0.8):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}, "shared": None}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def _ret(decay, dim, vdim, rot, base=100.0, mlp=None):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay),
                                                       "rot": {"base": base, "dims": rot}}}


def _par(left, window, decay, dim, vdim, scales=(0.9, 0.4), base=50.0, scale=None, mlp=None):
    """left: (heads, key heads, key size, value size, rotated entries)."""
    H, G, D, E, rot = left
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": E, "mask": {"size": window},
                               "scale": scale or 1.0 / math.sqrt(D), "rot": {"base": base, "dims": rot}},
                      "right": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def _cfg(layers, vocab=97, width=72, eps=1e-6, scale=3.0, mult=0.6, loop=None):
    return {"architecture": "Buvesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "loop": loop, "layers": layers}


CONFIGS = {
    # every size differs from every other; the loop runs over one layer of each kind and one without a feed-forward
    "mixed": _cfg([_ret([0.5, 0.97], 12, 20, 8, mlp=_moe(6, 2, 20, 33)), _par((4, 2, 16, 12, 8), 7, [0.6, 0.9, 0.999], 10, 14, mlp=_moe(5, 3, 12)),
                   _ret([0.8, 0.99, 0.3], 16, 8, 16, base=30.0), _par((3, 1, 10, 10, 10), 25, [0.95], 24, 6, mlp=_moe(3, 1, 40, 9))],
                  loop={"start": 1, "stop": 3, "times": 2}),
    # nothing a multiple of 4, decays of 0 and 1, an eps that counts beside the squares, a window of one key, the loop over
    # everything but the first layer, a small residual weight, a mixture that uses all of its experts, one of one expert
    "odd_sizes": _cfg([_par((3, 1, 6, 5, 4), 1, [0.0, 1.0], 7, 5, scales=(-0.5, 1.3), mlp=_moe(1, 1, 9, 7, limit=0.3, shared_limit=4.0)),
                       _ret([1.0, 0.0, 0.7], 10, 3, 6, mlp=_moe(3, 3, 11)), _par((2, 2, 9, 9, 2), 300, [0.9], 5, 9, base=1000.0)],
                      vocab=33, width=51, eps=0.2, scale=0.7, mult=0.3, loop={"start": 1, "stop": 3, "times": 3}),
    # sizes of the tensor-core routes; the loop runs over the last layer alone
    "tiles": _cfg([_ret([0.9, 0.98, 0.995, 0.9995], 32, 32, 32, base=1e4, mlp=_moe(5, 3, 64, 72)),
                   _par((4, 2, 32, 32, 16), 48, [0.7, 0.99], 64, 48, base=1e5, mlp=_moe(9, 2, 72, 64)),
                   _par((4, 4, 16, 16, 16), 100, [0.999, 0.9, 0.5], 16, 16, mlp=_moe(4, 2, 80))],
                  vocab=120, width=128, loop={"start": 2, "stop": 3, "times": 2}),
    # no loop at all, the embedding as it is
    "no_loop": _cfg([_ret([0.9] * 3, 8, 16, 4, mlp=_moe(4, 2, 16)), _par((2, 1, 8, 24, 8), 10, [0.99, 0.8], 8, 16)], width=48, scale=1.0),
    # the loop over all layers, once; residual weight 1
    "one_pass": _cfg([_par((2, 1, 16, 16, 8), 12, [0.97, 0.6], 12, 12, mlp=_moe(3, 2, 24, 16)), _ret([0.95], 20, 28, 12)],
                     width=64, mult=1.0, loop={"start": 0, "stop": 2, "times": 1}),
}


def _model(cfg, W, dtype):
    from llark_b200.models.buvesun import BuvesunConfig, BuvesunForCausalLM

    return BuvesunForCausalLM(BuvesunConfig.from_dict(cfg), W, device="cuda:0", dtype=dtype)


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class _Stores:
    """Stand-in cache for mixers used alone: recurrent states at zero, everything else garbage."""

    def __init__(self, n_slots=4, positions=512):
        self.t, self.n, self.positions = [], n_slots, positions

    def add_store(self, shape, dtype, zero_on_alloc, per_position=False):
        lead = (self.positions,) if per_position else ()
        self.t.append(torch.full((self.n,) + lead + tuple(shape), 0.0 if zero_on_alloc else float("nan"), device=_dev(), dtype=dtype))
        return len(self.t) - 1

    def view(self, h):
        return self.t[h]


def _run_mixer(W, kind, spec, width, h, portions, act, eps=1e-5, slot=2, max_positions=None):
    """One mixer ('m.' in W) on a stand-in cache, one request in `slot` whose input h [T, width] is cut into `portions`."""
    from llark_b200.mixers import MIXERS
    from llark_b200.models.buvesun import MIXER_TYPES

    cls = MIXERS[MIXER_TYPES.get(kind, kind)]
    stores = _Stores()
    mix = cls(cls.Weights({k: v.to(F32) for k, v in W.items()}, "m.", spec, width, _dev(), act), stores, eps, act, max_positions)
    outs, at = [], 0
    for n in portions:
        outs.append(mix.forward(h[at:at + n].to(_dev(), act).contiguous(), _layout([n], [at], [slot]), stores).cpu())
        at += n
    assert at == h.shape[0]
    return torch.cat(outs)


def _mixer_weights(layer, width, seed):
    W = bo.random_weights(_cfg([dict(layer, mlp=None)], width=width), seed=seed)
    return {"m" + k[len("l0.mix"):]: v for k, v in W.items() if k.startswith("l0.mix.")}


def _input(T, width, seed):
    return torch.randn(T, width, generator=torch.Generator().manual_seed(seed), dtype=F64).to(BF16).to(F64)


def _bf16_numbers(t):
    return t.to(BF16).to(F64)


PORTIONS = ([150], [1] * 150, [100] + [1] * 50, [31, 2, 2, 65, 1, 1, 30, 18])


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("C", [8, 51, 72, 1024, 1028, 2048, 4100, 8200])
def test_layer_norm_and_the_sum_with_the_next_input_norm(C):
    """The plain norm with and without chosen rows; x + norm(f) * w, f of a result and / or expert rows (weighted or as they
    are); then the next norm, the sum itself in the other dtype, or nothing."""
    from llark_b200 import ops

    g = torch.Generator().manual_seed(C)
    n, d, eps = 13, _dev(), 1e-3

    def rand(*s):
        return torch.randn(*s, generator=g, dtype=F64).to(F32).to(F64)

    x, y, wp, wn = 2.0 * rand(n, C) + 5.0, 3.0 * rand(n, C) - 1.0, rand(C), rand(C)
    x[0] *= 100.0        # a large mean beside the spread
    y[1] *= 1e-3         # squares that eps counts beside
    y[2, 0] = 1000.0     # one entry far off
    rows = torch.tensor([5, 0, 12, 1], dtype=torch.int32, device=d)
    dx, dy, dp, dn = (t.to(d, F32) for t in (x, y, wp, wn))
    for act, tol in ((F32, 3e-5), (BF16, 4e-3)):
        got = ops.seq_layer_norm(dx, dn, eps, act)
        assert got.dtype == act and _rel(got[1:], bo.layer_norm(x[1:], wn, eps)) < tol
        assert _rel(got[0], bo.layer_norm(x[0], wn, eps)) < max(tol, 2e-4)
        assert torch.equal(ops.seq_layer_norm(dx, dn, eps, act, rows=rows), got[rows.long()])
    for top in (0, 1, 3, 6):
        for with_y in (True, False):
            if not with_y and not top:
                continue
            z = rand(n * max(top, 1), C)
            pos = torch.randperm(n * top, generator=g).to(torch.int32) if top else None
            for wts in ((None, torch.rand(n, top, generator=g, dtype=F64)) if top else (None,)):
                f = y.clone() if with_y else torch.zeros_like(x)
                for t in range(n):
                    for k in range(top):
                        f[t] += (wts[t, k] if wts is not None else 1.0) * z[int(pos[t * top + k])]
                want = x + bo.layer_norm(f, wp, eps)
                kw = {"y": dy if with_y else None}
                if top:
                    kw.update(z=z.to(d, F32), pos_of=pos.to(d), top=top, wts=wts.to(d, F32) if wts is not None else None)
                assert _rel(ops.seq_layer_norm_add(dx, eps, w_post=dp, **kw), want) < 2e-6
                assert _rel(ops.seq_layer_norm_add(dx, eps, **kw), x + f) < 2e-6
                for act, tol in ((F32, 3e-5), (BF16, 4e-3)):
                    got, nxt = ops.seq_layer_norm_add(dx, eps, w_post=dp, w_next=dn, act=act, **kw)
                    assert _rel(got, want) < 2e-6 and nxt.dtype == act and _rel(nxt[1:], bo.layer_norm(want[1:], wn, eps)) < tol
                    got, same = ops.seq_layer_norm_add(dx, eps, w_post=dp, act=act, keep_sum=False, **kw)
                    assert same.dtype == act and _rel(same, want) < tol and (got is None) == (act == BF16)


@pytest.mark.parametrize("M", [1, 2, 7, 8, 9, 70, 300])
@pytest.mark.parametrize("N,K", [(6, 10), (64, 64), (136, 72), (264, 512), (5000, 64)])
def test_clamped_gated_unit_in_the_products(M, N, K):
    """Gate and up rows alternating, through the weight-streaming kernel (up to 8 rows), the tcgen05 core and the tiled
    kernel, with and without a bias, on a column slice; limits that cut most entries, some and none."""
    from llark_b200 import ops

    g = torch.Generator().manual_seed(M + N)
    x = 2.0 * torch.randn(M, K + 8, generator=g, dtype=F64).to(BF16).to(F64)
    w = (torch.randn(N, K, generator=g, dtype=F64) / math.sqrt(K)).to(BF16).to(F64)
    bias = torch.randn(N, generator=g, dtype=F64).to(F32).to(F64)
    d = _dev()
    for bb in (None, bias):
        z = x[:, :K] @ w.T + (bb if bb is not None else 0.0)
        for limit in (0.25, 2.0, 50.0):
            gate, up = z[:, 0::2].clamp(max=limit), z[:, 1::2].clamp(-limit, limit)
            y = gate * torch.sigmoid(1.702 * gate) * (up + 1.0)
            for dt, out, tol in ((F32, F32, 1e-5), (BF16, F32, 1e-5), (BF16, BF16, 4e-3)):
                got = ops.linear(x.to(d, dt)[:, :K], w.to(d, dt), bias=bb.to(d, F32) if bb is not None else None, out_dtype=out,
                                 act="clamp_glu", act_limit=limit)
                assert got.shape == y.shape and got.dtype == out and _rel(got, y) < tol, (limit, dt, out)


@pytest.mark.parametrize("H,D,E,rot,neighbours,lens,off", [
    (2, 128, 128, 128, False, [300, 65], 0), (3, 32, 32, 32, False, [40, 33, 1], 0), (2, 48, 64, 16, False, [70], 0),
    (2, 24, 20, 8, True, [100, 17], 0), (2, 10, 6, 6, False, [50], 1), (1, 128, 200, 0, False, [600], 0),
    (3, 100, 144, 40, False, [33], 4), (2, 64, 7, 64, True, [64], 2), (4, 16, 16, 4, False, [530, 20], 0),
    (2, 144, 40, 96, False, [45], 0), (1, 300, 33, 10, False, [20, 2], 0), (2, 1, 1, 0, False, [37], 3)])
@pytest.mark.parametrize("silu", [False, True])
def test_decay_scan_on_stored_states(H, D, E, rot, neighbours, lens, off, silu):
    """S <- d S + k v^T, o = S^T q from states that are not zero, in unordered slots, at positions that do not start at 0:
    blocks of 32 tokens on the tensor cores with one request per item and cut into chunks, and token by token (full_fp32,
    heads wider than 128). Both orders of rotary pairs, partial rotation, columns off the 16-byte boundary, decays 0 and 1."""
    from llark_b200 import ops

    g = torch.Generator().manual_seed(D + E)
    n, W = sum(lens), 2 * H * D + H * E + off
    W += (-W) % 4 if off % 4 == 0 else 0
    src = torch.randn(n, W, generator=g, dtype=F64).to(F32).to(F64)
    dec, pos0, slots = [0.9, 0.999, 1.0, 0.0][:H], [5 * i for i in range(len(lens))], [3, 1, 6][:len(lens)]
    S0 = torch.randn(8, H, D, E, generator=g, dtype=F64).to(F32).to(F64)
    f = bo.frequencies(rot, 100.0) if rot and not silu else None
    want, S1, at = [], S0.clone(), 0
    for b, L in enumerate(lens):
        x = src[at:at + L, off:]
        q, k = x[:, :H * D].reshape(L, H, D), x[:, H * D:2 * H * D].reshape(L, H, D)
        v = x[:, 2 * H * D:2 * H * D + H * E].reshape(L, H, E)
        if silu:
            q, k, v = bo.silu(q), bo.silu(k), bo.silu(v)
        elif f is not None:
            p = torch.arange(L) + pos0[b]
            q, k = bo.turn(q, p, f, neighbours), bo.turn(k, p, f, neighbours)
        o, S1[slots[b]] = bo.decayed_memory(q, 0.3 * k, v, dec, S0[slots[b]])
        want.append(o.reshape(L, -1))
        at += L
    d = _dev()
    powers, saved = ops.decay_powers(dec, d), ops.decay_chunk_rows
    for full, rows in ((True, None), (False, None), (False, 32), (False, 128)):
        ops.decay_chunk_rows = lambda *a, rows=rows: rows
        try:
            state = S0.to(d, F32)
            got = ops.seq_decay_scan(src.to(d, F32), off, off + H * D, off + 2 * H * D, powers, state, _layout(lens, pos0, slots), H,
                                     D, E, freq=f.to(d, F32) if f is not None else None, interleaved=neighbours, k_scale=0.3,
                                     silu=silu, full_fp32=full)
        finally:
            ops.decay_chunk_rows = saved
        assert _rel(got, torch.cat(want)) < 1e-5 and _rel(state, S1) < 1e-5, (full, rows)
        untouched = [s for s in range(8) if s not in slots]
        assert torch.equal(state[untouched].cpu(), S0[untouched].to(F32))


def test_chunk_length_follows_the_step():
    from llark_b200 import ops

    assert ops.decay_chunk_rows([40], 4, 32) is None                 # shorter than any chunk
    assert ops.decay_chunk_rows([2048] * 64, 16, 128) is None        # enough requests to fill the GPU
    assert ops.decay_chunk_rows([8192], 8, 64) in ops.DECAY_CHUNKS   # one long prompt is cut
    assert ops.decay_powers([0.5, 0.0, 1.0], "cpu").shape == (3, ops.DECAY_CHUNKS[-1] + 1)
    assert ops.decay_powers([0.5, 0.0, 1.0], "cpu")[:, :3].tolist() == [[1.0, 0.5, 0.25], [1.0, 0.0, 0.0], [1.0, 1.0, 1.0]]


@pytest.mark.parametrize("H,E,off", [(1, 64, 0), (3, 20, 0), (2, 7, 3), (4, 128, 8), (2, 200, 4), (1, 512, 0), (1, 513, 0), (1, 2048, 0),
                                     (1, 3000, 8), (1, 8192, 0), (1, 9000, 0)])
def test_read_out_norm_and_gate_into_a_column_slice(H, E, off):
    """Heads divided by their root mean square, with and without a weight (shared by the heads or one per head), times a SiLU
    or a sigmoid of the gate; written beside other columns, which stay as they are."""
    from llark_b200 import ops

    g = torch.Generator().manual_seed(E)
    T, d = 5, _dev()
    x = torch.randn(T, H * E, generator=g, dtype=F64)
    x[1] *= 0.01
    gate, w = torch.randn(T, H * E + 8, generator=g, dtype=F64), torch.randn(H * E, generator=g, dtype=F64)
    for weight in (None, w[:E], w):
        for silu in (True, False):
            gv = gate[:, off // 2:off // 2 + H * E]
            y = bo.rms(x.view(T, H, E), 1e-3).reshape(T, -1) * (bo.silu(gv) if silu else bo.sigmoid(gv))
            if weight is not None:
                y = y * (weight.repeat(H) if weight.numel() == E else weight)
            for act, tol in ((F32, 2e-6), (BF16, 4e-3)):
                out = torch.full((T, H * E + off + 5), 7.0, device=d, dtype=act)
                got = ops.seq_head_norm_gate(x.to(d, F32), weight.to(d, F32).contiguous() if weight is not None else None, H, E, 1e-3, act,
                                             gate=gate.to(d, F32)[:, off // 2:off // 2 + H * E],
                                             w_per_head=weight is not None and weight.numel() == H * E, gate_silu=silu,
                                             out=out[:, off:off + H * E])
                assert _rel(got, y) < tol
                assert (out[:, :off] == 7.0).all() and (out[:, off + H * E:] == 7.0).all()


def _tol(act):
    return 2e-5 if act == F32 else 2e-2


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("spec", [(_ret([0.5, 0.97], 12, 20, 8)), (_ret([1.0, 0.0, 0.7], 10, 3, 6)), (_ret([0.9, 0.995], 64, 64, 64, base=1e4)),
                                  (_ret([0.99], 136, 16, 32)), (_ret([0.98] * 5, 8, 132, 0))])
def test_retention_alone(spec, act):
    width, m = 40, spec["mixer"]
    W, h = _mixer_weights(spec, width, 1), _input(150, 40, 2)
    want = bo.retention_mixer(h, W, "m.", m, 1e-5)
    for portions in PORTIONS:
        got = _run_mixer(W, "retention", m, width, h, portions, act)
        assert _rel(got, want) < _tol(act), portions
        assert max(_rel(got[i], want[i]) for i in range(150)) < 5 * _tol(act), portions


PARALLELS = [_par((4, 2, 16, 12, 8), 7, [0.6, 0.9, 0.999], 10, 14), _par((3, 1, 6, 5, 4), 1, [0.0, 1.0], 7, 5, scales=(-0.5, 1.3)),
             _par((4, 2, 32, 32, 16), 48, [0.7, 0.99], 64, 48, base=1e5), _par((2, 2, 16, 16, 16), 500, [0.95] * 3, 16, 16, scales=(0.0, 2.0)),
             _par((8, 1, 64, 64, 24), 33, [0.9], 24, 6, scales=(1.0, 1.0)), _par((1, 1, 9, 3, 2), 16, [0.99], 130, 20, scales=(2.0, 0.0))]


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("case", range(len(PARALLELS)))
def test_parallel_mixers_alone(case, act):
    """Both sides through one projection in and one out; portions; a bound on the positions shorter and longer than the window."""
    width, m = 40, PARALLELS[case]["mixer"]
    W, h = _mixer_weights(PARALLELS[case], width, case), _input(150, 40, case)
    want = bo.parallel_mixer(h, W, "m.", m, 1e-5)
    for portions in PORTIONS:
        for bound in (None, 150):
            got = _run_mixer(W, "parallel", m, width, h, portions, act, max_positions=bound)
            assert _rel(got, want) < _tol(act), portions


@pytest.mark.parametrize("act", [F32, BF16])
def test_window_attention_and_lightning_attention_by_themselves(act):
    """The two sides are mixers of their own; a window attention without a mask sees everything before."""
    m, width = PARALLELS[0]["mixer"], 40
    W, h = _mixer_weights(PARALLELS[0], width, 3), _input(90, 40, 3)
    left = {k.replace("m.left.", "m."): v for k, v in W.items() if ".left." in k}
    right = {k.replace("m.right.", "m."): v for k, v in W.items() if ".right." in k}
    open_left = {k: v for k, v in m["left"].items() if k != "mask"}
    for portions in ([90], [1] * 90, [40, 2, 3, 45]):
        assert _rel(_run_mixer(right, "lightning", m["right"], width, h, portions, act), bo.lightning_mixer(h, right, "m.", m["right"], 1e-5)) < _tol(act)
        for spec in (m["left"], open_left):
            got = _run_mixer(left, "rotary_attention_window", spec, width, h, portions, act)
            assert _rel(got, bo.window_mixer(h, left, "m.", spec)) < _tol(act)


# ------------------------------------------------------------------------------------------------ single keys that count
def _spotlight(W, pfx, heads, kv, dim, channel, width):
    """Entry `channel` of every query head becomes input channel 0, of every key head input channel 1, and no other entry
    reads those two: a query with a large channel 0 picks out the key with a large channel 1."""
    for name, n, c in ((pfx + "q", heads, 0), (pfx + "k", kv, 1)):
        W[name] = 0.1 * W[name]
        W[name][:, :2] = 0.0
        for h in range(n):
            W[name][h * dim + channel] = 0.0
            W[name][h * dim + channel, c] = 1.0
        W[name] = _bf16_numbers(W[name])


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("dim,window", [(16, 5), (16, 64), (16, 65), (10, 12), (32, 33), (16, 128)])
def test_a_key_just_inside_and_just_outside_the_window(dim, window, act):
    """One query asks for one key with a score far above the others: at the distances window - 1 (the last that is seen) and
    window (the first that is not), in prompts, across the border of portions and in decoding, also after the ring has gone
    round several times."""
    width, T = 24, 3 * 128 + 20
    layer = _par((4, 2, dim, dim, dim // 4 * 2), window, [0.5], 4, 4, scales=(1.0, 0.0))
    m = layer["mixer"]
    base = _mixer_weights(layer, width, dim + window)
    _spotlight(base, "m.left.", 4, 2, dim, dim - 2, width)
    for i in (window, 64 + window, T - 1, T - 130):
        if not window <= i < T:
            continue
        for dist in (window - 1, window, 0, 1):
            h = _input(T, width, i)
            h[:, :2] = 0.0
            h[i, 0], h[i - dist, 1] = 20.0, 20.0
            want = bo.parallel_mixer(h, base, "m.", m, 1e-5)[i]
            # the restatement with a window one shorter or longer shows that this position tells them apart
            near = dict(m, left=dict(m["left"], mask={"size": window + (1 if dist == window else -1)}))
            if dist >= window - 1 and window > 1:
                assert _rel(bo.parallel_mixer(h, base, "m.", near, 1e-5)[i], want) > 0.3
            for portions in ([T], [i, T - i], [i + 1, T - i - 1] if i + 1 < T else [T], [max(1, i - dist)] + [1] * (T - max(1, i - dist)),
                             [i - 1, 2] + ([T - i - 1] if i + 1 < T else [])):
                got = _run_mixer(base, "parallel", m, width, h, portions, act)[i]
                assert _rel(got, want) < 3 * _tol(act), (i, dist, portions)


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("kind", ["retention", "parallel"])
def test_a_key_far_back_in_the_recurrent_state(kind, act):
    """A state that keeps what it is told (decay 1, or next to it) is asked for one key hundreds of tokens back: at the first
    position, around the borders of the 32-token blocks and of the chunks of long prompts, and right beside the query. What a
    state loses at a portion's border, a chunk's or in decoding would show."""
    width, T, i = 24, 600, 599
    decay = [1.0, 0.9999]
    layer = _ret(decay, 16, 12, 8) if kind == "retention" else _par((1, 1, 4, 4, 2), 3, decay, 16, 12, scales=(0.0, 1.0))
    pfx = "m." if kind == "retention" else "m.right."
    W = _mixer_weights(layer, width, 5)
    _spotlight(W, pfx, 2, 2, 16, 12, width)
    for j in (0, 1, 31, 32, 255, 256, 300, 511, 512, 597, 598, 599):
        h = _input(T, width, j)
        h[:, :2] = 0.0
        h[i, 0], h[j, 1] = 20.0, 20.0
        run = bo.retention_mixer if kind == "retention" else bo.parallel_mixer
        want = run(h, W, "m.", layer["mixer"], 1e-5)[i]
        gone = h.clone()
        gone[j, 1] = 0.0
        assert _rel(run(gone, W, "m.", layer["mixer"], 1e-5)[i], want) > 0.3
        for portions in ([T], [300, 300], [T - 40] + [1] * 40, [j + 1, T - j - 1] if j + 1 < T else [j, 1], [17, 2, 513, 68]):
            got = _run_mixer(W, kind, layer["mixer"], width, h, portions, act)[i]
            assert _rel(got, want) < 2 * _tol(act), (j, portions)


@pytest.mark.parametrize("act", [F32, BF16])
def test_decays_are_per_head_and_act_once_per_token(act):
    """One write at position 0, nothing after it: the read-out d tokens later is decay^d of it, for every head its own decay,
    in prompts and in decoding (whole projection read before any norm)."""
    from llark_b200 import ops

    H, D, E, T = 4, 8, 8, 300
    decay = [0.0, 0.5, 0.97, 1.0]
    src = torch.zeros(T, 2 * H * D + H * E, dtype=F64)
    src[:, :H * D] = 1.0
    src[0, H * D:] = 1.0
    want = torch.tensor(decay, dtype=F64)[None, :] ** torch.arange(T, dtype=F64)[:, None] * D
    d = _dev()
    for portions in ([T], [1] * T, [33, 2, 265]):
        state, at, out = torch.zeros(1, H, D, E, device=d), 0, []
        for n in portions:
            out.append(ops.seq_decay_scan(src[at:at + n].to(d, F32).contiguous(), 0, H * D, 2 * H * D, ops.decay_powers(decay, d), state,
                                          _layout([n], [at], [0]), H, D, E, full_fp32=act == F32))
            at += n
        got = torch.cat(out).view(T, H, E).double().cpu()
        assert ((got - want[:, :, None]).abs() <= 1e-4 * want[:, :, None] + 1e-30).all()


# ------------------------------------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("n_exp,top", [(1, 1), (3, 3), (5, 2), (16, 1), (64, 8), (200, 32)])
def test_router_takes_the_largest_scores_as_they_are(n_exp, top):
    from llark_b200 import ops

    g = torch.Generator().manual_seed(n_exp)
    z = 3.0 * torch.randn(50, n_exp + 4, generator=g, dtype=F64)
    z[0] = 40.0 + torch.arange(n_exp + 4, dtype=F64)   # sigmoids that round to 1: the order is the logits'
    z[1] = -200.0 - torch.arange(n_exp + 4, dtype=F64)
    ids, wts = ops.seq_moe_route_top(z.to(_dev(), F32)[:, :n_exp], top, sigmoid=True)
    best = torch.topk(z.to(F32)[:, :n_exp], top, dim=-1)
    assert torch.equal(ids.cpu().long(), best.indices)
    assert (wts.double().cpu() - torch.sigmoid(best.values.double())).abs().max() < 1e-6


@pytest.mark.parametrize("T", [1, 5, 60, 300, 800, 2100])
@pytest.mark.parametrize("width,m", [(40, _moe(6, 2, 20, 33)), (51, _moe(3, 3, 11)), (96, _moe(9, 3, 64, 72, limit=0.5)), (30, _moe(1, 1, 5, 3)),
                                     (64, _moe(33, 1, 67)), (64, _moe(4, 1, 64, 64, limit=9.0, shared_limit=0.1))])
def test_mixture_of_experts_alone(T, width, m):
    """Few tokens (weight-streaming kernels), some hundreds (grouped kernels) and, in bf16 with sizes for it, the tcgen05
    core's runs of rows. The weights multiply the inputs: a unit is not linear, so on the outputs they would give another sum."""
    from llark_b200 import ops
    from llark_b200.mixers import FEED_FORWARDS
    from llark_b200.models.buvesun import FEED_FORWARD_KINDS

    W = bo.random_weights(_cfg([_ret([0.5], 2, 2, 2, mlp=m)], width=width), seed=T)
    W = {k[len("l0.mlp."):]: v for k, v in W.items() if k.startswith("l0.mlp.")}
    W["router"] = 0.25 * W["router"]  # scores that are no ones
    h = _input(T, width, T)
    want = bo.expert_mixture(h, W, "", m)
    ids, wts = bo.route(h, W, "", m)
    lim = m["expert"]["limit"]
    outside, inside = (sum(a * bo.clamped_unit(b * h[0], W, f"e{e}.", lim) for e, a, b in zip(ids[0].tolist(), *two))
                       for two in ((wts[0], torch.ones(m["router"]["top"])), (torch.ones(m["router"]["top"]), wts[0])))
    assert _rel(outside, inside) > 0.05
    cls, d = FEED_FORWARDS[FEED_FORWARD_KINDS["moe"]], _dev()
    for act, tol in ((F32, 1e-5), (BF16, 2e-2)):
        ff = cls(cls.Weights({k: v.to(F32) for k, v in W.items()}, "", m, width, d, act), act)
        t = ff.terms(h.to(d, act))
        assert (t["y"] is None) == (not m["shared"])
        got = ops.seq_layer_norm_add(torch.zeros(T, width, device=d), 1e-6, **t)
        assert _rel(got, want) < tol


# ------------------------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_the_residual_after_every_layer_run(name):
    cfg = CONFIGS[name]
    W = bo.random_weights(cfg, seed=3)
    toks = _tokens(75, cfg["vocab"], 1)
    want, want_layers = bo.forward(cfg, W, toks, return_residuals=True)
    m = _model(cfg, W, F32)
    cache = m.new_cache()
    logits, res = m.engine.step(cache, [cache.alloc()], [toks], want=[list(range(75))], return_residuals=True)
    assert len(res) == len(want_layers)
    for i, r in enumerate(res):
        assert _rel(r, want_layers[i]) < 3e-5, f"residual after layer run {i}"
    _agree(logits, want, F32)
    assert _rel(logits, want) < 1e-4
    s = cache.alloc()
    again = m.engine.step(cache, [s], [toks], want=[list(range(75))])  # nobody asks for the residuals
    assert _rel(again, logits) < 1e-5
    m16 = _model(cfg, W, BF16)
    c16 = m16.new_cache()
    lg, res = m16.engine.step(c16, [c16.alloc()], [toks], want=[list(range(75))], return_residuals=True)
    _agree(lg, want, BF16)
    assert all(r.dtype == F32 for r in res)
    _agree(m16.engine.step(c16, [c16.alloc()], [toks], want=[list(range(75))]), want, BF16)


def test_every_pass_of_a_loop_has_stores_of_its_own():
    cfg = CONFIGS["mixed"]
    m = _model(cfg, bo.random_weights(cfg, seed=1), F32)
    cache = m.new_cache(n_slots=2)
    cache.alloc()
    assert [e["enters"] for e in cache.layers] == [False, True, False, True, False, False]
    assert cache.layers[1]["pk"] is cache.layers[3]["pk"] and cache.layers[1]["mixer"] is not cache.layers[3]["mixer"]
    right = [cache.layers[i]["mixer"].right.h_state for i in (1, 3)]
    assert right[0] != right[1] and cache.view(right[0]).data_ptr() != cache.view(right[1]).data_ptr()
    ret = lambda h, d, e: h * d * e
    par = lambda w, g, d, e, h, dm, em: w * g * (d + e) + h * dm * em
    floats = (ret(2, 12, 20) + 2 * (par(7, 2, 16, 12, 3, 10, 14) + ret(3, 16, 8)) + par(25, 1, 10, 10, 1, 24, 6))
    assert cache.bytes_per_slot() == 4 * floats and not cache.has_per_position


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prefill_portions_and_decoding_agree(name, dtype):
    """The same 90 tokens: in one step; as a prompt and then token by token; token by token from the start; in portions."""
    cfg = CONFIGS[name]
    W = bo.random_weights(cfg, seed=3)
    toks = _tokens(90, cfg["vocab"], 2)
    m = _model(cfg, W, dtype)
    want = bo.forward(cfg, W, toks)
    for portions in ([90], [30] + [1] * 60, [1] * 90, [2] * 45, [7, 2, 2, 30, 1, 1, 2, 3, 2, 40]):
        cache = m.new_cache()
        s = cache.alloc()
        out, at = [], 0
        for n in portions:
            out.append(m.engine.step(cache, [s], [toks[at:at + n]], want=[list(range(n))]))
            at += n
        assert at == 90 and cache.length[s] == 90
        _agree(torch.cat(out), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tiles", "one_pass"])
def test_unequal_batch_equals_each_request_alone_and_slots_are_reused(name, dtype):
    cfg = CONFIGS[name]
    W = bo.random_weights(cfg, seed=4)
    m = _model(cfg, W, dtype)
    prompts = [_tokens(n, cfg["vocab"], 10 + n) for n in (1, 33, 5, 70, 12)]
    tails = [_tokens(6, cfg["vocab"], 50 + i) for i in range(5)]
    stop_after = [2, 6, 1, 4, 6]  # decode steps each request takes part in
    want = [bo.forward(cfg, W, p + t[:k]) for p, t, k in zip(prompts, tails, stop_after)]

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


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_steps_of_prompts_portions_and_single_tokens(dtype):
    """One step in which a request decodes a token, another goes on by a portion of its prompt and a third starts."""
    cfg = CONFIGS["mixed"]
    W = bo.random_weights(cfg, seed=11)
    m = _model(cfg, W, dtype)
    a, b, c = (_tokens(n, cfg["vocab"], n) for n in (41, 60, 17))
    la, lb, lc = (bo.forward(cfg, W, q) for q in (a, b, c))
    cache = m.new_cache(n_slots=1)
    sa, sb = cache.alloc(), cache.alloc()
    m.engine.step(cache, [sa, sb], [a[:40], b[:20]], want=[[], []])
    sc = cache.alloc()
    lg = m.engine.step(cache, [sb, sa, sc], [b[20:50], [a[40]], c], want=[list(range(30)), [0], list(range(17))])
    _agree(lg, torch.cat([lb[20:50], la[40:], lc]), dtype)
    _agree(m.engine.step(cache, [sb], [b[50:]], want=[list(range(10))]), lb[50:], dtype)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_of_a_sequence(name):
    """Position 0 alone, and every prompt length up to a dozen."""
    cfg = CONFIGS[name]
    W = bo.random_weights(cfg, seed=6)
    m = _model(cfg, W, F32)
    toks = _tokens(12, cfg["vocab"], 6)
    want = bo.forward(cfg, W, toks)
    cache = m.new_cache()
    for n in range(1, 13):
        s = cache.alloc()
        _agree(m.engine.step(cache, [s], [toks[:n]], want=[list(range(n))]), want[:n], F32)
        cache.release(s)


def test_long_prompt_and_long_decoding():
    """520 tokens, the last 140 decoded one by one; the prompt is longer than the tiles, the windows and a chunk of the scan."""
    cfg = CONFIGS["tiles"]
    W = bo.random_weights(cfg, seed=7)
    toks = _tokens(520, cfg["vocab"], 7)
    want = bo.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = _model(cfg, W, dtype)
        cache = m.new_cache()
        s = cache.alloc()
        idx = [0, 1, 31, 32, 47, 48, 62, 63, 64, 65, 99, 100, 127, 128, 255, 256, 299, 300, 379]
        out = [m.engine.step(cache, [s], [toks[:380]], want=[idx])]
        for t in range(380, 520):
            out.append(m.engine.step(cache, [s], [[toks[t]]]))
        _agree(torch.cat(out), want[idx + list(range(380, 520))], dtype)


def test_a_large_step_takes_the_tensor_core_route_of_the_experts():
    """700 tokens at once: tokens x choices passes the bound from which the experts' rows run through the tcgen05 core."""
    from llark_b200 import ops

    cfg = _cfg([_ret([0.9, 0.99], 16, 16, 16, mlp=_moe(6, 3, 64, 64)), _par((2, 1, 16, 16, 16), 40, [0.97], 16, 16, mlp=_moe(4, 4, 80))],
               vocab=64, width=64, loop={"start": 0, "stop": 1, "times": 2})
    assert 700 * 3 >= ops.MOE_DENSE_MIN_ENTRIES
    W = bo.random_weights(cfg, seed=5)
    toks = _tokens(700, 64, 5)
    want = bo.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = _model(cfg, W, dtype)
        cache = m.new_cache()
        _agree(m.engine.step(cache, [cache.alloc()], [toks], want=[list(range(700))]), want, dtype)


def _random_config(seed):
    """A configuration drawn at random: 1 to 5 layers of either kind, widths and head sizes on and off the 16-byte and
    tensor-core routes, any window, any decays, any feed-forward or none, any loop or none."""
    import random

    r = random.Random(seed)

    def decays():
        return [r.choice([0.0, 0.3, 0.9, 0.99, 0.9999, 1.0]) for _ in range(r.choice([1, 2, 3, 5, 8]))]

    layers = []
    for _ in range(r.randint(1, 5)):
        n = r.choice([1, 2, 5, 8, 16])
        mlp = None if r.random() < 0.2 else _moe(n, r.randint(1, min(n, 4)), r.choice([9, 24, 64]), r.choice([None, 13, 64, 80]),
                                                 limit=r.choice([0.5, 2.0, 7.0]), shared_limit=r.choice([0.3, 1.0, 10.0]))
        D, E = r.choice([6, 8, 12, 16, 32, 64, 80]), r.choice([4, 10, 16, 32, 64, 100])
        if r.random() < 0.5:
            layers.append(_ret(decays(), D, E, r.choice([D, D // 4 * 2, 2]), base=r.choice([10.0, 1e4, 3e6]), mlp=mlp))
            continue
        H = r.choice([1, 2, 4, 6, 8])
        G = r.choice([g for g in (1, 2, 3, 4, 6, 8) if H % g == 0])
        A = r.choice([8, 12, 16, 32, 64])
        layers.append(_par((H, G, A, r.choice([A, A, 10, 24]), r.choice([A, A // 4 * 2, 4])), r.choice([1, 2, 9, 40, 64, 1000]), decays(), D, E,
                           scales=(r.choice([1.0, 0.8, -0.3]), r.choice([1.0, 0.5, 1.7])), base=r.choice([20.0, 1e6]),
                           scale=r.choice([None, 0.05, 0.3]), mlp=mlp))
    loop = None
    if r.random() < 0.8:
        a = r.randrange(len(layers))
        loop = {"start": a, "stop": r.randint(a + 1, len(layers)), "times": r.randint(1, 3)}
    return _cfg(layers, vocab=r.choice([37, 100, 256]), width=r.choice([48, 51, 64, 100, 136]), eps=r.choice([1e-5, 1e-6, 0.1]),
                scale=r.choice([1.0, 0.3, 8.0]), mult=r.choice([1.0, 0.3, 0.7]), loop=loop)


def _draw(seed):
    """A random model and requests that do not blow up rounding: a head whose state decays at once can read out next to nothing
    and be divided by that, which a loop then repeats. Where the restatement itself, run in 32 bits, is off by more than the
    bound, the next one is drawn."""
    while True:
        cfg = _random_config(seed)
        W = bo.random_weights(cfg, seed=seed)
        reqs = [_tokens(n, cfg["vocab"], seed + n) for n in (5, 70, 150)]
        want = [bo.forward(cfg, W, q) for q in reqs]
        W32 = {k: v.to(F32) for k, v in W.items()}
        if max(_errors(bo.forward(cfg, W32, q), w).max() for q, w in zip(reqs, want)) < 3e-6:
            return cfg, W, reqs, want
        seed += 100


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed):
    """Each request alone in one step, as a prompt with its last tokens decoded, and three unequal requests together."""
    cfg, W, reqs, want = _draw(seed)
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

    W = bo.random_weights(cfg, seed=seed)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(BF16) for k, v in W.items()}, str(folder / "model.safetensors"))
    return W


def _oracle_greedy(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(bo.forward(cfg, W, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_checkpoint_folder_registry_and_greedy_generation(tmp_path):
    """config.json + model.safetensors -> the registry picks the class; generate() and the scheduler reproduce the
    restatement's greedy continuation (fp32, so that the argmax is the restatement's)."""
    from llark_b200.models.registry import load_model
    from llark_b200.scheduler import BatchScheduler, Request

    cfg = CONFIGS["mixed"]
    W = _checkpoint(tmp_path, cfg, 8)
    m = load_model(str(tmp_path), dtype=F32)
    assert type(m).__name__ == "BuvesunForCausalLM"
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
    la, lb, lc = bo.forward(cfg, W, a), bo.forward(cfg, W, b), bo.forward(cfg, W, c)

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
