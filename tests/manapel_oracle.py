"""Plain, slow restatement of the Manapel decoder for the tests: one function per mechanism, whole sequences only (no
cache, no batching, no kernels), PyTorch on the CPU in whatever float dtype the weights come in (the tests use float64).
Nothing here is imported by the package and nothing of the package is imported here.

Notation: T tokens, C = width, H query heads, G key / value heads, D = per-head query / key size, E = per-head value size.
Weights are a dict name -> tensor, linear weights stored [out, in]; `m` is a mixer's (or a feed-forward's) dictionary of
sizes and constants as the configuration carries it.
"""
import math

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    """An element-wise squashing in the place of a norm: one number alpha, a weight and an offset per coordinate."""
    return torch.tanh(alpha * x) * w + b


def named_norm(x, W, name):
    return tanh_norm(x, W[name + ".alpha"], W[name], W[name + ".b"])


def relu(z):
    return torch.clamp(z, min=0.0)


def frequencies(dims, base):
    """base^(-2 i / dims) for the dims / 2 pairs."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return float(base) ** (-2.0 * i / dims)


def turn(x, positions, f):
    """Rotates the first 2 * len(f) entries of every head of x [T, n_heads, n]: entry i and entry i + len(f) form pair i,
    which turns by positions[t] * f_i. The rest of the head passes."""
    n = f.numel()
    if n == 0:
        return x
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    co, si = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * co - v * si, v * co + u * si, x[..., 2 * n:]], dim=-1)


def attend(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]: causal softmax attention, head h on key / value head
    floor(h / (H / G))."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    heads = []
    for h in range(H):
        s = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(later, -math.inf)
        heads.append(torch.softmax(s, dim=-1) @ v[:, h // per])
    return torch.stack(heads, dim=1)


# ------------------------------------------------------------------------------------------------ mixer "attention"
def turned_unit(x, m, eps):
    """Rotation first, then each head divided by its root mean square (no weight)."""
    rot = m["rot"]
    return rms(turn(x, torch.arange(x.shape[0]), frequencies(int(rot["dims"]), rot["base"])), eps)


def queries(h, W, pfx, m, eps):
    H, D = int(m["heads"]), int(m["dim"])
    return turned_unit((h @ W[pfx + "q"].T + W[pfx + "q.b"]).view(-1, H, D), m, eps)


def keys_values(h, W, pfx, m, eps):
    G, D, E = int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    k = turned_unit((h @ W[pfx + "k"].T + W[pfx + "k.b"]).view(-1, G, D), m, eps)
    return k, (h @ W[pfx + "v"].T + W[pfx + "v.b"]).view(-1, G, E)


def attention_mixer(h, W, pfx, m, eps, kv=None):
    """kv: keys and values of another layer; None: the mixer's own. Returns (output, the keys and values used)."""
    if kv is None:
        kv = keys_values(h, W, pfx, m, eps)
    o = attend(queries(h, W, pfx, m, eps), kv[0], kv[1], float(m["scale"]))
    return o.reshape(h.shape[0], -1) @ W[pfx + "o"].T, kv


# ------------------------------------------------------------------------------------------------ feed-forwards
def relu_gated_ff(h, W, pfx):
    return (relu(h @ W[pfx + "gate"].T) * (h @ W[pfx + "up"].T)) @ W[pfx + "down"].T


def relu_squared_ff(h, W, pfx):
    return relu(h @ W[pfx + "up"].T) ** 2 @ W[pfx + "down"].T


def route(h, W, pfx, m):
    """(expert numbers [T, top], weights [T, top]): the experts of the largest logits, softmax over those logits only."""
    z = h @ W[pfx + "router"].T + W[pfx + "router.b"]
    best = torch.topk(z, int(m["router"]["top"]), dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def expert_mixture(h, W, pfx, m):
    ids, wts = route(h, W, pfx, m)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), wts[t]):
            out[t] += wt * relu_squared_ff(h[t], W, f"{pfx}e{e}.")
    if m.get("shared"):
        out = out + relu_squared_ff(h, W, pfx + "shared.")
    return out


def feed_forward(h, W, pfx, m):
    return {"dense": lambda: relu_gated_ff(h, W, pfx), "moe": lambda: expert_mixture(h, W, pfx, m)}[m["kind"]]()


# ------------------------------------------------------------------------------------------------ model
def forward(cfg, W, tokens, return_residuals=False):
    """cfg: the configuration as a dict; tokens: list of ids -> logits [T, vocab] (and the stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    residuals, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        y, kept[i] = attention_mixer(named_norm(x, W, p + "norm1"), W, p + "mix.", m, eps, kept.get(m.get("kv_from")))
        x = x + named_norm(y, W, p + "norm1b")
        if layer.get("mlp"):
            y = feed_forward(named_norm(x, W, p + "norm2"), W, p + "mlp.", layer["mlp"])
            x = x + named_norm(y, W, p + "norm2b")
        residuals.append(x)
    logits = (named_norm(x, W, "final.norm") @ W["head"].T) * float(cfg.get("logit_scale", 1.0))
    return (logits, residuals) if return_residuals else logits


# ------------------------------------------------------------------------------------------------ random checkpoints
def random_weights(cfg, seed=0, dtype=torch.float64):
    """Random weights of every tensor a configuration names, as bf16 numbers held in `dtype` (a checkpoint stores bf16)."""
    gen = torch.Generator().manual_seed(seed)
    C, V = int(cfg["width"]), int(cfg["vocab"])
    W = {}

    def mat(name, n_out, n_in, gain=1.0):
        W[name] = torch.randn(n_out, n_in, generator=gen) * (gain / math.sqrt(n_in))

    def vec(name, n, mean=0.0, spread=1.0):
        W[name] = mean + spread * torch.randn(n, generator=gen)

    def norm(name, w=1.0):
        vec(name, C, w, 0.2)
        vec(name + ".b", C, 0.0, 0.2)
        W[name + ".alpha"] = (0.7 + 0.2 * torch.rand((), generator=gen)).reshape(())

    W["embed"] = torch.randn(V, C, generator=gen)
    mat("head", V, C)
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, G, D, E = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        norm(p + "norm1"), norm(p + "norm1b", 0.6)
        x = p + "mix."
        mat(x + "q", H * D, C, 2.0), vec(x + "q.b", H * D, 0.0, 0.5), mat(x + "o", C, H * E, 2.0)
        if m.get("kv_from") is None:
            mat(x + "k", G * D, C, 2.0), vec(x + "k.b", G * D, 0.0, 0.5), mat(x + "v", G * E, C, 2.0), vec(x + "v.b", G * E, 0.0, 0.5)
        if not mlp:
            continue
        norm(p + "norm2"), norm(p + "norm2b", 0.6)
        x = p + "mlp."
        if mlp["kind"] == "dense":
            F = int(mlp["ff"])
            mat(x + "gate", F, C, 1.5), mat(x + "up", F, C, 1.5), mat(x + "down", C, F)
        else:
            n, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            mat(x + "router", n, C, 3.0), vec(x + "router.b", n, 0.0, 1.0)
            for e in range(n):
                mat(f"{x}e{e}.up", F, C, 1.5), mat(f"{x}e{e}.down", C, F)
            if mlp.get("shared"):
                F = int(mlp["shared"]["ff"])
                mat(x + "shared.up", F, C, 1.5), mat(x + "shared.down", C, F)
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in W.items()}
