"""Plain, slow restatement of the Buvesun decoder for the tests: one function per mechanism, whole sequences only (no cache,
no batching, no kernels, recurrences token by token), PyTorch on the CPU in whatever float dtype the weights come in (the
tests use float64). Nothing here is imported by the package and nothing of the package is imported here.

Notation: T tokens, C = width, H heads, G key / value heads, D = per-head query / key size, E = per-head value size. Weights
are a dict name -> tensor, linear weights stored [out, in]; `m` is a mixer's (or a feed-forward's) dictionary of sizes and
constants as the configuration carries it.
"""
import math

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def layer_norm(x, w, eps):
    """Mean taken off, divided by the root of the mean squared deviation + eps, a weight and no offset."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def frequencies(dims, base):
    """base^(-2 i / dims) for the dims / 2 pairs."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return float(base) ** (-2.0 * i / dims)


def turn(x, positions, f, neighbours):
    """Rotates the first 2 * len(f) entries of every head of x [T, n_heads, n], pair i by positions[t] * f_i. The pair is
    (2i, 2i + 1) with `neighbours`, (i, i + len(f)) without. The rest of the head passes."""
    n = f.numel()
    out = x.clone()
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    for i in range(n):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + n)
        co, si = torch.cos(ang[:, i]).to(x.dtype)[:, None], torch.sin(ang[:, i]).to(x.dtype)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a] = u * co - v * si
        out[..., b] = v * co + u * si
    return out


def turned(x, m, neighbours):
    rot = m.get("rot")
    if not rot:
        return x
    return turn(x, torch.arange(x.shape[0]), frequencies(int(rot["dims"]), rot["base"]), neighbours)


def decayed_memory(q, k, v, decay, S=None):
    """q, k [T, H, D], v [T, H, E], decay: one number per head. A matrix per head is multiplied by its decay and gets
    k_t v_t^T added, then q_t is read out of it. Returns ([T, H, E], final matrices [H, D, E])."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    d = torch.tensor([float(z) for z in decay], dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(dim=1))
    return torch.stack(out), S


def windowed_attention(q, k, v, scale, window):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]: softmax over the last `window` positions (the query's own among
    them; None: everything before), head h on key / value head floor(h / (H / G))."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    hidden = (back < 0) | (back >= (window if window is not None else T))
    heads = []
    for h in range(H):
        s = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(hidden, -math.inf)
        heads.append(torch.softmax(s, dim=-1) @ v[:, h // per])
    return torch.stack(heads, dim=1)


# ------------------------------------------------------------------------------------------------ mixers
def retention_mixer(h, W, pfx, m, eps):
    T, H, D, E = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = turned((h @ W[pfx + "q"].T).view(T, H, D), m, False)
    k = turned((h @ W[pfx + "k"].T).view(T, H, D), m, False) / math.sqrt(D)
    v = (h @ W[pfx + "v"].T).view(T, H, E)
    o, _ = decayed_memory(q, k, v, m["decay"])
    o = rms(o, eps).reshape(T, H * E) * silu(h @ W[pfx + "g"].T)
    return o @ W[pfx + "o"].T


def window_mixer(h, W, pfx, m):
    T, H, G, D, E = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = turned((h @ W[pfx + "q"].T).view(T, H, D), m, True)
    k = turned((h @ W[pfx + "k"].T).view(T, G, D), m, True)
    v = (h @ W[pfx + "v"].T).view(T, G, E)
    window = int(m["mask"]["size"]) if m.get("mask") else None
    return windowed_attention(q, k, v, float(m["scale"]), window).reshape(T, H * E) @ W[pfx + "o"].T


def lightning_mixer(h, W, pfx, m, eps):
    T, H, D, E = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(h @ W[pfx + n].T).view(T, H, z) for n, z in (("q", D), ("k", D), ("v", E)))
    o, _ = decayed_memory(q, k, v, m["decay"])
    o = rms(o.reshape(T, H * E), eps) * W[pfx + "norm"] * sigmoid(h @ W[pfx + "g"].T)
    return o @ W[pfx + "o"].T


def parallel_mixer(h, W, pfx, m, eps):
    return (float(m["left_scale"]) * window_mixer(h, W, pfx + "left.", m["left"])
            + float(m["right_scale"]) * lightning_mixer(h, W, pfx + "right.", m["right"], eps))


def mixer(h, W, pfx, kind, m, eps):
    return {"retention": retention_mixer, "parallel": parallel_mixer}[kind](h, W, pfx, m, eps)


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_unit(h, W, pfx, limit):
    g = torch.clamp(h @ W[pfx + "gate"].T, max=limit)
    u = torch.clamp(h @ W[pfx + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[pfx + "down"].T


def route(h, W, pfx, m):
    """(expert numbers [T, top], weights [T, top]): sigmoid scores, the largest chosen, their scores as they are."""
    s = sigmoid(h @ W[pfx + "router"].T)
    best = torch.topk(s, int(m["router"]["top"]), dim=-1)
    return best.indices, best.values


def expert_mixture(h, W, pfx, m):
    """Every chosen expert works on the token multiplied by its weight; the results are added as they are."""
    ids, wts = route(h, W, pfx, m)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), wts[t]):
            out[t] += clamped_unit(wt * h[t], W, f"{pfx}e{e}.", float(m["expert"]["limit"]))
    if m.get("shared"):
        out = out + clamped_unit(h, W, pfx + "shared.", float(m["shared"]["limit"]))
    return out


# ------------------------------------------------------------------------------------------------ model
def layer_runs(cfg):
    """[(layer number, whether a pass of the loop begins with it)] in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    runs = [(i, False) for i in range(a)]
    for _ in range(int(loop["times"])):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens, return_residuals=False):
    """cfg: the configuration as a dict; tokens: list of ids -> logits [T, vocab] (and the stream after every layer run)."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = first = W["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    residuals = []
    for i, enters in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if enters:
            x = torch.cat([x, first], dim=-1) @ W["loop.in"].T
        y = mixer(layer_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["type"], layer["mixer"], eps)
        x = x + mult * (layer_norm(y, W[p + "norm1b"], eps) * W[p + "ls1"])
        if layer.get("mlp"):
            y = expert_mixture(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
            x = x + mult * (layer_norm(y, W[p + "norm2b"], eps) * W[p + "ls2"])
        residuals.append(x)
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, residuals) if return_residuals else logits


# ------------------------------------------------------------------------------------------------ random checkpoints
def random_weights(cfg, seed=0, dtype=torch.float64):
    """Random weights of every tensor a configuration names, as bf16 numbers held in `dtype` (a checkpoint stores bf16)."""
    gen = torch.Generator().manual_seed(seed)
    C, V = int(cfg["width"]), int(cfg["vocab"])
    W = {}

    def mat(name, n_out, n_in, gain=1.0):
        W[name] = torch.randn(n_out, n_in, generator=gen) * (gain / math.sqrt(n_in))

    def vec(name, n, mean=1.0, spread=0.3):
        W[name] = mean + spread * torch.randn(n, generator=gen)

    def unit(pfx, F):
        mat(pfx + "gate", F, C, 1.5), mat(pfx + "up", F, C, 1.5), mat(pfx + "down", C, F)

    def memory(pfx, m):
        H, D, E = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        mat(pfx + "q", H * D, C, 1.5), mat(pfx + "k", H * D, C, 1.5), mat(pfx + "v", H * E, C, 1.5)
        mat(pfx + "g", H * E, C, 1.5), mat(pfx + "o", C, H * E)

    W["embed"] = torch.randn(V, C, generator=gen)
    mat("head", V, C)
    vec("final.norm", C)
    if cfg.get("loop"):
        mat("loop.in", C, 2 * C)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for n in ("norm1", "norm1b", "ls1") + (("norm2", "norm2b", "ls2") if mlp else ()):
            vec(p + n, C)
        x = p + "mix."
        if layer["type"] == "retention":
            memory(x, m)
        else:
            a = m["left"]
            H, G, D, E = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
            mat(x + "left.q", H * D, C, 2.0), mat(x + "left.k", G * D, C, 2.0), mat(x + "left.v", G * E, C, 2.0)
            mat(x + "left.o", C, H * E, 2.0)
            memory(x + "right.", m["right"])
            vec(x + "right.norm", int(m["right"]["heads"]) * int(m["right"]["vdim"]))
        if mlp:
            x = p + "mlp."
            mat(x + "router", int(mlp["router"]["experts"]), C, 2.0)
            for e in range(int(mlp["router"]["experts"])):
                unit(f"{x}e{e}.", int(mlp["expert"]["ff"]))
            if mlp.get("shared"):
                unit(x + "shared.", int(mlp["shared"]["ff"]))
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in W.items()}
