"""Execution schedule of the Manapel decoder on the generation path: a list of layers, each sublayer between two tanh norms,

    x = x + norm1b(mixer(norm1(x)))
    x = x + norm2b(ff(norm2(x)))                only in layers that have a feed-forward

with norm(z) = tanh(alpha z) * w + b. The mixer comes from llark_b200.mixers.MIXERS through
llark_b200.models.manapel.MIXER_TYPES (attention with unit query / key heads; a layer may read an earlier layer's keys and
values), the feed-forward from FEED_FORWARDS (a ReLU-gated unit, or routed squared-ReLU experts with a shared one). Logits
are head(final_norm(x)) * logit_scale.

The norm of a sublayer's result, the residual sum AND the next sublayer's input norm are ONE kernel
(llark_seq_tanh_norm_add): the stream is read and written once per sublayer, and it takes the weighted sum over a token's
chosen experts and the shared expert's output itself, so that the mixture's result is never written out. The activations of
the feed-forwards sit in the epilogue of their first product. The scale of the logits is folded into the final norm. The step
function is llark_b200.engine_seq.LayerListEngine.step; keys and values live in per-position stores of a
llark_b200.state_cache.StateCache that grow. Precision: the residual stream, norms, rotation angles, the heads' root mean
squares, attention scores and softmax, and the router are fp32 in both modes, and every projection that feeds one of them is
written in fp32 by its GEMM; matrix products and the activations between them are bf16 with fp32 accumulation
(dtype=torch.bfloat16) or true fp32 (dtype=torch.float32).
"""
import torch

from . import ops
from .engine_seq import LayerListEngine
from .mixers import FEED_FORWARDS, MIXERS, _pad_rows
from .models.manapel import FEED_FORWARD_KINDS, MIXER_TYPES
from .state_cache import StateCache

F32 = torch.float32


class ManapelEngine(LayerListEngine):
    def __init__(self, config, weights, device, dtype=torch.bfloat16):
        """config: llark_b200.models.manapel.ManapelConfig; weights: name -> tensor (any device / float dtype)."""
        dev = self._init_device(device, dtype)
        self.cfg = config
        C = config.width

        def norm(name, scale=1.0):
            """(alpha, w, b) of a tanh norm; scale multiplies its result."""
            alpha, w, b = (weights[name + s].to(device=dev, dtype=F32) for s in (".alpha", "", ".b"))
            if alpha.numel() != 1 or tuple(w.shape) != (C,) or tuple(b.shape) != (C,):
                raise ValueError(f"{name} does not fit: one number alpha, w and b of the width")
            return float(alpha), (w * scale).contiguous(), (b * scale).contiguous()

        self.embed = weights["embed"].to(device=dev, dtype=dtype).contiguous()
        head = weights["head"].to(device=dev, dtype=dtype)
        if tuple(self.embed.shape) != (config.vocab, C) or tuple(head.shape) != (config.vocab, C):
            raise ValueError("embed / head do not fit vocab x width")
        self.head = _pad_rows(head)  # logits of the padding rows are cut off
        self.final_norm = norm("final.norm", config.logit_scale)
        self._packed = []
        for i, layer in enumerate(config.layers):
            p = f"l{i}."
            pk = {"mixer": MIXERS[MIXER_TYPES[layer.type]].Weights(weights, p + "mix.", layer.mixer, C, dev, dtype),
                  "norm1": norm(p + "norm1"), "norm1b": norm(p + "norm1b"), "ff": None}
            if layer.mlp is not None:
                pk["ff_kind"] = FEED_FORWARD_KINDS[layer.mlp["kind"]]
                pk["ff"] = FEED_FORWARDS[pk["ff_kind"]].Weights(weights, p + "mlp.", layer.mlp, C, dev, dtype)
                pk["norm2"], pk["norm2b"] = norm(p + "norm2"), norm(p + "norm2b")
            self._packed.append(pk)

    # ------------------------------------------------------------------------------------------ state
    def new_cache(self, n_slots=4):
        """A StateCache with the stores of every layer that has keys and values of its own declared. The per-position
        stores start with room for max_positions tokens per request when that is set, and grow otherwise."""
        cfg = self.cfg
        cache = StateCache(self.device, n_slots=n_slots, positions=self.max_positions or 256)
        layers = []
        for pk, layer in zip(self._packed, cfg.layers):
            j = layer.mixer.get("kv_from")
            mixer = MIXERS[MIXER_TYPES[layer.type]](pk["mixer"], cache, cfg.eps, self.act, self.max_positions,
                                                    lender=layers[int(j)]["mixer"] if j is not None else None)
            layers.append({"pk": pk, "mixer": mixer,
                           "ff": FEED_FORWARDS[pk["ff_kind"]](pk["ff"], self.act) if pk["ff"] is not None else None})
        cache.layers = layers
        return cache

    # ------------------------------------------------------------------------------------------ one step (hooks)
    def _embed(self, ids, st):
        return ops.seq_embed(ids, st, self.embed, None, 1.0)

    def _run_layers(self, cache, x, st, residuals):
        entries = cache.layers
        # the first input norm; every later one rides on a residual kernel
        h = ops.seq_tanh_norm(x, entries[0]["pk"]["norm1"], self.act)
        for i, entry in enumerate(entries):
            pk = entry["pk"]
            nxt = entries[i + 1]["pk"]["norm1"] if i + 1 < len(entries) else None
            y = entry["mixer"].forward(h, st, cache)
            if entry["ff"] is None:
                x, h = self._residual(x, pk["norm1b"], nxt, y=y)
            else:
                x, h = self._residual(x, pk["norm1b"], pk["norm2"], y=y)
                x, h = self._residual(x, pk["norm2b"], nxt, **entry["ff"].terms(h))
            if residuals is not None:
                residuals.append(x)
        for entry in entries:
            entry["mixer"].end_step()
        return x

    def _residual(self, x, post, nxt, **terms):
        if nxt is None:
            return ops.seq_tanh_norm_add(x, post, **terms), None
        return ops.seq_tanh_norm_add(x, post, next_norm=nxt, act=self.act, **terms)

    def _logits(self, x, rows):
        return ops.linear(ops.seq_tanh_norm(x, self.final_norm, self.act, rows=rows), self.head, out_dtype=F32)[:, :self.cfg.vocab]
