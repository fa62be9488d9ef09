"""Execution schedule of the Buvesun decoder on the generation path: a list of layer RUNS (a loop runs some of the layers several
times on the same weights, every pass with stores of its own), each sublayer between two layer norms,

    x = x + m * ls1 * norm1b(mixer(norm1(x)))
    x = x + m * ls2 * norm2b(ff(norm2(x)))      only in layers that have a feed-forward

and, in front of the first layer of every pass of the loop, x = W_in [x; x0] with x0 the embedding. The mixer comes from
llark_b200.mixers.MIXERS through llark_b200.models.buvesun.MIXER_TYPES (retention, or window attention beside lightning
attention), the feed-forward from FEED_FORWARDS. Logits are head(final_norm(x)).

The norm of a sublayer's result, layer scale, m, the residual sum AND the next input norm are ONE kernel
(llark_seq_layer_norm_add): the stream is read and written once per sublayer, and it adds up a token's chosen experts and the
shared expert itself. In front of a pass it writes the stream only as the operand of W_in. W_in's part for x0 is the same in
every pass: its product is taken once per step and joins in the kernel that norms the pass's first input. The step function is
llark_b200.engine_seq.LayerListEngine.step; recurrent states and rings of the last `mask.size` keys live in a
llark_b200.state_cache.StateCache. Precision: the residual stream, norms, rotation angles, attention scores and softmax, the
router, q / k / v, decays and states of the recurrences are fp32 in both modes, and every projection that feeds one of them is
written in fp32 by its GEMM; matrix products and the activations between them are bf16 with fp32 accumulation
(dtype=torch.bfloat16) or true fp32 (dtype=torch.float32).
"""
import torch

from . import ops
from .engine_seq import LayerListEngine
from .mixers import FEED_FORWARDS, MIXERS, _pad_rows
from .models.buvesun import FEED_FORWARD_KINDS, MIXER_TYPES
from .state_cache import StateCache

F32 = torch.float32


class BuvesunEngine(LayerListEngine):
    def __init__(self, config, weights, device, dtype=torch.bfloat16):
        """config: llark_b200.models.buvesun.BuvesunConfig; weights: name -> tensor (any device / float dtype)."""
        dev = self._init_device(device, dtype)
        self.cfg = config
        C, m = config.width, config.residual_mult

        def vector(name):
            v = weights[name].to(device=dev, dtype=F32).contiguous()
            if tuple(v.shape) != (C,):
                raise ValueError(f"{name} does not fit the width")
            return v

        self.embed = weights["embed"].to(device=dev, dtype=dtype).contiguous()
        head = weights["head"].to(device=dev, dtype=dtype)
        if tuple(self.embed.shape) != (config.vocab, C) or tuple(head.shape) != (config.vocab, C):
            raise ValueError("embed / head do not fit vocab x width")
        self.head = _pad_rows(head)  # logits of the padding rows are cut off
        self.final_norm = vector("final.norm")
        if config.loop:
            w_in = weights["loop.in"].to(device=dev, dtype=dtype)
            if tuple(w_in.shape) != (C, 2 * C):
                raise ValueError("loop.in does not fit width x 2 width")
            self.loop_x, self.loop_first = w_in[:, :C].contiguous(), w_in[:, C:].contiguous()
        self._packed = []
        for i, layer in enumerate(config.layers):
            p = f"l{i}."
            pk = {"mixer": MIXERS[MIXER_TYPES[layer.type]].Weights(weights, p + "mix.", layer.mixer, C, dev, dtype),
                  "norm1": vector(p + "norm1"), "post1": (m * vector(p + "ls1") * vector(p + "norm1b")).contiguous(), "ff": None}
            if layer.mlp is not None:
                pk["ff_kind"] = FEED_FORWARD_KINDS[layer.mlp["kind"]]
                pk["ff"] = FEED_FORWARDS[pk["ff_kind"]].Weights(weights, p + "mlp.", layer.mlp, C, dev, dtype)
                pk["norm2"], pk["post2"] = vector(p + "norm2"), (m * vector(p + "ls2") * vector(p + "norm2b")).contiguous()
            self._packed.append(pk)

    # ------------------------------------------------------------------------------------------ state
    def new_cache(self, n_slots=4):
        """A StateCache with the stores of every layer run declared (a looped layer: one set per pass)."""
        cfg = self.cfg
        cache = StateCache(self.device, n_slots=n_slots, positions=self.max_positions or 256)
        entries = []
        for i, _, enters in cfg.layer_runs():
            pk = self._packed[i]
            entries.append({"pk": pk, "enters": enters,
                            "mixer": MIXERS[MIXER_TYPES[cfg.layers[i].type]](pk["mixer"], cache, cfg.eps, self.act,
                                                                             self.max_positions),
                            "ff": FEED_FORWARDS[pk["ff_kind"]](pk["ff"], self.act) if pk["ff"] is not None else None})
        cache.layers = entries
        return cache

    # ------------------------------------------------------------------------------------------ one step (hooks)
    def _embed(self, ids, st):
        if not self.cfg.loop:
            return ops.seq_embed(ids, st, self.embed, None, self.cfg.embedding_scale), None
        return ops.seq_embed(ids, st, self.embed, None, self.cfg.embedding_scale, copy=True)

    def _run_layers(self, cache, embedded, st, residuals):
        eps = self.cfg.eps
        x, operand = embedded  # the stream in fp32; in front of a pass also as the operand of W_in
        first = ops.linear(operand, self.loop_first, out_dtype=F32) if self.cfg.loop else None
        entries, h = cache.layers, None
        for i, entry in enumerate(entries):
            pk = entry["pk"]
            if entry["enters"]:
                x, h = ops.seq_layer_norm_add(first, eps, y=ops.linear(operand, self.loop_x, out_dtype=F32), w_next=pk["norm1"],
                                              act=self.act)
            elif h is None:
                h = ops.seq_layer_norm(x, pk["norm1"], eps, self.act)
            last, nxt = i + 1 == len(entries), None
            if not last and not entries[i + 1]["enters"]:
                nxt = entries[i + 1]["pk"]["norm1"]
            # what leaves the layer: the next input norm, the stream as the operand of W_in, or the stream alone
            leave = {"w_next": nxt, "act": None if last else self.act,
                     "keep_sum": last or nxt is not None or residuals is not None}
            terms, post = {"y": entry["mixer"].forward(h, st, cache)}, pk["post1"]
            if entry["ff"] is not None:
                x, h = ops.seq_layer_norm_add(x, eps, w_post=post, w_next=pk["norm2"], act=self.act, **terms)
                terms, post = entry["ff"].terms(h), pk["post2"]
            left = ops.seq_layer_norm_add(x, eps, w_post=post, **leave, **terms)
            x, out = left if not last else (left, None)
            h, operand = (out, None) if nxt is not None else (None, out)
            if residuals is not None:
                residuals.append(x)
        return x

    def _logits(self, x, rows):
        return ops.linear(ops.seq_layer_norm(x, self.final_norm, self.cfg.eps, self.act, rows=rows), self.head,
                          out_dtype=F32)[:, :self.cfg.vocab]
