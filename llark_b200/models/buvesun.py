"""Buvesun: a small decoder-only language model built around linear attention with a fixed decay per head and a loop over some
of its layers. Every sublayer sits between two layer norms (a weight, no offset), its normed result is multiplied by a vector
(layer scale) and by one number before it joins the residual stream:

    x <- x + m * ls * norm_b(sublayer(norm_a(x)))

The layers loop.start .. loop.stop - 1 run loop.times times in a row on the same weights, each pass with a cache or state of its
own; in front of every pass the stream becomes a linear mix of itself and the embedding. A mixer is a retention (rotary q and
k, a matrix state per head that decays by a fixed factor, heads divided by their root mean square, SiLU gate), or two mixers
side by side whose results are weighed and added: grouped-query attention in a sliding window with rotary positions, and
lightning attention (the same kind of recurrence on SiLU'd q, k and v with an RMS norm over all heads and a sigmoid gate). The
feed-forward is a mixture of clamped gated units: the largest router scores (sigmoid) are chosen and multiply their experts'
INPUTS; a shared unit with constants of its own is added for every token. The reference has no such model; it is served the
way the other native decoders are: configuration and weights from a checkpoint folder (config.json + model.safetensors), the
CUDA engine (llark_b200.engine_buvesun), the slot cache (llark_b200.state_cache), `generate()` through llark_b200.generate and
batches through llark_b200.scheduler.

config.json keys: architecture ("Buvesun"), vocab, width, embedding.scale, norm.eps, residual_mult, loop (null | {start, stop,
times}), layers[] with type ("retention" | "parallel"), mixer {...}, mlp (null | {kind: "moe", expert {ff, limit}, router
{experts, top}, shared (null | {ff, limit})}).
  retention:  heads, dim, vdim, decay[heads], rot {base, dims};  tensors q, k, v, g, o
  parallel:   left_scale, right_scale;  left {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims}}: left.q / k / v /
              o;  right {heads, dim, vdim, decay[heads]}: right.q / k / v / g / o / norm
Other tensors: embed, head, final.norm, loop.in, l<i>.norm1 / norm1b / ls1 / norm2 / norm2b / ls2, l<i>.mlp.router,
l<i>.mlp.e<j>.gate / up / down, l<i>.mlp.shared.gate / up / down.
"""
from dataclasses import dataclass, field
from typing import List, Optional

from llark_b200.models.layer_loop import layer_runs, read_loop
from llark_b200.models.native import NativeCausalLM

ARCHITECTURE = "Buvesun"
# the configuration's layer types and feed-forward kinds -> entries of llark_b200.mixers.MIXERS / FEED_FORWARDS
MIXER_TYPES = {"retention": "retention", "parallel": "parallel_weighted"}
FEED_FORWARD_KINDS = {"moe": "moe_sigmoid_input"}


@dataclass
class BuvesunLayer:
    type: str
    mixer: dict
    mlp: Optional[dict] = None


@dataclass
class BuvesunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    layers: List[BuvesunLayer] = field(default_factory=list)
    loop: Optional[dict] = None
    eos_token_id: Optional[int] = None
    pad_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d):
        from llark_b200.mixers import FEED_FORWARDS, MIXERS

        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture = {d.get('architecture')!r}")
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXER_TYPES or MIXER_TYPES[e["type"]] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r} (known: {sorted(MIXER_TYPES)})")
            mixer, mlp = dict(e["mixer"]), e.get("mlp")
            memory = mixer if e["type"] == "retention" else mixer["right"]
            if len(memory["decay"]) != int(memory["heads"]) or not all(0.0 <= float(z) <= 1.0 for z in memory["decay"]):
                raise ValueError(f"layer {i}: one decay between 0 and 1 per head")
            if mlp is not None and (mlp.get("kind") not in FEED_FORWARD_KINDS
                                    or FEED_FORWARD_KINDS[mlp["kind"]] not in FEED_FORWARDS):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r} (known: {sorted(FEED_FORWARD_KINDS)})")
            layers.append(BuvesunLayer(type=e["type"], mixer=mixer, mlp=dict(mlp) if mlp else None))
        if not layers:
            raise ValueError("a model needs at least one layer")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), layers=layers,
                   loop=read_loop(d.get("loop"), len(layers)),
                   eos_token_id=d.get("eos_token_id"), pad_token_id=d.get("pad_token_id"))

    def to_dict(self):
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "loop": self.loop,
                "layers": [{"type": l.type, "mixer": l.mixer, "mlp": l.mlp} for l in self.layers]}

    def layer_runs(self):
        """(layer, pass, first layer of a pass?) in the order the layers run; pass is None outside the loop."""
        return layer_runs(self.loop, len(self.layers))


class BuvesunForCausalLM(NativeCausalLM):
    """Inference-only model object: configuration + engine (llark_b200.models.native.NativeCausalLM)."""
    config_class = BuvesunConfig

    @staticmethod
    def engine_class():
        from llark_b200.engine_buvesun import BuvesunEngine

        return BuvesunEngine
