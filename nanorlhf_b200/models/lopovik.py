"""Lopovik: a decoder of latent-attention layers with mixer and feed-forward side by side, a token shift in front of every mixer
and a range of layers that runs several times with the same weights.

* Embedding: ``x = embed[token]``; ``x0`` is kept.
* Loop: layers ``loop.start .. loop.stop - 1`` run ``loop.times`` times in a row, then the rest; every pass begins with
  ``x = loop.in [x; x0]`` and has pages and state of its own.
* Layer: ``x += mixer(shifted) + ff(norm2(x))``, ``h = norm1(x)``, ``shifted = h + (h_prev - h) * shift`` with the previous token's ``h``
  (zeros for the first); RMS norms whose weight is stored around zero.
* ``latent_attention`` mixer: queries ``uq rmsnorm(dq h)``, per head ``dim`` unrotated and ``rot_dim`` rotated columns; one projection
  ``dkv`` gives a latent of ``kv_rank`` columns (RMS-normed) and one rotated key part shared by all heads; unrotated keys ``uk latent``
  and values ``uv latent`` per head; causal softmax of ``(q.k) * scale`` whose denominator also holds ``exp(sink_h)``; interleaved
  rotation; the concatenated heads times ``sigmoid(g h)``, element by element; output projection ``o``.
* Feed-forward: ``down relu(up h)^2``; or ``experts`` SwiGLU experts of which the ``top`` with the largest ``sigmoid(router h)`` read
  ``score * h`` and are summed; or none.
* Output: ``logits = embed norm(x)`` (tied).

This module holds the configuration (every size and constant is read from ``config.json`` or a tensor's shape) and the
checkpoint tensors under their own names; it describes the layers as generic specs (models/hybrid_spec.py) that the step
engine (sampler/hybrid_sampler.py) executes.  There is no forward loop here.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from .hybrid_spec import LayerSpec, MixerSpec, StreamSpec, TensorModel
from .registry import register_model


@dataclass
class LopovikConfig:
    vocab: int = 256
    width: int = 128
    norm_eps: float = 1e-6
    loop: Optional[dict] = None                              # {"start", "stop", "times"}; None: every layer runs once
    layers: List[dict] = field(default_factory=list)         # the checkpoint's own layer descriptions
    model_type: str = "lopovik"
    architecture: str = "Lopovik"
    pad_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None
    max_positions: int = 1 << 30                             # positions are rotations: nothing bounds a sequence's length

    @classmethod
    def from_dict(cls, d: dict) -> "LopovikConfig":
        layers = list(d["layers"])
        for i, layer in enumerate(layers):
            if layer["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown layer type {layer['type']!r}")
            m, mlp = layer["mixer"], layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            if mlp is not None and mlp["kind"] == "moe" and not 1 <= int(mlp["router"]["top"]) <= int(mlp["router"]["experts"]):
                raise ValueError(f"layer {i}: router.top must lie between 1 and router.experts")
            if int(m["rot"]["dims"]) % 2 or int(m["rot"]["dims"]) > int(m["rot_dim"]):
                raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
        loop = d.get("loop")
        if loop is not None and not (0 <= int(loop["start"]) < int(loop["stop"]) <= len(layers) and int(loop["times"]) >= 1):
            raise ValueError("loop must name a range of layers and run it at least once")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]), loop=dict(loop) if loop else None,
                   layers=layers, pad_token_id=d.get("pad_token_id"), eos_token_id=d.get("eos_token_id"))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "layers": self.layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
               "width": self.width}
        if self.loop:
            out["loop"] = self.loop
        for k in ("pad_token_id", "eos_token_id"):
            if getattr(self, k) is not None:
                out[k] = getattr(self, k)
        return out

    @classmethod
    def from_pretrained(cls, path: str) -> "LopovikConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    # ---- names the engines share with the other model families ----
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def stream_spec(self) -> StreamSpec:
        loop = (int(self.loop["start"]), int(self.loop["stop"]), int(self.loop["times"])) if self.loop else None
        return StreamSpec(kind="parallel", positions=False, token_shift=True, centred_norm=True, loop=loop, tied_head=True)

    def layer_specs(self) -> List[LayerSpec]:
        specs = []
        for i, layer in enumerate(self.layers):
            m, rot = layer["mixer"], layer["mixer"]["rot"]
            mixer = MixerSpec("latent_attention", f"l{i}.mix.", heads=int(m["heads"]), kv_heads=1, dim=int(m["dim"]), vdim=int(m["vdim"]),
                              scale=float(m["scale"]), kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), rot_dim=int(m["rot_dim"]),
                              rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_layout="interleaved", head_sink=True, out_gate=True)
            spec = LayerSpec(i, [mixer])
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] == "dense":
                spec.ff, spec.ff_act = int(mlp["ff"]), "relu2"
            elif mlp is not None:
                spec.ff, spec.ff_act, spec.ff_kind = int(mlp["expert"]["ff"]), "swiglu", "moe"
                spec.experts, spec.top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
                spec.route, spec.weight_input = "sigmoid", True
            specs.append(spec)
        return specs

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every checkpoint tensor."""
        W = self.width
        out: Dict[str, tuple] = {"embed": (self.vocab, W)}
        if self.loop:
            out["loop.in"] = (W, 2 * W)
        for spec in self.layer_specs():
            p, m = f"l{spec.index}.", spec.mixers[0]
            q, f, n = m.prefix, p + "mlp.", m.heads * m.vdim
            out[p + "norm1"], out[p + "shift"] = (W,), (W,)
            out.update({q + "dq": (m.q_rank, W), q + "dq.norm": (m.q_rank,), q + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                        q + "dkv": (m.kv_rank + m.rot_dim, W), q + "dkv.norm": (m.kv_rank,), q + "uk": (m.heads * m.dim, m.kv_rank),
                        q + "uv": (n, m.kv_rank), q + "sink": (m.heads,), q + "g": (n, W), q + "o": (W, n)})
            if spec.ff:
                out[p + "norm2"] = (W,)
            if spec.ff and spec.ff_kind == "dense":
                out.update({f + "up": (spec.ff, W), f + "down": (W, spec.ff)})
            elif spec.ff:
                for e in range(spec.experts):
                    out.update({f"{f}e{e}.gate": (spec.ff, W), f"{f}e{e}.up": (spec.ff, W), f"{f}e{e}.down": (W, spec.ff)})
                out[f + "router"] = (spec.experts, W)
        out["final.norm"] = (W,)
        return out


@register_model("Lopovik", "lopovik", sampler="hybrid")
class LopovikForCausalLM(TensorModel):
    """Lopovik checkpoint tensors under their own names; executed by ``sampler.hybrid_sampler.HybridSampler``."""
    config_class = LopovikConfig
    ignore_extra = True                                    # e.g. the second norm of a layer without a feed-forward

    @staticmethod
    def init_value(n: str, t: torch.Tensor, g: torch.Generator) -> torch.Tensor:
        """Random weights (benchmarks, smoke tests): projections ~ N(0, 1/fan_in), norm weights around zero, shifts in [0, 1]."""
        leaf = n.rsplit(".", 1)[-1]
        if t.dim() == 2:
            return torch.randn(t.shape, generator=g) / (1.0 if leaf == "embed" else t.shape[1] ** 0.5)
        if leaf == "sink":
            return torch.randn(t.shape, generator=g)
        if leaf == "shift":
            return torch.rand(t.shape, generator=g)
        if n.endswith("dq.norm") or n.endswith("dkv.norm"):
            return torch.rand(t.shape, generator=g) * 0.5 + 0.75
        return torch.randn(t.shape, generator=g) * 0.1
