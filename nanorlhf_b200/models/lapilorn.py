"""Lapilorn: a decoder whose layers feed a mixer and a feed-forward from one norm and add both results.

* Embedding: ``x = embed[token]``; output: ``logits = embed norm(x)`` (tied).
* Layer: ``h = norm1(x)``, ``x += mixer(h) + ff(h)``; RMS norms whose weight is stored around zero.
* ``attention`` mixer: grouped heads; interleaved rotation of the first ``rot.dims`` columns of q and k, long wavelengths stretched by
  ``rot.scaling``; scores ``softcap * tanh((q.k) scale / softcap)``; causal softmax; the concatenated heads times ``sigmoid(g h)``;
  output projection ``o``.  With ``kv_from: j`` the layer has no key / value projections and reads layer j's pages.
* ``lightning`` mixer: linear attention with a constant decay per head, ``S = decay_h S + k v^T``, ``o = S^T q``, with q, k, v = silu of their
  projections; the concatenated heads RMS-normed together (weight ``norm``), times ``sigmoid(g h)``, output projection ``o``.
* Feed-forward: a clamped gated unit ``down (g sigmoid(1.702 g) (u + 1))`` with ``g = min(gate h, limit)``, ``u = clamp(up h, limit)``; or squared-ReLU
  experts, ``top`` of them chosen by ``sigmoid(router h) + correction`` among the experts of the best ``groups.keep`` groups (a group's score
  is the sum of its two largest), weighed by their sigmoids over their sum times ``scale``, plus a shared expert; or none.

This module holds the configuration (every size and constant is read from ``config.json``) and the checkpoint tensors under their
own names; it describes the layers as generic specs (models/hybrid_spec.py) that the step engine (sampler/hybrid_sampler.py)
executes.  There is no forward loop here.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from .hybrid_spec import LayerSpec, MixerSpec, StreamSpec, TensorModel
from .registry import register_model

LAYER_TYPES = ("attention", "lightning")
GATE_ALPHA, UP_SHIFT = 1.702, 1.0                              # the dense feed-forward's gate slope and the offset of its linear half


def _rot_fields(rot: Optional[dict]) -> dict:
    if not rot or not int(rot.get("dims", 0)):
        return dict(rot_dims=0)
    return dict(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_layout="interleaved",
                rot_scaling=dict(rot["scaling"]) if rot.get("scaling") else None)


@dataclass
class LapilornConfig:
    vocab: int = 256
    width: int = 128
    norm_eps: float = 1e-6
    layers: List[dict] = field(default_factory=list)         # the checkpoint's own layer descriptions
    model_type: str = "lapilorn"
    architecture: str = "Lapilorn"
    pad_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None
    max_positions: int = 1 << 30                             # positions are rotations: nothing bounds a sequence's length

    @classmethod
    def from_dict(cls, d: dict) -> "LapilornConfig":
        layers = list(d["layers"])
        for i, layer in enumerate(layers):
            if layer["type"] not in LAYER_TYPES:
                raise ValueError(f"layer {i}: unknown layer type {layer['type']!r}")
            m, mlp = layer["mixer"], layer.get("mlp")
            if layer["type"] == "lightning":
                if len(m["decay"]) != int(m["heads"]):
                    raise ValueError(f"layer {i}: decay must hold one number per head")
            else:
                cls._check_attention(layers, i)
            if mlp is None:
                continue
            if mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            if mlp["kind"] == "dense" and not float(mlp["limit"]) > 0:
                raise ValueError(f"layer {i}: limit must be positive")
            if mlp["kind"] == "moe":
                r = mlp["router"]
                n, top, g = int(r["experts"]), int(r["top"]), r.get("groups")
                if not 1 <= top <= n:
                    raise ValueError(f"layer {i}: router.top must lie between 1 and router.experts")
                if g and (n % int(g["count"]) or not 1 <= int(g["keep"]) <= int(g["count"]) or int(g["keep"]) * (n // int(g["count"])) < top):
                    raise ValueError(f"layer {i}: the router's groups do not fit its experts")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=layers,
                   pad_token_id=d.get("pad_token_id"), eos_token_id=d.get("eos_token_id"))

    @staticmethod
    def _check_attention(layers: List[dict], i: int):
        m = layers[i]["mixer"]
        rot, src = m.get("rot"), m.get("kv_from")
        if int(m["heads"]) % int(m["kv_heads"]):
            raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
        if rot and (int(rot["dims"]) % 2 or int(rot["dims"]) > int(m["dim"])):
            raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
        if src is None:
            return
        src = int(src)
        if not 0 <= src < i or layers[src]["type"] != "attention" or layers[src]["mixer"].get("kv_from") is not None:
            raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with projections of its own")
        o = layers[src]["mixer"]
        if any(int(o[k]) != int(m[k]) for k in ("kv_heads", "dim", "vdim")):
            raise ValueError(f"layer {i}: kv_from layer {src} has other key / value sizes")

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "layers": self.layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
               "width": self.width}
        for k in ("pad_token_id", "eos_token_id"):
            if getattr(self, k) is not None:
                out[k] = getattr(self, k)
        return out

    @classmethod
    def from_pretrained(cls, path: str) -> "LapilornConfig":
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
        return StreamSpec(kind="parallel", positions=False, shared_norm=True, centred_norm=True, tied_head=True)

    def layer_specs(self) -> List[LayerSpec]:
        specs = []
        for i, layer in enumerate(self.layers):
            m, p = layer["mixer"], f"l{i}.mix."
            if layer["type"] == "attention":
                src = m.get("kv_from")
                mixer = MixerSpec("rot_attention", p, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                  scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), out_gate=True,
                                  kv_from=-1 if src is None else int(src), **_rot_fields(m.get("rot")))
            else:
                mixer = MixerSpec("lightning", p, heads=int(m["heads"]), kv_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                  decay=tuple(float(x) for x in m["decay"]))
            spec = LayerSpec(i, [mixer])
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] == "dense":
                spec.ff, spec.ff_act, spec.ff_limit = int(mlp["ff"]), "swiglu", float(mlp["limit"])
                spec.ff_alpha, spec.ff_up_shift = GATE_ALPHA, UP_SHIFT
            elif mlp is not None:
                r, g = mlp["router"], mlp["router"].get("groups")
                spec.ff, spec.ff_act, spec.ff_kind = int(mlp["expert"]["ff"]), "relu2", "moe"
                spec.experts, spec.top = int(r["experts"]), int(r["top"])
                spec.route, spec.route_scale, spec.group_score = "sigmoid_all", float(r.get("scale", 1.0)), "top2"
                if g:
                    spec.route_groups, spec.route_keep = int(g["count"]), int(g["keep"])
                if mlp.get("shared"):
                    spec.shared_ff = int(mlp["shared"]["ff"])
            specs.append(spec)
        return specs

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every checkpoint tensor."""
        W = self.width
        out: Dict[str, tuple] = {"embed": (self.vocab, W)}
        for spec in self.layer_specs():
            p, m = f"l{spec.index}.", spec.mixers[0]
            q, f, n = m.prefix, p + "mlp.", m.heads * m.vdim
            out[p + "norm1"] = (W,)
            out[q + "q"] = (m.heads * m.dim, W)
            if m.kv_from < 0:
                out[q + "k"], out[q + "v"] = (m.kv_heads * m.dim, W), (m.kv_heads * m.vdim, W)
            out[q + "g"], out[q + "o"] = (n, W), (W, n)
            if m.kind == "lightning":
                out[q + "norm"] = (n,)
            if spec.ff and spec.ff_kind == "dense":
                out.update({f + "gate": (spec.ff, W), f + "up": (spec.ff, W), f + "down": (W, spec.ff)})
            elif spec.ff:
                for e in range(spec.experts):
                    out.update({f"{f}e{e}.up": (spec.ff, W), f"{f}e{e}.down": (W, spec.ff)})
                out[f + "router"], out[f + "correction"] = (spec.experts, W), (spec.experts,)
                if spec.shared_ff:
                    out.update({f + "shared.up": (spec.shared_ff, W), f + "shared.down": (W, spec.shared_ff)})
        out["final.norm"] = (W,)
        return out


@register_model("Lapilorn", "lapilorn", sampler="hybrid")
class LapilornForCausalLM(TensorModel):
    """Lapilorn checkpoint tensors under their own names; executed by ``sampler.hybrid_sampler.HybridSampler``."""
    config_class = LapilornConfig
    ignore_extra = True

    @staticmethod
    def init_value(n: str, t: torch.Tensor, g: torch.Generator) -> torch.Tensor:
        """Random weights (benchmarks, smoke tests): projections ~ N(0, 1/fan_in), norm weights around zero (the mixer's own around one)."""
        leaf = n.rsplit(".", 1)[-1]
        if t.dim() == 2:
            return torch.randn(t.shape, generator=g) / (1.0 if leaf == "embed" else t.shape[1] ** 0.5)
        if n.endswith("mix.norm"):
            return torch.rand(t.shape, generator=g) * 0.5 + 0.75
        return torch.randn(t.shape, generator=g) * (0.02 if leaf == "correction" else 0.1)
