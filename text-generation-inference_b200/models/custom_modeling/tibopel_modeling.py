"""Tibopel: a decoder on one fp32 residual stream whose layers read the stream once and add a mixer and a routed feed-forward side by side,
x += mixer(N1(x)) + ff(N2(x)), with N = x / sqrt(mean x^2 + eps) * w; x_0 = embed[token], logits = cap tanh(head N_final(x) / cap).  A layer
may use another layer's tensors (`weights_of`) with a cache of its own.

Mixers: grouped-query attention with projection biases, an interleaved rotation of a part of every head (optionally slowed by
wavelength), a chunked causal mask and a gate per head; latent attention with a sink logit per head.  Feed-forward: squared-ReLU experts
by corrected soft-max scores, identity experts, and a shared expert with a gate per token; or none.

config.json: {"architecture": "Tibopel", "vocab", "width", "norm": {"eps"}, "logit_softcap", "layers": [{"type": "attention" |
"latent_attention", "mixer": {...}, "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "identity", "top"}, "shared":
null | {"ff"}} [, "weights_of": j]}, ...]}.
  attention:        heads, kv_heads, dim, vdim, scale [, rot {base, dims [, scaling {factor, low, high, original}]}] [, mask {size}]
  latent_attention: heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims [, scaling]}
Checkpoint tensors: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.

The mixers and feed-forwards (utils/mixers.py) and their kernels know nothing of this family; this file reads the configuration,
loads the tensors under the family's names and composes the layers.  Steps are ragged (ragged_decoder.py).
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, List, Optional

import torch
from torch import nn

from ... import ops_seq as ops
from ...utils.mixers import LatentAttention, RoutedSharedFeedForward, ScaledRotaryTables, SinkRotaryAttention
from ...utils.paged import HybridCacheManager
from .ragged_decoder import RaggedDecoderForCausalLM

ARCHITECTURE = "Tibopel"
MIXER_TYPES = ("attention", "latent_attention")


class TibopelConfig:
    """config.json of the family, with the attribute names the runtime reads on any model config."""
    model_type = "tibopel"

    def __init__(self, raw: Dict[str, Any]):
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration")
        self.raw = raw
        self.architecture = ARCHITECTURE
        self.vocab_size = int(raw["vocab"])
        self.hidden_size = int(raw["width"])
        self.layers: List[Dict[str, Any]] = list(raw["layers"])
        self.num_hidden_layers = len(self.layers)
        self.norm_eps = float(raw["norm"]["eps"])
        self.logit_softcap = float(raw.get("logit_softcap") or 0.0)
        self.eos_token_id = raw.get("eos_token_id")
        self.pad_token_id = raw.get("pad_token_id")
        self.quantize = None
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXER_TYPES:
                raise NotImplementedError(f"mixer type {layer['type']!r}")
            f = layer.get("mlp")
            if f and f.get("kind") != "moe":
                raise NotImplementedError(f"mlp kind {f.get('kind')!r}")
            j = self.weight_layer(i)
            if j != i:
                own = self.layers[j]
                if own["type"] != layer["type"] or own["mixer"] != layer["mixer"] or own.get("mlp") != layer.get("mlp"):
                    raise ValueError(f"layer {i}: weights_of {j} names a layer of another shape")

    def weight_layer(self, i: int) -> int:
        """the layer whose tensors layer i uses (itself unless `weights_of` says otherwise)"""
        seen = set()
        while self.layers[i].get("weights_of") is not None:
            if i in seen or not 0 <= int(self.layers[i]["weights_of"]) < len(self.layers):
                raise ValueError(f"layer {i}: weights_of does not lead to a layer with tensors")
            seen.add(i)
            i = int(self.layers[i]["weights_of"])
        return i

    @classmethod
    def from_pretrained(cls, model_path: str) -> "TibopelConfig":
        with open(os.path.join(model_path, "config.json")) as f:
            return cls(json.load(f))


def tensor_shapes(raw: Dict[str, Any]) -> Dict[str, tuple]:
    """name -> shape of every checkpoint tensor of a configuration (synthetic checkpoints)"""
    W, V = int(raw["width"]), int(raw["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(raw["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, pre = layer["mixer"], f"l{i}"
        H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        if layer["type"] == "attention":
            G = int(m["kv_heads"])
            mix = {"q": (H * d, W), "q.b": (H * d,), "k": (G * d, W), "k.b": (G * d,), "v": (G * dv, W), "v.b": (G * dv,), "g": (H, W),
                   "o": (W, H * dv), "o.b": (W,)}
        else:
            R, Q, r = int(m["kv_rank"]), int(m["q_rank"]), int(m["rot_dim"])
            mix = {"dq": (Q, W), "dq.norm": (Q,), "uq": (H * (d + r), Q), "dkv": (R + r, W), "dkv.norm": (R,), "uk": (H * d, R), "uv": (H * dv, R),
                   "sink": (H,), "o": (W, H * dv)}
        out[f"{pre}.norm1"] = (W,)
        out.update({f"{pre}.mix.{k}": v for k, v in mix.items()})
        f = layer.get("mlp")
        if not f:
            continue
        E, n, ff = int(f["router"]["experts"]), int(f["router"]["experts"]) + int(f["router"].get("identity") or 0), int(f["expert"]["ff"])
        out.update({f"{pre}.norm2": (W,), f"{pre}.mlp.router": (n, W), f"{pre}.mlp.correction": (n,)})
        for e in range(E):
            out.update({f"{pre}.mlp.e{e}.up": (ff, W), f"{pre}.mlp.e{e}.down": (W, ff)})
        if f.get("shared"):
            sf = int(f["shared"]["ff"])
            out.update({f"{pre}.mlp.shared.up": (sf, W), f"{pre}.mlp.shared.down": (W, sf), f"{pre}.mlp.shared.sg": (1, W)})
    return out


def _rotary(rot: Optional[Dict[str, Any]]) -> Optional[ScaledRotaryTables]:
    return ScaledRotaryTables(int(rot["dims"]), float(rot["base"]), rot.get("scaling")) if rot and int(rot.get("dims", 0)) > 0 else None


def build_mixer(kind: str, prefix: str, m: Dict[str, Any], weights, eps: float) -> nn.Module:
    if kind == "attention":
        mask = m.get("mask")
        return SinkRotaryAttention(prefix, weights, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                   scale=float(m["scale"]), rotary=_rotary(m.get("rot")), value_rotary=None, qk_pairs="interleaved",
                                   chunk=int(mask["size"]) if mask else None, sink=False, head_gate=True, qk_norm=False, bias=True, out_bias=True,
                                   eps=eps)
    if kind == "latent_attention":
        return LatentAttention(prefix, weights, heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), scale=float(m["scale"]), window=None, rotary=_rotary(m["rot"]),
                               eps=eps, gate=False, sink=True, out_dtype=torch.float32)
    raise NotImplementedError(f"mixer type {kind!r}")


class TibopelLayer(nn.Module):
    """the modules of one layer: its own, or another layer's; the cache is this layer's in any case (looked up by `index`)"""

    def __init__(self, index: int, config: TibopelConfig, weights, share: Optional["TibopelLayer"] = None):
        super().__init__()
        self.index = index
        if share is not None:
            self.mixer, self.mlp, self.norm1, self.norm2 = share.mixer, share.mlp, share.norm1, share.norm2
            return
        spec, pre, eps = config.layers[index], f"l{index}", config.norm_eps
        self.mixer = build_mixer(spec["type"], f"{pre}.mix", spec["mixer"], weights, eps)
        self.norm1 = weights.get_tensor(f"{pre}.norm1").contiguous()
        self.mlp = self.norm2 = None
        f = spec.get("mlp")
        if f:
            self.mlp = RoutedSharedFeedForward(f"{pre}.mlp", weights, experts=int(f["router"]["experts"]),
                                               identity=int(f["router"].get("identity") or 0), top=int(f["router"]["top"]), shared=bool(f.get("shared")))
            self.norm2 = weights.get_tensor(f"{pre}.norm2").contiguous()

    def halves(self, h1: torch.Tensor, h2: Optional[torch.Tensor], step: ops.RaggedStep, manager: HybridCacheManager, max_s: int) -> Dict[str, Any]:
        """what the layer adds to the stream, as arguments of `ops.halves_step`; in a captured decoding step the two halves run side by side"""
        out: Dict[str, Any] = {}
        with ops.beside(h1.device) as side:
            if self.mlp is not None:
                out.update(self.mlp(h2))
        if isinstance(self.mixer, LatentAttention):
            y = self.mixer(h1, step, manager.layer_pages(self.index), max_s)
        else:
            y = self.mixer(h1, step, manager.layer_pages(self.index), None, max_s)
        side.join()
        out["y1"] = y
        return out


class _PlainNorm(nn.Module):
    def __init__(self, name: str, weights, eps: float):
        super().__init__()
        self.w, self.eps = weights.get_tensor(name).contiguous(), eps

    def forward(self, x):
        return ops.rmsnorm_rows(x, self.w, self.eps)


class TibopelModel(nn.Module):
    def __init__(self, config: TibopelConfig, weights):
        super().__init__()
        self.config = config
        self.embed = weights.get_tensor("embed").contiguous()
        self.dtype = self.embed.dtype
        layers: List[Optional[TibopelLayer]] = [None] * config.num_hidden_layers
        for i in range(config.num_hidden_layers):      # layers with tensors first: a sharing layer may come before its source
            if config.weight_layer(i) == i:
                layers[i] = TibopelLayer(i, config, weights)
        for i in range(config.num_hidden_layers):
            if layers[i] is None:
                layers[i] = TibopelLayer(i, config, weights, share=layers[config.weight_layer(i)])
        self.layers = nn.ModuleList(layers)
        self.final_norm = _PlainNorm("final.norm", weights, config.norm_eps)
        self.kv_cache_manager: Optional[HybridCacheManager] = None
        self.residual_probe: Optional[list] = None  # when a list: receives a copy of the stream after every layer (tests)

    def forward(self, input_ids, step: ops.RaggedStep, max_s: int) -> torch.Tensor:
        """-> the fp32 stream [T, W].  Between two layers ONE launch adds everything the last layer's halves bring and reads the stream
        through both norms of the next one."""
        x0 = ops.embed_scale(self.embed, input_ids, 1.0)
        x, eps = torch.empty_like(x0), self.config.norm_eps
        joins: Dict[str, Any] = {"init": x0}
        for layer in self.layers:
            h1, h2 = ops.halves_step(x, norm_a=layer.norm1, norm_b=layer.norm2, eps=eps, dtype=self.dtype, **joins)
            if self.residual_probe is not None and "init" not in joins:
                self.residual_probe.append(x.clone())
            joins = layer.halves(h1, h2, step, self.kv_cache_manager, max_s)
        ops.halves_step(x, eps=eps, dtype=self.dtype, **joins)
        if self.residual_probe is not None:
            self.residual_probe.append(x.clone())
        return x


class TibopelForCausalLM(RaggedDecoderForCausalLM):
    def __init__(self, config: TibopelConfig, weights):
        super().__init__(config, weights, TibopelModel(config, weights))
        self.logit_softcap = config.logit_softcap
