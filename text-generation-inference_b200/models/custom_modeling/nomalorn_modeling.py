"""Nomalorn: a pre-norm decoder on one fp32 residual stream whose layers each put attention and a recurrent memory side by side, with
a run of layers that repeats with the same tensors.

x_0 = embed[token]; every layer is x += mixer(N1(x)), then x += ff(N2(x)), with N = x / sqrt(mean x^2 + eps) * w.  Layers loop.start ..
loop.stop - 1 run loop.times times in a row with the same tensors; ahead of pass t the stream takes x_0 once more (t > 0) and the vector
step[t] (every t).  Every pass is a layer run with a cache and state of its own.  logits = embed (N_final x): the embedding table
is the vocabulary head.

Mixer "parallel": 1/2 (unit_rms(left(h)) * w_left + unit_rms(right(h)) * w_right); left = grouped-query attention with projection biases,
partly rotated heads, a chunked causal mask and a gate per head; right = the gated delta rule with a decay per head and key channel.
Feed-forward: up / squared ReLU / down with biases, or none.

config.json: {"architecture": "Nomalorn", "vocab", "width", "norm": {"eps"}, ["loop": {"start", "stop", "times"},] "layers": [{"type":
"parallel", "mixer": {"left": {heads, kv_heads, dim, vdim, scale, [rot {base, dims},] [mask {size}]}, "right": {heads, kv_heads, dim, vdim,
conv}}, "mlp": null | {"kind": "dense", "ff"}}, ...]}.
Checkpoint tensors: `embed`, `loop.step` [times, width], `l<i>.norm1|norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `final.norm`.

The mixers and feed-forwards (utils/mixers.py) and their kernels know nothing of this family; this file reads the configuration,
loads the tensors under the family's names and composes the layer runs.  Steps are ragged (ragged_decoder.py).
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, List, Optional, Tuple

import torch
from torch import nn

from ... import ops_seq as ops
from ...utils.mixers import ChannelDeltaMixer, NormedParallelMixers, PlainMLP, ScaledRotaryTables, SinkRotaryAttention
from ...utils.paged import HybridCacheManager
from .ragged_decoder import RaggedDecoderForCausalLM

ARCHITECTURE = "Nomalorn"
MIXER_TYPES = ("parallel",)


class NomalornConfig:
    """config.json of the family, with the attribute names the runtime reads on any model config."""
    model_type = "nomalorn"

    def __init__(self, raw: Dict[str, Any]):
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration")
        self.raw = raw
        self.architecture = ARCHITECTURE
        self.vocab_size = int(raw["vocab"])
        self.hidden_size = int(raw["width"])
        self.layers: List[Dict[str, Any]] = list(raw["layers"])
        self.norm_eps = float(raw["norm"]["eps"])
        self.eos_token_id = raw.get("eos_token_id")
        self.pad_token_id = raw.get("pad_token_id")
        self.quantize = None
        n, loop = len(self.layers), raw.get("loop")
        # (layer, pass): the layer of every run in order; pass t only where a run opens pass t of the loop
        self.layer_runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(n)]
        self.loop_times = 0
        if loop:
            a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
            if not (0 <= a <= b <= n) or times < 1:
                raise ValueError("loop: need 0 <= start <= stop <= number of layers and times >= 1")
            self.loop_times = times
            inner = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
            self.layer_runs = [(i, None) for i in range(a)] + inner + [(i, None) for i in range(b, n)]
        self.num_hidden_layers = len(self.layer_runs)     # what the cache manager books: one entry per layer run
        for layer in self.layers:
            if layer["type"] not in MIXER_TYPES:
                raise NotImplementedError(f"mixer type {layer['type']!r}")
            f = layer.get("mlp")
            if f and f.get("kind") != "dense":
                raise NotImplementedError(f"mlp kind {f.get('kind')!r}")

    @classmethod
    def from_pretrained(cls, model_path: str) -> "NomalornConfig":
        with open(os.path.join(model_path, "config.json")) as f:
            return cls(json.load(f))


def tensor_shapes(raw: Dict[str, Any], decay_rank: int = 64, gate_rank: int = 64) -> Dict[str, tuple]:
    """name -> shape of every checkpoint tensor of a configuration (synthetic checkpoints).  The ranks of the decay and gate projections
    are not part of the configuration: a checkpoint's `a1` / `g1` decide them, a synthetic one takes these."""
    W, V = int(raw["width"]), int(raw["vocab"])
    out = {"embed": (V, W), "final.norm": (W,)}
    if raw.get("loop"):
        out["loop.step"] = (int(raw["loop"]["times"]), W)
    for i, layer in enumerate(raw["layers"]):
        pre = f"l{i}"
        a, r = ({k: v if isinstance(v, dict) else int(v) for k, v in layer["mixer"][side].items() if k != "scale"} for side in ("left", "right"))
        H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        mix = {"left.q": (H * d, W), "left.q.b": (H * d,), "left.k": (G * d, W), "left.k.b": (G * d,), "left.v": (G * dv, W), "left.v.b": (G * dv,),
               "left.g": (H, W), "left.o": (W, H * dv), "left.out": (W,)}
        H, G, d, dv, taps = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
        mix.update({"right.q": (G * d, W), "right.q.conv": (G * d, taps), "right.k": (G * d, W), "right.k.conv": (G * d, taps),
                    "right.v": (H * dv, W), "right.v.conv": (H * dv, taps), "right.b": (H, W), "right.A_log": (H,), "right.norm": (dv,),
                    "right.a1": (int(decay_rank), W), "right.a2": (H * d, int(decay_rank)), "right.dt_bias": (H * d,),
                    "right.g1": (int(gate_rank), W), "right.g2": (H * dv, int(gate_rank)), "right.o": (W, H * dv), "right.out": (W,)})
        out[f"{pre}.norm1"] = (W,)
        out.update({f"{pre}.mix.{k}": v for k, v in mix.items()})
        f = layer.get("mlp")
        if f:
            ff = int(f["ff"])
            out.update({f"{pre}.norm2": (W,), f"{pre}.mlp.up": (ff, W), f"{pre}.mlp.up.b": (ff,), f"{pre}.mlp.down": (W, ff), f"{pre}.mlp.down.b": (W,)})
    return out


def build_mixer(kind: str, prefix: str, m: Dict[str, Any], weights, eps: float) -> nn.Module:
    if kind != "parallel":
        raise NotImplementedError(f"mixer type {kind!r}")
    a, r = m["left"], m["right"]
    rot, mask = a.get("rot"), a.get("mask")
    rotary = ScaledRotaryTables(int(rot["dims"]), float(rot["base"])) if rot and int(rot.get("dims", 0)) > 0 else None
    left = SinkRotaryAttention(f"{prefix}.left", weights, heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                               scale=float(a["scale"]), rotary=rotary, value_rotary=None, chunk=int(mask["size"]) if mask else None, sink=False,
                               head_gate=True, qk_norm=False, bias=True, eps=eps)
    right = ChannelDeltaMixer(f"{prefix}.right", weights, heads=int(r["heads"]), kv_heads=int(r["kv_heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]),
                              conv=int(r["conv"]), eps=eps)
    return NormedParallelMixers(prefix, weights, left, right, out_scale=0.5)


class NomalornLayer(nn.Module):
    """one layer run: `index` is the run (its cache and state), `entering` the pass of the loop that it opens; the modules may be
    another run's (a looped layer)"""

    def __init__(self, index: int, layer: int, entering: Optional[int], config: NomalornConfig, weights, share: Optional["NomalornLayer"] = None):
        super().__init__()
        self.index, self.entering = index, entering
        if share is not None:
            self.mixer, self.mlp, self.norm1, self.norm2 = share.mixer, share.mlp, share.norm1, share.norm2
            return
        spec, pre, eps = config.layers[layer], f"l{layer}", config.norm_eps
        self.mixer = build_mixer(spec["type"], f"{pre}.mix", spec["mixer"], weights, eps)
        self.norm1 = weights.get_tensor(f"{pre}.norm1").contiguous()
        self.mlp = self.norm2 = None
        if spec.get("mlp"):
            self.mlp = PlainMLP(f"{pre}.mlp", weights, activation="relu2", bias=True)
            self.norm2 = weights.get_tensor(f"{pre}.norm2").contiguous()


class _PlainNorm(nn.Module):
    def __init__(self, name: str, weights, eps: float):
        super().__init__()
        self.w, self.eps = weights.get_tensor(name).contiguous(), eps

    def forward(self, x):
        return ops.rmsnorm_rows(x, self.w, self.eps)


class NomalornModel(nn.Module):
    def __init__(self, config: NomalornConfig, weights):
        super().__init__()
        self.config = config
        self.embed = weights.get_tensor("embed").contiguous()
        self.dtype = self.embed.dtype
        self.step_vecs = []
        if config.loop_times:
            steps = weights.get_tensor("loop.step")
            if steps.shape != (config.loop_times, config.hidden_size):
                raise ValueError("loop.step: one vector of the model's width per pass expected")
            self.step_vecs = [v.contiguous() for v in steps]
        first: Dict[int, NomalornLayer] = {}
        runs = []
        for index, (layer, entering) in enumerate(config.layer_runs):
            run = NomalornLayer(index, layer, entering, config, weights, share=first.get(layer))
            first.setdefault(layer, run)
            runs.append(run)
        self.layers = nn.ModuleList(runs)
        self.final_norm = _PlainNorm("final.norm", weights, config.norm_eps)
        self.kv_cache_manager: Optional[HybridCacheManager] = None
        self.residual_probe: Optional[list] = None  # when a list: receives a copy of the stream after every layer run (tests)

    def _ahead_of(self, run: Optional[NomalornLayer], x0: torch.Tensor) -> Dict[str, Any]:
        """what joins the stream between the run before and `run`, and the norm that `run` reads it through"""
        if run is None:
            return {}
        out: Dict[str, Any] = {"norm_w": run.norm1}
        if run.entering is not None:
            out["step_vec"] = self.step_vecs[run.entering]
            if run.entering > 0:
                out["add"] = x0
        return out

    def forward(self, input_ids, step: ops.RaggedStep, max_s: int) -> torch.Tensor:
        """-> the fp32 stream [T, W].  Between two sublayers ONE launch norms and adds the last result's branches, adds what the loop
        puts ahead of a pass and reads the next sublayer's normed input."""
        x0 = ops.embed_scale(self.embed, input_ids, 1.0)
        x = torch.empty_like(x0)
        eps, manager = self.config.norm_eps, self.kv_cache_manager
        runs: List[Optional[NomalornLayer]] = list(self.layers) + [None]
        h = ops.branches_step(x, init=x0, eps=eps, **self._ahead_of(runs[0], x0))
        for run, following in zip(self.layers, runs[1:]):
            branches, scale = run.mixer(h, step, manager.layer_pages(run.index), manager.layer_state(run.index), max_s), run.mixer.out_scale
            if run.mlp is not None:
                h = ops.branches_step(x, branches=branches, y_scale=scale, norm_w=run.norm2, eps=eps)
                branches, scale = [(run.mlp(h), None)], 1.0
            if self.residual_probe is not None:   # the stream before anything joins it for the next run: written by a launch of its own
                ops.branches_step(x, branches=branches, y_scale=scale, eps=eps)
                self.residual_probe.append(x.clone())
                branches = []
            h = ops.branches_step(x, branches=branches, y_scale=scale, eps=eps, **self._ahead_of(following, x0))
        return x


class NomalornForCausalLM(RaggedDecoderForCausalLM):
    def __init__(self, config: NomalornConfig, weights):
        super().__init__(config, weights, NomalornModel(config, weights), head_tensor="embed")
