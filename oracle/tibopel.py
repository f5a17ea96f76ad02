"""Slow reference of the Tibopel decoder: plain PyTorch on the CPU, one function per mechanism, whole sequences at once.

Test infrastructure only.  It shares no code with the product path (no paged cache, no absorbed products, no row plans, no kernels):
every mixer recomputes a sequence from its first token with dense score matrices and every expert runs on every token, so a test
can compare any cut of a prompt, any batch and any reuse of pages in the product against it.  `dtype` is torch.float64 by default.

The model: x_0 = embed[token]; a layer reads the stream once and adds both of its halves, x += mixer(N1(x)) + ff(N2(x)), N = unit-RMS
times a weight.  Mixers: grouped-query attention (projection biases, interleaved rotation of a part of the head with slowed low
frequencies, a mask that cuts the sequence into chunks, a sigmoid gate per head), and latent attention (keys and values are
up-projections of one normed latent per token, one rotated key part for all heads, a sink logit per head).  Feed-forward: experts
W_down relu(W_up h)^2 picked by corrected soft-max scores, some of the router's outputs being the identity, plus a shared expert
times a sigmoid gate per token.  logits = cap tanh(head N_final(x) / cap).

Checkpoint naming: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""
from __future__ import annotations

import copy
import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sub(sd: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


def turn_rates(dims: int, base: float, scaling: Optional[dict] = None) -> List[float]:
    """radians per position of every rotated pair.  `scaling` {factor, low, high, original}: a pair whose period is shorter than
    original / high keeps its rate, one whose period is longer than original / low is slowed by factor, in between the two are blended
    by where original / period lies between low and high"""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[n]) for n in ("factor", "low", "high", "original"))
            period = 2.0 * math.pi / f
            if period > original / low:
                f = f / factor
            elif period >= original / high:
                s = (original / period - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_neighbours(x, positions, rates: List[float]):
    """x [L, heads, n]: columns 2i and 2i + 1 of every head are turned by position * rates[i]; the other columns pass"""
    dims = 2 * len(rates)
    if dims == 0:
        return x
    ang = positions.to(F64)[:, None] * torch.tensor(rates, dtype=F64)[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2] = a * c - b * s
    y[..., 1:dims:2] = b * c + a * s
    return y


# ------------------------------------------------------------------------------------------------ mixers
def chunk_attention(h, p, m: dict):
    """h [L, W] -> [L, W]"""
    L, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(L)
    q = (h @ p["q"].T + p["q.b"]).view(L, H, d)
    k = (h @ p["k"].T + p["k.b"]).view(L, G, d)
    v = (h @ p["v"].T + p["v.b"]).view(L, G, dv)
    if m.get("rot"):
        rates = turn_rates(int(m["rot"]["dims"]), float(m["rot"]["base"]), m["rot"].get("scaling"))
        q, k = rotate_neighbours(q, pos, rates), rotate_neighbours(k, pos, rates)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * float(m["scale"])
    see = pos[None, :] <= pos[:, None]
    if m.get("mask"):
        size = int(m["mask"]["size"])
        see = see & ((pos[None, :] // size) == (pos[:, None] // size))
    a = torch.softmax(s.masked_fill(~see, float("-inf")), -1)
    o = torch.einsum("hij,jhv->ihv", a, v.repeat_interleave(H // G, dim=1))
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(L, H * dv) @ p["o"].T + p["o.b"]


def sink_softmax(s, sink):
    """s [H, L, L] scores (-inf where a key is hidden), sink [H]: exp(sink) takes weight in the denominator and gives none out"""
    m = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def latent_attention(h, p, m: dict, eps: float):
    """h [L, W] -> [L, W]; keys and values are written out per head"""
    L, H, d, r, dv, R = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(L)
    rates = turn_rates(int(m["rot"]["dims"]), float(m["rot"]["base"]), m["rot"].get("scaling"))
    q = ((unit_rms(h @ p["dq"].T, eps) * p["dq.norm"]) @ p["uq"].T).view(L, H, d + r)
    down = h @ p["dkv"].T
    c = unit_rms(down[:, :R], eps) * p["dkv.norm"]
    k_rot = rotate_neighbours(down[:, None, R:], pos, rates)[:, 0]
    q_rot = rotate_neighbours(q[..., d:], pos, rates)
    k = (c @ p["uk"].T).view(L, H, d)
    v = (c @ p["uv"].T).view(L, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihr,jr->hij", q_rot, k_rot)) * float(m["scale"])
    s = s.masked_fill(~(pos[None, :] <= pos[:, None]), float("-inf"))
    o = torch.einsum("hij,jhv->ihv", sink_softmax(s, p["sink"]), v)
    return o.reshape(L, H * dv) @ p["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def squared_relu_expert(h, p, prefix: str):
    return torch.clamp(h @ p[prefix + "up"].T, min=0.0) ** 2 @ p[prefix + "down"].T


def pick_experts(scores, correction, top: int):
    """scores [L, E] (soft-max over all router outputs) -> ids [L, top], weights [L, top]: picked by score + correction, weighed by the
    plain scores of the picks over their sum"""
    ids = torch.topk(scores + correction, top, dim=-1).indices
    w = torch.gather(scores, 1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def routed_experts(h, p, f: dict):
    """h [L, W] -> [L, W]: every expert on every token, times its weight (0 where it was not picked)"""
    E, top = int(f["router"]["experts"]), int(f["router"]["top"])
    scores = torch.softmax(h @ p["router"].T, -1)
    ids, w = pick_experts(scores, p["correction"], top)
    full = torch.zeros_like(scores).scatter_add_(1, ids, w)
    y = torch.zeros_like(h)
    for e in range(scores.shape[1]):
        y = y + full[:, e:e + 1] * (squared_relu_expert(h, p, f"e{e}.") if e < E else h)
    if f.get("shared"):
        y = y + torch.sigmoid(h @ p["shared.sg"].T) * squared_relu_expert(h, p, "shared.")
    return y


# ------------------------------------------------------------------------------------------------ the model
def weight_layer(config: dict, i: int) -> int:
    while config["layers"][i].get("weights_of") is not None:
        i = int(config["layers"][i]["weights_of"])
    return i


def soft_cap(z, cap: float):
    return cap * torch.tanh(z / cap)


def forward(config: dict, sd: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, residuals: Optional[list] = None):
    """logits [L, vocab] of one sequence; `residuals`, when a list, receives the stream after every layer"""
    sd = {k: v.to(dtype) for k, v in sd.items() if v.is_floating_point()}
    eps = float(config["norm"]["eps"])
    x = sd["embed"][torch.tensor(tokens, dtype=torch.int64)]
    for i, layer in enumerate(config["layers"]):
        pre = f"l{weight_layer(config, i)}."
        h, p = unit_rms(x, eps) * sd[pre + "norm1"], sub(sd, pre + "mix.")
        y = chunk_attention(h, p, layer["mixer"]) if layer["type"] == "attention" else latent_attention(h, p, layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + routed_experts(unit_rms(x, eps) * sd[pre + "norm2"], sub(sd, pre + "mlp."), layer["mlp"])
        x = x + y
        if residuals is not None:
            residuals.append(x)
    z = (unit_rms(x, eps) * sd["final.norm"]) @ sd["head"].T
    return soft_cap(z, float(config["logit_softcap"])) if config.get("logit_softcap") else z


# ------------------------------------------------------------------------------------------------ random models
def random_config(*, width: int = 40, vocab: int = 72, order=("attention", "latent_attention", "attention", "latent_attention"), shares=(None, None, None, 1),
                  heads: int = 6, kv_heads: int = 2, dim: int = 10, vdim: int = 12, rot_dims=6, base: float = 500.0,
                  scaling=(4.0, 1.0, 3.0, 60), chunk=20, sharp: float = 1.0, l_heads: int = 3, l_dim: int = 8, rot_dim: int = 6, l_rot_dims=None,
                  l_base: float = 200.0, l_vdim: int = 14, kv_rank: int = 20, q_rank: int = 18, mlp=("moe",), experts: int = 5, identity: int = 2,
                  top: int = 3, ff: int = 12, shared=28, cap=15.0, eps: float = 1e-5, other: Optional[dict] = None) -> dict:
    """a small configuration; `rot_dims` / `scaling` (factor, low, high, original) / `chunk` / `shared` / `cap` None leave the entry out, `sharp`
    multiplies the score scales, `other` = {layer: changed entries of its mixer}, `shares` names the layer whose tensors a layer uses"""
    layers = []
    for i, kind in enumerate(order):
        if kind == "attention":
            m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": dim ** -0.5 * sharp}
            if chunk:
                m["mask"] = {"size": chunk}
            if rot_dims:
                m["rot"] = {"base": base, "dims": rot_dims}
                if scaling:
                    m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        else:
            m = {"dim": l_dim, "heads": l_heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": l_base, "dims": l_rot_dims or rot_dim},
                 "rot_dim": rot_dim, "scale": (l_dim + rot_dim) ** -0.5 * sharp, "vdim": l_vdim}
        m.update((other or {}).get(i, {}))
        f = None
        if mlp[i % len(mlp)]:
            f = {"kind": "moe", "expert": {"ff": ff + 4 * (i % 2)}, "router": {"experts": experts + i % 2, "identity": identity, "top": top},
                 "shared": {"ff": shared} if shared else None}
        layer = {"type": kind, "mixer": m, "mlp": f}
        if i < len(shares) and shares[i] is not None:
            layer = {**copy.deepcopy(layers[shares[i]]), "weights_of": shares[i]}
        layers.append(layer)
    cfg = {"architecture": "Tibopel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


def tensor_shapes(config: dict) -> Dict[str, tuple]:
    W, V = int(config["width"]), int(config["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, f, H, dv = layer["mixer"], layer.get("mlp"), layer["mixer"]["heads"], layer["mixer"]["vdim"]
        if layer["type"] == "attention":
            nq, nk, nv = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * dv
            mix = {"q": (nq, W), "q.b": (nq,), "k": (nk, W), "k.b": (nk,), "v": (nv, W), "v.b": (nv,), "g": (H, W), "o": (W, H * dv), "o.b": (W,)}
        else:
            R, Q, r = m["kv_rank"], m["q_rank"], m["rot_dim"]
            mix = {"dq": (Q, W), "dq.norm": (Q,), "uq": (H * (m["dim"] + r), Q), "dkv": (R + r, W), "dkv.norm": (R,), "uk": (H * m["dim"], R),
                   "uv": (H * dv, R), "sink": (H,), "o": (W, H * dv)}
        out[f"l{i}.norm1"] = (W,)
        out.update({f"l{i}.mix.{name}": shape for name, shape in mix.items()})
        if f:
            E, ff, n = f["router"]["experts"], f["expert"]["ff"], f["router"]["experts"] + f["router"]["identity"]
            out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.router": (n, W), f"l{i}.mlp.correction": (n,)})
            for e in range(E):
                out.update({f"l{i}.mlp.e{e}.up": (ff, W), f"l{i}.mlp.e{e}.down": (W, ff)})
            if f.get("shared"):
                sf = f["shared"]["ff"]
                out.update({f"l{i}.mlp.shared.up": (sf, W), f"l{i}.mlp.shared.down": (W, sf), f"l{i}.mlp.shared.sg": (1, W)})
    return out


def random_state_dict(config: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """weights that are exactly representable in bfloat16, so that every element type starts from the same numbers"""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if leaf == "correction":
            t = torch.randn(shape, generator=g) * 0.15
        elif leaf == "sink":
            t = torch.randn(shape, generator=g) + 0.5
        elif leaf == "b":
            t = torch.randn(shape, generator=g) * 0.7
        elif leaf == "router":
            t = torch.randn(shape, generator=g) * (1.5 / math.sqrt(shape[1]))
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) * (0.7 if name == "embed" else (2.5 if name == "head" else 1.2) / math.sqrt(shape[1]))
        else:  # norm weights
            t = 1.0 + torch.randn(shape, generator=g) * 0.3
        sd[name] = t.to(torch.bfloat16).to(torch.float32)
    return sd
