"""Slow reference of the Nomalorn decoder: plain PyTorch on the CPU, one function per mechanism, whole sequences at once.

Test infrastructure only.  It shares no code with the product path (no paged cache, no state slots, no kernels): every mixer
recomputes a sequence from its first token (dense score matrices, a token-by-token recurrence), so a test can compare any cut
of a prompt, any batch and any reuse of pages and slots in the product against it.  `dtype` is torch.float64 by default.

The model: x_0 = embed[token]; every layer is x += mixer(N1(x)) then x += ff(N2(x)), N = unit-RMS times a weight.  A run of layers
repeats `times` times with the same tensors; ahead of pass t the stream takes x_0 once more (t > 0) and the vector step[t].  The
mixer puts two memories side by side, y = 1/2 (unit_rms(left(h)) * w_left + unit_rms(right(h)) * w_right): grouped-query attention
with projection biases, a partly rotated head (rotate-half pairs), a mask that cuts the sequence into chunks of equal length and
a sigmoid gate per head; and a gated delta rule whose decay has an entry per head and key channel, from a low-rank projection,
behind short convolutions + SiLU on q / k / v, with a sigmoid gate from a second low-rank projection.  The feed-forward is
W_down relu(W_up h + b_up)^2 + b_down.  logits = embed N_final(x).

Checkpoint naming: `embed`, `loop.step`, `l<i>.norm1|norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.up|down` (+ `.b`),
`final.norm`.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-torch.abs(z)))


def short_conv(u, w):
    """u [L, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the first row"""
    L, taps = u.shape[0], w.shape[1]
    pad = torch.cat([u.new_zeros(taps - 1, u.shape[1]), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + w[:, j] * pad[j:j + L]
    return y


def sub(sd: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


def rotate_halves(x, positions, dims: int, base: float):
    """x [L, heads, n]: the first `dims` columns of every head, column i paired with column i + dims / 2, pair i turned by
    position * base^(-2i / dims); the other columns pass"""
    i = torch.arange(dims // 2, dtype=x.dtype)
    ang = positions.to(x.dtype)[:, None] * base ** (-2.0 * i / dims)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


# ------------------------------------------------------------------------------------------------ mixers
def chunk_attention(h, p, m: dict):
    """h [L, W] -> [L, W]: the left half of the mixer"""
    L, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(L)
    q = (h @ p["q"].T + p["q.b"]).view(L, H, d)
    k = (h @ p["k"].T + p["k.b"]).view(L, G, d)
    v = (h @ p["v"].T + p["v.b"]).view(L, G, dv)
    if m.get("rot"):
        q, k = (rotate_halves(t, pos, int(m["rot"]["dims"]), float(m["rot"]["base"])) for t in (q, k))
    rep = H // G
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, dim=1)) * float(m["scale"])
    see = pos[None, :] <= pos[:, None]
    if m.get("mask"):
        size = int(m["mask"]["size"])
        see = see & ((pos[None, :] // size) == (pos[:, None] // size))
    a = torch.softmax(s.masked_fill(~see, float("-inf")), -1)
    o = torch.einsum("hij,jhv->ihv", a, v.repeat_interleave(rep, dim=1))
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(L, H * dv) @ p["o"].T


def delta_memory(q, k, v, beta, g):
    """q, k, g [L, H, d], v [L, H, dv], beta [L, H] -> o [L, H, dv]: S <- diag(g) S, then S += k (beta (v - S^T k))^T, o = S^T q"""
    L, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(L):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def channel_delta(h, p, m: dict, eps: float):
    """h [L, W] -> [L, W]: the right half of the mixer"""
    L, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(short_conv(h @ p["q"].T, p["q.conv"])).view(L, G, d)
    k = silu(short_conv(h @ p["k"].T, p["k.conv"])).view(L, G, d)
    v = silu(short_conv(h @ p["v"].T, p["v.conv"])).view(L, H, dv)
    rep = H // G
    q = (unit_length(q) * d ** -0.5).repeat_interleave(rep, dim=1)
    k = unit_length(k).repeat_interleave(rep, dim=1)
    beta = torch.sigmoid(h @ p["b"].T)
    raw = ((h @ p["a1"].T) @ p["a2"].T + p["dt_bias"]).view(L, H, d)
    g = torch.exp(-torch.exp(p["A_log"])[None, :, None] * softplus(raw))
    o = unit_rms(delta_memory(q, k, v, beta, g), eps) * p["norm"]
    o = o * torch.sigmoid((h @ p["g1"].T) @ p["g2"].T).view(L, H, dv)
    return o.reshape(L, H * dv) @ p["o"].T


def parallel_mixer(h, p, m: dict, eps: float):
    left = unit_rms(chunk_attention(h, sub(p, "left."), m["left"]), eps) * p["left.out"]
    right = unit_rms(channel_delta(h, sub(p, "right."), m["right"], eps), eps) * p["right.out"]
    return 0.5 * (left + right)


def squared_relu_mlp(h, p):
    return torch.clamp(h @ p["up"].T + p["up.b"], min=0.0) ** 2 @ p["down"].T + p["down.b"]


# ------------------------------------------------------------------------------------------------ the model
def layer_runs(config: dict) -> List[tuple]:
    """(layer, pass) of every layer run in order; the pass is None except for the first layer of a pass of the loop"""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    inner = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
    return [(i, None) for i in range(a)] + inner + [(i, None) for i in range(b, n)]


def forward(config: dict, sd: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, residuals: Optional[list] = None):
    """logits [L, vocab] of one sequence; `residuals`, when a list, receives the stream after every layer run"""
    sd = {k: v.to(dtype) for k, v in sd.items() if v.is_floating_point()}
    eps = float(config["norm"]["eps"])
    x0 = sd["embed"][torch.tensor(tokens, dtype=torch.int64)]
    x = x0
    for i, entering in layer_runs(config):
        layer, pre = config["layers"][i], f"l{i}."
        if entering is not None:
            if entering > 0:
                x = x + x0
            x = x + sd["loop.step"][entering]
        x = x + parallel_mixer(unit_rms(x, eps) * sd[pre + "norm1"], sub(sd, pre + "mix."), layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + squared_relu_mlp(unit_rms(x, eps) * sd[pre + "norm2"], sub(sd, pre + "mlp."))
        if residuals is not None:
            residuals.append(x)
    return (unit_rms(x, eps) * sd["final.norm"]) @ sd["embed"].T


# ------------------------------------------------------------------------------------------------ random models
def random_config(*, width: int = 40, vocab: int = 72, layers: int = 3, loop=(1, 3, 2), heads: int = 6, kv_heads: int = 2, dim: int = 10,
                  vdim: int = 12, rot_dims=6, base: float = 100.0, chunk=20, sharp: float = 1.0, r_heads: int = 4, r_kv_heads: int = 2,
                  r_dim: int = 12, r_vdim: int = 14, conv: int = 3, mlp=("dense", None, "dense"), ff: int = 28, eps: float = 1e-5,
                  other: Optional[dict] = None) -> dict:
    """a small configuration; `loop` = (start, stop, times) or None, `rot_dims` / `chunk` None to leave the entry out, `sharp`
    multiplies the attention's score scale, `other` = {layer: {side: changed sizes}} for layers unlike the rest"""
    out = []
    for i in range(layers):
        left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": dim ** -0.5 * sharp}
        if rot_dims:
            left["rot"] = {"base": base, "dims": rot_dims}
        if chunk:
            left["mask"] = {"size": chunk}
        right = {"conv": conv, "dim": r_dim, "heads": r_heads, "kv_heads": r_kv_heads, "vdim": r_vdim}
        for side, changes in (other or {}).get(i, {}).items():
            {"left": left, "right": right}[side].update(changes)
        f = mlp[i % len(mlp)]
        out.append({"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff + 4 * i} if f else None})
    cfg = {"architecture": "Nomalorn", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def tensor_shapes(config: dict, decay_rank: int = 5, gate_rank: int = 7) -> Dict[str, tuple]:
    W, V = int(config["width"]), int(config["vocab"])
    out = {"embed": (V, W), "final.norm": (W,)}
    if config.get("loop"):
        out["loop.step"] = (int(config["loop"]["times"]), W)
    for i, layer in enumerate(config["layers"]):
        a, r = layer["mixer"]["left"], layer["mixer"]["right"]
        q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
        cqk, n, nv = r["kv_heads"] * r["dim"], r["heads"] * r["dim"], r["heads"] * r["vdim"]
        mix = {"left.q": (q, W), "left.q.b": (q,), "left.k": (k, W), "left.k.b": (k,), "left.v": (v, W), "left.v.b": (v,),
               "left.g": (a["heads"], W), "left.o": (W, a["heads"] * a["vdim"]), "left.out": (W,),
               "right.q": (cqk, W), "right.q.conv": (cqk, r["conv"]), "right.k": (cqk, W), "right.k.conv": (cqk, r["conv"]),
               "right.v": (nv, W), "right.v.conv": (nv, r["conv"]), "right.b": (r["heads"], W), "right.A_log": (r["heads"],),
               "right.norm": (r["vdim"],), "right.a1": (decay_rank, W), "right.a2": (n, decay_rank), "right.dt_bias": (n,),
               "right.g1": (gate_rank, W), "right.g2": (nv, gate_rank), "right.o": (W, nv), "right.out": (W,)}
        out.update({f"l{i}.mix.{name}": shape for name, shape in mix.items()})
        out[f"l{i}.norm1"] = (W,)
        if layer.get("mlp"):
            ff = int(layer["mlp"]["ff"])
            out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.up.b": (ff,), f"l{i}.mlp.down": (W, ff), f"l{i}.mlp.down.b": (W,)})
    return out


def random_state_dict(config: dict, seed: int = 0, decay_rank: int = 5, gate_rank: int = 7) -> Dict[str, torch.Tensor]:
    """weights that are exactly representable in bfloat16, so that every element type starts from the same numbers"""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in tensor_shapes(config, decay_rank, gate_rank).items():
        leaf = name.split(".")[-1]
        if leaf == "conv":
            t = torch.randn(shape, generator=g) * 0.6
        elif leaf == "A_log":
            t = torch.randn(shape, generator=g) * 0.7 - 1.5
        elif leaf == "dt_bias":
            t = torch.randn(shape, generator=g) * 1.5 - 1.0
        elif name == "loop.step":
            t = torch.randn(shape, generator=g) * 0.5
        elif leaf == "b" and len(shape) == 1:
            t = torch.randn(shape, generator=g) * 0.7
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) * (0.7 if name == "embed" else 1.5 / math.sqrt(shape[1]))
        else:  # norm weights
            t = 1.0 + torch.randn(shape, generator=g) * 0.3
        sd[name] = t.to(torch.bfloat16).to(torch.float32)
    return sd
