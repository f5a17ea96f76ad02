"""Nomalorn on the GPU against the slow CPU reference (oracle/nomalorn.py, float64): each mechanism alone, then the model through
the engine's step function and cache manager - whole prompts, token-by-token decoding, portions down to two tokens, ragged
batches, pages and state slots that are freed and used again - and greedy generation through FlashCausalLM.generate_token.

The configurations are small and uneven (key size != value size, other head counts left and right, several key heads and one,
layers of different sizes, loops of one to three passes anywhere in the stack and none, one to eight convolution taps).  Where
random weights would hide a fault the test makes it show: a key that must win the soft-max from just inside the chunk, from just
outside it, at a page border or at position 0; keys written again while the memory still holds their old value; decays that
forget at once on some rows and never on others; recurrent states, pages and convolution inputs filled with garbage before use."""
import math

import pytest
import torch

from oracle import nomalorn as orc
from tests.test_gpu_nasozen import _DictWeights, _feed, _model, _rel, _run_cut, _step, _tokens, _vary

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL32, TOL16 = 1e-4, 0.1


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("W", [44, 37, 1028])
def test_branches_step_every_combination(W):
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(W)
    T, eps = 5, 1e-3
    x0, y1, y2, add = (torch.randn(T, W, generator=g) * s for s in (2.0, 3.0, 0.02, 1.0))
    d = lambda t: None if t is None else t.to(DEV)  # noqa: E731
    for dtype in (torch.float32, torch.bfloat16):
        w1, w2, vec, nw = ((1 + 0.4 * torch.randn(W, generator=g)).to(dtype) for _ in range(4))
        for branches, scale, more, normed, start in (
                ([(y1, w1), (y2, w2)], 0.5, (), True, False), ([(y1, w1), (y2, w2)], 0.5, ("add", "vec"), True, False),
                ([(y1, None)], 1.0, ("vec",), True, False), ([(y1, None), (y2, w2)], -0.3, ("add",), False, False),
                ([], 1.0, ("vec",), True, True), ([], 1.0, (), True, False), ([(y2, w2)], 2.0, (), False, True)):
            want = x0.double()
            for y, w in branches:
                want = want + scale * (y.double() if w is None else orc.unit_rms(y.double(), eps) * w.double())
            if "add" in more:
                want = want + add.double()
            if "vec" in more:
                want = want + vec.double()
            x = torch.full((T, W), float("nan")) if start else x0.clone()      # a started stream never reads what was there
            x = x.to(DEV)
            h = ops.branches_step(x, init=d(x0) if start else None, branches=[(d(y), d(w)) for y, w in branches], y_scale=scale,
                                  add=d(add) if "add" in more else None, step_vec=d(vec) if "vec" in more else None,
                                  norm_w=d(nw) if normed else None, eps=eps, dtype=dtype)
            assert float((x.cpu().double() - want).abs().max()) < 2e-5
            if normed:
                ref = orc.unit_rms(want, eps) * nw.double()
                assert h.dtype == dtype and float((h.cpu().double() - ref).abs().max()) < (2e-5 if dtype == torch.float32 else 0.03)
            else:
                assert h is None


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_squared_relu_mlp_and_plain_copy(dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    from tgis_b200.utils.mixers import PlainMLP
    g = torch.Generator().manual_seed(3)
    wide = torch.randn(9, 50, generator=g) * 2
    ref = torch.clamp(wide[:, 7:30].double(), min=0) ** 2
    assert float((ops.ff_act(wide.to(DEV)[:, 7:30], ops.ACT_RELU2).cpu().double() - ref).abs().max()) < 1e-5
    assert torch.equal(ops.ff_act(wide.to(DEV)[:, 7:30], ops.ACT_NONE, out_dtype=dtype).cpu(), wide[:, 7:30].to(dtype))
    for rows, F in ((3, 64), (70, 1000)):     # whole 16-byte pieces, and sizes that leave a rest
        x = (torch.randn(rows, F, generator=g) * 2).to(dtype)
        want = torch.clamp(x.double(), min=0) ** 2
        err = (ops.ff_act(x.to(DEV), ops.ACT_RELU2).cpu().double() - want).abs()
        assert float((err / (want + 1e-3)).max()) < (1e-6 if dtype == torch.float32 else 0.005)
    for W, ff in ((24, 30), (64, 200)):
        sd = {"m.up": torch.randn(ff, W, generator=g) / math.sqrt(W), "m.up.b": torch.randn(ff, generator=g), "m.down": torch.randn(W, ff, generator=g) / ff,
              "m.down.b": torch.randn(W, generator=g)}
        sd = {k: v.to(torch.bfloat16).float() for k, v in sd.items()}
        h = torch.randn(11, W, generator=g).to(torch.bfloat16).float()
        want = orc.squared_relu_mlp(h.double(), {k[2:]: v.double() for k, v in sd.items()})
        got = PlainMLP("m", _DictWeights(sd, dtype), activation="relu2", bias=True)(h.to(dtype).to(DEV))
        assert got.dtype == torch.float32 and float((got.cpu().double() - want).abs().max()) < (1e-4 if dtype == torch.float32 else 0.05)


def _delta_inputs(g, L, H, G, d, dv, channels, wild=False):
    """conv-free inputs of the memory: u columns, beta and decay logits; `wild`: keys come back, some rows forget at once"""
    u = torch.randn(L, 2 * G * d + H * dv, generator=g)
    raw = torch.randn(L, H + 3, generator=g) * 2
    dec = torch.randn(L, (H * d if channels else H) + 2, generator=g) * 2
    if wild:
        u[1::2, G * d:2 * G * d] = u[0:1, G * d:2 * G * d] * 1.3        # every second token writes at one and the same key
        raw[:, :] = 6.0                                                # ... replacing nearly all of what is there
        dec[:, ::3] = 60.0                                             # rows (or heads) that forget everything
        dec[:, 1::3] = -40.0                                           # and rows that forget nothing
    return u, raw, dec


@pytest.mark.parametrize("H,G,d,dv,channels", [(4, 2, 12, 14, True), (3, 3, 10, 9, True), (2, 1, 72, 80, True), (1, 1, 132, 36, True), (2, 2, 256, 40, True),
                                               (2, 1, 64, 130, True), (3, 3, 64, 64, True), (6, 2, 16, 200, True), (1, 1, 5, 1, True),
                                               (4, 2, 12, 14, False), (2, 1, 128, 128, False), (3, 1, 68, 10, False)])
def test_delta_memory_alone(H, G, d, dv, channels):
    """preparation and memory against the token-by-token recurrence: whole sequences, single rows, ragged groups whose sizes leave one to
    three tokens over, several sequences in one step, garbage in the slots; gentle inputs and wild ones"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(H * 1000 + d + dv)
    n_dec = H * d if channels else H
    A_log, dt_bias = torch.randn(H, generator=g) * 0.5, torch.randn(n_dec, generator=g)
    taps = 3
    conv_w = torch.randn(2 * G * d + H * dv, taps, generator=g) * 0.6
    for wild in (False, True):
        seqs = [_delta_inputs(g, L, H, G, d, dv, channels, wild) for L in (37, 18, 1)]
        want = []
        for u, raw, dec in seqs:
            L = u.shape[0]
            c = orc.silu(orc.short_conv(u.double(), conv_w.double()))
            rep = H // G
            q = (orc.unit_length(c[:, :G * d].view(L, G, d)) * d ** -0.5).repeat_interleave(rep, dim=1)
            k = orc.unit_length(c[:, G * d:2 * G * d].view(L, G, d)).repeat_interleave(rep, dim=1)
            v = c[:, 2 * G * d:].view(L, H, dv)
            gg = torch.exp(-torch.exp(A_log.double())[:, None] * orc.softplus((dec[:, 2:].double() + dt_bias.double()).view(L, H, -1))).expand(L, H, d)
            want.append(orc.delta_memory(q, k, v, torch.sigmoid(raw[:, 3:].double()), gg).reshape(L, H * dv))

        def run(plan):
            """plan: steps, each a list of (sequence, count) -> outputs per sequence"""
            S = torch.full((5, H, d, dv), float("nan"), device=DEV)
            cs = torch.full((5, taps - 1, 2 * G * d + H * dv), float("nan"), device=DEV)
            slot = {0: 3, 1: 0, 2: 4}
            at, out = {0: 0, 1: 0, 2: 0}, {0: [], 1: [], 2: []}
            for entries in plan:
                st = _step([(at[i], n) for i, n in entries], [[0] * 3 for _ in entries], slots=[slot[i] for i, _ in entries])
                parts = [[t[at[i]:at[i] + n] for t in seqs[i]] for i, n in entries]
                u, raw, dec = (torch.cat([p[j] for p in parts]).to(DEV) for j in range(3))
                rows = ops.delta_prepare(u, 0, conv_w.t().contiguous().to(DEV), cs, raw, 3, dec, 2, A_log.to(DEV), dt_bias.to(DEV), d ** -0.5, st, H, G, d, dv, channels)
                y = ops.delta_rows_scan(rows, S, st, H, G, d, dv, channels)
                o = 0
                for i, n in entries:
                    out[i].append(y[o:o + n].cpu().double())
                    o, at[i] = o + n, at[i] + n
            return [torch.cat(out[i]) for i in range(3)]

        plans = {
            "whole": [[(0, 37), (1, 18), (2, 1)]],
            "single rows": [[(0, 1), (1, 1)]] * 18 + [[(2, 1), (0, 1)]] + [[(0, 1)]] * 18,
            "ragged": [[(0, 2)], [(0, 5), (1, 1)], [(0, 16), (2, 1), (1, 2)], [(1, 15), (0, 1)], [(0, 2)], [(0, 11)]],
            "pairs and threes": [[(0, 2), (1, 2)], [(0, 2)], [(0, 3), (1, 3)], [(1, 13), (0, 13)], [(0, 17), (2, 1)]],
        }
        for name, plan in plans.items():
            for i, got in enumerate(run(plan)):
                assert float((got - want[i]).abs().max()) < 2e-5 * max(1.0, float(want[i].abs().max())), (wild, name, i)


@pytest.mark.parametrize("taps", [1, 2, 4, 8])
def test_delta_convolution_inputs_across_steps(taps):
    """the first tokens of a sequence, steps shorter than the taps, one row per sequence (the launch that also moves the state on)
    beside many: the prepared rows equal the whole sequence's, and the state holds the last taps - 1 inputs"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(taps)
    H, G, d, dv, L = 2, 1, 7, 5, 30
    C = 2 * G * d + H * dv
    u, raw, dec = _delta_inputs(g, L, H, G, d, dv, True)
    conv_w, A_log, dt = torch.randn(C, taps, generator=g), torch.randn(H, generator=g), torch.randn(H * d, generator=g)
    c = orc.silu(orc.short_conv(u.double(), conv_w.double()))
    want_q = orc.unit_length(c[:, :G * d]) * d ** -0.5
    want_k, want_v = orc.unit_length(c[:, G * d:2 * G * d]), c[:, 2 * G * d:]
    want_g = torch.exp(-torch.exp(A_log.double())[:, None] * orc.softplus((dec[:, 2:].double() + dt.double()).view(L, H, d))).reshape(L, H * d)
    want = torch.cat([want_q, want_k, want_v, want_g, torch.sigmoid(raw[:, 3:].double())], 1)
    for cuts in ([L], [1] * L, [2, 1, 3, 1, 1, 9, 2, 11], [1, 29]):
        cs = torch.full((3, max(taps - 1, 1), C), float("nan"), device=DEV)
        at, got = 0, []
        for n in cuts:
            st = _step([(at, n)], [[0] * 2], slots=[1])
            got.append(ops.delta_prepare(u[at:at + n].to(DEV), 0, conv_w.t().contiguous().to(DEV), cs, raw[at:at + n].to(DEV), 3, dec[at:at + n].to(DEV), 2, A_log.to(DEV),
                                         dt.to(DEV), d ** -0.5, st, H, G, d, dv, True).cpu().double())
            at += n
        got = torch.cat(got)[:, :want.shape[1]]
        assert float((got - want).abs().max()) < 2e-5, cuts
        if taps > 1:
            assert torch.equal(cs[1].cpu(), u[L - taps + 1:])
        assert torch.isnan(cs[0]).all() and torch.isnan(cs[2]).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,conv,ranks", [(4, 2, 12, 14, 3, (5, 7)), (2, 2, 48, 32, 4, (20, 8)), (3, 1, 20, 70, 1, (60, 13)), (1, 1, 8, 6, 2, (1, 2))])
def test_channel_delta_mixer_any_cut(H, G, d, dv, conv, ranks, dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200.utils.mixers import ChannelDeltaMixer
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "conv": conv}
    cfg = orc.random_config(layers=1, loop=None, width=64, r_heads=H, r_kv_heads=G, r_dim=d, r_vdim=dv, conv=conv)
    sd = {k[13:]: v for k, v in orc.random_state_dict(cfg, seed=d, decay_rank=ranks[0], gate_rank=ranks[1]).items() if k.startswith("l0.mix.right.")}
    g = torch.Generator().manual_seed(1)
    L, eps = 45, 1e-5
    h = torch.randn(L, 64, generator=g).to(torch.bfloat16).float()
    ref = orc.channel_delta(h.double(), {k: v.double() for k, v in sd.items()}, m, eps)
    mixer = ChannelDeltaMixer("m", _DictWeights({"m." + k: v for k, v in sd.items()}, dtype), heads=H, kv_heads=G, dim=d, vdim=dv, conv=conv, eps=eps)
    tol = 1e-4 if dtype == torch.float32 else 0.06
    for cuts in ([L], [], [2, 2, 30, 3], [1, 43], [7, 9, 2]):
        got = _feed(mixer, mixer.cache_spec(), h, cuts, dtype)
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max()), cuts


def test_delta_memory_long_run():
    """300 single steps against the recurrence: the memory does not drift from the form that prompts take"""
    import tgis_b200  # noqa: F401
    from tgis_b200.utils.mixers import ChannelDeltaMixer
    cfg = orc.random_config(layers=1, loop=None, width=24)
    m = cfg["layers"][0]["mixer"]["right"]
    sd = {k[13:]: v for k, v in orc.random_state_dict(cfg, seed=5).items() if k.startswith("l0.mix.right.")}
    sd["A_log"] = (sd["A_log"] - 4.0).to(torch.bfloat16).float()     # long memory
    h = torch.randn(300, 24, generator=torch.Generator().manual_seed(2)).to(torch.bfloat16).float()
    ref = orc.channel_delta(h.double(), {k: v.double() for k, v in sd.items()}, m, 1e-5)
    mixer = ChannelDeltaMixer("m", _DictWeights({"m." + k: v for k, v in sd.items()}, torch.float32), heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"],
                              vdim=m["vdim"], conv=m["conv"], eps=1e-5)
    for cuts in ([], [150, 150], [299]):
        assert float((_feed(mixer, mixer.cache_spec(), h, cuts, torch.float32) - ref).abs().max()) < 1e-4 * float(ref.abs().max()), cuts


ATTENTION_CASES = [  # heads, kv heads, dim, vdim, rotated columns, chunk
    (6, 2, 10, 12, 6, 20),        # the plain kernel: sizes that are no multiples of 16
    (4, 4, 16, 48, 16, 37),       # as many key heads as heads, full rotation
    (8, 1, 32, 96, 8, 16),        # one key head, a chunk of exactly one page
    (16, 4, 16, 112, 0, 50),      # no rotation
    (8, 2, 48, 80, 2, 0),         # no chunks
    (3, 1, 8, 8, 4, 5),           # a chunk shorter than a page
    (4, 2, 64, 128, 32, 64),
    (2, 1, 16, 144, 16, 24),      # a value size beyond the tensor-core kernel
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,rot,chunk", ATTENTION_CASES)
def test_attention_half_any_cut(H, G, d, dv, rot, chunk, dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200.utils.mixers import ScaledRotaryTables, SinkRotaryAttention
    cfg = orc.random_config(layers=1, loop=None, width=32, heads=H, kv_heads=G, dim=d, vdim=dv, rot_dims=rot or None, chunk=chunk or None, sharp=1.5)
    m = cfg["layers"][0]["mixer"]["left"]
    sd = {k[12:]: v for k, v in orc.random_state_dict(cfg, seed=dv).items() if k.startswith("l0.mix.left.")}
    L = 70
    h = torch.randn(L, 32, generator=torch.Generator().manual_seed(3)).to(torch.bfloat16).float()
    ref = orc.chunk_attention(h.double(), {k: v.double() for k, v in sd.items()}, m)
    mixer = SinkRotaryAttention("a", _DictWeights({"a." + k: v for k, v in sd.items()}, dtype), heads=H, kv_heads=G, dim=d, vdim=dv, scale=m["scale"],
                                rotary=ScaledRotaryTables(rot, m["rot"]["base"]) if rot else None, value_rotary=None, chunk=chunk or None, sink=False,
                                qk_norm=False, bias=True)
    tol = 1e-4 if dtype == torch.float32 else 0.08
    for cuts in ([L], [], [2, 33, 2, 31], [16, 16, 16, 16], [1, 20, 47]):
        got = _feed(mixer, mixer.cache_spec(), h, cuts, dtype)
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max()), cuts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,chunk", [(6, 3, 10, 14, 100), (6, 2, 16, 80, 70), (8, 2, 32, 48, 33), (16, 4, 16, 96, 150), (2, 2, 64, 112, 17)])
def test_loud_keys_at_chunk_edges(dtype, H, G, d, dv, chunk):
    """One key is made to win the soft-max of every head: the output must be that key's value when the key is the chunk's first
    position, at a page border or the query itself, and must not move when the key is the last position of the chunk before - for a
    decoded token and for a row inside a portion that crosses the border."""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(chunk)
    L = 420
    edge = (300 // chunk) * chunk
    cases = [(edge + min(chunk - 1, L - 1 - edge), edge, True), (edge, edge, True), (edge, edge - 1, False), (edge + min(5, chunk - 1), edge - 1, False),
             (edge - 1, edge - chunk, True), (edge - 1, edge - chunk - 1, False), (chunk - 1, 0, True), (chunk, 0, False), (0, 0, True),
             (L - 1, L - 1, True), (edge - 1, (edge - 1) // 16 * 16, (edge - 1) // 16 * 16 >= edge - chunk)]
    cases = [c for c in cases if 0 <= c[1] <= c[0] < L]
    blocks = (L + 15) // 16
    table = [(7 * i + 1) % (blocks + 3) for i in range(blocks)]
    assert len(set(table)) == blocks
    RW = G * d + G * dv
    for qpos, kpos, inside in cases:
        q, k, v = torch.randn(L, H, d, generator=g) * 0.3, torch.randn(L, G, d, generator=g) * 0.3, torch.randn(L, G, dv, generator=g)
        direction = torch.nn.functional.normalize(torch.randn(d, generator=g), dim=0)
        q[qpos] = direction * 9.0
        k[kpos] = direction * 9.0
        pool = torch.full((blocks + 3, 16, RW), float("nan"), dtype=dtype, device=DEV)
        rows = torch.tensor([table[p // 16] * 16 + p % 16 for p in range(L)], device=DEV)
        pool.view(-1, RW)[rows] = torch.cat([k.reshape(L, -1), v.reshape(L, -1)], 1).to(dtype).to(DEV)
        for start, n in ((qpos, 1), (max(qpos - 40, 0), min(41, qpos + 1) + (3 if qpos + 3 < L else 0))):
            st = _step([(start, n)], [table])
            got = ops.talk_attn(q[start:start + n].contiguous().to(DEV), pool, st, kv_heads=G, vdim=dv, k_off=0, v_off=G * d, scale=1.0,
                                chunk=chunk)[qpos - start].cpu()
            vv = v.to(dtype).float()
            loud = vv[kpos].repeat_interleave(H // G, dim=0)
            if inside:
                assert float((got - loud).abs().max()) < 1e-3, (qpos, kpos, n)
            else:
                lo = (qpos // chunk) * chunk
                s = torch.einsum("hd,jhd->hj", q[qpos].double(), k[lo:qpos + 1].to(dtype).double().repeat_interleave(H // G, dim=1))
                ref = torch.einsum("hj,jhv->hv", torch.softmax(s, 1), vv[lo:qpos + 1].double().repeat_interleave(H // G, dim=1))
                assert float((got.double() - ref).abs().max()) < (1e-4 if dtype == torch.float32 else 0.03), (qpos, kpos, n)
                assert float((got - loud).abs().max()) > 0.3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_normed_parallel_mixer(dtype):
    """both halves of one layer over a shared input product: their results with the norm weights, joined by the stream's launch"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    from tgis_b200.models.custom_modeling.nomalorn_modeling import build_mixer
    cfg = orc.random_config(layers=1, loop=None, width=64, sharp=1.5)
    layer, eps = cfg["layers"][0], 1e-5
    sd = {k: v for k, v in orc.random_state_dict(cfg, seed=9).items() if k.startswith("l0.mix.")}
    sd["l0.mix.left.o"] = sd["l0.mix.left.o"] * 30.0             # the norms take the halves' sizes away: a scaled output product changes nothing
    L = 50
    h = torch.randn(L, 64, generator=torch.Generator().manual_seed(4)).to(torch.bfloat16).float()
    ref = orc.parallel_mixer(h.double(), {k[7:]: v.double() for k, v in sd.items()}, layer["mixer"], eps)
    mixer = build_mixer("parallel", "l0.mix", layer["mixer"], _DictWeights(sd, dtype), eps)

    def joined(*args):
        out = mixer(*args)
        x = torch.zeros(args[0].shape[0], 64, device=DEV)
        ops.branches_step(x, branches=out, y_scale=mixer.out_scale, eps=eps)
        return x
    tol = 1e-4 if dtype == torch.float32 else 0.06
    for cuts in ([L], [], [2, 33, 2]):
        got = _feed(joined, mixer.cache_spec(), h, cuts, dtype)
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max()), cuts


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_prompt_portions_and_decoding_agree_with_reference(tmp_path, dtype):
    cfg = orc.random_config(sharp=3.0, chunk=24)
    sd = orc.random_state_dict(cfg, seed=2)
    model = _model(tmp_path, cfg, sd, dtype)
    toks = _tokens(1, 90, cfg["vocab"])
    ref = orc.forward(cfg, sd, toks)
    tol = TOL32 if dtype == torch.float32 else TOL16
    whole = _run_cut(model, toks, [len(toks)])
    assert _rel(whole, ref) < tol
    if dtype == torch.float32:
        # what the configuration and the tensors say is live in this test: each of these, when wrong, is far outside the tolerance
        def changed(fn):
            c2, s2 = _vary(cfg, sd, fn)
            return _rel(orc.forward(c2, s2, toks), ref)
        left = lambda c, i=0: c["layers"][i]["mixer"]["left"]  # noqa: E731
        scaled = lambda name, f: (lambda c, s: s.update({name: s[name] * f}))  # noqa: E731
        # one part of a weight only: a common factor would vanish in the norm behind it
        halved = lambda name, f: (lambda c, s: s.update({name: torch.cat([s[name][:4] * f, s[name][4:]])}))  # noqa: E731
        for fn in (lambda c, s: left(c)["mask"].update(size=25), lambda c, s: left(c)["mask"].update(size=23), lambda c, s: left(c)["rot"].update(dims=4),
                   lambda c, s: left(c)["rot"].update(base=90.0), lambda c, s: left(c).update(scale=left(c)["scale"] * 1.05),
                   scaled("l0.mix.left.g", 0.5), scaled("l1.mix.left.q.b", 0.0), scaled("l1.mix.left.k.b", 0.0), scaled("l0.mix.left.v.b", 0.0),
                   scaled("l2.mix.left.out", 1.1), scaled("l2.mix.right.out", 1.1), halved("l0.mix.right.norm", 1.1), scaled("l0.mix.right.A_log", 0.8),
                   scaled("l1.mix.right.dt_bias", 0.8), scaled("l1.mix.right.a2", 0.8), scaled("l1.mix.right.g2", 0.8), scaled("l0.mix.right.b", 0.8),
                   lambda c, s: s.update({"l0.mix.right.k.conv": s["l0.mix.right.k.conv"].flip(1)}),
                   scaled("l0.mlp.up.b", 0.9), scaled("l0.mlp.down.b", 0.9), scaled("loop.step", 0.9),
                   lambda c, s: s.update({"loop.step": s["loop.step"].flip(0)}), lambda c, s: c["loop"].update(stop=2),
                   lambda c, s: (c["loop"].update(times=3), s.update({"loop.step": torch.cat([s["loop.step"], s["loop.step"][:1]])}))):
            assert changed(fn) > 20 * TOL32
    for cuts in ([], [40], [2, 2, 2, 19, 3, 16, 17, 2], [16, 16, 16, 16], [24, 24, 24], [23, 2, 23, 2], [1, 25, 22, 31]):
        got = _run_cut(model, toks, cuts)
        assert _rel(got, ref) < tol, cuts
        if dtype == torch.float32:
            assert _rel(got, whole.cpu()) < 1e-5, cuts  # the cut itself changes nothing beyond rounding
    assert model.kv_cache_manager.free_blocks == model.kv_cache_manager.total_num_gpu_blocks
    assert model.kv_cache_manager.free_state_slots == 4


def test_tensor_core_shapes_through_the_engine(tmp_path):
    """bfloat16 with head sizes in 16s: prompts, portions and decoded tokens take the tensor-core attention kernel and the
    tensor-core products; a step mixes a long portion (several query tiles) with single tokens"""
    cfg = orc.random_config(width=64, layers=2, loop=(0, 2, 2), heads=8, kv_heads=2, dim=32, vdim=80, rot_dims=16, chunk=60, sharp=2.0, r_heads=4, r_kv_heads=4,
                            r_dim=32, r_vdim=48, conv=4, ff=128)
    sd = orc.random_state_dict(cfg, seed=12, decay_rank=40, gate_rank=24)
    model = _model(tmp_path, cfg, sd, torch.bfloat16)
    toks, other = _tokens(3, 150, cfg["vocab"]), _tokens(4, 90, cfg["vocab"])
    ref, ref_o = orc.forward(cfg, sd, toks), orc.forward(cfg, sd, other)
    for cuts in ([150], [100, 2, 40], [1, 70, 33], [5]):
        assert _rel(_run_cut(model, toks, cuts), ref) < TOL16, cuts
    (a,), la = model.step_ragged([None], [toks[:20]])
    (a, b), l2 = model.step_ragged([a, None], [toks[20:21], other[:80]])
    (b, a), l3 = model.step_ragged([b, a], [other[80:], toks[21:150]])
    model.kv_cache_manager.free_sequences([a, b])
    assert _rel(torch.cat([la, l2[:1], l3[10:]]), ref) < TOL16
    assert _rel(torch.cat([l2[1:], l3[:10]]), ref_o) < TOL16


def test_stream_after_every_layer_run(tmp_path):
    """the stream as a layer leaves it: what the loop adds ahead of the next pass is not in it yet"""
    cfg = orc.random_config(loop=(1, 3, 3))
    sd = orc.random_state_dict(cfg, seed=4)
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(5, 30, cfg["vocab"])
    want = []
    ref = orc.forward(cfg, sd, toks, residuals=want)
    probe = []
    model.model.model.residual_probe = probe
    sids, lg = model.step_ragged([None], [toks])
    model.model.model.residual_probe = None
    model.kv_cache_manager.free_sequences(sids)
    assert len(probe) == len(want) == 7 and _rel(lg, ref) < TOL32
    for i, (a, b) in enumerate(zip(probe, want)):
        assert float((a.cpu().double() - b).abs().max()) < 1e-4 * float(b.abs().max()), i


OTHER_SIZES = {
    "no_loop_one_key_head": dict(loop=None, heads=5, kv_heads=1, r_heads=3, r_kv_heads=1, conv=2),
    "one_pass_equal_heads": dict(loop=(0, 3, 1), heads=4, kv_heads=4, dim=14, vdim=14, rot_dims=14, r_heads=4, r_kv_heads=4, r_dim=14, r_vdim=14, chunk=2),
    "loop_at_the_end": dict(loop=(2, 3, 3), width=56, chunk=31, conv=1, r_dim=70, r_vdim=5, r_heads=1, r_kv_heads=1, mlp=(None, "dense", "dense")),
    "loop_of_everything": dict(loop=(0, 2, 3), layers=2, heads=1, kv_heads=1, rot_dims=2, chunk=33, mlp=("dense", None), conv=8),
    "no_rotation_no_chunks": dict(rot_dims=None, chunk=None, layers=2, loop=(1, 2, 2), mlp=(None,), vdim=20),
    "layers_unlike_each_other": dict(other={1: {"left": {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 16, "scale": 1.1, "mask": {"size": 7},
                                                           "rot": {"base": 10.0, "dims": 4}},
                                                  "right": {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 10, "conv": 5}}}, loop=(0, 2, 2), eps=1e-3),
    "an_empty_loop": dict(loop=(1, 1, 4)),
}


@pytest.mark.parametrize("variant", sorted(OTHER_SIZES))
def test_other_sizes(tmp_path, variant):
    """sizes that a usual configuration makes equal or 1, and entries it may leave out"""
    cfg = orc.random_config(**{"sharp": 3.0, **OTHER_SIZES[variant]})
    sd = orc.random_state_dict(cfg, seed=31, decay_rank=3, gate_rank=9)
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(6, 60, cfg["vocab"])
    ref = orc.forward(cfg, sd, toks)
    for cuts in ([60], [3, 30, 2], [17]):
        assert _rel(_run_cut(model, toks, cuts), ref) < TOL32, (variant, cuts)


def test_ragged_batches_reused_pages_and_slots(tmp_path):
    """four requests of unequal length run as mixed steps (portions beside decoded tokens, requests joining and leaving) in a pool
    that is too small for all of them at once and is filled with garbage first: every request equals its run alone"""
    cfg = orc.random_config(sharp=3.0)
    sd = orc.random_state_dict(cfg, seed=21)
    model = _model(tmp_path, cfg, sd, torch.float32, blocks=12, slots=2)
    mgr = model.kv_cache_manager
    assert len(mgr.pages) == 5   # one store per layer run
    for p in mgr.pages:
        p.fill_(float("nan"))
    for st in mgr.states:
        for t in st.values():
            t.fill_(float("nan"))
    lens = {"a": 70, "b": 33, "c": 1, "d": 50}
    toks = {k: _tokens(30 + i, n, cfg["vocab"]) for i, (k, n) in enumerate(lens.items())}
    refs = {k: orc.forward(cfg, sd, v) for k, v in toks.items()}
    plan = [[("a", 20), ("b", 2)], [("a", 1), ("b", 31)], [("a", 30)], [("a", 1)], [("a", 18), ("c", 1)],   # b ends at step 1, a at 4
            [("d", 17)], [("d", 2)], [("d", 1)], [("d", 30)]]
    got, at, live = {k: [] for k in lens}, {k: 0 for k in lens}, {}
    for step in plan:
        sids, lg = model.step_ragged([live.get(k) for k, _ in step], [toks[k][at[k]:at[k] + n] for k, n in step])
        o = 0
        for (k, n), sid in zip(step, sids):
            live[k] = sid
            got[k].append(lg[o:o + n])
            o += n
            at[k] += n
            if at[k] == lens[k]:
                mgr.free_sequences([live.pop(k)])
        assert len(live) <= 2
    for k in lens:
        assert at[k] == lens[k]
        assert _rel(torch.cat(got[k]), refs[k]) < TOL32, k
    assert mgr.free_blocks == mgr.total_num_gpu_blocks and mgr.free_state_slots == 2


def test_long_decoding_and_first_tokens(tmp_path):
    """three prompt tokens, then 197 single steps: chunks begin and end among decoded tokens only; the first tokens have fewer
    inputs than taps"""
    cfg = orc.random_config(sharp=3.0, chunk=40, conv=4)
    sd = orc.random_state_dict(cfg, seed=8)
    for i in range(3):
        sd[f"l{i}.mix.right.A_log"] = (sd[f"l{i}.mix.right.A_log"] - 3.0).to(torch.bfloat16).float()   # the memory reaches back over the chunks
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(9, 200, cfg["vocab"])
    ref = orc.forward(cfg, sd, toks)
    c2, _ = _vary(cfg, sd, lambda c, s: [layer["mixer"]["left"]["mask"].update(size=41) for layer in c["layers"]])
    assert _rel(orc.forward(c2, sd, toks)[45:], ref[45:]) > 20 * TOL32          # the chunk's edge is live
    swapped = list(toks)
    swapped[3] = toks[3] % (cfg["vocab"] - 5) + 5
    assert swapped[3] != toks[3] and _rel(orc.forward(cfg, sd, swapped)[180:], ref[180:]) > 20 * TOL32   # and so is a token far back
    got = _run_cut(model, toks, [3])
    assert _rel(got[:8], ref[:8]) < TOL32
    assert _rel(got, ref) < TOL32
    one = _run_cut(model, toks[:1], [1])  # a request of a single token
    assert _rel(one, ref[:1]) < TOL32


def test_greedy_generation_through_generate_token(tmp_path):
    """from_pb -> generate_token (prefill, decode steps, a second batch joined by concatenate, prune of a finished request):
    the engine's own scheduler path picks the reference's greedy tokens wherever the reference's top-2 gap is decisive"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import pb
    cfg = orc.random_config()
    sd = orc.random_state_dict(cfg, seed=13)
    model = _model(tmp_path, cfg, sd, torch.float32, blocks=64, slots=6)
    tok, V = model.tokenizer, cfg["vocab"]

    def batch_of(bid, prompts, n_new, first_id):
        text = lambda ids: " ".join("test" if i == 3 else f"<tok{i}>" for i in ids)  # noqa: E731
        reqs = [pb.Request(id=first_id + i, inputs=text(p), input_length=len(p), truncate=False, max_output_length=n_new,
                           parameters=pb.NextTokenChooserParameters(temperature=0.0, top_p=1.0, min_new_tokens=n_new))
                for i, p in enumerate(prompts)]
        return pb.Batch(id=bid, requests=reqs)

    def oracle_greedy(prompt, n_new):
        seq, out, sure = list(prompt), [], n_new
        for s in range(n_new):
            lg = orc.forward(cfg, sd, seq)[-1]
            lg[2] = float("-inf")  # min_new_tokens bans EOS
            top = lg.topk(2).values
            if float(top[0] - top[1]) < 1e-3 * float(lg[torch.isfinite(lg)].std()):
                sure = min(sure, s)
            out.append(int(lg.argmax()))
            seq.append(out[-1])
        return out, sure

    n_new = 7
    p1, p2 = [_tokens(40, 9, V), _tokens(41, 23, V)], [_tokens(42, 5, V)]
    got = {0: [], 1: [], 2: []}
    with torch.inference_mode():
        b1, errs = model.batch_type.from_pb(batch_of(0, p1, n_new, 0), tok, model.dtype, model.device, None, None, True)
        assert not errs
        for t in model.generate_token(b1, first=True)[0]:
            got[t.request_id].append(t.token_id)
        for _ in range(2):
            for t in model.generate_token(b1)[0]:
                got[t.request_id].append(t.token_id)
        b2, errs = model.batch_type.from_pb(batch_of(1, p2, n_new, 2), tok, model.dtype, model.device, None, None, True)
        assert not errs
        for t in model.generate_token(b2, first=True, for_concat=True)[0]:
            got[t.request_id].append(t.token_id)
        both = model.batch_type.concatenate([b1, b2])
        for _ in range(n_new - 3):
            for t in model.generate_token(both)[0]:
                got[t.request_id].append(t.token_id)
        assert len(got[0]) == n_new and len(got[1]) == n_new
        rest = model.batch_type.prune(both, [0, 1])
        assert len(rest) == 1
        while len(got[2]) < n_new:
            for t in model.generate_token(rest)[0]:
                got[t.request_id].append(t.token_id)
        model.kv_cache_manager.free_sequences(rest.sequence_ids)
    sure_total = 0
    for rid, prompt in enumerate(p1 + p2):
        ref, sure = oracle_greedy(prompt, n_new)
        assert got[rid][:sure] == ref[:sure], (rid, got[rid], ref)
        sure_total += sure
    assert sure_total >= 12
    mgr = model.kv_cache_manager
    assert mgr.free_blocks == mgr.total_num_gpu_blocks and mgr.free_state_slots == 6


def test_replayed_trace_writes_the_reference_logits(tmp_path):
    """bin/trace_run as a user calls it, in both element types: portions and single tokens of two requests, one admitted after the other
    ended, in a pool for one of them"""
    import json
    import os
    import subprocess
    import sys
    from safetensors.torch import save_file
    cfg = orc.random_config(width=48, heads=4)
    sd = orc.random_state_dict(cfg, seed=3)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in sd.items()}, str(tmp_path / "model.safetensors"))
    a, b = _tokens(1, 40, cfg["vocab"]), _tokens(2, 25, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:21], "want": [0, 20]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[21:38], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[38:39], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[39:], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
             {"step": 5, "entries": [{"id": "b", "tokens": b[2:], "want": [22]}], "end": ["b"]}]
    ra, rb = orc.forward(cfg, sd, a), orc.forward(cfg, sd, b)
    want = {0: ra[[0, 20]], 2: ra[38:39], 3: ra[39:], 4: rb[1:2], 5: rb[24:]}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, tol in (("bfloat16", TOL16), ("float32", TOL32)):
        out = tmp_path / dtype
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(6)]
        assert sorted(os.listdir(out)) == sorted(f"{i}.f32" for i in want)
        for i, ref in want.items():
            got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
            assert _rel(got, ref) < tol, (dtype, i)
