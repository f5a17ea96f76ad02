"""Tibopel on the GPU against the slow CPU reference (oracle/tibopel.py, float64): each mechanism alone, then the model through the
engine's step function and cache manager - whole prompts, token-by-token decoding, portions down to two tokens, ragged batches,
pages that are freed and used again - and greedy generation through FlashCausalLM.generate_token.

The configurations are small and uneven (key size != value size, other head counts in the two mixers, one key head and several, ranks
that do and do not suit the tensor cores, layers unlike each other, no and several identity outputs, with and without a shared expert).
Where random weights would hide a fault the test makes it show: a key that must win the soft-max from just inside the chunk, from just
outside it, at a page border or hundreds of tokens back; sinks that take nearly all weight or none; picks that only the correction
decides, picks of identity outputs only; pages filled with garbage before use."""
import math

import pytest
import torch

from oracle import tibopel as orc
from tests.test_gpu_nasozen import _DictWeights, _feed, _model, _rel, _run_cut, _step, _tokens, _vary

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL32, TOL16 = 1e-4, 0.1


def _fixed_picks(cfg, sd, seed=0):
    """corrections far apart: every token of a layer has the same picks, so that a bfloat16 run cannot pick other experts than the reference"""
    g = torch.Generator().manual_seed(seed)
    for name, t in sd.items():
        if name.endswith(".correction"):
            sd[name] = torch.randperm(t.numel(), generator=g).float() * 4.0
    return sd


# ------------------------------------------------------------------------------------------------ mechanisms alone
def test_wavelength_scaled_rotary_tables():
    import tgis_b200  # noqa: F401
    from tgis_b200.utils.mixers import ScaledRotaryTables
    for dims, base, sc in ((16, 5000.0, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60}), (64, 1e5, {"factor": 32.0, "low": 2.0, "high": 8.0, "original": 1024}),
                           (6, 30.0, {"factor": 2.5, "low": 0.5, "high": 40.0, "original": 100}), (2, 10.0, None)):
        rates = torch.tensor(orc.turn_rates(dims, base, sc), dtype=torch.float64)
        plain = torch.tensor(orc.turn_rates(dims, base), dtype=torch.float64)
        if sc:   # kept, blended and slowed pairs
            kept, slowed = int((rates == plain).sum()), int((rates == plain / sc["factor"]).sum())
            assert dims < 16 or (kept >= 1 and slowed >= 1 and kept + slowed < dims // 2)
        cos, sin = ScaledRotaryTables(dims, base, sc).tables(700, DEV)
        ang = torch.arange(700, dtype=torch.float64)[:, None] * rates
        assert float((cos[:700].cpu().double() - torch.cos(ang)).abs().max()) < 1e-6 and float((sin[:700].cpu().double() - torch.sin(ang)).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_interleaved_rotation_into_the_cache(dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    from tgis_b200.utils.mixers import ScaledRotaryTables
    g = torch.Generator().manual_seed(1)
    H, G, d, dv, rot, base = 6, 2, 10, 7, 6, 40.0
    u = torch.randn(9, H * d + G * d + G * dv + 5, generator=g)
    pos = torch.tensor([0, 1, 2, 3, 40, 41, 7, 300, 5])
    st = _step([(0, 4), (40, 2), (7, 1), (300, 1), (5, 1)], [[1, 3], [5, 2, 9], [4], list(range(30, 50)), [8]])
    rates = orc.turn_rates(rot, base)
    q_ref = orc.rotate_neighbours(u[:, 5:5 + H * d].double().view(9, H, d), pos, rates)
    k_ref = orc.rotate_neighbours(u[:, 5 + H * d:5 + (H + G) * d].double().view(9, G, d), pos, rates).reshape(9, -1)
    cos, sin = ScaledRotaryTables(rot, base).tables(400, DEV)
    pages = torch.full((50, 16, G * (d + dv)), float("nan"), dtype=dtype, device=DEV)
    q = ops.qk_rot_prepare(u.to(DEV), col_q=5, col_k=5 + H * d, col_v=5 + (H + G) * d, heads=H, kv_heads=G, dim=d, vdim=dv, q_norm_w=None, k_norm_w=None,
                           whole_norm=False, eps=0.0, cos=cos, sin=sin, rot=rot, step=st, cache=pages, k_off=0, v_off=G * d, interleaved=True)
    assert float((q.cpu().double() - q_ref).abs().max()) < 1e-5
    rows = pages.view(-1, G * (d + dv))[st.slot_mapping].cpu().double()
    tol = 1e-5 if dtype == torch.float32 else 0.03
    assert float((rows[:, :G * d] - k_ref).abs().max()) < tol and float((rows[:, G * d:] - u[:, 5 + (H + G) * d:].double()).abs().max()) < tol
    assert int(torch.isnan(pages).all(-1).sum()) == 50 * 16 - 9


@pytest.mark.parametrize("W", [44, 37, 1028])
def test_halves_step_every_combination(W):
    """mixer, gated second addend, picked rows, passed rows, both norms - together and each alone; a started stream never reads x"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(W)
    T, eps, E, ident, top = 70, 1e-3, 5, 2, 3
    z = torch.randn(T, E + ident + 1, generator=g) * 2
    x0, y1, y2 = (torch.randn(T, W, generator=g) * s for s in (2.0, 1.0, 3.0))
    rows = torch.randn(T * top, W, generator=g)
    d = lambda t: None if t is None else t.to(DEV)  # noqa: E731
    for dtype in (torch.float32, torch.bfloat16):
        na, nb = ((1 + 0.4 * torch.randn(W, generator=g)).to(dtype) for _ in range(2))
        h = torch.randn(T, W, generator=g).to(dtype)
        for n in (T, 3):   # a step of many tokens and of few: two forms of the routing
            zd = d(z[:n])
            r = ops.moe_route(zd[:, :E + ident], top, softmax_scores=True, identity=ident)
            ids, wts = orc.pick_experts(torch.softmax(z[:n, :E + ident].double(), -1), torch.zeros(E + ident), top)
            # a token's place among the rows of its expert is free: read it back
            lib_rows = _row_of(r)
            routed = torch.zeros(n, W, dtype=torch.float64)
            for t in range(n):
                for k in range(top):
                    j = ids[t].tolist().index(int(r.ids[t, k]))
                    src = rows[lib_rows[t][k]].double() if int(r.ids[t, k]) < E else h[t].double()
                    routed[t] += wts[t, j] * src
            for use_y1, use_y2, gated, picks, norms, start in ((1, 1, 1, 1, "ab", 0), (1, 0, 0, 0, "a", 0), (0, 1, 0, 0, "b", 1), (1, 1, 1, 1, "", 1), (0, 0, 0, 1, "ab", 0),
                                                             (0, 0, 0, 0, "ab", 1)):
                want = x0[:n].double()
                want = want + y1[:n].double() if use_y1 else want
                if use_y2:
                    want = want + y2[:n].double() * (torch.sigmoid(z[:n, -1:].double()) if gated else 1.0)
                want = want + routed if picks else want
                x = d(torch.full((n, W), float("nan")) if start else x0[:n].clone())
                a, b = ops.halves_step(x, init=d(x0[:n]).contiguous() if start else None, y1=d(y1[:n]) if use_y1 else None, y2=d(y2[:n]) if use_y2 else None,
                                       gate=zd[:, -1] if gated else None, rows=d(rows[:n * top]) if picks else None, routing=r if picks else None,
                                       passed=d(h[:n]) if picks else None, norm_a=d(na) if "a" in norms else None, norm_b=d(nb) if "b" in norms else None,
                                       eps=eps, dtype=dtype)
                assert float((x.cpu().double() - want).abs().max()) < 3e-5
                for out, w in ((a, na if "a" in norms else None), (b, nb if "b" in norms else None)):
                    assert (out is None) == (w is None)
                    if w is not None:
                        ref = orc.unit_rms(want, eps) * w.double()
                        assert out.dtype == dtype and float((out.cpu().double() - ref).abs().max()) < (2e-5 if dtype == torch.float32 else 0.04)


def _row_of(r):
    """the plan's row of every pick, from its expert-ordered token list (what the library's row_of must say)"""
    import ctypes
    from tgis_b200 import _lib
    p = _lib.load_seq().b200_seq_moe_row_of(r.plan.data_ptr(), r.T, r.experts, r.top)
    at = (p - r.plan.data_ptr()) // ctypes.sizeof(ctypes.c_int32)
    return r.plan[at:at + r.T * r.top].view(r.T, r.top).tolist()


@pytest.mark.parametrize("T", [1, 9, 64, 65, 300])
@pytest.mark.parametrize("E,ident,top", [(5, 2, 3), (1, 0, 1), (3, 4, 5), (70, 9, 6), (240, 16, 16), (2, 1, 3)])
def test_softmax_routing_with_identity_outputs(T, E, ident, top):
    """ids, weights and the plan: rows of an expert are contiguous and all different, identity picks have none; corrections move the
    picks but not the weights"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(T * 1000 + E)
    z = torch.randn(T, E + ident + 3, generator=g) * 2
    corr = torch.randn(E + ident, generator=g) * 0.5
    for dtype in (torch.float32, torch.bfloat16):
        c = corr.to(dtype)
        r = ops.moe_route(z.to(DEV)[:, 2:2 + E + ident], top, softmax_scores=True, correction=c.to(DEV), identity=ident)   # a column slice
        s = torch.softmax(z[:, 2:2 + E + ident].double(), -1)
        ids, w = orc.pick_experts(s, c.double(), top)
        assert torch.equal(r.ids.cpu().long().sort(-1).values, ids.sort(-1).values)
        full = torch.zeros(T, E + ident, dtype=torch.float64).scatter_(1, r.ids.cpu().long(), r.weights.cpu().double())
        assert float((full - torch.zeros_like(full).scatter_(1, ids, w)).abs().max()) < 1e-6
        rows = torch.tensor(_row_of(r))
        experts = r.ids.cpu() < E
        assert bool((rows[~experts] == -1).all())
        n = int(experts.sum())
        assert sorted(rows[experts].tolist()) == list(range(n))
        order = r.ids.cpu()[experts][torch.argsort(rows[experts])]
        assert bool((order[1:] >= order[:-1]).all()) and r.experts == E and r.identity == ident
    if E >= 3:    # a correction that outweighs any score decides alone
        big = torch.zeros(E + ident)
        big[E - 1] = 5.0
        r = ops.moe_route(z.to(DEV)[:, 2:2 + E + ident].contiguous(), 1, softmax_scores=True, correction=big.to(DEV), identity=ident)
        assert bool((r.ids == E - 1).all()) and float((r.weights - 1).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,ident,top,W,ff,shared", [(5, 2, 3, 40, 12, 28), (6, 0, 2, 64, 72, None), (3, 5, 4, 128, 40, 64), (8, 3, 2, 96, 136, 200), (1, 1, 2, 64, 64, 16)])
def test_routed_feed_forward(dtype, E, ident, top, W, ff, shared):
    """steps of one row to several hundred: the plain products, the grouped tensor-core ones and the tcgen05 groups"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    from tgis_b200.utils.mixers import RoutedSharedFeedForward
    f = {"router": {"experts": E, "identity": ident, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}
    cfg = orc.random_config(width=W, order=("attention",), shares=(), experts=E, identity=ident, top=top, ff=ff, shared=shared)
    sd = {k[3:]: v for k, v in orc.random_state_dict(cfg, seed=E).items() if ".mlp." in k}
    if dtype == torch.bfloat16:
        sd = _fixed_picks(cfg, sd)
    m = RoutedSharedFeedForward("mlp", _DictWeights(sd, dtype), experts=E, identity=ident, top=top, shared=shared is not None)
    for T in (1, 33, 130, 700):
        h = torch.randn(T, W, generator=torch.Generator().manual_seed(T)).to(torch.bfloat16).float()
        ref = orc.routed_experts(h.double(), {k[4:]: v.double() for k, v in sd.items()}, f)
        x = torch.zeros(T, W, device=DEV)
        ops.halves_step(x, dtype=dtype, **m(h.to(dtype).to(DEV)))
        assert float((x.cpu().double() - ref).abs().max()) < (2e-5 if dtype == torch.float32 else 0.02) * float(ref.abs().max()), T
    from tgis_b200 import _lib
    assert _lib.load_seq().b200_seq_group_gemm_gave_up() == 0


@pytest.mark.parametrize("E,N,K,T,top", [(4, 130, 72, 500, 2), (7, 256, 64, 90, 3), (3, 40, 200, 1500, 2), (1, 128, 128, 260, 1)])
def test_experts_on_tensor_core_groups(E, N, K, T, top):
    """uneven and empty experts, feature tiles and k-blocks that end inside a tile, both results and the squared ReLU"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(N)
    z = torch.randn(T, E, generator=g) * 3
    if E > 2:
        z[:, 1] = -100.0        # an expert without rows
    r = ops.moe_route(z.to(DEV), top if E > 2 else 1)
    a = torch.randn(T, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(E, N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    rows, ids = torch.tensor(_row_of(r)), r.ids.cpu().long()
    want = torch.zeros(T * r.top, N, dtype=torch.float64)
    for k in range(r.top):
        want[rows[:, k]] = torch.einsum("tk,tnk->tn", a.double(), w[ids[:, k]].double())
    c = ops.moe_gather_rows(a.to(DEV), r)
    for act, fn in ((ops.ACT_NONE, lambda v: v), (ops.ACT_RELU2, lambda v: torch.clamp(v, min=0) ** 2)):
        for dt in (torch.float32, torch.bfloat16):
            got = ops.experts_linear(c, w.to(DEV), r, dt, act=act).cpu().double()
            assert float((got - fn(want)).abs().max()) < (1e-4 if dt == torch.float32 else 0.01) * float(fn(want).abs().max())
        assert float((ops.moe_linear(a.to(DEV), w.to(DEV), r, True, torch.float32, act=act).cpu().double() - fn(want)).abs().max()) < 1e-4 * float(fn(want).abs().max())


@pytest.mark.parametrize("T,Z,N,K,gap", [(1, 3, 40, 8, 8), (20, 5, 130, 72, 0), (50, 2, 96, 64, 24), (100, 4, 128, 128, 64), (300, 3, 72, 80, 16), (700, 2, 256, 192, 0)])
def test_per_head_products_on_tensor_core_groups(T, Z, N, K, gap):
    """slices of wider rows on both sides: what lies between the heads is neither read into a result nor written"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(T)
    wide = torch.randn(T, Z, K + gap, generator=g).to(torch.bfloat16)
    w = (torch.randn(Z, N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    ref = torch.einsum("tzk,znk->tzn", wide[:, :, :K].double(), w.double())
    for dt in (torch.float32, torch.bfloat16):
        out = torch.full((T, Z, N + 4), 7.0, dtype=dt, device=DEV)
        ops.linear_per_head(wide.to(DEV)[:, :, :K], w.to(DEV), out[:, :, :N])
        assert float((out[:, :, :N].cpu().double() - ref).abs().max()) < (1e-4 if dt == torch.float32 else 0.02) * float(ref.abs().max())
        assert bool((out[:, :, N:] == 7.0).all())


def test_soft_cap_and_squared_relu_epilogue():
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    g = torch.Generator().manual_seed(5)
    z = torch.randn(7, 133, generator=g) * 40
    assert float((ops.soft_cap(z.to(DEV).clone(), 12.5).cpu().double() - orc.soft_cap(z.double(), 12.5)).abs().max()) < 1e-5
    for M, N, K in ((3, 200, 64), (40, 96, 136), (600, 320, 256), (5, 30, 20)):
        x, w, b = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((M, K), (N, K), (N,)))
        ref = torch.clamp(x.double() @ w.double().T + b.double(), min=0) ** 2
        for dt in (torch.bfloat16, torch.float32):
            got = ops.linear(x.to(dt).to(DEV), w.to(dt).to(DEV), b.to(dt).to(DEV), act=ops.ACT_RELU2).cpu().double()
            assert float(((got - ref).abs() / (ref + ref.abs().mean())).max()) < (0.01 if dt == torch.bfloat16 else 1e-4)


ATTENTION_CASES = [  # heads, kv heads, dim, vdim, rotated columns, chunk
    (6, 2, 10, 12, 6, 20),        # the plain kernel: sizes that are no multiples of 16
    (4, 4, 16, 48, 16, 37),       # as many key heads as heads, full rotation
    (8, 1, 32, 96, 8, 16),        # one key head, a chunk of exactly one page
    (16, 4, 16, 112, 0, 50),      # no rotation
    (8, 2, 48, 80, 2, 0),         # no chunks
    (3, 1, 8, 8, 4, 5),           # a chunk shorter than a page
    (2, 1, 16, 144, 16, 24),      # a value size beyond the tensor-core kernel
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,rot,chunk", ATTENTION_CASES)
def test_chunk_attention_any_cut(H, G, d, dv, rot, chunk, dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.tibopel_modeling import build_mixer
    cfg = orc.random_config(order=("attention",), shares=(), width=32, heads=H, kv_heads=G, dim=d, vdim=dv, rot_dims=rot or None, chunk=chunk or None, sharp=1.5)
    m = cfg["layers"][0]["mixer"]
    sd = {k: v for k, v in orc.random_state_dict(cfg, seed=dv).items() if k.startswith("l0.mix.")}
    L = 70
    h = torch.randn(L, 32, generator=torch.Generator().manual_seed(3)).to(torch.bfloat16).float()
    ref = orc.chunk_attention(h.double(), {k[7:]: v.double() for k, v in sd.items()}, m)
    mixer = build_mixer("attention", "l0.mix", m, _DictWeights(sd, dtype), 1e-5)
    tol = 1e-4 if dtype == torch.float32 else 0.08
    for cuts in ([L], [], [2, 33, 2, 31], [16, 16, 16, 16], [1, 20, 47]):
        got = _feed(mixer, mixer.cache_spec(), h, cuts, dtype)
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max()), cuts


LATENT_CASES = [  # heads, dim, rotated part, rotated columns, vdim, kv rank, q rank
    (3, 8, 6, 6, 14, 20, 18),         # the plain kernel
    (5, 24, 16, 16, 40, 48, 72),      # tensor-core tiles: heads that do not divide a tile, three 16-column pieces
    (1, 16, 16, 8, 8, 16, 64),        # one head, a partly rotated key part, one piece
    (20, 8, 32, 32, 16, 80, 24),      # more rows per token than one row group
    (33, 16, 16, 16, 24, 144, 40),    # decoded tokens of several row groups
    (8, 64, 64, 64, 32, 512, 128),    # the widest latent of the tensor-core kernel
    (4, 16, 12, 12, 16, 272, 32),     # a rotated part that is no multiple of 16: the plain kernel in bfloat16 too
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,r,rot,dv,R,Q", LATENT_CASES)
def test_latent_attention_any_cut(H, d, r, rot, dv, R, Q, dtype):
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.tibopel_modeling import build_mixer
    cfg = orc.random_config(order=("latent_attention",), shares=(), width=32, l_heads=H, l_dim=d, rot_dim=r, l_rot_dims=rot, l_vdim=dv, kv_rank=R, q_rank=Q,
                            sharp=1.5)
    m = cfg["layers"][0]["mixer"]
    sd = {k: v for k, v in orc.random_state_dict(cfg, seed=R).items() if k.startswith("l0.mix.")}
    L = 75
    h = torch.randn(L, 32, generator=torch.Generator().manual_seed(3)).to(torch.bfloat16).float()
    ref = orc.latent_attention(h.double(), {k[7:]: v.double() for k, v in sd.items()}, m, 1e-5)
    mixer = build_mixer("latent_attention", "l0.mix", m, _DictWeights(sd, dtype), 1e-5)
    run = lambda x, st, pages, state, max_s: mixer(x, st, pages, max_s)  # noqa: E731
    tol = 1e-4 if dtype == torch.float32 else 0.08
    for cuts in ([L], [], [2, 33, 2, 31], [16, 16, 16, 16], [1, 20, 52]):
        got = _feed(run, mixer.cache_spec(), h, cuts, dtype)
        assert got.shape == ref.shape and float((got - ref).abs().max()) < tol * float(ref.abs().max()), cuts


def _latent_case(dtype, H, R, r, L, seed):
    """a pool of latent rows out of order, NaN everywhere else"""
    g = torch.Generator().manual_seed(seed)
    D, blocks = R + r, (L + 15) // 16
    rows = (torch.randn(L, D, generator=g) * 0.3).to(dtype)
    table = [(7 * i + 1) % (blocks + 3) for i in range(blocks)]
    assert len(set(table)) == blocks
    pool = torch.full((blocks + 3, 16, D), float("nan"), dtype=dtype, device=DEV)
    where = torch.tensor([table[p // 16] * 16 + p % 16 for p in range(L)], device=DEV)
    pool.view(-1, D)[where] = rows.to(DEV)
    return g, rows, pool, table


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,R,r", [(3, 40, 8), (5, 48, 16), (16, 64, 16), (24, 96, 32), (40, 128, 16), (8, 512, 64)])
def test_loud_keys_far_back_and_sinks(dtype, H, R, r):
    """One key wins the soft-max of every head from hundreds of tokens back, a page border or the query itself - for a decoded token (the
    keys split over blocks) and for a row inside a portion; the sink takes all of it away, half of it or nothing, per head."""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    L = 430
    g, rows, pool, table = _latent_case(dtype, H, R, r, L, R)
    for qpos, kpos in ((429, 0), (429, 15), (428, 16), (429, 429), (300, 31), (17, 16), (64, 1), (0, 0), (33, 32)):
        q = torch.randn(L, H, R + r, generator=g) * 0.1
        loud = rows[kpos].float()
        q[qpos] = loud / loud.norm() ** 2 * 30.0
        q = q.to(dtype)
        score = (q[qpos].double() @ rows[kpos].double())                     # per head, about 30
        for sink in (None, torch.full((H,), -50.0), score.float(), score.float() + 12.0 * (torch.arange(H) % 3 - 1.0)):
            s = q[qpos].double() @ rows[:qpos + 1].double().T                  # [H, keys]
            if sink is not None:
                s = torch.cat([s, sink.double()[:, None]], 1)
            want = torch.softmax(s, 1)[:, :qpos + 1] @ rows[:qpos + 1, :R].double()
            for start, n in ((qpos, 1), (max(qpos - 40, 0), min(41, qpos + 1) + (1 if qpos + 1 < L else 0))):
                st = _step([(start, n)], [table])
                got = ops.latent_attn(q[start:start + n].contiguous().to(DEV), pool, st, R, r, 0, 1.0, None if sink is None else sink.to(DEV))[qpos - start]
                assert float((got.cpu().double() - want).abs().max()) < (1e-4 if dtype == torch.float32 else 0.02), (qpos, kpos, n)
        if qpos > 40:
            assert float((want - rows[kpos, :R].double()).abs().max()) > 0.05   # the last sinks did take weight


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_ragged_batch_and_windows(dtype):
    """portions beside decoded tokens of unlike lengths in one launch, with and without a window whose edge a loud key sits at"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq as ops
    H, R, r = 6, 64, 16
    g, rows, pool, table = _latent_case(dtype, H, R, r, 300, 9)
    entries = [(0, 1), (250, 50), (77, 1), (100, 3), (0, 33), (299, 1), (16, 16)]
    q = torch.cat([torch.randn(n, H, R + r, generator=g) for _, n in entries]) * 0.2
    pos = [p for s, n in entries for p in range(s, s + n)]
    sink = torch.randn(H, generator=g)
    for window in (0, 40, 16):
        for i, p in enumerate(pos):       # just inside (even rows) and just outside (odd rows)
            j = p - window + (1 if i % 2 == 0 else 0)
            if window and 0 <= j <= p:
                q[i, i % H] = rows[j].float() / rows[j].float().norm() ** 2 * 20.0
        qt = q.to(dtype)
        st = _step(entries, [table] * len(entries))
        got = ops.latent_attn(qt.to(DEV), pool, st, R, r, window, 0.9, sink.to(DEV)).cpu().double()
        for i, p in enumerate(pos):
            lo = max(0, p - window + 1) if window else 0
            s = torch.cat([qt[i].double() @ rows[lo:p + 1].double().T * 0.9, sink.double()[:, None]], 1)
            want = torch.softmax(s, 1)[:, :-1] @ rows[lo:p + 1, :R].double()
            assert float((got[i] - want).abs().max()) < (1e-4 if dtype == torch.float32 else 0.02), (window, i, p)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,chunk", [(6, 3, 10, 14, 100), (8, 2, 32, 48, 33), (2, 2, 64, 112, 17)])
def test_loud_keys_at_chunk_edges_through_the_mixer(dtype, H, G, d, dv, chunk):
    """the same through projection, rotation and cache: biases make one key loud for every query of the sequence; rows of its chunk after
    it carry its value, rows of the next chunk do not"""
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.tibopel_modeling import build_mixer
    cfg = orc.random_config(order=("attention",), shares=(), width=32, heads=H, kv_heads=G, dim=d, vdim=dv, rot_dims=None, chunk=chunk)
    m = cfg["layers"][0]["mixer"]
    m["scale"] = 1.0
    sd = {k: v for k, v in orc.random_state_dict(cfg, seed=chunk).items() if k.startswith("l0.mix.")}
    L, edge = 2 * chunk + 20, chunk
    h = (torch.randn(L, 32, generator=torch.Generator().manual_seed(1)) * 0.3).to(torch.bfloat16).float()
    for kpos in (edge, edge - 1, 2 * edge - 1):
        hk = h.clone()
        hk[kpos, :8] = 6.0                                    # a direction that only this row has
        s2 = dict(sd)
        s2["l0.mix.q.b"] = torch.ones(H * d)
        k = sd["l0.mix.k"].clone() * 0.1
        k[:, :8] = 0.5
        s2["l0.mix.k"] = k.to(torch.bfloat16).float()
        ref = orc.chunk_attention(hk.double(), {n[7:]: v.double() for n, v in s2.items()}, m)
        calm = orc.chunk_attention(h.double(), {n[7:]: v.double() for n, v in s2.items()}, m)
        moved = (ref - calm).abs().amax(1) > 1e-9
        assert bool(moved[kpos:(kpos // chunk + 1) * chunk].all()) and not bool(moved[(kpos // chunk + 1) * chunk:].any())
        mixer = build_mixer("attention", "l0.mix", m, _DictWeights(s2, dtype), 1e-5)
        for cuts in ([L], [kpos - 1, 2, 2], [kpos, L - kpos - 3], [chunk, chunk]):
            got = _feed(mixer, mixer.cache_spec(), hk, cuts, dtype)
            assert float((got - ref).abs().max()) < (1e-4 if dtype == torch.float32 else 0.08) * float(ref.abs().max()), (kpos, cuts)


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_prompt_portions_and_decoding_agree_with_reference(tmp_path, dtype):
    cfg = orc.random_config(sharp=3.0, chunk=24)
    sd = orc.random_state_dict(cfg, seed=2)
    if dtype == torch.bfloat16:
        sd = _fixed_picks(cfg, sd)
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
        mix = lambda c, i=0: c["layers"][i]["mixer"]  # noqa: E731
        scaled = lambda name, f: (lambda c, s: s.update({name: s[name] * f}))  # noqa: E731
        shared = lambda fn: (lambda c, s: [fn(c["layers"][i]) for i in (1, 3)])  # noqa: E731
        for fn in (lambda c, s: mix(c)["mask"].update(size=25), lambda c, s: mix(c)["mask"].update(size=23), lambda c, s: mix(c)["rot"].update(dims=4),
                   lambda c, s: mix(c)["rot"].update(base=450.0), lambda c, s: mix(c)["rot"].pop("scaling"), lambda c, s: mix(c)["rot"]["scaling"].update(factor=5.0),
                   lambda c, s: mix(c)["rot"]["scaling"].update(original=80), lambda c, s: mix(c)["rot"]["scaling"].update(low=1.4),
                   lambda c, s: mix(c)["rot"]["scaling"].update(high=4.5),
                   lambda c, s: mix(c).update(scale=mix(c)["scale"] * 1.05), scaled("l0.mix.g", 0.5), scaled("l0.mix.q.b", 0.0), scaled("l2.mix.k.b", 0.0),
                   scaled("l0.mix.v.b", 0.0), scaled("l0.mix.o.b", 0.5), scaled("l1.mix.sink", 0.5), shared(lambda l: l["mixer"].update(scale=l["mixer"]["scale"] * 1.05)),
                   shared(lambda l: l["mixer"]["rot"].update(base=150.0)), scaled("l1.mix.dq.norm", 1.1), scaled("l1.mix.dkv.norm", 1.1),
                   lambda c, s: c["layers"][3].update(type="attention", mixer=c["layers"][2]["mixer"], mlp=c["layers"][2]["mlp"], weights_of=2),
                   scaled("l0.norm1", 1.05), scaled("l0.norm2", 1.05), scaled("l1.mlp.router", 0.9), scaled("l0.mlp.correction", 0.0),
                   scaled("l1.mlp.shared.sg", 0.5), scaled("l0.mlp.shared.up", 0.9), scaled("l0.mlp.e1.up", 0.9), lambda c, s: c["layers"][0]["mlp"]["router"].update(top=2),
                   lambda c, s: c.update(logit_softcap=16.0), lambda c, s: c["norm"].update(eps=1e-1)):
            assert changed(fn) > 20 * TOL32
    for cuts in ([], [40], [2, 2, 2, 19, 3, 16, 17, 2], [16, 16, 16, 16], [24, 24, 24], [23, 2, 23, 2], [1, 25, 22, 31]):
        got = _run_cut(model, toks, cuts)
        assert _rel(got, ref) < tol, cuts
        if dtype == torch.float32:
            assert _rel(got, whole.cpu()) < 1e-5, cuts  # the cut itself changes nothing beyond rounding
    assert model.kv_cache_manager.free_blocks == model.kv_cache_manager.total_num_gpu_blocks
    assert model.kv_cache_manager.free_state_slots == 4


def test_tensor_core_shapes_through_the_engine(tmp_path):
    """bfloat16 with sizes in 16s: prompts, portions and decoded tokens take the tensor-core attention kernels, the per-head and experts'
    groups and the fused epilogues; a step mixes a long portion (several row tiles) with single tokens"""
    cfg = orc.random_config(width=64, heads=8, kv_heads=2, dim=32, vdim=80, rot_dims=16, chunk=60, sharp=2.0, l_heads=6, l_dim=24, rot_dim=16, l_vdim=40,
                            kv_rank=96, q_rank=64, experts=3, identity=2, top=3, ff=64, shared=96)
    sd = _fixed_picks(cfg, orc.random_state_dict(cfg, seed=12))
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


def test_stream_after_every_layer(tmp_path):
    cfg = orc.random_config(mlp=("moe", "moe", None))
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
    assert len(probe) == len(want) == 4 and _rel(lg, ref) < TOL32
    for i, (a, b) in enumerate(zip(probe, want)):
        assert float((a.cpu().double() - b).abs().max()) < 1e-4 * float(b.abs().max()), i


OTHER_SIZES = {
    "one_key_head_no_identity": dict(heads=5, kv_heads=1, identity=0, top=1, experts=3, l_heads=1),
    "equal_sizes": dict(heads=4, kv_heads=4, dim=14, vdim=14, rot_dims=14, l_heads=4, l_dim=14, l_vdim=14, rot_dim=14, kv_rank=28, q_rank=28, chunk=2),
    "one_expert": dict(experts=1, identity=3, top=4, shared=None, scaling=None, width=56, chunk=31),
    "mostly_identity": dict(experts=2, identity=9, top=5, cap=4.0, shares=(None, None, 0, 1, 0), order=("attention", "latent_attention", "attention", "latent_attention", "attention")),
    "no_rotation_no_chunks_no_cap": dict(rot_dims=None, chunk=None, cap=None, vdim=20, mlp=(None, "moe")),
    "latent_only": dict(order=("latent_attention",) * 3, shares=(None, 0, None), l_rot_dims=4, rot_dim=10, kv_rank=7, q_rank=5, eps=1e-3),
    "attention_only": dict(order=("attention",) * 2, shares=(None, None), scaling=(2.0, 0.5, 6.0, 200), base=30.0, rot_dims=10, experts=7, top=7, identity=0),
    "layers_unlike_each_other": dict(shares=(), other={2: {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 16, "scale": 1.1, "mask": {"size": 7},
                                                           "rot": {"base": 10.0, "dims": 4}},
                                                       3: {"heads": 5, "kv_rank": 11, "vdim": 6, "scale": 0.9}}),
    "many_experts": dict(experts=40, identity=1, top=8, ff=4, vocab=130),
}


@pytest.mark.parametrize("variant", sorted(OTHER_SIZES))
def test_other_sizes(tmp_path, variant):
    """sizes that a usual configuration makes equal or 1, and entries it may leave out"""
    cfg = orc.random_config(**{"sharp": 3.0, **OTHER_SIZES[variant]})
    sd = orc.random_state_dict(cfg, seed=31)
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(6, 60, cfg["vocab"])
    ref = orc.forward(cfg, sd, toks)
    for cuts in ([60], [3, 30, 2], [17]):
        assert _rel(_run_cut(model, toks, cuts), ref) < TOL32, (variant, cuts)


def test_layer_may_share_with_a_later_one(tmp_path):
    cfg = orc.random_config(shares=())
    cfg["layers"][0] = {**cfg["layers"][2], "weights_of": 2}
    sd = orc.random_state_dict(cfg, seed=8)
    assert not any(k.startswith("l0.") for k in sd)
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(2, 40, cfg["vocab"])
    assert _rel(_run_cut(model, toks, [25]), orc.forward(cfg, sd, toks)) < TOL32
    layers = model.model.model.layers
    assert layers[0].mixer is layers[2].mixer and model.kv_cache_manager.layer_pages(0).data_ptr() != model.kv_cache_manager.layer_pages(2).data_ptr()


def test_ragged_batches_and_reused_pages(tmp_path):
    """four requests of unequal length run as mixed steps (portions beside decoded tokens, requests joining and leaving) in a pool
    that is too small for all of them at once and is filled with garbage first: every request equals its run alone"""
    cfg = orc.random_config(sharp=3.0)
    sd = orc.random_state_dict(cfg, seed=21)
    model = _model(tmp_path, cfg, sd, torch.float32, blocks=12, slots=2)
    mgr = model.kv_cache_manager
    for p in mgr.pages:
        p.fill_(float("nan"))
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
    """three prompt tokens, then 197 single steps: chunks begin and end among decoded tokens only, the latent layers look back over all of them"""
    cfg = orc.random_config(sharp=3.0, chunk=40)
    sd = orc.random_state_dict(cfg, seed=8)
    model = _model(tmp_path, cfg, sd, torch.float32)
    toks = _tokens(9, 200, cfg["vocab"])
    ref = orc.forward(cfg, sd, toks)
    c2, _ = _vary(cfg, sd, lambda c, s: [l["mixer"]["mask"].update(size=41) for l in c["layers"] if "mask" in l["mixer"]])
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
    sd = _fixed_picks(cfg, orc.random_state_dict(cfg, seed=3))
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


def test_captured_decoding_runs_the_halves_side_by_side(tmp_path, monkeypatch):
    """bfloat16 decoding through generate_token: the captured step (mixer and feed-forward as parallel branches of the graph) and the same
    with one branch after the other choose the same tokens, step for step"""
    import tgis_b200  # noqa: F401
    from tgis_b200 import ops_seq, pb
    cfg = orc.random_config(width=128, heads=8, kv_heads=2, dim=32, vdim=48, rot_dims=16, chunk=60, l_heads=6, l_dim=24, rot_dim=16, l_vdim=40, kv_rank=96,
                            q_rank=64, experts=6, identity=2, top=3, ff=72, shared=96)
    model = _model(tmp_path, cfg, orc.random_state_dict(cfg, seed=5), torch.bfloat16, blocks=64, slots=6)
    forks = []
    enter = ops_seq.beside.__enter__

    def counting(self):
        enter(self)
        forks.append(self.side is not None)
        return self
    monkeypatch.setattr(ops_seq.beside, "__enter__", counting)
    outs = []
    for on in (True, False):
        monkeypatch.setattr(ops_seq, "SIDE_STREAM", on)
        forks.clear()
        prompts, n_new = [_tokens(60 + i, n, cfg["vocab"]) for i, n in enumerate((9, 40, 77))], 24
        reqs = [pb.Request(id=i, inputs=" ".join("test" if t == 3 else f"<tok{t}>" for t in p), input_length=len(p), truncate=False, max_output_length=n_new,
                           parameters=pb.NextTokenChooserParameters(temperature=0.0, top_p=1.0, min_new_tokens=n_new)) for i, p in enumerate(prompts)]
        got = {i: [] for i in range(3)}
        with torch.inference_mode():
            b, errs = model.batch_type.from_pb(pb.Batch(id=0, requests=reqs), model.tokenizer, model.dtype, model.device, None, None, True)
            assert not errs
            for step in range(n_new):
                for t in model.generate_token(b, first=step == 0)[0]:
                    got[t.request_id].append(t.token_id)
            model.kv_cache_manager.free_sequences(b.sequence_ids)
        outs.append(got)
        assert any(forks) == on
    assert outs[0] == outs[1] and all(len(v) == 24 for v in outs[0].values())
