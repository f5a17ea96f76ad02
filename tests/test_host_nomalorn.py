"""Nomalorn without a GPU: the configuration reader (layer runs of a loop, optional entries) and its refusals, the checkpoint table
against the reference's, the cache manager's bookkeeping for a stack whose looped layers keep a store per pass, and properties of
the slow reference itself (so that a GPU test that agrees with it agrees with the mechanism)."""
import copy
import json

import pytest
import torch

from oracle import nomalorn as orc


def test_config_reader_layer_runs_and_refusals():
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.nomalorn_modeling import NomalornConfig, tensor_shapes
    raw = orc.random_config()
    cfg = NomalornConfig(raw)
    assert cfg.model_type == "nomalorn" and cfg.hidden_size == 40 and cfg.vocab_size == 72 and cfg.norm_eps == 1e-5
    assert cfg.layer_runs == orc.layer_runs(raw) == [(0, None), (1, 0), (2, None), (1, 1), (2, None)]
    assert cfg.num_hidden_layers == 5 and cfg.loop_times == 2
    assert tensor_shapes(raw, 5, 7) == orc.tensor_shapes(raw) and "head" not in tensor_shapes(raw)   # the embedding table is the head
    plain = orc.random_config(loop=None, rot_dims=None, chunk=None)
    assert NomalornConfig(plain).layer_runs == [(0, None), (1, None), (2, None)] and "loop.step" not in tensor_shapes(plain)
    assert NomalornConfig(orc.random_config(loop=(0, 3, 1))).layer_runs == [(0, 0), (1, None), (2, None)]
    assert NomalornConfig(orc.random_config(loop=(2, 3, 3))).layer_runs == [(0, None), (1, None), (2, 0), (2, 1), (2, 2)]
    assert NomalornConfig(orc.random_config(loop=(2, 2, 5))).layer_runs == [(0, None), (1, None), (2, None)]   # an empty run repeats nothing
    with pytest.raises(ValueError):
        NomalornConfig(dict(raw, architecture="Other"))
    for loop in ({"start": 3, "stop": 2, "times": 2}, {"start": 0, "stop": 4, "times": 2}, {"start": 0, "stop": 1, "times": 0}):
        with pytest.raises(ValueError):
            NomalornConfig(dict(raw, loop=loop))
    bad = copy.deepcopy(raw)
    bad["layers"][1]["type"] = "conv_only"
    with pytest.raises(NotImplementedError):
        NomalornConfig(bad)
    bad = copy.deepcopy(raw)
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(NotImplementedError):
        NomalornConfig(bad)


def test_engine_recognises_the_architecture(tmp_path):
    import tgis_b200  # noqa: F401
    from tgis_b200.inference_engine import FLASH_TYPES, OWN_CONFIG_ARCHITECTURES, load_config
    with open(tmp_path / "config.json", "w") as f:
        json.dump(orc.random_config(), f)
    cfg = load_config(str(tmp_path))
    assert cfg.model_type == "nomalorn" and cfg.model_type in FLASH_TYPES and cfg.architecture in OWN_CONFIG_ARCHITECTURES


class _Weights:
    def __init__(self, sd):
        from tgis_b200.utils.dist import FakeGroup
        self.sd, self.dtype, self.device, self.process_group = sd, torch.float32, "cpu", FakeGroup(0, 1)

    def get_tensor(self, name):
        return self.sd[name]


def test_modules_specs_and_stores_per_layer_run():
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.nomalorn_modeling import NomalornConfig, NomalornForCausalLM
    from tgis_b200.utils.paged import HybridCacheManager
    cfg = orc.random_config()
    sd = orc.random_state_dict(cfg)
    model = NomalornForCausalLM(NomalornConfig(cfg), _Weights(sd))
    runs = model.model.layers
    assert len(runs) == 5 and runs[1].mixer is runs[3].mixer and runs[2].mixer is runs[4].mixer and runs[1].mixer is not runs[2].mixer
    assert [r.index for r in runs] == [0, 1, 2, 3, 4] and [r.entering for r in runs] == [None, 0, None, 1, None]
    assert runs[0].mlp is not None and runs[1].mlp is None and model.head is model.model.embed
    m = runs[0].mixer
    # one input product: the attention's rows with their biases, then the memory's rows without; the two low ranks share one padded latent
    assert m.w_in.shape == (6 * 10 + 2 * 10 + 2 * 12 + 6 + 2 * 2 * 12 + 4 * 14 + 64 + 4, 40) and m.b_in.shape == (m.w_in.shape[0],)
    assert torch.equal(m.b_in[:60], sd["l0.mix.left.q.b"]) and float(m.b_in[104:].abs().max()) == 0.0
    low = m.right.w_low
    assert low.shape == (4 * 12 + 4 * 14, 64) and torch.equal(low[:48, :5], sd["l0.mix.right.a2"]) and torch.equal(low[48:, 5:12], sd["l0.mix.right.g2"])
    assert float(low[:48, 5:].abs().max()) == 0.0 and float(low[48:, :5].abs().max()) == 0.0 and float(low[:, 12:].abs().max()) == 0.0
    mgr = HybridCacheManager([r.mixer.cache_spec() for r in runs], torch.float32, "cpu", total_num_gpu_blocks=5, num_state_slots=2)
    assert mgr.layer_pages(0).shape == (5, 16, 2 * (10 + 12))
    assert mgr.layer_state(0)["right.S"].shape == (2, 4, 12, 14) and mgr.layer_state(0)["right.conv"].shape == (2, 2, 2 * 2 * 12 + 4 * 14)
    assert mgr.layer_state(1)["right.S"].data_ptr() != mgr.layer_state(3)["right.S"].data_ptr()     # two passes of one layer
    assert mgr.layer_pages(1).data_ptr() != mgr.layer_pages(3).data_ptr()
    bad = dict(sd, **{"loop.step": sd["loop.step"][:1]})
    with pytest.raises(ValueError):
        NomalornForCausalLM(NomalornConfig(cfg), _Weights(bad))
    bad = dict(sd, **{"l0.mix.right.a2": sd["l0.mix.right.a2"][:, :4]})
    with pytest.raises(ValueError):
        NomalornForCausalLM(NomalornConfig(cfg), _Weights(bad))


def _halves(seed=1, **kw):
    cfg = orc.random_config(layers=1, loop=None, **kw)
    sd = {k: v.double() for k, v in orc.random_state_dict(cfg, seed=seed).items()}
    m = cfg["layers"][0]["mixer"]
    return cfg, m, orc.sub(sd, "l0.mix.left."), orc.sub(sd, "l0.mix.right.")


def test_reference_attention_properties():
    cfg, m, p, _ = _halves(chunk=8)
    g = torch.Generator().manual_seed(0)
    h = torch.randn(30, cfg["width"], dtype=torch.float64, generator=g)
    full = orc.chunk_attention(h, p, m["left"])
    # a row sees its own chunk up to itself: rows from 16 on do not move when rows 0 .. 15 change, row 15 does
    h2 = h.clone()
    h2[:16] = torch.randn(16, cfg["width"], dtype=torch.float64, generator=g)
    other = orc.chunk_attention(h2, p, m["left"])
    assert torch.allclose(other[16:], full[16:], atol=1e-12) and not torch.allclose(other[15], full[15], atol=1e-4)
    h2 = h.clone()
    h2[16] += 1.0
    assert not torch.allclose(orc.chunk_attention(h2, p, m["left"])[23], full[23], atol=1e-6)
    # the first row of a chunk sees itself only: its result is its own value
    v = (h[8:9] @ p["v"].T + p["v.b"]).view(1, 2, 12).repeat_interleave(3, dim=1) * torch.sigmoid(h[8:9] @ p["g"].T)[:, :, None]
    assert torch.allclose(full[8:9], v.reshape(1, -1) @ p["o"].T)
    # rotation: only position differences count, columns beyond the rotated ones pass
    x, pos = torch.randn(4, 2, 10, dtype=torch.float64, generator=g), torch.tensor([3, 9, 0, 100])
    a, b = orc.rotate_halves(x, pos, 6, 50.0), orc.rotate_halves(x, pos + 17, 6, 50.0)
    assert torch.equal(a[..., 6:], x[..., 6:]) and torch.equal(a[2], x[2])
    assert torch.allclose((a[0] * a[1]).sum(), (b[0] * b[1]).sum())


def test_reference_delta_memory():
    d, dv = 4, 3
    f = dict(dtype=torch.float64)
    k = torch.eye(d, **f)
    one = torch.ones(1, 1, **f)
    keep = torch.ones(1, 1, d, **f)
    # full strength and no decay: a second write at the same key replaces the first, another key's value stays
    ks = torch.stack([k[1], k[2], k[1]])[:, None, :]
    v = torch.arange(9.0, **f).view(3, 1, dv)
    o = orc.delta_memory(torch.stack([k[1], k[2], k[2]])[:, None, :], ks, v, one.expand(3, 1), keep.expand(3, 1, d))
    assert torch.allclose(o, torch.stack([v[0], v[1], v[1]]))            # the read-out sees the token's own write
    o = orc.delta_memory(k[1].expand(3, 1, d), ks, v, one.expand(3, 1), keep.expand(3, 1, d))
    assert torch.allclose(o, torch.stack([v[0], v[0], v[2]]))
    # a decay of zero on row 1 forgets what was written there, and only that
    gone = keep.expand(3, 1, d).clone()
    gone[2, 0, 1] = 0.0
    ks = torch.stack([k[1], k[2], k[3]])[:, None, :]
    o = orc.delta_memory((k[1] + k[2]).expand(3, 1, d), ks, v, one.expand(3, 1), gone)
    assert torch.allclose(o[1], v[0] + v[1]) and torch.allclose(o[2], v[1])
    # the decay comes before the prediction: a forgotten row is not subtracted from the new value
    ks = torch.stack([k[1], k[1]])[:, None, :]
    o = orc.delta_memory(k[1].expand(2, 1, d), ks, v[:2], one.expand(2, 1) * 0.5, gone[1:])
    assert torch.allclose(o[0], 0.5 * v[0]) and torch.allclose(o[1], 0.5 * v[1])
    # no strength: nothing is written
    assert float(orc.delta_memory(k[1].expand(2, 1, d), ks, v[:2], one.expand(2, 1) * 0.0, keep.expand(2, 1, d)).abs().max()) == 0.0
    cfg, m, _, p = _halves(seed=3)
    h = torch.randn(20, cfg["width"], dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    full = orc.channel_delta(h, p, m["right"], 1e-5)
    assert torch.allclose(orc.channel_delta(h[:12], p, m["right"], 1e-5), full[:12], atol=1e-12)      # causal
    # the head norm takes the memory's size away, up to eps: values twice as large give nearly the same result
    twice = orc.channel_delta(h, dict(p, **{"norm": p["norm"] * 2.0}), m["right"], 1e-5)
    assert torch.allclose(twice, 2.0 * full)


def test_reference_loop_steps_and_norms():
    """ahead of every pass its vector, ahead of every pass but the first the embedding output; a loop shares tensors, not memory"""
    base = orc.random_config(loop=(1, 3, 2))
    sd = orc.random_state_dict(base, seed=6)
    toks = list(range(5, 25))
    ref = orc.forward(base, sd, toks)
    assert torch.allclose(orc.forward(base, sd, toks[:9]), ref[:9], atol=1e-12)                # causal
    # with zero vectors and a zero embedding added, the loop is its unrolled stack; a loop of one pass with a zero vector is no loop
    zero = dict(sd, **{"loop.step": torch.zeros_like(sd["loop.step"])})
    once = dict(base, loop={"start": 1, "stop": 3, "times": 1})
    no_loop = {k: v for k, v in base.items() if k != "loop"}
    assert torch.allclose(orc.forward(once, dict(zero, **{"loop.step": zero["loop.step"][:1]}), toks), orc.forward(no_loop, sd, toks), atol=1e-12)
    assert not torch.allclose(orc.forward(once, sd, toks), orc.forward(no_loop, sd, toks), atol=1e-3)
    res, eps = [], 1e-5
    orc.forward(base, sd, toks, residuals=res)
    assert len(res) == 5
    d = {k: v.double() for k, v in sd.items()}
    x0 = d["embed"][torch.tensor(toks)]
    # the stream ahead of the second pass, rebuilt by hand from what the first pass left
    x = res[2] + x0 + d["loop.step"][1]
    x = x + orc.parallel_mixer(orc.unit_rms(x, eps) * d["l1.norm1"], orc.sub(d, "l1.mix."), base["layers"][1]["mixer"], eps)
    assert torch.allclose(x, res[3])                                                        # layer 1 has no feed-forward
    y = x + orc.squared_relu_mlp(orc.unit_rms(x + orc.parallel_mixer(orc.unit_rms(x, eps) * d["l2.norm1"], orc.sub(d, "l2.mix."),
                                                                     base["layers"][2]["mixer"], eps), eps) * d["l2.norm2"], orc.sub(d, "l2.mlp."))
    assert torch.allclose(y + orc.parallel_mixer(orc.unit_rms(x, eps) * d["l2.norm1"], orc.sub(d, "l2.mix."), base["layers"][2]["mixer"], eps), res[4])
    # each half is normed before the sum: scaling one half's output product changes next to nothing
    loud = dict(sd, **{"l0.mix.left.o": sd["l0.mix.left.o"] * 50.0})
    assert float((orc.forward(base, loud, toks) - ref).abs().max()) < 1e-2 * float(ref.std())
