"""Tibopel without a GPU: the configuration reader and its refusals, the checkpoint table against the reference's, joined weights and shared
modules, the cache manager's bookkeeping, and properties of the slow reference itself (so that a GPU test that agrees with it agrees
with the mechanism)."""
import copy
import json
import math

import pytest
import torch

from oracle import tibopel as orc


def test_config_reader_and_refusals():
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.tibopel_modeling import TibopelConfig, tensor_shapes
    raw = orc.random_config()
    cfg = TibopelConfig(raw)
    assert cfg.model_type == "tibopel" and cfg.hidden_size == 40 and cfg.vocab_size == 72 and cfg.norm_eps == 1e-5 and cfg.logit_softcap == 15.0
    assert cfg.num_hidden_layers == 4 and [cfg.weight_layer(i) for i in range(4)] == [0, 1, 2, 1]
    assert tensor_shapes(raw) == orc.tensor_shapes(raw)
    for other in (dict(mlp=(None, "moe")), dict(shared=None, identity=0), dict(shares=(), scaling=None, chunk=None, rot_dims=None, cap=None)):
        c = orc.random_config(**other)
        assert tensor_shapes(c) == orc.tensor_shapes(c) and TibopelConfig(c).num_hidden_layers == 4
    assert TibopelConfig(orc.random_config(cap=None)).logit_softcap == 0.0
    chain = copy.deepcopy(raw)
    chain["layers"].append({**chain["layers"][3], "weights_of": 3})
    assert TibopelConfig(chain).weight_layer(4) == 1
    with pytest.raises(ValueError):
        TibopelConfig(dict(raw, architecture="Other"))
    for change in (lambda c: c["layers"][3].update(weights_of=9), lambda c: c["layers"][3].update(weights_of=3), lambda c: c["layers"][3].update(weights_of=0),
                   lambda c: c["layers"][3]["mixer"].update(heads=7)):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ValueError):
            TibopelConfig(bad)
    for change in (lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0]["mlp"].update(kind="dense")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(NotImplementedError):
            TibopelConfig(bad)


def test_engine_recognises_the_architecture(tmp_path):
    import tgis_b200  # noqa: F401
    from tgis_b200.inference_engine import FLASH_TYPES, OWN_CONFIG_ARCHITECTURES, load_config
    with open(tmp_path / "config.json", "w") as f:
        json.dump(orc.random_config(), f)
    cfg = load_config(str(tmp_path))
    assert cfg.model_type == "tibopel" and cfg.model_type in FLASH_TYPES and cfg.architecture in OWN_CONFIG_ARCHITECTURES


class _Weights:
    def __init__(self, sd):
        from tgis_b200.utils.dist import FakeGroup
        self.sd, self.dtype, self.device, self.process_group = sd, torch.float32, "cpu", FakeGroup(0, 1)

    def get_tensor(self, name):
        return self.sd[name]


def test_modules_joined_weights_and_stores():
    import tgis_b200  # noqa: F401
    from tgis_b200.models.custom_modeling.tibopel_modeling import TibopelConfig, TibopelForCausalLM
    from tgis_b200.utils.paged import HybridCacheManager
    cfg = orc.random_config()
    sd = orc.random_state_dict(cfg)
    model = TibopelForCausalLM(TibopelConfig(cfg), _Weights(sd))
    layers = model.model.layers
    assert layers[3].mixer is layers[1].mixer and layers[3].mlp is layers[1].mlp and layers[0].mixer is not layers[2].mixer
    assert [l.index for l in layers] == [0, 1, 2, 3] and model.logit_softcap == 15.0
    a, r, m = layers[0].mixer, layers[1].mixer, layers[0].mlp
    # the gate's rows run with q / k / v, without a bias; the shared expert's gate row runs with the router
    assert a.w_in.shape == (6 * 10 + 2 * 10 + 2 * 12 + 6, 40) and torch.equal(a.b_in[:60], sd["l0.mix.q.b"]) and float(a.b_in[104:].abs().max()) == 0.0
    assert torch.equal(a.b_o, sd["l0.mix.o.b"]) and a.qk_interleaved
    assert m.routed.w_router.shape == (5 + 2 + 1, 40) and torch.equal(m.routed.w_router[7:], sd["l0.mlp.shared.sg"]) and m.routed.n_route == 7
    assert m.routed.w_gate_up.shape == (5, 12, 40) and m.routed.w_down.shape == (5, 40, 12)
    assert r.w_in.shape == (18 + 20 + 6, 40) and r.sink.dtype == torch.float32 and torch.equal(r.w_uk_t[1].t(), sd["l1.mix.uk"][8:16])
    mgr = HybridCacheManager([l.mixer.cache_spec() for l in layers], torch.float32, "cpu", total_num_gpu_blocks=5, num_state_slots=2)
    assert mgr.layer_pages(0).shape == (5, 16, 2 * (10 + 12)) and mgr.layer_pages(1).shape == (5, 16, 20 + 6)
    assert mgr.layer_pages(1).data_ptr() != mgr.layer_pages(3).data_ptr()      # shared tensors, a store each
    for name, bad in (("l1.mix.sink", sd["l1.mix.sink"][:2]), ("l0.mlp.router", sd["l0.mlp.router"][:5]), ("l1.mix.uq", sd["l1.mix.uq"][:-1])):
        with pytest.raises(ValueError):
            TibopelForCausalLM(TibopelConfig(cfg), _Weights(dict(sd, **{name: bad})))


def test_rotary_scaling_rules_do_not_mix():
    import tgis_b200  # noqa: F401
    from tgis_b200.utils.mixers import ScaledRotaryTables
    wave = ScaledRotaryTables(16, 5000.0, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60})
    rates = torch.tensor(orc.turn_rates(16, 5000.0, wave.scaling), dtype=torch.float64)
    assert torch.allclose(wave.frequencies(), rates, rtol=1e-12) and wave.amplitude() == 1.0
    yarn = ScaledRotaryTables(16, 5000.0, {"factor": 4.0, "fast": 16.0, "slow": 1.0, "original": 60})
    assert yarn.amplitude() == pytest.approx(0.1 * math.log(4.0) + 1.0) and not torch.allclose(yarn.frequencies(), rates)
    assert ScaledRotaryTables(16, 5000.0).amplitude() == 1.0


# ------------------------------------------------------------------------------------------------ the reference itself
def _layer(kind, seed=1, **kw):
    cfg = orc.random_config(order=(kind,), shares=(), **kw)
    sd = {k: v.double() for k, v in orc.random_state_dict(cfg, seed=seed).items()}
    return cfg, cfg["layers"][0]["mixer"], orc.sub(sd, "l0.mix."), orc.sub(sd, "l0.mlp.")


def _rows(n, width, seed=0):
    return torch.randn(n, width, dtype=torch.float64, generator=torch.Generator().manual_seed(seed))


def test_reference_chunks_and_rotation():
    cfg, m, p, _ = _layer("attention", chunk=8)
    h = _rows(30, 40)
    full = orc.chunk_attention(h, p, m)
    h2 = h.clone()
    h2[:16] = _rows(16, 40, 5)
    other = orc.chunk_attention(h2, p, m)
    assert torch.allclose(other[16:], full[16:], atol=1e-12) and not torch.allclose(other[15], full[15], atol=1e-4)
    # scores depend on position differences: a chunk at other positions gives the same rows (the rotation is the only use of the position)
    assert torch.allclose(orc.chunk_attention(h[8:16], p, m), full[8:16], atol=1e-9)
    x = _rows(3, 6).view(3, 1, 6)
    y = orc.rotate_neighbours(x, torch.tensor([0, 1, 7]), [0.3, 0.01])
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    assert torch.allclose(torch.complex(y[2, 0, 0], y[2, 0, 1]), torch.complex(x[2, 0, 0], x[2, 0, 1]) * torch.exp(torch.tensor(2.1j, dtype=torch.complex128)))


def test_reference_latent_attention_and_sink():
    cfg, m, p, _ = _layer("latent_attention")
    h = _rows(20, 40)
    full = orc.latent_attention(h, p, m, 1e-5)
    assert torch.allclose(orc.latent_attention(h[:12], p, m, 1e-5), full[:12], atol=1e-12)      # causal
    gone = orc.latent_attention(h, dict(p, sink=torch.full_like(p["sink"], 200.0)), m, 1e-5)
    assert float(gone.abs().max()) < 1e-12                                                       # a sink that takes everything
    s = torch.tensor([[[1.0, -math.inf], [0.5, 2.0]]], dtype=torch.float64)
    w = orc.sink_softmax(s, torch.tensor([1.0], dtype=torch.float64))
    assert w[0, 0, 0] == pytest.approx(0.5) and w[0, 0, 1] == 0.0
    assert w[0, 1, 1] == pytest.approx(math.exp(2.0) / (math.exp(0.5) + math.exp(2.0) + math.exp(1.0)))
    # the last head's output alone, rebuilt in the absorbed form
    H, d, r, R, dv = 3, 8, 6, 20, 14
    q = ((orc.unit_rms(h @ p["dq"].T, 1e-5) * p["dq.norm"]) @ p["uq"].T).view(20, H, d + r)[:, 2]
    down = h @ p["dkv"].T
    c = orc.unit_rms(down[:, :R], 1e-5) * p["dkv.norm"]
    rates, pos = orc.turn_rates(6, 200.0), torch.arange(20)
    qr, kr = orc.rotate_neighbours(q[:, None, d:], pos, rates)[:, 0], orc.rotate_neighbours(down[:, None, R:], pos, rates)[:, 0]
    sc = ((q[:, :d] @ p["uk"][2 * d:]) @ c.T + qr @ kr.T) * m["scale"]
    sc = sc.masked_fill(torch.triu(torch.ones(20, 20, dtype=torch.bool), 1), -math.inf)
    o = (orc.sink_softmax(sc[None], p["sink"][2:])[0] @ c) @ p["uv"][2 * dv:].T
    mine = dict(p, o=torch.eye(H * dv, dtype=torch.float64))
    assert torch.allclose(orc.latent_attention(h, mine, m, 1e-5)[:, 2 * dv:], o, atol=1e-10)


def test_reference_routing():
    s = torch.tensor([[0.4, 0.3, 0.2, 0.1]], dtype=torch.float64)
    ids, w = orc.pick_experts(s, torch.tensor([0.0, 0.0, 0.15, 0.0]), 2)
    assert sorted(ids[0].tolist()) == [0, 2] and float(w[0, ids[0].tolist().index(2)]) == pytest.approx(0.2 / 0.6)
    cfg, _, _, p = _layer("attention", experts=2, identity=3, top=2, shared=None)
    h, f = _rows(5, 40), cfg["layers"][0]["mlp"]
    only = dict(p, correction=torch.tensor([0.0, 0.0, 9.0, 0.0, 9.0], dtype=torch.float64))
    assert torch.allclose(orc.routed_experts(h, only, f), h, atol=1e-12)          # identity picks only: the weights sum to one
    one = dict(p, correction=torch.tensor([0.0, 9.0, 0.0, 0.0, 9.0], dtype=torch.float64))
    sc = torch.softmax(h @ p["router"].T, -1)
    a = (sc[:, 1] / (sc[:, 1] + sc[:, 4]))[:, None]
    want = a * (torch.relu(h @ p["e1.up"].T) ** 2 @ p["e1.down"].T) + (1 - a) * h
    assert torch.allclose(orc.routed_experts(h, one, f), want, atol=1e-10)


def test_reference_layer_reads_the_stream_once():
    """both halves of a layer read the same stream, and a layer that shares tensors is computed like its source"""
    cfg = orc.random_config(order=("attention", "attention"), shares=(None, 0), cap=None)
    sd = orc.random_state_dict(cfg, seed=3)
    toks, res = [5, 9, 11, 60], []
    lg = orc.forward(cfg, sd, toks, residuals=res)
    s = {k: v.double() for k, v in sd.items()}
    x = s["embed"][toks]
    for i in range(2):
        layer, eps = cfg["layers"][i], 1e-5
        x = x + orc.chunk_attention(orc.unit_rms(x, eps) * s["l0.norm1"], orc.sub(s, "l0.mix."), layer["mixer"]) + \
            orc.routed_experts(orc.unit_rms(x, eps) * s["l0.norm2"], orc.sub(s, "l0.mlp."), layer["mlp"])
        assert torch.allclose(res[i], x, atol=1e-12)
    z = (orc.unit_rms(x, 1e-5) * s["final.norm"]) @ s["head"].T
    assert torch.allclose(lg, z, atol=1e-12)
    capped = orc.forward(dict(cfg, logit_softcap=2.0), sd, toks)
    assert torch.allclose(capped, 2.0 * torch.tanh(z / 2.0), atol=1e-12) and float(capped.abs().max()) <= 2.0
