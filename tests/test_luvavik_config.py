"""Configuration of the Luvavik decoder, its weight list, schedule and cache needs, and the plain functions against
hand-made cases (every other test of this design leans on them)."""
import copy
import math

import pytest
import torch

import luvavik_models as M
from plain import luvavik_plain as P
from plain.llama_plain import read_model_folder
from spissa_b200.cache import CacheManager
from spissa_b200.config import ConfigError, LuvavikConfig, config_from_dict
from spissa_b200.engine.model import Model
from spissa_b200.parts import CacheBundle, KVCacheRequest, StateRequest
from spissa_b200.weights import write_random_model

CFG = M.model(40, 90, [M.layer(M.rec(24, 3, 5), M.dense(56)),
                       M.layer(M.lat(3, 8, 4, 12, 20, base=100.0), M.moe(6, 2, 16, identity=3)),
                       M.layer(M.lat(2, 6, 0, 10, 14)),
                       M.layer(M.rec(32, 1, 1), M.moe(4, 4, 8))],
              loop=(1, 3, 3), mult=0.4, scale=1.7, eps=1e-4)


def test_registry_finds_the_architecture_and_the_configuration_round_trips():
    cfg = config_from_dict(CFG)
    assert isinstance(cfg, LuvavikConfig)
    assert cfg.to_dict() == CFG
    again = config_from_dict(LuvavikConfig(**{**cfg.__dict__, "raw": None}).to_dict())
    assert again.layers == cfg.layers and again.loop == (1, 3, 3)
    assert again.residual_mult == 0.4 and again.logit_scale == 1.7 and again.norm_eps == 1e-4


def test_absent_keys_mean_not_there():
    bare = dict(architecture="Luvavik", vocab=30, width=16, norm=dict(eps=1e-5),
                layers=[dict(type="rglru", mixer=dict(width=8), mlp=None),
                        dict(type="latent_attention", mixer=dict(heads=2, dim=8, kv_rank=6, scale=0.3),
                             mlp=dict(kind="moe", expert=dict(ff=4), router=dict(experts=2, top=1)))])
    cfg = config_from_dict(bare)
    assert cfg.residual_mult == 1.0 and cfg.logit_scale == 1.0 and cfg.loop is None
    model = Model(cfg.to_spec())
    shapes = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert "loop.step" not in shapes and "l0.norm2" not in shapes
    assert shapes["l0.mix.ra"] == (1, 8, 8) and shapes["l0.mix.conv"] == (8, 1)
    assert shapes["l1.mix.q"] == (16, 16) and shapes["l1.mix.dkv"] == (6, 16) and shapes["l1.mix.uv"] == (16, 6)
    assert shapes["l1.mlp.router"] == (2, 16) and shapes["l1.mlp.correction"] == (2,)
    assert model.cache_requests() == {0: CacheBundle.of(state=StateRequest((8,), torch.float32)),
                                      1: KVCacheRequest(1, 6, None, keys_only=True)}


def test_weight_list():
    shapes = {s.name: tuple(s.shape) for s in Model(config_from_dict(CFG).to_spec()).weight_specs()}
    assert shapes["embed"] == (90, 40) and shapes["head"] == (90, 40) and shapes["final.norm"] == (40,)
    assert shapes["loop.step"] == (3, 40)
    assert shapes["l0.mix.y"] == shapes["l0.mix.x"] == (24, 40) and shapes["l0.mix.o"] == (40, 24)
    assert shapes["l0.mix.y.b"] == shapes["l0.mix.x.b"] == shapes["l0.mix.conv.b"] == shapes["l0.mix.lam"] == (24,)
    assert shapes["l0.mix.conv"] == (24, 5) and shapes["l0.mix.ra"] == shapes["l0.mix.ri"] == (3, 8, 8)
    assert shapes["l0.mix.ra.b"] == shapes["l0.mix.ri.b"] == (3, 8)
    assert shapes["l0.mlp.gate"] == (56, 40) and shapes["l0.mlp.down"] == (40, 56)
    assert shapes["l1.mix.q"] == (36, 40) and shapes["l1.mix.dkv"] == (24, 40) and shapes["l1.mix.dkv.norm"] == (20,)
    assert shapes["l1.mix.uk"] == (24, 20) and shapes["l1.mix.uv"] == (36, 20)
    assert shapes["l1.mix.g"] == (36, 40) and shapes["l1.mix.o"] == (40, 36)           # a gate per element of the heads
    assert shapes["l1.mlp.router"] == (9, 40) and shapes["l1.mlp.correction"] == (9,)   # six experts and three identities
    assert shapes["l1.mlp.e5.up"] == (16, 40) and shapes["l1.mlp.e5.down"] == (40, 16)
    assert "l1.mlp.e6.up" not in shapes and "l1.mlp.e0.gate" not in shapes and "l2.norm2" not in shapes
    assert shapes["l2.mix.q"] == (12, 40) and shapes["l2.mix.dkv"] == (14, 40)


def test_schedule_gives_every_pass_a_cache_of_its_own_and_its_row():
    spec = config_from_dict(CFG).to_spec()
    runs = [(e.layer, e.cache, e.writes_cache, e.adds_row) for e in spec.schedule]
    assert runs == [(0, 0, True, None), (1, 1, True, 0), (2, 2, True, None), (1, 3, True, 1), (2, 4, True, None), (1, 5, True, 2),
                    (2, 6, True, None), (3, 7, True, None)]
    reqs = Model(spec).cache_requests()
    assert reqs[0] == CacheBundle.of(conv=StateRequest((5, 24), torch.float32), state=StateRequest((24,), torch.float32))
    assert reqs[1] == reqs[3] == reqs[5] == KVCacheRequest(1, 24, None, keys_only=True)
    assert reqs[2] == KVCacheRequest(1, 14, None, keys_only=True)
    assert reqs[7] == CacheBundle.of(state=StateRequest((32,), torch.float32))
    cache = CacheManager(reqs, max_tokens=64 * 4, max_seqs=2, page_size=64, dtype=torch.float32, device="cpu")
    step = type("S", (), dict(page_tables={g: None for g in cache.kv_groups}, token_seq=None, positions=None, seq_row=None))
    pools = [cache.view(c, step, True).k_pool.data_ptr() for c in (1, 3, 5, 2)]
    assert len(set(pools)) == 4
    assert tuple(cache.view(0, step, True)["conv"].state.shape[1:]) == (5, 24)
    assert cache.view(7, step, True).get("conv") is None and tuple(cache.view(7, step, True)["state"].state.shape[1:]) == (32,)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="attention"), "known mixers"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=5), "blocks"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("width"), "width"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=3), "rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=2), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=10), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "top|identit"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("start"), "start"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(residual_mult="half"), "residual_mult"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_bad_configurations_are_refused_with_the_field_named(change, word):
    bad = copy.deepcopy(CFG)
    change(bad)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(bad)


# ---------------------------------------------------------------------------------------------- the plain functions
def test_plain_convolution_and_parts():
    z = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]], dtype=torch.float64)
    taps = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 2.0]], dtype=torch.float64)
    out = P.causal_conv(z, taps, torch.tensor([0.5, 0.0], dtype=torch.float64))
    assert out[:, 0].tolist() == [1.5, 12.5, 123.5] and out[:, 1].tolist() == [20.0, 40.0, 60.0]
    mats = torch.tensor([[[0.0, 1.0], [2.0, 0.0]], [[1.0, 1.0], [0.0, 3.0]]], dtype=torch.float64)
    got = P.part_products(torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=torch.float64), mats, torch.tensor([[0.0, 1.0], [0.0, 0.0]], dtype=torch.float64))
    assert got[0].tolist() == [2.0, 3.0, 7.0, 12.0]


def test_plain_recurrence_by_hand():
    r, lam = torch.tensor([[0.5], [0.25]], dtype=torch.float64), torch.tensor([0.0], dtype=torch.float64)
    la = P.decays(r, lam)
    assert math.isclose(float(la[0]), -4.0 * math.log(2.0)) and math.isclose(float(la[1]), -2.0 * math.log(2.0))
    S = P.linear_recurrence(la, torch.tensor([[2.0], [3.0]], dtype=torch.float64))
    d0, d1 = 2.0 ** -4, 2.0 ** -2
    first = math.sqrt(1 - d0 ** 2) * 2.0                           # the first token is weighed like every other
    assert math.isclose(float(S[0]), first) and math.isclose(float(S[1]), d1 * first + math.sqrt(1 - d1 ** 2) * 3.0)


def test_plain_rotation_and_router():
    v = torch.zeros(3, 1, 4, dtype=torch.float64)
    v[:, 0, 1] = 1.0                                               # dim 1 pairs with dim 3, at base^(−1/2)
    r = P.rotate_halves(v, 16.0)
    assert torch.allclose(r[2, 0], torch.tensor([0.0, math.cos(0.5), 0.0, math.sin(0.5)], dtype=torch.float64))
    w = {"router": torch.zeros(3, 2, dtype=torch.float64), "correction": torch.tensor([0.0, 1.0, 2.0], dtype=torch.float64),
         "e0.up": torch.ones(1, 2, dtype=torch.float64), "e0.down": torch.ones(2, 1, dtype=torch.float64),
         "e1.up": torch.tensor([[1.0, -3.0]], dtype=torch.float64), "e1.down": torch.tensor([[1.0], [0.0]], dtype=torch.float64)}
    a = torch.tensor([[5.0, 1.0], [1.0, 5.0]], dtype=torch.float64)
    # equal scores of a third; the correction picks the identity (place 2) and expert 1, whose relu cuts the second token
    out = P.routed_experts(a, w, "", dict(experts=2, identity=1, top=2))
    assert torch.allclose(out, torch.tensor([[(5.0 + 4.0) / 3, 1.0 / 3], [1.0 / 3, 5.0 / 3]], dtype=torch.float64))


def test_plain_layer_runs_and_a_model_from_a_random_folder(tmp_path):
    assert P.layer_runs(CFG) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert P.layer_runs(dict(layers=[1, 2])) == [(0, None), (1, None)]
    write_random_model(config_from_dict(CFG), tmp_path, seed=4, std=0.1, norm_std=0.1)
    cfg, w = read_model_folder(tmp_path)
    toks = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5, 8, 9, 7, 9]
    layers = []
    full = P.forward(cfg, w, toks, layers_out=layers)
    assert full.shape == (15, 90) and len(layers) == 8
    assert torch.allclose(P.forward(cfg, w, toks[:9]), full[:9], atol=1e-12)          # a later token changes nothing earlier
    assert not torch.allclose(P.forward(cfg, w, [8] + toks[1:])[14], full[14], atol=1e-9)
