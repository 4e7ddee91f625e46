"""Configuration of the Lazulix decoder, its weight list, schedule and cache needs, and the plain functions against
hand-made cases (every other test of this design leans on them)."""
import copy
import math

import pytest
import torch

import lazulix_models as M
from plain import lazulix_plain as P
from plain.llama_plain import read_model_folder
from spissa_b200.cache import CacheManager
from spissa_b200.config import ConfigError, LazulixConfig, config_from_dict
from spissa_b200.engine.model import Model
from spissa_b200.parts import CacheBundle, KVCacheRequest, StateRequest
from spissa_b200.parts.rope import rotary_amplitude, rotary_inv_freq
from spissa_b200.weights import write_random_model

CFG = M.model(40, 90, [M.layer("attention_2", M.att(4, 2, 12, 8, rot=6, base=100.0, scaling=(2.0, 64, 8.0, 1.0)), M.dense(56, 0.7)),
                       M.layer("mlstm", M.mem(3, 6, 10, 5.0)),
                       M.layer("attention_2", M.att(6, 2, 12, 8, rot=6, base=100.0, kv_from=0), M.dense(24)),
                       M.layer("attention", M.att(2, 1, 14, 14))], scale=3.5, eps=1e-4)


def test_registry_finds_the_architecture_and_the_configuration_round_trips():
    cfg = config_from_dict(CFG)
    assert isinstance(cfg, LazulixConfig)
    assert cfg.to_dict() == CFG
    again = config_from_dict(LazulixConfig(**{**cfg.__dict__, "raw": None}).to_dict())
    assert again.layers == cfg.layers and again.embedding_scale == 3.5 and again.norm_eps == 1e-4


def test_absent_keys_mean_not_there():
    bare = dict(architecture="Lazulix", vocab=30, width=16, norm=dict(eps=1e-5),
                layers=[dict(type="attention", mixer=dict(heads=2, dim=8, scale=0.3)), dict(type="mlstm", mixer=dict(heads=2, dim=4, gate_cap=3.0))])
    cfg = config_from_dict(bare)
    assert cfg.embedding_scale == 1.0
    model = Model(cfg.to_spec())
    shapes = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert "l0.norm2" not in shapes and "l0.mlp.up" not in shapes and "l0.mix.g" not in shapes and "l0.mix.q.norm" not in shapes
    assert shapes["l0.mix.k"] == shapes["l0.mix.v"] == (16, 16) and shapes["l1.mix.v"] == (8, 16)
    assert model.cache_requests()[0] == KVCacheRequest(2, 8, None)


def test_weight_list():
    shapes = {s.name: tuple(s.shape) for s in Model(config_from_dict(CFG).to_spec()).weight_specs()}
    assert shapes["embed"] == (90, 40) and shapes["final.norm"] == (40,) and "head" not in shapes
    for i in range(4):
        assert shapes[f"l{i}.norm1"] == shapes[f"l{i}.norm1b"] == (40,)
    assert shapes["l0.norm2"] == shapes["l0.norm2b"] == (40,) and "l1.norm2b" not in shapes
    assert shapes["l0.mix.q"] == (48, 40) and shapes["l0.mix.k"] == (24, 40) and shapes["l0.mix.v"] == (16, 40)
    assert shapes["l0.mix.q.b"] == (48,) and shapes["l0.mix.k.b"] == (24,) and shapes["l0.mix.v.b"] == (16,)
    assert shapes["l0.mix.q.norm"] == shapes["l0.mix.k.norm"] == (12,)
    assert shapes["l0.mix.g"] == (32, 40) and shapes["l0.mix.o"] == (40, 32)
    assert shapes["l1.mix.q"] == shapes["l1.mix.k"] == (18, 40) and shapes["l1.mix.v"] == shapes["l1.mix.g"] == (30, 40)
    assert shapes["l1.mix.norm"] == (30,) and shapes["l1.mix.i"] == shapes["l1.mix.f"] == (3, 40)
    assert shapes["l1.mix.i.b"] == shapes["l1.mix.f.b"] == (3,) and shapes["l1.mix.o"] == (40, 30)
    assert {k for k in shapes if k.startswith("l2.mix.")} == {"l2.mix." + k for k in ("q", "q.b", "q.norm", "g", "o")}
    assert shapes["l2.mix.q"] == (72, 40) and shapes["l2.mix.o"] == (40, 48)
    assert shapes["l0.mlp.gate"] == shapes["l0.mlp.up"] == (56, 40) and shapes["l0.mlp.down"] == (40, 56)
    assert {k for k in shapes if k.startswith("l3.mix.")} == {"l3.mix." + k for k in ("q", "k", "v", "q.b", "k.b", "v.b", "o")}


def test_schedule_and_caches():
    spec = config_from_dict(CFG).to_spec()
    assert [(e.layer, e.cache, e.writes_cache) for e in spec.schedule] == [(0, 0, True), (1, 1, True), (2, 0, False), (3, 3, True)]
    reqs = Model(spec).cache_requests()
    assert reqs == {0: KVCacheRequest(2, 12, None, v_head_dim=8), 3: KVCacheRequest(1, 14, None),
                    1: CacheBundle.of(state=StateRequest((3, 6, 10), torch.float32), nm=StateRequest((3, 7), torch.float32))}
    cache = CacheManager(reqs, max_tokens=64 * 4, max_seqs=2, page_size=64, dtype=torch.float32, device="cpu")
    step = type("S", (), dict(page_tables={g: None for g in cache.kv_groups}, token_seq=None, positions=None, seq_row=None))
    mine, its = cache.view(0, step, True), cache.view(0, step, False)
    assert mine.k_pool.data_ptr() == its.k_pool.data_ptr() and mine.writes and not its.writes
    assert tuple(mine.v_pool.shape[1:]) == (2, 64, 8)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="attention_3"), "known mixers"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "scaling"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=-1.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["embedding"].update(scale="big"), "scale"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_bad_configurations_are_refused_with_the_field_named(change, word):
    bad = copy.deepcopy(CFG)
    change(bad)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(bad)


# ---------------------------------------------------------------------------------------------- the plain functions
def test_plain_memory_by_hand():
    one = torch.ones(2, 1, 1, dtype=torch.float64)
    i, f = torch.tensor([[-1.0], [0.5]], dtype=torch.float64), torch.tensor([[-0.25], [-0.5]], dtype=torch.float64)
    k, v = torch.tensor([[[2.0]], [[3.0]]], dtype=torch.float64), torch.tensor([[[5.0]], [[7.0]]], dtype=torch.float64)
    o, S, n, m = P.matrix_memory(one, k, v, i, f)
    # the maximum starts at 0: after the first token it is max(−0.25 + 0, −1), not −1
    assert math.isclose(float(m), 0.5) and math.isclose(float(n), math.exp(-2.0) * 2.0 + 3.0)
    first = math.exp(-0.75)
    assert math.isclose(float(o[0]), first * 10.0 / (max(first * 2.0, math.exp(0.25)) + 1e-6))
    n1 = math.exp(-0.25 - 0.5 - 0.5) * first * 2.0 + 3.0
    assert math.isclose(float(o[1]), (math.exp(-1.25) * first * 10.0 + 21.0) / (max(n1, math.exp(-0.5)) + 1e-6))


def test_plain_gates_norms_and_unit():
    w = {"i": torch.tensor([[100.0]], dtype=torch.float64), "i.b": torch.zeros(1, dtype=torch.float64),
         "f": torch.tensor([[-100.0]], dtype=torch.float64), "f.b": torch.zeros(1, dtype=torch.float64)}
    i, f = P.capped_gates(torch.ones(1, 1, dtype=torch.float64), w, "", 2.0)
    assert math.isclose(float(i), 2.0) and math.isclose(float(f), -math.log(1 + math.exp(2.0)))
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    assert torch.allclose(P.layer_norm(x, torch.tensor([2.0, 5.0], dtype=torch.float64), 3.0), torch.tensor([[-1.0, 2.5]], dtype=torch.float64))
    u = {"gate": torch.tensor([[3.0]], dtype=torch.float64), "up": torch.tensor([[-4.0]], dtype=torch.float64), "down": torch.ones(1, 1, dtype=torch.float64)}
    got = P.clamped_unit(torch.ones(1, 1, dtype=torch.float64), u, "", 0.5)       # gate 0.5 (only from above), up −0.5
    assert math.isclose(float(got), 0.5 / (1 + math.exp(-0.851)) * 0.5)
    low = P.clamped_unit(-torch.ones(1, 1, dtype=torch.float64), u, "", 0.5)
    assert math.isclose(float(low), -3.0 / (1 + math.exp(1.702 * 3.0)) * 1.5)


def test_plain_rotation_and_the_librarys_tables_agree():
    for dims, base, sc in ((24, 20.0, (2.0, 64, 8.0, 1.0)), (8, 1e4, (4.0, 4096, 32.0, 1.0)), (6, 30.0, (5.0, 40, 3.0, 1.0)), (16, 70.0, None)):
        scaling = dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None
        f, amp = P.pair_frequencies(dict(dims=dims, base=base, scaling=scaling))
        lib = rotary_inv_freq(base, dims, dict(scaling, type="ramp") if sc else None)
        assert torch.allclose(lib.double(), torch.tensor(f, dtype=torch.float64), rtol=1e-6)
        assert math.isclose(amp, rotary_amplitude(dict(scaling, type="ramp") if sc else None))
    v = torch.zeros(3, 1, 5, dtype=torch.float64)
    v[:, 0, 1] = v[:, 0, 4] = 1.0                                  # dim 1 pairs with dim 3, at base^(−1/2); dim 4 passes
    r = P.rotate_halves(v, dict(dims=4, base=16.0))
    assert torch.allclose(r[2, 0], torch.tensor([0.0, math.cos(0.5), 0.0, math.sin(0.5), 1.0], dtype=torch.float64))


def test_plain_grouped_heads_and_a_model_from_a_random_folder(tmp_path):
    q, k = torch.zeros(1, 4, 2, dtype=torch.float64), torch.zeros(1, 2, 2, dtype=torch.float64)
    v = torch.tensor([[[1.0], [2.0]]], dtype=torch.float64)
    assert P.causal_mix(q, k, v, 1.0)[0, :, 0].tolist() == [1.0, 1.0, 2.0, 2.0]
    write_random_model(config_from_dict(CFG), tmp_path, seed=4, std=0.1, norm_std=0.1)
    cfg, w = read_model_folder(tmp_path)
    toks = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5, 8, 9, 7, 9]
    layers = []
    full = P.forward(cfg, w, toks, layers_out=layers)
    assert full.shape == (15, 90) and len(layers) == 4
    assert torch.allclose(P.forward(cfg, w, toks[:9]), full[:9], atol=1e-12)          # a later token changes nothing earlier
    assert not torch.allclose(P.forward(cfg, w, [8] + toks[1:])[14], full[14], atol=1e-9)
