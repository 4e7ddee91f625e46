"""Small Lazulix configurations with random weights for tests, and models whose weights make one token stand out."""
import math
import os

import torch

from plain.llama_plain import read_model_folder


def mem(heads, dim, vdim, cap=11.0):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def att(heads, kv, dim, vdim, rot=0, base=10000.0, scale=None, scaling=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 1.0 / math.sqrt(dim))
    if rot:
        m["rot"] = dict(dims=rot, base=base)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff, limit=1.5):
    return dict(kind="dense", ff=ff, limit=limit)


def layer(kind, mixer, mlp=None):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def model(width, vocab, layers, scale=6.0, eps=1e-5):
    return dict(architecture="Lazulix", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


# sizes that differ from one another everywhere: memories of one head and of many, key sizes above and below the value sizes,
# odd sizes, values beyond one column block; attentions of one size and of two, multiples of eight and not, grouped and not,
# wholly, partly and not rotated, with and without interpolated frequencies; a layer that reads another's keys and values,
# directly behind it and far from it, with other head counts and another scale; feed-forwards whose limits bite or hardly do
CONFIGS = {
    "a": model(64, 200, [layer("attention_2", att(4, 2, 24, 16, rot=8, base=100.0, scaling=(2.0, 64, 4.0, 1.0)), dense(64, 0.7)),
                         layer("attention_2", att(6, 2, 24, 16, rot=8, base=100.0, scaling=(2.0, 64, 4.0, 1.0), scale=0.4, kv_from=0), dense(40)),
                         layer("mlstm", mem(2, 16, 24)),
                         layer("attention", att(3, 1, 16, 16, rot=16, base=50.0), dense(48, 5.0)),
                         layer("mlstm", mem(3, 24, 8, 3.0), dense(72))], eps=1e-4),
    "b": model(128, 333, [layer("mlstm", mem(4, 32, 64, 15.0), dense(128)),
                          layer("attention", att(4, 4, 48, 32, rot=16, scaling=(4.0, 32, 8.0, 1.0)), dense(192, 0.5)),
                          layer("mlstm", mem(1, 64, 32)),
                          layer("attention_2", att(4, 2, 32, 64, rot=32, base=500.0), dense(64)),
                          layer("attention_2", att(2, 2, 32, 64, rot=16, base=70.0, scaling=(3.0, 16, 2.0, 0.5), kv_from=3))], scale=2.0),
    # nothing a multiple of four: the paths without wide accesses
    "c": model(50, 97, [layer("attention_2", att(3, 3, 10, 7, rot=6, base=30.0, scaling=(5.0, 40, 3.0, 1.0)), dense(30)),
                        layer("mlstm", mem(3, 5, 9, 7.0)),
                        layer("attention", att(2, 1, 9, 11), dense(22, 0.6)),
                        layer("attention_2", att(6, 3, 10, 7, rot=2, base=30.0, kv_from=0)),
                        layer("mlstm", mem(1, 7, 3, 2.0), dense(26))], scale=1.0, eps=1e-3),
    "d": model(96, 150, [layer("attention", att(4, 1, 72, 40, rot=24), dense(64)),
                         layer("mlstm", mem(2, 72, 40)),
                         layer("attention_2", att(20, 1, 16, 8, rot=4), dense(96, 0.9)),
                         layer("attention", att(2, 2, 16, 24, rot=16, base=200.0, scaling=(2.0, 128, 16.0, 2.0)))], scale=9.0),
    "e": model(72, 120, [layer("mlstm", mem(5, 8, 12, 1.0), dense(40, 0.3)),
                         layer("attention_2", att(5, 5, 12, 20, rot=4, base=20.0))], scale=0.5),
}
INIT = {"a": dict(seed=5, std=0.1), "b": dict(seed=9, std=0.07), "c": dict(seed=13, std=0.12), "d": dict(seed=17, std=0.09),
        "e": dict(seed=21, std=0.1)}


def make(cfg, folder, seed, std, patch=None):
    """A model folder from the library's random-weights mode, with the tensors that it draws too tamely spread out."""
    from spissa_b200.config import config_from_dict
    from spissa_b200.weights import write_random_model, write_safetensors
    write_random_model(config_from_dict(cfg), folder, seed=seed, std=std, norm_std=0.1)
    pcfg, w = read_model_folder(folder)
    g = torch.Generator().manual_seed(seed)

    def draw(name, spread, mean=0.0):
        w[name] = (mean + spread * torch.randn(w[name].shape, generator=g)).to(w[name].dtype)
    for name in sorted(w):
        parts = name.split(".")
        last = parts[-1]
        if name == "embed":
            draw(name, 0.3)
        elif name.endswith("mix.i.b"):                # input gates from "hardly takes" to "takes a lot"
            draw(name, 1.5, 0.5)
        elif name.endswith("mix.f.b"):                # forget gates from "keeps hundreds of tokens" to "forgets at once"
            draw(name, 3.0, 3.0)
        elif last in ("i", "f"):
            draw(name, 1.5 / math.sqrt(w[name].shape[-1]))
        elif last == "b":
            draw(name, 0.5)
        elif last in ("g", "gate", "up"):
            w[name] = (4.0 * w[name].float()).to(w[name].dtype)
        elif "norm" in last:
            w[name] = (w[name].float() + 0.3 * torch.randn(w[name].shape, generator=g)).to(w[name].dtype)
    for name in w:
        # a memory's keys lie near its queries: where k · q is a difference of large terms, the unit rms blows its rounding up
        # (a first token whose k · q is close to zero turns its output's sign round)
        if name.endswith("mix.k") and name[:-1] + "i" in w:
            w[name] = (w[name[:-1] + "q"].float() + 0.4 * w[name].float()).to(w[name].dtype)
    if patch:
        patch(w)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    return read_model_folder(folder)


# ---------------------------------------------------------------------------------------------- one token that stands out
NEEDLE = 7


def _mark_embedding(w, width):
    """Token ``NEEDLE`` alone has a large entry along dim 3 (the mean of its row stays near the others')."""
    w["embed"][:, 3] = 0.0
    w["embed"][NEEDLE] = 0.0
    w["embed"][NEEDLE, 3], w["embed"][NEEDLE, 4] = 6.0, -6.0


def key_needle_model(kind="attention", heads=2, kv=1, dim=16, vdim=8, shared=False):
    """An attention that gives almost all its weight to the key of token ``NEEDLE``, however far back it lies: its key is
    large along one dim that every query's bias points along (behind the rotated dims)."""
    rot = dim // 4 * 2
    layers = [layer(kind, att(heads, kv, dim, vdim, rot=rot, base=50.0, scale=1.0))]
    if shared:
        layers.append(layer("attention_2", att(heads, kv, dim, vdim, rot=rot, base=50.0, scale=1.0, kv_from=0)))
    cfg = model(32, 64, layers, scale=1.0)

    def patch(w):
        _mark_embedding(w, 32)
        for i in range(len(layers)):
            p = f"l{i}.mix."
            w[f"l{i}.norm1"][:] = 1.0
            for h in range(heads):
                w[p + "q"][h * dim:(h + 1) * dim] *= 0.2
                w[p + "q.b"][h * dim:(h + 1) * dim] = 0.0
                w[p + "q.b"][h * dim + dim - 1] = 4.0
            if i == 0:
                w[p + "k.b"][:] = 0.0
                w[p + "k"][:] *= 0.5
                for g in range(kv):
                    w[p + "k"][g * dim + dim - 1] = 0.0
                    w[p + "k"][g * dim + dim - 1, 3] = 3.0
                w[p + "v"][:, 3] = 2.0
            if (p + "q.norm") in w:
                w[p + "q.norm"][:] = 1.0
                if i == 0:
                    w[p + "k.norm"][:] = 1.0
                    w[p + "k.norm"][dim - 1] = 4.0

    return cfg, patch


def memory_needle_model(heads=2, dim=8, vdim=12, slow=True):
    """A matrix memory into which token ``NEEDLE`` alone writes something large (its input gate opens wide). ``slow``: forget
    gates so open that it is still there hundreds of tokens later; else the memory forgets at once."""
    cfg = model(32, 64, [layer("mlstm", mem(heads, dim, vdim, 13.0))], scale=1.0)

    def patch(w):
        _mark_embedding(w, 32)
        p = "l0.mix."
        w["l0.norm1"][:] = 1.0
        w[p + "i"][:] = 0.1 * w[p + "i"]
        w[p + "i"][:, 3] = 2.5                                   # the needle alone opens the input gate
        w[p + "i.b"][:] = -3.0
        w[p + "f"][:] = 0.05 * w[p + "f"]
        w[p + "f"][:, 3] = 0.0
        w[p + "f.b"][:] = 9.0 if slow else -9.0
        w[p + "o"][:] = 4.0 * w[p + "o"]
        w[p + "g"][:] = 0.0

    return cfg, patch


def with_needle(base, place):
    toks = list(base)
    toks[place] = NEEDLE
    return toks
