"""Small Luvavik configurations with random weights for tests, and models whose weights make one token stand out."""
import math
import os

import torch

from plain.llama_plain import read_model_folder


def rec(width, blocks, taps):
    return dict(width=width, blocks=blocks, conv=taps)


def lat(heads, dim, rot_dim, vdim, rank, base=10000.0, scale=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale or 1.0 / math.sqrt(dim + rot_dim))
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
    return m


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, identity=0):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, identity=identity, top=top))


def layer(mixer, mlp=None):
    return dict(type="rglru" if "blocks" in mixer else "latent_attention", mixer=mixer, mlp=mlp)


def model(width, vocab, layers, loop=None, mult=0.8, scale=1.5, eps=1e-5):
    out = dict(architecture="Luvavik", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, logit_scale=scale,
               layers=layers)
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# sizes that differ from one another everywhere: recurrences of one part and of many, parts whose size is a multiple of
# eight and not, convolutions of 1 to 6 taps; latent rows whose size the tensor-core kernels take and not, key and value
# sizes equal or not, no rotated part, a single head; dense, routed and absent feed-forwards; experts with and without
# identity experts, one expert per token, as many as there are; loops of one, two and three passes over one, two or all
# layers, with a mixer of either kind first, or no loop; multipliers of 1, below and above it
CONFIGS = {
    "a": model(64, 200, [layer(lat(3, 8, 4, 12, 20, base=100.0), dense(56)),
                         layer(rec(96, 4, 3), moe(6, 2, 24, identity=3)),
                         layer(lat(2, 16, 6, 8, 24, base=500.0)),
                         layer(rec(40, 1, 1), dense(48))],
               loop=(1, 3, 3), mult=0.6, scale=0.5, eps=1e-4),
    "b": model(128, 333, [layer(rec(128, 8, 4), moe(5, 1, 64)),
                          layer(lat(5, 16, 16, 32, 112), moe(9, 4, 40, identity=1)),
                          layer(rec(160, 5, 2), dense(96)),
                          layer(lat(2, 32, 16, 16, 80, base=50.0), dense(64))],
               loop=(0, 2, 2), mult=1.3, scale=3.0),
    # nothing a multiple of four: the paths without wide accesses; a latent without a rotated part; every expert chosen
    "c": model(50, 97, [layer(lat(3, 5, 6, 7, 11, base=30.0), moe(3, 3, 10)),
                        layer(rec(30, 3, 6), moe(2, 3, 14, identity=2)),
                        layer(lat(1, 6, 0, 3, 13)),
                        layer(rec(55, 5, 4))],
               loop=(3, 4, 2), mult=0.9, scale=1.0, eps=1e-3),
    "d": model(96, 150, [layer(rec(64, 2, 5), dense(64)), layer(lat(4, 24, 8, 24, 248), moe(12, 3, 32, identity=4)),
                         layer(rec(136, 17, 4), moe(4, 2, 72, identity=7))],
               mult=1.0, scale=1.0),
    "e": model(72, 120, [layer(lat(6, 12, 4, 20, 28, base=20.0), dense(40)), layer(rec(48, 6, 2), moe(7, 5, 16, identity=2))],
               loop=(0, 2, 1), mult=0.5, scale=0.25),
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
        last = name.split(".")[-1]
        if last == "embed":
            draw(name, 1.0)
        elif name == "loop.step":
            draw(name, 0.7)
        elif last == "lam":                          # decays from "keeps hundreds of tokens" to "forgets the last one"
            draw(name, 2.5, -4.0)
        elif last in ("ra", "ri"):
            draw(name, 1.5 / math.sqrt(w[name].shape[-1]))
        elif last == "conv":
            draw(name, 0.6)
        elif last == "b":
            draw(name, 0.4)
        elif last == "router":                       # so that few choices are close calls
            w[name] = (8.0 * w[name].float()).to(w[name].dtype)
        elif last == "correction":
            draw(name, 0.15)
        elif last == "g":
            w[name] = (5.0 * w[name].float()).to(w[name].dtype)
        elif "norm" in last:
            w[name] = (w[name].float() + 0.3 * torch.randn(w[name].shape, generator=g)).to(w[name].dtype)
    if patch:
        patch(w)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    return read_model_folder(folder)


# ---------------------------------------------------------------------------------------------- one token that stands out
NEEDLE, DIRECTION, CONST = 7, 3, 5


def _mark_embedding(w):
    """Token ``NEEDLE`` alone has a large entry along ``DIRECTION``; every token the same large one along ``CONST``."""
    w["embed"][:, DIRECTION] = 0.0
    w["embed"][:, CONST] = 5.0
    w["embed"][NEEDLE, DIRECTION] = 6.0
    for name in ("l0.norm1",):
        w[name][DIRECTION] = w[name][CONST] = 1.0


def rows_needle_model(heads=2, dim=8, rot_dim=4, vdim=6, rank=20):
    """An attention that gives almost all its weight to the row of token ``NEEDLE``, however far back it lies."""
    cfg = model(32, 64, [layer(lat(heads, dim, rot_dim, vdim, rank, base=100.0, scale=1.0))], mult=1.0, scale=1.0)

    def patch(w):
        _mark_embedding(w)
        p = "l0.mix."
        qd = dim + rot_dim
        w[p + "dkv"][:, [DIRECTION, CONST]] = 0.0
        w[p + "q"][:, [DIRECTION, CONST]] = 0.0
        w[p + "dkv"][0] = 0.0
        w[p + "dkv"][0, DIRECTION] = 4.0                         # the needle's row points along entry 0, nobody else's does
        w[p + "dkv.norm"][0] = 2.0
        for h in range(heads):
            w[p + "uk"][h * dim + dim - 1] = 0.0
            w[p + "uk"][h * dim + dim - 1, 0] = 1.0              # key dim d − 1 reads entry 0 of the row
            w[p + "q"][h * qd + dim - 1] = 0.0
            w[p + "q"][h * qd + dim - 1, CONST] = 1.0            # and every query looks along it
        w[p + "uv"][:, 0] = 3.0                                  # the needle's value stands out
        w[p + "g"][:] = 0.0                                      # every gate half open

    return cfg, patch


def recurrence_needle_model(width=24, blocks=2, taps=3, slow=True):
    """A recurrence in which token ``NEEDLE`` alone puts something large into the state. ``slow``: decays so close to one
    that it is still there hundreds of tokens later; else the state forgets at once and only the convolution's taps
    reach back."""
    cfg = model(32, 64, [layer(rec(width, blocks, taps))], mult=1.0, scale=1.0)

    def patch(w):
        _mark_embedding(w)
        p = "l0.mix."
        w[p + "x"][:] = 0.2 * w[p + "x"]
        w[p + "x"][:, CONST] = 0.0
        w[p + "x"][:, DIRECTION] = 2.0                           # u is large at the needle and at the taps behind it
        w[p + "x.b"][:] = w[p + "conv.b"][:] = 0.0               # ... and small everywhere else
        w[p + "lam"][:] = -9.0 if slow else 4.0
        w[p + "ra"][:] = 0.05 * w[p + "ra"]
        w[p + "ra.b"][:] = 0.0 if slow else 3.0
        w[p + "conv"][:] = 1.0
        w[p + "y"][:, CONST] = 0.4
        w[p + "o"][:] = 4.0 * w[p + "o"]

    return cfg, patch


def with_needle(base, place):
    toks = list(base)
    toks[place] = NEEDLE
    return toks
