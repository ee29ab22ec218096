"""Small Bipulorn configurations with random weights for the tests, and their plain float64 logits.

Configurations that differ from each other in every size.  ``B1``: all three mixers, grouped key/value heads beside grouped
B and C, a window that is no multiple of a page, a rotation over part of a head slowed down, norm parts that cross heads, a
feed-forward behind most layers and one layer without.  ``B2``: one key/value head a query head, a window wider than most
requests, a rotation over whole heads, a one-tap convolution, one group of B and C, one norm part, a temperature of 1 (decays
that forget within a few tokens), a low gate cap, no identity experts, no scale of the routing weights, a cap on the logits
that bites.  ``B3``: sizes that are multiples of two at most, a window of three places and one of one place, no rotation, no
window, no cap on the logits, one head, one expert of each kind.
"""
import json
import os

import torch

import plain_bipulorn


def gla(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}


def mlstm(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def att(heads, kv_heads, dim, vdim, scale, window=None, rot=None, base=10000.0, factor=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    return m


def ssd(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def pair(left, right):
    return {"left": left, "right": right}


def moe(experts, top, ff, identity=None, scale=None, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if identity is not None:
        m["router"]["identity"] = identity
    if scale is not None:
        m["router"]["scale"] = scale
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    kind = "parallel" if "left" in mixer else ("gla" if "tau" in mixer else "mlstm")
    return {"type": kind, "mixer": mixer, "mlp": mlp}


B1 = {"architecture": "Bipulorn", "vocab": 311, "width": 72, "norm": {"eps": 1e-5}, "logit_softcap": 20.0,
      "layers": [layer(pair(att(4, 2, 16, 24, 0.3, window=21, rot=8, base=700.0, factor=3.0), ssd(6, 16, 24, 3, 4, 4)),
                       moe(5, 2, 24, identity=3, scale=1.7, shared=40)),
                 layer(gla(3, 16, 40, 8.0, 10), moe(4, 3, 32, identity=2, scale=0.8, shared=24)),
                 layer(mlstm(2, 24, 16, 9.0)),
                 layer(pair(att(3, 1, 24, 16, 0.25, window=40, rot=24, base=50.0), ssd(4, 24, 16, 2, 1, 2)),
                       moe(6, 1, 16, identity=1, scale=2.2, shared=56))]}
B2 = {"architecture": "Bipulorn", "vocab": 263, "width": 64, "norm": {"eps": 1e-6}, "logit_softcap": 3.0,
      "layers": [layer(mlstm(3, 8, 48, 2.5), moe(7, 4, 40, shared=16)),
                 layer(pair(att(3, 3, 8, 40, 0.5, window=90, rot=8, base=20.0, factor=0.5), ssd(2, 40, 72, 1, 1, 1)),
                       moe(3, 2, 24, identity=4)),
                 layer(gla(2, 72, 16, 1.0, 33), moe(4, 2, 72, identity=0, scale=1.0, shared=8))]}
B3 = {"architecture": "Bipulorn", "vocab": 83, "width": 50, "norm": {"eps": 1e-5},
      "layers": [layer(gla(1, 10, 6, 3.0, 1), moe(1, 1, 14, identity=1, scale=0.5, shared=10)),
                 layer(pair(att(3, 1, 10, 6, 0.4, window=3, rot=6, base=30.0), ssd(3, 6, 5, 3, 3, 3)), moe(2, 2, 22)),
                 layer(mlstm(1, 6, 10, 4.0), moe(3, 1, 10, identity=2, scale=3.0, shared=18)),
                 layer(pair(att(2, 2, 6, 10, 0.3), ssd(1, 14, 3, 1, 2, 5))),
                 layer(pair(att(1, 1, 2, 4, -0.7, window=1), ssd(2, 3, 1, 2, 2, 2)))]}
CONFIGS = {"B1": B1, "B2": B2, "B3": B3}
SIGMA = {"B1": 0.15, "B2": 0.15, "B3": 0.2}


def single_layer(mixer, mlp=None, **changes):
    """A model of ONE layer (a mechanism alone)."""
    raw = {"architecture": "Bipulorn", "vocab": 120, "width": 48, "norm": {"eps": 1e-5}, "logit_softcap": 15.0,
           "layers": [layer(mixer, mlp)]}
    raw.update(changes)
    return raw


def write_model(folder, raw, seed, sigma):
    from pih_b200.config import config_from_dict
    from pih_b200.weights import write_random_model
    return write_random_model(str(folder), config_from_dict(raw), seed=seed, sigma=sigma)


def load_plain(model_dir):
    from pih_b200.weights.safetensors_io import SafetensorsFile
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with SafetensorsFile(os.path.join(model_dir, "model.safetensors")) as sf:
        w = {n: sf.read_tensor(n).to(torch.float64) for n in sf.names()}
    return cfg, w


_LOGITS = {}


def plain_logits(model_dir, requests):
    """{rid: float64 logits [len, vocab]} of the plain implementation, cached per (folder, request)."""
    cfg = w = None
    out = {}
    for rid, toks in requests.items():
        key = (model_dir, tuple(toks))
        if key not in _LOGITS:
            if cfg is None:
                cfg, w = load_plain(model_dir)
            _LOGITS[key] = plain_bipulorn.model_layers(cfg, w, toks)[1]
        out[rid] = _LOGITS[key]
    return out


def random_config(seed):
    """A configuration drawn at random: sizes (also odd ones and ones that no fast kernel takes), the order of layers,
    every constant."""
    import random
    rnd = random.Random(seed)
    layers = []
    for _ in range(rnd.randint(2, 5)):
        kind = rnd.random()
        if kind < 0.3:
            mixer = gla(rnd.choice([1, 2, 3, 5]), rnd.choice([4, 8, 16, 20, 40, 64, 72]), rnd.choice([4, 8, 24, 40, 66, 136]),
                        rnd.choice([1.0, 4.0, 16.0]), rnd.choice([1, 6, 16, 40]))
        elif kind < 0.6:
            mixer = mlstm(rnd.choice([1, 2, 3]), rnd.choice([4, 8, 16, 20, 40, 64, 72]), rnd.choice([4, 8, 24, 40, 66, 136]),
                          rnd.choice([1.5, 6.0, 15.0]))
        else:
            kv, g = rnd.choice([1, 2, 3]), rnd.choice([1, 2, 4])
            dim = rnd.choice([4, 8, 12, 16, 24, 32, 40, 64, 72])
            left = att(kv * g, kv, dim, rnd.choice([4, 8, 12, 16, 24, 40, 64, 72, 130]), rnd.uniform(0.1, 0.6),
                       window=rnd.choice([1, 2, 5, 8, 17, 31, 64, 300]),
                       rot=rnd.choice([None] + [d for d in (2, 4, 8, 12, 16, 24, 32, 40, 64, 72) if d <= dim]),
                       base=rnd.choice([10.0, 1e4, 2e5]), factor=rnd.choice([None, 2.0, 8.0]))
            groups, per = rnd.choice([1, 2, 3]), rnd.choice([1, 2, 4])
            vdim = rnd.choice([4, 6, 8, 16, 24, 40, 64])
            inner = groups * per * vdim
            right = ssd(groups * per, vdim, rnd.choice([1, 4, 8, 16, 20, 40, 72]), groups,
                        rnd.choice([n for n in (1, 2, 3, 4, 6, 8) if inner % n == 0 and inner >= 4 * n]), rnd.choice([1, 2, 4]))
            mixer = pair(left, right)
        experts, identity = rnd.choice([1, 3, 6, 9]), rnd.choice([None, 0, 2, 5])
        mlp = moe(experts, rnd.randint(1, experts + (identity or 0)), rnd.choice([8, 24, 50]), identity=identity,
                  scale=rnd.choice([None, 0.7, 2.0]), shared=rnd.choice([None, 16, 40, 62]))
        layers.append(layer(mixer, rnd.choice([None, mlp, mlp])))
    raw = {"architecture": "Bipulorn", "vocab": rnd.choice([97, 256, 301]), "width": rnd.choice([40, 56, 64, 74, 96, 136]),
           "norm": {"eps": rnd.choice([1e-5, 1e-6])}, "layers": layers}
    if rnd.random() < 0.8:
        raw["logit_softcap"] = rnd.choice([2.0, 10.0, 40.0])
    return raw
