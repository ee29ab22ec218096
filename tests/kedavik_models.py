"""Small Kedavik configurations with random weights for the tests, and their plain float64 logits.

Configurations that differ from each other in every size.  ``K1``: a loop of two layers in the middle run three times,
grouped key/value heads on both sides, a rotation over part of a head, chunks that are no multiple of a page, narrow
projections of unequal widths, values wider than keys on the left and narrower on the right, a scan with a feed-forward
and a pair without one.  ``K2``: a loop that begins with the first layer and ends with the last, one key/value head a
query head, a rotation over whole heads, a one-tap convolution beside a five-tap one, chunks wider than most requests, a
negative scale.  ``K3``: no loop, no factor on embedding or residual, sizes that are multiples of two at most, chunks of
three places, a pair that sees every key and does not rotate.
"""
import json
import os

import torch

import plain_kedavik


def scan(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def pair(left, right, left_scale, right_scale):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def att(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    return m


def dlt(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
            "gate_rank": gate_rank}


def ff(n):
    return {"kind": "dense", "ff": n}


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "mamba1", "mixer": mixer, "mlp": mlp}


K1 = {"architecture": "Kedavik", "vocab": 307, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.7},
      "residual_mult": 0.45, "loop": {"start": 1, "stop": 3, "times": 3},
      "layers": [layer(scan(88, 5, 6, 4)),
                 layer(pair(att(4, 2, 16, 24, 0.3, chunk=20, rot=8, base=500.0), dlt(4, 2, 16, 12, 3, 10, 14), 0.7, 1.3), ff(100)),
                 layer(scan(56, 20, 3, 3), ff(60)),
                 layer(pair(att(3, 1, 24, 40, 0.25, chunk=37, rot=24), dlt(2, 1, 32, 40, 4, 24, 8), 1.1, 0.6))]}
K2 = {"architecture": "Kedavik", "vocab": 259, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 2.5},
      "residual_mult": 0.8, "loop": {"start": 0, "stop": 3, "times": 2},
      "layers": [layer(pair(att(3, 3, 8, 16, 0.5, chunk=50, rot=8, base=50.0), dlt(3, 3, 8, 24, 1, 5, 7), -0.5, 0.9), ff(48)),
                 layer(scan(40, 33, 9, 5)),
                 layer(pair(att(2, 1, 64, 72, 0.2, chunk=16, rot=32, base=1e6), dlt(1, 1, 64, 8, 2, 33, 4), 0.9, 0.4), ff(130))]}
K3 = {"architecture": "Kedavik", "vocab": 77, "width": 50, "norm": {"eps": 1e-5},
      "layers": [layer(pair(att(3, 1, 10, 6, 0.4, chunk=3, rot=6, base=20.0), dlt(2, 2, 6, 10, 2, 3, 5), 1.0, 1.0), ff(30)),
                 layer(scan(22, 3, 2, 2), ff(26)),
                 layer(pair(att(2, 2, 6, 10, 0.3), dlt(4, 2, 10, 6, 3, 1, 2), 0.8, 0.5)),
                 layer(scan(18, 1, 1, 1))]}
CONFIGS = {"K1": K1, "K2": K2, "K3": K3}
SIGMA = {"K1": 0.15, "K2": 0.15, "K3": 0.2}


def single_layer(mixer, mlp=None, **changes):
    """A model of ONE layer (a mechanism alone)."""
    raw = {"architecture": "Kedavik", "vocab": 120, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5},
           "residual_mult": 0.9, "layers": [layer(mixer, mlp)]}
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
            _LOGITS[key] = plain_kedavik.model_layers(cfg, w, toks)[1]
        out[rid] = _LOGITS[key]
    return out


def random_config(seed):
    """A configuration drawn at random: sizes (also odd ones and ones that no fast kernel takes), the order of layers,
    the loop, every constant."""
    import random
    rnd = random.Random(seed)
    layers = []
    for _ in range(rnd.randint(2, 5)):
        if rnd.random() < 0.4:
            mixer = scan(rnd.choice([12, 24, 40, 64, 70, 96]), rnd.choice([1, 2, 5, 8, 16, 24, 48]), rnd.choice([1, 4, 7, 16, 32]),
                         rnd.choice([1, 2, 4, 6]))
        else:
            kv, g = rnd.choice([1, 2, 3]), rnd.choice([1, 2, 4])
            dim = rnd.choice([4, 8, 12, 16, 24, 32, 40, 64, 72])
            left = att(kv * g, kv, dim, rnd.choice([4, 8, 12, 16, 24, 40, 64, 72, 130]), rnd.uniform(0.1, 0.6),
                       chunk=rnd.choice([1, 2, 5, 8, 16, 31, 64, 300]),
                       rot=rnd.choice([None] + [d for d in (2, 4, 8, 12, 16, 24, 32, 40, 64, 72) if d <= dim]),
                       base=rnd.choice([10.0, 1e4, 2e5]))
            kv, g = rnd.choice([1, 2]), rnd.choice([1, 2, 3])
            right = dlt(kv * g, kv, rnd.choice([4, 8, 16, 20, 32, 64]), rnd.choice([6, 8, 12, 16, 20, 40, 48]), rnd.choice([1, 2, 4]),
                        rnd.choice([1, 6, 16, 24, 40]), rnd.choice([2, 8, 24]))
            mixer = pair(left, right, rnd.uniform(-1.5, 1.5), rnd.uniform(0.2, 1.5))
        layers.append(layer(mixer, rnd.choice([None, ff(rnd.choice([24, 50, 64, 130]))])))
    raw = {"architecture": "Kedavik", "vocab": rnd.choice([97, 256, 301]), "width": rnd.choice([40, 56, 64, 74, 96, 136]),
           "norm": {"eps": rnd.choice([1e-5, 1e-6])}, "embedding": {"scale": rnd.choice([1.0, 0.3, 4.0])},
           "residual_mult": rnd.choice([1.0, 0.25, 0.6]), "layers": layers}
    if rnd.random() < 0.8:
        a = rnd.randrange(len(layers))
        raw["loop"] = {"start": a, "stop": rnd.randint(a + 1, len(layers)), "times": rnd.choice([1, 2, 3])}
    return raw
