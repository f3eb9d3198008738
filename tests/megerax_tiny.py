"""Small Megerax configurations of the tests' own (config.json dictionaries) and helpers to write model folders whose
weights make faults show: peaked attention with scores near the cap, decays of a channel from fast to nearly one (a token
far back still counts), sinks of the scores' size.

MG_A: attention whose value heads are wider than its key heads (window 40), a delta layer whose heads share q and k two by
two and that has no feed-forward, latent attention, attention that reads the first layer's keys and values behind a longer
window and with another cap.
MG_B: a width that is no multiple of 8 (the plain products serve it); latent attention of one head with ranks of odd sizes;
attention with one kv head a head, a head size that is no multiple of 16, narrower values, five taps, no rotation, a window
shorter than a page; a delta layer with a convolution of one tap.
MG_C: sizes the tensor cores take: heads of 64 and of 128 (with values of 32), a latent of 64, a delta layer of 128 x 64;
two readers of one layer's keys, one with a shorter window than its owner's, one with a longer.
MG_D: delta layers only (no cache of keys): key sizes 136, 8 and 33, one and two taps, one q/k head for all heads.
"""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def _att(heads, kv, dim, vdim, conv, scale, cap, rot_dims, base, size, scaling=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "softcap": cap,
         "mask": {"size": size}, "rot": {"base": base, "dims": rot_dims}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _delta(heads, kv, dim, vdim, conv, ranks=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}
    if ranks:
        m["decay_rank"], m["gate_rank"] = ranks
    return m


def _lat(heads, dim, rot, vdim, q_rank, kv_rank, scale, base):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot}}


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


MG_A: Dict = {
    "architecture": "Megerax", "vocab": 311, "width": 96, "logit_scale": 0.75, "norm": {"eps": 1e-6},
    "layers": [
        _layer("attention", _att(4, 2, 32, 48, 4, 0.2, 6.0, 16, 10000.0, 40, (8.0, 1.0, 4.0, 64)), 72),
        _layer("channel_delta", _delta(6, 3, 24, 40, 3, (20, 12)), None),
        _layer("latent_attention", _lat(3, 16, 16, 24, 40, 32, 0.25, 1000.0), 104),
        _layer("attention", _att(4, 2, 32, 48, 4, 0.15, 20.0, 16, 10000.0, 70, (8.0, 1.0, 4.0, 64), kv_from=0), None),
    ],
}

MG_B: Dict = {
    "architecture": "Megerax", "vocab": 257, "width": 100, "logit_scale": 1.5, "norm": {"eps": 1e-5},
    "layers": [
        _layer("latent_attention", _lat(1, 9, 6, 12, 13, 20, 0.3, 100.0), 60),
        _layer("attention", _att(3, 3, 40, 20, 5, 0.16, 10.0, 0, 3000.0, 7), None),
        _layer("channel_delta", _delta(2, 2, 40, 20, 1, (7, 9)), 44),
    ],
}

MG_C: Dict = {
    "architecture": "Megerax", "vocab": 200, "width": 128, "logit_scale": 1.0, "norm": {"eps": 1e-6},
    "layers": [
        _layer("attention", _att(8, 2, 64, 64, 4, 0.125, 15.0, 64, 5000.0, 70), 136),
        _layer("latent_attention", _lat(4, 32, 16, 48, 64, 64, 0.2, 20000.0), None),
        _layer("attention", _att(4, 1, 128, 32, 2, 0.09, 30.0, 48, 100000.0, 130, (4.0, 2.0, 3.0, 512)), 64),
        _layer("channel_delta", _delta(4, 2, 128, 64, 4, (16, 24)), 72),
        _layer("attention", _att(8, 2, 64, 64, 3, 0.1, 9.0, 64, 5000.0, 20, kv_from=0), None),
        _layer("attention", _att(8, 2, 64, 64, 4, 0.125, 15.0, 64, 5000.0, 97, kv_from=0), 40),
    ],
}

MG_D: Dict = {
    "architecture": "Megerax", "vocab": 128, "width": 64, "logit_scale": 0.3, "norm": {"eps": 1e-6},
    "layers": [
        _layer("channel_delta", _delta(3, 1, 136, 36, 2, (8, 8)), None),
        _layer("channel_delta", _delta(8, 4, 8, 8, 4, (33, 5)), 96),
        _layer("channel_delta", _delta(2, 2, 33, 70, 3), None),
    ],
}

MG_CONFIGS = {"A": MG_A, "B": MG_B, "C": MG_C, "D": MG_D}
MG_SEEDS = {"A": 5, "B": 19, "C": 23, "D": 43}

# factors on the drawn tensors, by the end of their names (the first that fits)
GAINS = {"head": 8.0, "embed": 10.0, ".q.b": 20.0, ".k.b": 20.0, ".v.b": 20.0, ".mix.q": 8.0, ".mix.k": 8.0, ".mix.v": 10.0, ".mix.o": 8.0,
         ".mix.g": 15.0, ".mix.dq": 8.0, ".mix.uq": 12.0, ".mix.dkv": 8.0, ".mix.uk": 12.0, ".mix.uv": 12.0, ".mix.sink": 1.5, ".mix.b": 12.0,
         ".mix.a1": 10.0, ".mix.a2": 15.0, ".mix.g1": 10.0, ".mix.g2": 15.0, ".mix.dt_bias": 1.5, ".mix.A_log": 2.0, ".gate": 8.0, ".up": 8.0,
         ".down": 8.0}


def shape_weights(tensors: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    out = {}
    for n, t in tensors.items():
        x = t.float()
        if n.endswith("norm") or n.endswith(".norm1") or n.endswith(".norm2"):
            x = 1.0 + (x - 1.0) * 10.0
        else:
            x = x * next((v for k, v in GAINS.items() if n.endswith(k)), 1.0)
            if n.endswith(".dt_bias"):
                x = x - 3.0                    # most channels remember dozens to hundreds of tokens, some forget at once
        out[n] = x.to(t.dtype)
    return out


def make_megerax_folder(tmp_path, name: str, cfg: Dict = None, seed: int = None) -> str:
    """Write a model folder for configuration `name` (or `cfg`) with shaped random weights."""
    from braidinfer_b200.weights import open_model_folder, save_file, write_random_model
    cfg = dict(cfg if cfg is not None else MG_CONFIGS[name])
    seed = MG_SEEDS.get(name, 1) if seed is None else seed
    folder = os.path.join(str(tmp_path), f"megerax_{name}")
    write_random_model(cfg, folder, seed)
    tensors = {n: f.tensor(k).clone() for n, (f, k) in open_model_folder(folder).items()}
    save_file(shape_weights(tensors), os.path.join(folder, "model.safetensors"))
    return folder


def random_config(seed: int) -> Dict:
    """A configuration drawn from a seed: sizes, head counts, the order and number of layers, windows, who reads whose keys
    and the constants all vary, within what a test can afford."""
    import random
    r = random.Random(seed)

    def divisor(n):
        return r.choice([d for d in range(1, n + 1) if n % d == 0])

    layers, owners = [], []
    for i in range(r.randint(2, 7)):
        ff = r.choice([None, 24, 40, 60, 72, 100])
        u = r.random()
        window = r.choice([1, 2, 5, 17, 33, 63, 64, 65, 100, 129, 500])
        if u < 0.25 and owners:
            j = r.choice(owners)
            m = json.loads(json.dumps(layers[j]["mixer"]))
            m.update(kv_from=j, softcap=r.choice([4.0, 12.0, 50.0]), scale=r.choice([0.3, 0.1]), mask={"size": window}, conv=r.randint(1, 5))
            layers.append(_layer("attention", m, ff))
        elif u < 0.5:
            heads, dim = r.choice([1, 2, 3, 4, 6, 8]), r.choice([8, 16, 20, 24, 32, 40, 64, 80, 128])
            dims = r.choice([d for d in (0, 2, 8, 16, 20, 32, 64) if d <= dim] + [dim])
            scaling = (r.choice([2.0, 4.0, 16.0]), r.choice([1.0, 1.5]), r.choice([2.0, 4.0, 8.0]), r.choice([16, 64, 512])) \
                if r.random() < 0.6 else None
            owners.append(i)
            layers.append(_layer("attention", _att(heads, divisor(heads), dim, r.choice([dim, dim, 8, 12, 24, 72]), r.randint(1, 5),
                                                   r.choice([dim ** -0.5, 0.25]), r.choice([5.0, 15.0, 50.0]), dims,
                                                   r.choice([100.0, 10000.0, 500000.0]), window, scaling), ff))
        elif u < 0.75:
            heads = r.choice([1, 2, 3, 4, 6])
            layers.append(_layer("channel_delta", _delta(heads, divisor(heads), r.choice([4, 8, 12, 20, 32, 40, 64, 72, 136]),
                                                         r.choice([4, 8, 12, 24, 36, 63, 64, 130]), r.randint(1, 5),
                                                         (r.randint(1, 40), r.randint(1, 40))), ff))
        else:
            rot = r.choice([2, 6, 8, 16, 32])
            layers.append(_layer("latent_attention", _lat(r.randint(1, 6), r.choice([4, 8, 15, 16, 32]), rot, r.choice([4, 8, 20, 36]),
                                                          r.choice([5, 16, 24, 60]), r.choice([8, 16, 20, 48, 64, 96]),
                                                          r.choice([0.3, 0.15]), r.choice([100.0, 10000.0])), ff))
    return {"architecture": "Megerax", "vocab": r.randint(90, 400), "width": r.choice([40, 48, 64, 72, 96, 100, 101]),
            "logit_scale": r.choice([0.2, 0.6, 1.0, 3.0]), "norm": {"eps": r.choice([1e-6, 1e-5])}, "layers": layers}


def folder_config(folder: str) -> Dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
