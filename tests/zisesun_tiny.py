"""Small Zisesun configurations of the tests' own (config.json dictionaries) and helpers to write model folders whose
weights make faults show: streams that differ and are mixed unsymmetrically, peaked attention with a distance bias of
weight, decays from a token's to hundreds of tokens' reach.

ZS_A: value heads wider than key heads (padded to one size) behind a window that ends inside a page; lightning heads whose
key and value sizes differ; a third layer that reads the first one's tensors with a cache of its own; a layer without a
feed-forward.
ZS_B: a width that is no multiple of 4 or 8 (the plain products serve it), two streams, lightning first with top = experts,
a head of its own for every kv head, of a size that is no multiple of 16, a window of 7.
ZS_C: attention only, of head sizes that the tcgen05 kernel takes (64, and keys of 128 with values of 64), one kv head,
windows of 70 and 130, four streams, a chain of layers that read the second layer's tensors.
ZS_D: lightning only (no cache of keys at all): a key size above 128, a value size that fills no tile, one head; a single
stream; one expert of one.
"""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def _att(heads, kv, dim, vdim, scale, window):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}


def _mem(dim, vdim, *decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def _moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


ZS_A: Dict = {
    "architecture": "Zisesun", "vocab": 311, "width": 96, "streams": 3, "max_positions": 400, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "attention", "mixer": _att(4, 2, 32, 48, 0.3, 40), "mlp": _moe(40, 6, 2)},
        {"type": "lightning", "mixer": _mem(24, 40, 0.4, 0.95, 0.998), "mlp": _moe(24, 5, 3)},
        {"type": "attention", "mixer": _att(4, 2, 32, 48, 0.3, 40), "mlp": _moe(40, 6, 2), "weights_of": 0},
        {"type": "lightning", "mixer": _mem(16, 16, 0.9, 0.99), "mlp": None},
    ],
}

ZS_B: Dict = {
    "architecture": "Zisesun", "vocab": 257, "width": 98, "streams": 2, "max_positions": 320, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "lightning", "mixer": _mem(40, 20, 0.97), "mlp": _moe(24, 4, 4)},
        {"type": "attention", "mixer": _att(3, 3, 40, 40, 0.25, 7), "mlp": _moe(20, 7, 2)},
    ],
}

ZS_C: Dict = {
    "architecture": "Zisesun", "vocab": 200, "width": 128, "streams": 4, "max_positions": 384, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "attention", "mixer": _att(8, 1, 64, 64, 0.2, 70), "mlp": _moe(64, 8, 3)},
        {"type": "attention", "mixer": _att(2, 1, 128, 64, 0.09, 130), "mlp": _moe(16, 3, 1)},
        {"type": "attention", "mixer": _att(2, 1, 128, 64, 0.09, 130), "mlp": _moe(16, 3, 1), "weights_of": 1},
        {"type": "attention", "mixer": _att(2, 1, 128, 64, 0.09, 130), "mlp": _moe(16, 3, 1), "weights_of": 2},
    ],
}

ZS_D: Dict = {
    "architecture": "Zisesun", "vocab": 128, "width": 64, "streams": 1, "max_positions": 330, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "lightning", "mixer": _mem(136, 8, 0.8, 0.9995), "mlp": None},
        {"type": "lightning", "mixer": _mem(48, 70, 0.3, 0.9, 0.99, 0.999), "mlp": _moe(96, 1, 1)},
        {"type": "lightning", "mixer": _mem(8, 24, 0.996), "mlp": _moe(32, 5, 3)},
    ],
}

ZS_CONFIGS = {"A": ZS_A, "B": ZS_B, "C": ZS_C, "D": ZS_D}
ZS_SEEDS = {"A": 5, "B": 19, "C": 23, "D": 43}

# factors on the drawn tensors, by the end of their names
GAINS = {"embed": 40.0, "pos": 15.0, "head": 4.0, ".mix.q": 10.0, ".mix.k": 10.0, ".mix.v": 10.0, ".mix.g": 20.0, ".mix.o": 6.0,
         ".q.b": 30.0, ".k.b": 30.0, ".v.b": 30.0, ".mlp.router": 12.0, ".gate": 10.0, ".up": 10.0, ".down": 10.0}
# tensors drawn around one: their distance from it is stretched
AROUND_ONE = {".norm1": 10.0, ".norm2": 10.0, "final.norm": 10.0, ".q.norm": 15.0, ".k.norm": 15.0, ".mix.norm": 15.0,
              ".r1": 4.0, ".r2": 4.0, ".in": 15.0, ".out": 15.0}


def shape_weights(tensors: Dict[str, torch.Tensor], cfg: Dict = None, steady: bool = False) -> Dict[str, torch.Tensor]:
    """The drawn tensors times their gains.  `steady`: the experts' choice rests on no close call, whatever the precision of
    the run: the corrections are multiples of two in a random order, more apart than any two softmax scores, so a layer
    always uses the same experts, weighted by scores that the corrections are no part of."""
    out = {}
    g = torch.Generator().manual_seed(77)
    for n, t in tensors.items():
        x = t.float()
        if n.endswith(".mix.norm") or n.endswith(".q.norm") or n.endswith(".k.norm"):
            x = 1.0 + (x - 1.0) * 15.0
        elif n.endswith(".hc1.mix") or n.endswith(".hc2.mix"):
            eye = torch.eye(x.shape[0])
            x = 0.9 * eye + (x - eye) * 12.0
        elif n.endswith(".correction"):
            x = 2.0 * torch.randperm(x.numel(), generator=g).float() if steady else 0.4 * torch.randn(x.shape, generator=g)
        elif any(n.endswith(k) for k in AROUND_ONE):
            x = 1.0 + (x - 1.0) * next(v for k, v in AROUND_ONE.items() if n.endswith(k))
            if n.endswith(".in"):
                x = x / x.numel()
            if n.endswith(".r1") or n.endswith(".r2"):
                x = x.abs() * (1.0 if n.endswith(".r1") else 0.3)
        else:
            x = x * next((v for k, v in GAINS.items() if n.endswith(k)), 1.0)
        out[n] = x.to(t.dtype)
    return out


def make_zisesun_folder(tmp_path, name: str, cfg: Dict = None, seed: int = None, steady: bool = False) -> str:
    """Write a model folder for configuration `name` (or `cfg`) with shaped random weights."""
    from braidinfer_b200.weights import open_model_folder, save_file, write_random_model
    cfg = dict(cfg if cfg is not None else ZS_CONFIGS[name])
    seed = ZS_SEEDS.get(name, 1) if seed is None else seed
    folder = os.path.join(str(tmp_path), f"zisesun_{name}" + ("_steady" if steady else ""))
    write_random_model(cfg, folder, seed)
    tensors = {n: f.tensor(k).clone() for n, (f, k) in open_model_folder(folder).items()}
    save_file(shape_weights(tensors, cfg, steady), os.path.join(folder, "model.safetensors"))
    return folder


def random_config(seed: int) -> Dict:
    """A configuration drawn from a seed: sizes, head counts, the order and number of layers, who reads whose tensors
    and the constants all vary, within what a test can afford."""
    import random
    r = random.Random(seed)

    def divisor(n):
        return r.choice([d for d in range(1, n + 1) if n % d == 0])

    layers = []
    for i in range(r.randint(2, 6)):
        if layers and r.random() < 0.25:
            j = r.randrange(len(layers))
            layers.append({**{k: v for k, v in layers[j].items() if k != "weights_of"}, "weights_of": j})
            continue
        experts = r.randint(1, 12)
        mlp = None if r.random() < 0.15 else _moe(r.choice([8, 16, 24, 36, 40, 72]), experts, r.randint(1, experts))
        if r.random() < 0.5:
            heads = r.choice([1, 2, 3, 4, 6, 8])
            dim = r.choice([8, 16, 24, 32, 36, 40, 64, 80, 128])
            layers.append({"type": "attention", "mlp": mlp,
                           "mixer": _att(heads, divisor(heads), dim, r.choice([dim, dim, 8, 20, 24, 64, 72]), r.choice([dim ** -0.5, 0.2, 0.07]),
                                         r.choice([1, 2, 5, 16, 33, 63, 64, 65, 100, 128, 129, 1000]))})
        else:
            layers.append({"type": "lightning", "mlp": mlp,
                           "mixer": _mem(r.choice([4, 8, 12, 20, 32, 40, 72, 136]), r.choice([4, 8, 12, 24, 36, 63, 64]),
                                         *[r.choice([0.1, 0.5, 0.8, 0.95, 0.99, 0.999, 1.0]) for _ in range(r.randint(1, 5))])})
    return {"architecture": "Zisesun", "vocab": r.randint(90, 400), "width": r.choice([40, 48, 64, 72, 96, 100, 101]),
            "streams": r.choice([1, 2, 3, 4, 5, 8, 9]), "max_positions": 256, "norm": {"eps": r.choice([1e-6, 1e-5])}, "layers": layers}


def folder_config(folder: str) -> Dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
