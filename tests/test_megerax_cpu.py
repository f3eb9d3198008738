"""Megerax without a GPU: configuration, recipe, cache plan, and the plain implementation's mechanisms by hand."""
import copy
import math

import pytest
import torch

import plain_megerax as P
from megerax_tiny import MG_A, MG_B, MG_C, MG_CONFIGS, MG_D, random_config
from braidinfer_b200.config import ConfigError, MegeraxConfig
from braidinfer_b200.config.megerax import DEFAULT_RANK
from braidinfer_b200.models import architecture_for, complete_config
from braidinfer_b200.weights import tensor_specs_of

D = torch.float64


def spec_of(cfg):
    arch = architecture_for(cfg)
    return arch.build_spec(arch.config_from_dict(cfg))


def runtime():
    from braidinfer_b200.parts.runtime import Runtime
    return Runtime(act_dtype=torch.bfloat16, device=torch.device("cpu"), kernels=None)


def plan_of(cfg):
    from braidinfer_b200.models import DecoderModel
    return DecoderModel(spec_of(cfg), runtime()).cache_plan()


def test_architecture_is_found_by_its_name_and_every_configuration_is_read():
    for cfg in MG_CONFIGS.values():
        assert architecture_for(cfg).name == "Megerax"
        c = MegeraxConfig.from_dict(cfg)
        assert (c.vocab, c.width, c.logit_scale, c.norm_eps) == (cfg["vocab"], cfg["width"], cfg["logit_scale"], cfg["norm"]["eps"])
        assert [L.type for L in c.layers] == [L["type"] for L in cfg["layers"]]
    c = MegeraxConfig.from_dict(MG_A)
    a, d, t, r = (L.mixer for L in c.layers)
    assert (a.window, a.vdim, a.softcap, a.conv, a.rot_scaling.high, a.kv_from) == (40, 48, 6.0, 4, 4.0, None)
    assert (d.heads, d.kv_heads, d.conv, d.decay_rank, d.gate_rank) == (6, 3, 3, 20, 12)
    assert (t.q_rank, t.kv_rank, t.rot_dim, t.vdim) == (40, 32, 16, 24) and r.kv_from == 0 and r.window == 70
    assert [L.ff for L in c.layers] == [72, None, 104, None]
    assert MegeraxConfig.from_dict(MG_D).layers[2].mixer.decay_rank == DEFAULT_RANK


@pytest.mark.parametrize("path, value", [
    ("layers.0.type", "conv"), ("layers.0.mixer.kv_heads", 3), ("layers.0.mixer.mask.size", 0), ("layers.0.mixer.mask", None),
    ("layers.0.mixer.softcap", None), ("layers.0.mixer.softcap", 0.0), ("layers.0.mixer.scale", None), ("layers.0.mixer.rot.dims", 34),
    ("layers.0.mixer.rot.dims", 15), ("layers.0.mixer.rot.scaling.high", 1.0), ("layers.0.mixer.rot.scaling.low", None),
    ("layers.0.mixer.conv", 0), ("layers.1.mixer.kv_heads", 4), ("layers.1.mixer.conv", None), ("layers.1.mixer.kv_from", 0),
    ("layers.2.mixer.q_rank", None), ("layers.2.mixer.rot.dims", 8), ("layers.2.mixer.rot.base", 0.0), ("layers.3.mixer.kv_from", 1),
    ("layers.3.mixer.kv_from", 3), ("layers.3.mixer.kv_from", True), ("layers.3.mixer.dim", 16), ("layers.3.mixer.rot.base", 5.0),
    ("layers.0.mlp.kind", "moe"), ("layers.0.mlp.ff", None), ("norm", None), ("logit_scale", None), ("vocab", None)])
def test_a_value_nothing_computes_is_an_error_that_names_its_key(path, value):
    cfg = copy.deepcopy(MG_A)
    cur, keys = cfg, path.split(".")
    for k in keys[:-1]:
        cur = cur[int(k)] if k.isdigit() else cur[k]
    if value is None:
        del cur[keys[-1]]
    else:
        cur[keys[-1]] = value
    with pytest.raises(ConfigError) as e:
        MegeraxConfig.from_dict(cfg)
    assert keys[-1] in str(e.value) or keys[-2] in str(e.value) or f"layers[{keys[1]}]" in str(e.value)


def test_a_reader_of_a_reader_is_refused():
    cfg = copy.deepcopy(MG_C)
    cfg["layers"][5]["mixer"]["kv_from"] = 4
    with pytest.raises(ConfigError, match="kv_from"):
        MegeraxConfig.from_dict(cfg)


def test_inner_sizes_of_the_low_rank_maps_come_from_the_tensors_shapes():
    cfg = complete_config(MG_D, {"l0.mix.a1": (5, 64), "l0.mix.g1": (6, 64), "l2.mix.a1": (50, 64)})
    m = [L.mixer for L in MegeraxConfig.from_dict(cfg).layers]
    assert (m[0].decay_rank, m[0].gate_rank, m[1].decay_rank, m[2].decay_rank, m[2].gate_rank) == (5, 6, 33, 50, DEFAULT_RANK)
    assert "decay_rank" not in MG_D["layers"][2]["mixer"]                    # the caller's dictionary is left alone
    with pytest.raises(ConfigError):
        complete_config(MG_D, {"l0.mix.a1": (5,)})


def test_recipe_names_the_tensors_of_the_design_and_the_parts_beside_the_existing_ones():
    spec = spec_of(MG_A)
    shapes = {n: t.shape for n, t in tensor_specs_of(spec).items()}
    want = {"embed": (311, 96), "embed.norm": (96,), "head": (311, 96), "final.norm": (96,), "l0.norm1": (96,), "l0.norm2": (96,),
            "l0.mix.q": (128, 96), "l0.mix.q.b": (128,), "l0.mix.q.conv": (128, 4), "l0.mix.q.norm": (32,), "l0.mix.k": (64, 96),
            "l0.mix.k.b": (64,), "l0.mix.k.conv": (64, 4), "l0.mix.k.norm": (32,), "l0.mix.v": (96, 96), "l0.mix.v.b": (96,),
            "l0.mix.v.conv": (96, 4), "l0.mix.g": (192, 96), "l0.mix.o": (96, 192), "l0.mlp.gate": (72, 96), "l0.mlp.down": (96, 72),
            "l1.mix.q": (72, 96), "l1.mix.q.conv": (72, 3), "l1.mix.v": (240, 96), "l1.mix.v.conv": (240, 3), "l1.mix.b": (6, 96),
            "l1.mix.A_log": (6,), "l1.mix.dt_bias": (144,), "l1.mix.a1": (20, 96), "l1.mix.a2": (144, 20), "l1.mix.g1": (12, 96),
            "l1.mix.g2": (240, 12), "l1.mix.norm": (40,), "l1.mix.o": (96, 240), "l2.mix.dq": (40, 96), "l2.mix.dq.norm": (40,),
            "l2.mix.uq": (96, 40), "l2.mix.dkv": (48, 96), "l2.mix.dkv.norm": (32,), "l2.mix.uk": (48, 32), "l2.mix.uv": (72, 32),
            "l2.mix.sink": (3,), "l2.mix.o": (96, 72), "l3.mix.q": (128, 96), "l3.mix.g": (192, 96)}
    for n, s in want.items():
        assert shapes[n] == s, n
    assert not any(n in shapes for n in ("l1.norm2", "l3.norm2", "l1.mlp.up", "l3.mix.k", "l3.mix.v", "l3.mix.k.b", "l3.mix.k.conv",
                                         "l3.mix.k.norm", "l2.mix.q", "l2.mix.g"))
    assert [L.mixer.kind for L in spec.layers] == ["gqa_attention", "channel_delta", "latent_attention", "gqa_attention"]
    assert [e.cache_of for e in spec.schedule] == [None, None, None, 0]
    assert spec.embedding.params["norm"].kind == "rmsnorm" and spec.final_norm.params["gain"] == 0.75


def test_cache_plan_keys_for_the_longest_window_among_the_readers_and_states():
    p = plan_of(MG_A)
    req, of, state = p[0]
    assert (req.kind, req.num_kv_heads, req.head_dim, req.window, req.planes) == ("window", 2, 48, 70, 2) and of is None
    assert state == 3 * (128 + 64 + 96) * 4
    assert p[1][0] is None and p[1][2] == 2 * (72 + 72 + 240) * 4 + 6 * 24 * 40 * 4
    assert (p[2][0].kind, p[2][0].head_dim, p[2][0].planes, p[2][2]) == ("full", 48, 1, 0)
    assert p[3][0] == req and p[3][1] == 0 and p[3][2] == 3 * 128 * 4            # the reader's own state: its queries' convolution
    p = plan_of(MG_B)
    assert p[1][0].head_dim == 48 and p[2][2] == 2 * 40 * 20 * 4               # padded heads; one tap keeps no inputs
    p = plan_of(MG_C)
    assert [x[0].window for x in (p[0], p[4], p[5])] == [97, 97, 97] and [x[1] for x in p] == [None, None, None, None, 0, 0]
    assert all(x[0] is None for x in plan_of(MG_D))


def test_configurations_drawn_from_a_seed_are_read():
    for seed in range(40):
        cfg = random_config(seed)
        assert len(plan_of(cfg)) == len(cfg["layers"])


def test_constant_factor_of_a_norm_is_kept_in_32_bits_and_norms_that_offset_refuse_it():
    from braidinfer_b200.parts.norm import RMSNorm
    n = RMSNorm({"width": 2, "eps": 1e-6, "name": "x", "gain": 0.3}, "", None)
    w = torch.tensor([1.0078125, -2.5], dtype=torch.bfloat16)
    n.load({"x": w})
    assert n.weight.dtype == torch.float32 and torch.equal(n.weight, w.float() * 0.3)
    with pytest.raises(ValueError):
        RMSNorm({"width": 2, "eps": 1e-6, "name": "x", "gain": 0.3, "offset": 1.0}, "", None)


@pytest.mark.parametrize("params", [{"head_gate": "g"}, {"keep_first": 3}, {"unit_v_eps": 1e-6}, {"conv": None, "column_gate": "g"},
                                    {"conv": None, "shared_kv": True}, {"softcap": -1.0}, {"cache_window": 10}, {"value_from_key": True}])
def test_options_of_attention_that_do_not_go_together_are_refused(params):
    from braidinfer_b200.parts.attention import GQAAttention
    from braidinfer_b200.parts.spec import PartSpec
    p = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "window": 20, "conv": 3,
         "position_encoding": PartSpec("rope", {"head_dim": 16, "theta": 100.0, "pairing": "adjacent"})}
    GQAAttention(p, "", runtime())
    with pytest.raises(ValueError):
        GQAAttention({**p, **params}, "", runtime())


def test_rotation_frequencies_by_bands():
    from braidinfer_b200.parts.rope import rotary_frequencies
    for dims, base, sc in ((32, 50000.0, (4.0, 1.0, 4.0, 512)), (64, 100.0, (8.0, 2.0, 3.0, 64)), (16, 1e6, (2.0, 1.0, 8.0, 100000))):
        sc = dict(zip(("factor", "low", "high", "original"), sc))
        f, amp = rotary_frequencies(dims, base, {"kind": "bands", **sc})
        want = P.frequencies({"dims": dims, "base": base, "scaling": sc})
        assert amp == 1.0 and torch.allclose(f, want, rtol=1e-12, atol=0)
        plain = P.frequencies({"dims": dims, "base": base})
        kinds = [(w == p_).item() for w, p_ in zip(want, plain)], [abs(w / p_ - 1 / sc["factor"]) < 1e-12 for w, p_ in zip(want, plain)]
        assert any(kinds[0]) and any(kinds[1])                                # the sizes of the test reach both ends of the scale
    with pytest.raises(ValueError):
        rotary_frequencies(16, 100.0, {"kind": "bands", "factor": 2.0, "low": 4.0, "high": 1.0, "original": 10})
    with pytest.raises(ValueError):
        rotary_frequencies(16, 100.0, {"kind": "other", "factor": 2.0, "original": 10})


# ---------------------------------------------------------------------------------------------- the oracle by hand
def test_convolution_by_hand():
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=D)
    assert P.causal_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=D)).view(-1).tolist() == [1.0, 12.0, 123.0]
    assert P.causal_conv(x, torch.tensor([[5.0]], dtype=D)).view(-1).tolist() == [5.0, 10.0, 15.0]


def test_delta_rule_by_hand():
    one = lambda *v: torch.tensor(v, dtype=D).view(-1, 1, 1)                   # noqa: E731  [T, 1 head, 1]
    # S1 = 0 + 1 * (0.5 * (4 - 0)) = 2, o1 = 3 * 2; S2: 0.5 * 2 = 1, u = 1 * (6 - 1 * 2) = 4, S2 = 1 + 2 * 4 = 9, o2 = 9
    o, S = P.delta_rule(one(3.0, 1.0), one(1.0, 2.0), one(4.0, 6.0), one(0.9, 0.5), torch.tensor([[0.5], [1.0]], dtype=D))
    assert o.view(-1).tolist() == [6.0, 9.0] and S.item() == 9.0
    o2, S2 = P.delta_rule(one(1.0), one(2.0), one(6.0), one(0.5), torch.tensor([[1.0]], dtype=D),
                          P.delta_rule(one(3.0), one(1.0), one(4.0), one(0.9), torch.tensor([[0.5]], dtype=D))[1])
    assert o2.item() == 9.0 and torch.equal(S, S2)


def test_delta_rule_recalls_a_key_and_a_second_write_replaces_it():
    e = torch.eye(3, dtype=D)
    k = torch.stack([e[0], e[1], e[0], e[2]])[:, None]
    v = torch.tensor([[1.0], [2.0], [5.0], [7.0]], dtype=D)[:, None]
    o, _ = P.delta_rule(torch.stack([e[0], e[0], e[0], e[1]])[:, None], k, v, torch.ones(4, 1, 3, dtype=D), torch.ones(4, 1, dtype=D))
    assert o.view(-1).tolist() == [1.0, 1.0, 5.0, 2.0]


def test_decay_of_a_channel_unit_heads_and_gate():
    w = {"a1": torch.tensor([[2.0]], dtype=D), "a2": torch.tensor([[1.0], [0.0]], dtype=D), "dt_bias": torch.tensor([0.0, -1.0], dtype=D),
         "A_log": torch.tensor([math.log(3.0)], dtype=D)}
    g = P.channel_decay(torch.tensor([[0.5]], dtype=D), w, 1, 2)
    assert torch.allclose(g.view(-1), torch.tensor([math.exp(-3 * math.log(1 + math.e)), math.exp(-3 * math.log(1 + math.exp(-1)))], dtype=D))
    u = P.unit_heads(torch.tensor([[3.0, 4.0], [0.0, 0.0]], dtype=D))
    assert torch.allclose(u[0], torch.tensor([0.6, 0.8], dtype=D)) and u[1].abs().max() == 0


def test_cap_window_and_sink_by_hand():
    assert P.capped(torch.tensor(1e9, dtype=D), 7.0).item() == 7.0 and abs(P.capped(torch.tensor(0.01, dtype=D), 7.0).item() - 0.01) < 1e-7
    assert P.visible(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    p = P.masked_softmax(torch.zeros(1, 2, 2, dtype=D), P.visible(2), torch.tensor([math.log(2.0)], dtype=D))
    assert torch.allclose(p[0], torch.tensor([[1 / 3, 0.0], [0.25, 0.25]], dtype=D))


def test_a_shared_layer_uses_its_owners_keys_with_its_own_mask():
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 1.0, "softcap": 50.0, "mask": {"size": 9}, "rot": {"base": 10.0, "dims": 2}}
    h = torch.tensor([[1.0], [2.0], [4.0]], dtype=D)
    one = torch.ones(1, 1, dtype=D)
    w = {"q": torch.zeros(2, 1, dtype=D), "q.b": torch.zeros(2, dtype=D), "q.conv": torch.ones(2, 1, dtype=D), "q.norm": torch.ones(2, dtype=D),
         "g": 1e3 * one, "o": one}
    keys, vals = torch.randn(3, 1, 2, dtype=D), torch.tensor([3.0, 5.0, 9.0], dtype=D).view(3, 1, 1)
    assert torch.allclose(P.attention(h, w, m, 1e-6, (keys, vals))[0].view(-1), torch.tensor([3.0, 4.0, 17 / 3], dtype=D))
    assert torch.allclose(P.attention(h, w, {**m, "mask": {"size": 2}}, 1e-6, (keys, vals))[0].view(-1), torch.tensor([3.0, 4.0, 7.0], dtype=D))
