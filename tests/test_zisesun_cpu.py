"""Zisesun without a GPU: configuration, recipe, cache plan, and the plain implementation's mechanisms by hand."""
import copy
import math

import pytest
import torch

import plain_zisesun as P
from zisesun_tiny import ZS_A, ZS_B, ZS_C, ZS_CONFIGS, ZS_D, random_config
from braidinfer_b200.config import ConfigError, ZisesunConfig
from braidinfer_b200.models import architecture_for
from braidinfer_b200.weights import draw_tensors, tensor_specs_of

D = torch.float64


def spec_of(cfg):
    arch = architecture_for(cfg)
    return arch.build_spec(arch.config_from_dict(cfg))


def test_architecture_is_found_by_its_name_and_every_configuration_is_read():
    for cfg in ZS_CONFIGS.values():
        assert architecture_for(cfg).name == "Zisesun"
        c = ZisesunConfig.from_dict(cfg)
        assert (c.vocab, c.width, c.streams, c.max_positions) == tuple(cfg[k] for k in ("vocab", "width", "streams", "max_positions"))
        assert len(c.layers) == len(cfg["layers"])
    c = ZisesunConfig.from_dict(ZS_A)
    assert c.layers[0].mixer.window == 40 and c.layers[0].mixer.vdim == 48 and c.layers[0].mlp.top == 2
    assert c.layers[1].mixer.decay == (0.4, 0.95, 0.998) and c.layers[1].mixer.heads == 3 and c.layers[3].mlp is None
    assert [L.weights_of for L in c.layers] == [0, 1, 0, 3]
    assert [L.weights_of for L in ZisesunConfig.from_dict(ZS_C).layers] == [0, 1, 1, 1]       # a chain ends at its owner


@pytest.mark.parametrize("path, value", [("layers.0.type", "conv"), ("layers.0.mixer.kv_heads", 3), ("layers.0.mixer.mask.size", 0),
                                         ("layers.0.mixer.mask", None), ("layers.1.mixer.decay", [0.5, 0.5]), ("layers.1.mixer.decay", None),
                                         ("layers.1.mixer.decay", 0.5), ("layers.0.mlp.kind", "dense"), ("layers.0.mlp.router.top", 7),
                                         ("layers.2.weights_of", 9), ("layers.2.mixer.heads", 2), ("norm", None), ("streams", None),
                                         ("streams", 0), ("max_positions", None), ("layers.0.mixer.scale", None), ("layers.1.mixer.vdim", None)])
def test_a_value_nothing_computes_is_an_error_that_names_its_key(path, value):
    cfg = copy.deepcopy(ZS_A)
    cur = cfg
    keys = path.split(".")
    for k in keys[:-1]:
        cur = cur[int(k)] if k.isdigit() else cur[k]
    if value is None:
        del cur[keys[-1]]
    else:
        cur[keys[-1]] = value
    with pytest.raises(ConfigError) as e:
        ZisesunConfig.from_dict(cfg)
    assert keys[-1] in str(e.value) or keys[-2] in str(e.value) or f"layers[{keys[1]}]" in str(e.value)


def test_layers_that_borrow_in_a_circle_are_refused():
    cfg = copy.deepcopy(ZS_C)
    cfg["layers"][1]["weights_of"] = 3
    with pytest.raises(ConfigError):
        ZisesunConfig.from_dict(cfg)


def test_recipe_names_the_tensors_of_the_design_and_the_parts_beside_the_existing_ones():
    spec = spec_of(ZS_A)
    specs = tensor_specs_of(spec)
    shapes = {n: t.shape for n, t in specs.items()}
    assert not any(n.startswith("l2.") for n in shapes)                  # the third layer reads the first one's tensors
    want = {"embed": (311, 96), "pos": (400, 96), "head": (311, 96), "final.norm": (), "l0.norm1": (), "l0.norm2": (),
            "l0.mix.q": (128, 96), "l0.mix.q.b": (128,), "l0.mix.q.norm": (128,), "l0.mix.k": (64, 96), "l0.mix.k.b": (64,),
            "l0.mix.k.norm": (64,), "l0.mix.v": (96, 96), "l0.mix.v.b": (96,), "l0.mix.r1": (4,), "l0.mix.r2": (4,), "l0.mix.o": (96, 192),
            "l0.mlp.router": (6, 96), "l0.mlp.correction": (6,), "l0.mlp.e0.gate": (40, 96), "l0.mlp.e5.down": (96, 40),
            "l0.hc1.in": (3,), "l0.hc1.mix": (3, 3), "l0.hc2.out": (3,), "l1.mix.q": (72, 96), "l1.mix.v": (120, 96), "l1.mix.g": (120, 96),
            "l1.mix.norm": (120,), "l1.mix.o": (96, 120), "l3.norm1": (), "l3.hc1.out": (3,)}
    for n, s in want.items():
        assert shapes[n] == s, n
    assert not any(n.startswith("l3.mlp") or n.startswith("l3.hc2") or n == "l3.norm2" for n in shapes)
    assert [e.layer for e in spec.schedule] == [0, 1, 0, 2] and len(spec.layers) == 3
    assert [L.mixer.kind for L in spec.layers] == ["gqa_attention", "lightning_attention", "lightning_attention"]
    assert all(L.block == "hyper_connected" and L.mixer_connection.kind == "hyper_connection" for L in spec.layers)
    assert [L.feed_forward.kind if L.feed_forward else None for L in spec.layers] == ["moe", "moe", None]
    assert spec.layers[2].feed_forward_connection is None and spec.streams.params == {"streams": 3} and spec.max_position == 400
    assert not spec.head.params["tied"] and spec.layers[0].mixer_norm.params["scalar"]
    assert [e.layer for e in spec_of(ZS_C).schedule] == [0, 1, 1, 1]


def test_cache_plan_gives_every_run_a_cache_or_state_of_its_own():
    from braidinfer_b200.models import DecoderModel
    from braidinfer_b200.parts.runtime import Runtime
    rt = Runtime(act_dtype=torch.bfloat16, device=torch.device("cpu"), kernels=None)
    plan = DecoderModel(spec_of(ZS_A), rt).cache_plan()
    assert len(plan) == 4 and all(cache_of is None for _, cache_of, _ in plan)
    req0, _, st0 = plan[0]
    assert (req0.kind, req0.num_kv_heads, req0.head_dim, req0.window, req0.planes) == ("window", 2, 48, 40, 2) and st0 == 0
    assert plan[2][0] == req0                                            # the borrowing layer: the same request, another entry
    assert plan[1][0] is None and plan[1][2] == 3 * 24 * 40 * 4 and plan[3][2] == 2 * 16 * 16 * 4
    assert DecoderModel(spec_of(ZS_B), rt).cache_plan()[1][0].head_dim == 48     # heads of 40 padded to the next size the kernels take
    plan = DecoderModel(spec_of(ZS_C), rt).cache_plan()
    assert [(p[0].head_dim, p[0].window) for p in plan] == [(64, 70)] + [(128, 130)] * 3
    assert all(p[0] is None for p in DecoderModel(spec_of(ZS_D), rt).cache_plan())


def test_configurations_drawn_from_a_seed_are_read():
    for seed in range(30):
        cfg = random_config(seed)
        spec = spec_of(cfg)
        assert len(spec.schedule) == len(cfg["layers"])
        assert len(spec.layers) == sum(1 for L in cfg["layers"] if L.get("weights_of") is None)


def test_random_weights_mix_the_streams_near_the_identity_and_a_scalar_norm_is_one_number():
    drawn = draw_tensors(tensor_specs_of(spec_of(ZS_A)), 3)
    assert (drawn["l0.hc1.mix"].float() - torch.eye(3)).abs().max().item() < 0.2 and drawn["l0.norm1"].shape == ()
    from braidinfer_b200.parts.norm import RMSNorm
    n = RMSNorm({"width": 5, "eps": 1e-6, "name": "x", "scalar": True}, "", None)
    n.load({"x": torch.tensor(1.5)})
    assert n.weight.tolist() == [1.5] * 5 and n.weight.is_contiguous()


@pytest.mark.parametrize("params, message", [({"unit_qk_eps": 1e-6}, "biases"), ({"unit_v_eps": 1e-4}, "one eps"),
                                             ({"position_encoding": "rope"}, "rotation")])
def test_options_of_attention_that_do_not_go_together_are_refused(params, message):
    from braidinfer_b200.parts.attention import GQAAttention
    from braidinfer_b200.parts.runtime import Runtime
    from braidinfer_b200.parts.spec import PartSpec
    rt = Runtime(act_dtype=torch.bfloat16, device=torch.device("cpu"), kernels=None)
    p = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "position_encoding": PartSpec("none", {"head_dim": 16}),
         "qkv_bias": True, "proj_norm": {"eps": 1e-6, "q_name": "qn", "k_name": "kn"}}
    if params.get("position_encoding") == "rope":
        params = {"position_encoding": PartSpec("rope", {"head_dim": 16, "theta": 100.0, "rope_dim": 16, "pairing": "half"})}
    with pytest.raises(ValueError, match=message):
        GQAAttention({**p, **params}, "", rt)


def test_several_streams_and_an_injection_are_refused():
    import dataclasses
    from braidinfer_b200.parts.spec import PartSpec
    with pytest.raises(ValueError, match="injection"):
        dataclasses.replace(spec_of(ZS_A), injection=PartSpec("concat_linear", {})).validate()


# ---------------------------------------------------------------------------------------------- the oracle by hand
def test_streams_by_hand():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=D)                                  # two streams, one token, width 2
    assert P.read_streams(X, torch.tensor([0.5, 2.0], dtype=D)).tolist() == [[20.5, 41.0]]
    M = torch.tensor([[1.0, 3.0], [0.0, -1.0]], dtype=D)                                       # [from, to]
    Y = P.write_streams(X, M, torch.tensor([1.0, 100.0], dtype=D), torch.tensor([[7.0, 8.0]], dtype=D))
    assert Y.tolist() == [[[1.0 + 7.0, 2.0 + 8.0]], [[3.0 - 10.0 + 700.0, 6.0 - 20.0 + 800.0]]]


def test_memory_with_a_constant_decay_by_hand():
    q, k = torch.tensor([[1.0], [2.0], [3.0]], dtype=D), torch.tensor([[1.0], [-1.0], [2.0]], dtype=D)
    v = torch.tensor([[4.0, 0.0], [0.0, 2.0], [1.0, 1.0]], dtype=D)
    o, S = P.decayed_memory(q, k, v, 0.5)
    # S1 = [4, 0]; S2 = [2, 0] - [0, 2] = [2, -2]; S3 = [1, -1] + [2, 2] = [3, 1]
    assert o.tolist() == [[4.0, 0.0], [4.0, -4.0], [9.0, 3.0]] and S.tolist() == [[3.0, 1.0]]
    o2, S2 = P.decayed_memory(q[2:], k[2:], v[2:], 0.5, P.decayed_memory(q[:2], k[:2], v[:2], 0.5)[1])
    assert o2.tolist() == [[9.0, 3.0]] and torch.equal(S2, S)


def test_lightning_norms_all_heads_together_before_the_gate():
    m = {"heads": 2, "dim": 1, "vdim": 1, "decay": [0.0, 0.0]}
    one = torch.ones(1, 1, dtype=D)
    w = {"q": torch.tensor([[1.0], [2.0]], dtype=D), "k": torch.tensor([[1.0], [1.0]], dtype=D), "v": torch.tensor([[1.0], [3.0]], dtype=D),
         "norm": torch.tensor([2.0, 1.0], dtype=D), "g": torch.tensor([[0.0], [1.0]], dtype=D), "o": torch.eye(2, dtype=D)}
    s = lambda z: z / (1 + math.exp(-z))       # noqa: E731
    o = [s(1) * s(1) * s(1), s(2) * s(1) * s(3)]
    rms = math.sqrt((o[0] ** 2 + o[1] ** 2) / 2)
    want = [o[0] / rms * 2 * 0.5, o[1] / rms / (1 + math.exp(-1))]
    assert torch.allclose(P.lightning(one, w, m, 0.0)[0], torch.tensor(want, dtype=D))


def test_distance_bias_window_and_value_norm_by_hand():
    d = P.distance_bias(torch.tensor([5, 5, 5]), torch.tensor([5, 3, 0]), torch.tensor(2.0, dtype=D), torch.tensor(0.5, dtype=D))
    assert torch.allclose(d, torch.tensor([0.0, 2 * math.log(2.0), 2 * math.log(3.5)], dtype=D))
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.5, "mask": {"size": 2}}
    h = torch.tensor([[1.0], [2.0], [3.0]], dtype=D)
    w = {"q": torch.zeros(2, 1, dtype=D), "q.b": torch.tensor([1.0, 1.0], dtype=D), "k": torch.zeros(2, 1, dtype=D), "k.b": torch.tensor([3.0, 4.0], dtype=D),
         "v": torch.tensor([[1.0], [0.0]], dtype=D), "v.b": torch.tensor([-2.0, 1.0], dtype=D), "q.norm": torch.tensor([1.0, 1.0], dtype=D),
         "k.norm": torch.tensor([1.0, 1.0], dtype=D), "r1": torch.tensor([1.0], dtype=D), "r2": torch.tensor([3.0], dtype=D), "o": torch.eye(2, dtype=D)}
    # all scores equal but for the bias: ln(1 + 3) at distance one, so weights 1 and 1/4; the key two back is out of the window
    v = [torch.tensor(t, dtype=D) for t in ([-1.0, 1.0], [0.0, math.sqrt(2.0)], [1.0, 1.0])]    # each of unit root mean square
    out = P.attention(h, w, m, 0.0)
    assert torch.allclose(out[0], v[0]) and torch.allclose(out[1], 0.8 * v[1] + 0.2 * v[0]) and torch.allclose(out[2], 0.8 * v[2] + 0.2 * v[1])


def test_query_norm_runs_over_all_heads_before_the_cut():
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 9}}
    h = torch.tensor([[1.0], [-1.0]], dtype=D)
    w = {"q": torch.tensor([[3.0], [4.0]], dtype=D), "q.b": torch.zeros(2, dtype=D), "k": torch.tensor([[1.0]], dtype=D), "k.b": torch.zeros(1, dtype=D),
         "v": torch.tensor([[1.0]], dtype=D), "v.b": torch.zeros(1, dtype=D), "q.norm": torch.tensor([1.0, 2.0], dtype=D),
         "k.norm": torch.tensor([1.0], dtype=D), "r1": torch.zeros(2, dtype=D), "r2": torch.ones(2, dtype=D), "o": torch.eye(2, dtype=D)}
    rms = math.sqrt(12.5)                                                                     # of (3, 4) together, not head by head
    out = P.attention(h, w, m, 0.0)[1]                                                        # values +1 and -1, keys +1 and -1
    for a, q in enumerate((-3.0 / rms, -8.0 / rms)):
        e = math.exp(q), math.exp(-q)
        assert abs(out[a].item() - (e[0] - e[1]) / (e[0] + e[1])) < 1e-12


def test_routing_by_hand():
    z = torch.tensor([[0.0, math.log(3.0), -1e9, math.log(4.0)]], dtype=D)                    # scores 1/8, 3/8, 0, 1/2
    idx, wgt = P.route(z, torch.tensor([0.5, 0.0, 0.0, 0.0], dtype=D), 2)
    assert idx.tolist() == [[0, 3]] and torch.allclose(wgt, torch.tensor([[0.125, 0.5]], dtype=D))     # the weights do not sum to one
    h = torch.tensor([[1.0, -2.0]], dtype=D)
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 0.0]], dtype=D), "correction": torch.tensor([0.0, 5.0], dtype=D)}
    for e in range(2):
        w[f"e{e}.gate"], w[f"e{e}.up"] = torch.tensor([[1.0 + e, 0.0]], dtype=D), torch.tensor([[0.0, 3.0]], dtype=D)
        w[f"e{e}.down"] = torch.tensor([[1.0], [2.0]], dtype=D)
    y = P.experts(h, w, {"router": {"experts": 2, "top": 1}})
    s1 = 1.0 / (1.0 + math.e)                                                                 # expert 1 is chosen and keeps its small score
    a = 2.0 / (1 + math.exp(-2.0)) * -6.0
    assert torch.allclose(y[0], torch.tensor([s1 * a, 2 * s1 * a], dtype=D))


def test_a_layer_that_borrows_reads_its_owners_tensors():
    assert [P.owner(ZS_A, i) for i in range(4)] == [0, 1, 0, 3]
    assert [P.owner(ZS_C, i) for i in range(4)] == [0, 1, 1, 1]
