"""Rusolorn without a GPU: the configuration and its errors, the model as data, tensor names and shapes, what
the layers ask of the cache (Python and C++ managers), state sizes, how parts keep their tensors, and the plain
implementation's own pieces."""
import copy
import math

import pytest
import torch

import plain_rusolorn as pr
import rusolorn_cases as rc
from rllm_b200.cache import CacheManager
from rllm_b200.cache.native import NativeCacheManager
from rllm_b200.config import ConfigError, RusolornConfig, config_from_dict
from rllm_b200.csrc import ops
from rllm_b200.models.model import DecoderModel, expected_tensors
from rllm_b200.parts import PagedKVNeed, Runtime, StateNeed
from rusolorn_cases import CASES

F64 = torch.float64


@pytest.mark.parametrize("name", list(CASES))
def test_configuration_round_trip_and_tensor_list(name):
    cfg = CASES[name]
    c = config_from_dict(cfg)
    assert isinstance(c, RusolornConfig)
    assert config_from_dict(c.to_dict()) == c
    exp = expected_tensors(c.model_spec())
    want = rc.tensor_shapes(cfg)
    assert set(exp) == set(want)
    for n, (shape, _) in want.items():
        assert tuple(exp[n][0]) == tuple(shape), n


def test_the_model_as_data():
    spec = config_from_dict(CASES["stack"]).model_spec()
    assert all(ls.block == "shared_norm" and ls.block_params["residual_mult"] == 0.6 for ls in spec.layers)
    assert all(ls.mixer.kind == "parallel" and ls.position is None and set(ls.norms) == {"mixer"} for ls in spec.layers)
    assert [None if ls.ffn is None else ls.ffn.kind for ls in spec.layers] == ["routed_experts", None, "routed_experts", "routed_experts"]
    m = spec.layers[1].mixer.params
    assert m["left_scale"] == m["right_scale"] == 0.5
    assert m["left_norm"].params["tensor"] == "l1.mix.left.out" and m["right_norm"].params["tensor"] == "l1.mix.right.out"
    left, right = m["left"].params, m["right"].params
    assert (left["num_heads"], left["num_kv_heads"], left["head_dim"], left["window"], left["scale"]) == (6, 3, 16, 30, 0.5)
    assert left["tie_values"] and left["qk_norm"] == "row" and not left.get("gate")
    assert spec.layers[3].mixer.params["left"].params["window"] == 0
    assert (right["num_heads"], right["num_kv_heads"], right["head_dim"], right["v_head_dim"], right["conv"]) == (2, 2, 48, 40, 3)
    assert right["q_scale"] == 48 ** -0.5 and right["unit_eps"] == 1e-6
    f = spec.layers[0].ffn.params
    assert f["expert_form"] == {"limit": 1.6, "alpha": 1.702, "shift": 1.0} and f["shared_form"]["limit"] == 1.1
    assert (f["n_groups"], f["keep_groups"], f["group_best"], f["score"], f["shared_gate"]) == (4, 2, 1, "softmax", False)
    assert spec.layers[2].ffn.params["shared_size"] == 0 and spec.layers[3].ffn.params["n_groups"] == 1
    assert [ls.side.params["part"] for ls in spec.layers] == [0, 1, 2, 3] and spec.layers[0].side.params["parts"] == 4
    assert spec.embedding.params["scale"] == 4.0 and spec.lm_head.params["tied_to"] == "embed"
    assert spec.final_norm.kind == "dynamic_tanh" and spec.max_position == 0
    bare = config_from_dict(CASES["mixers_alone"]).model_spec()
    assert all(ls.side is None and ls.ffn is None for ls in bare.layers)


def _broken(name, edit):
    cfg = copy.deepcopy(CASES[name])
    edit(cfg)
    return cfg


_left = lambda c: c["layers"][0]["mixer"]["left"]
_right = lambda c: c["layers"][0]["mixer"]["right"]
_mlp = lambda c: c["layers"][0]["mlp"]


@pytest.mark.parametrize("edit,word", [
    (lambda c: _left(c).update(kv_heads=3), "kv_heads"),
    (lambda c: _left(c).update(vdim=13), "vdim"),
    (lambda c: _left(c).pop("scale"), "scale"),
    (lambda c: _left(c)["mask"].update(size=0), "size"),
    (lambda c: _right(c).update(heads=4), "heads"),
    (lambda c: _right(c).update(conv=0), "conv"),
    (lambda c: _right(c).pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0].update(type="attention"), "attention"),
    (lambda c: _mlp(c).update(kind="dense"), "dense"),
    (lambda c: _mlp(c)["expert"].pop("limit"), "limit"),
    (lambda c: _mlp(c)["shared"].update(limit=0.0), "limit"),
    (lambda c: _mlp(c)["router"].update(top=5), "top"),
    (lambda c: _mlp(c)["router"]["groups"].update(count=3), "groups"),
    (lambda c: _mlp(c)["router"]["groups"].update(keep=5), "groups"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(edit, word):
    with pytest.raises(ConfigError) as e:
        config_from_dict(_broken("one_layer", edit))
    assert word in str(e.value)


def _model(name):
    return DecoderModel(config_from_dict(CASES[name]).model_spec(), Runtime(torch.device("cpu"), torch.float32))


def test_what_the_layers_ask_of_the_cache():
    needs, owners = _model("stack").cache_needs()
    assert len(needs) == 4 and owners == [None] * 4
    assert needs[0] == (PagedKVNeed(2, 32, 13, 0, 0), StateNeed((ops.delta_state_floats(4, 16, 24, 4),), torch.float32))
    assert needs[3] == (PagedKVNeed(4, 24, 0, 0, 0), StateNeed((ops.delta_state_floats(2, 64, 32, 2),), torch.float32))


def test_state_sizes():
    # per head: the key rows rounded up to 32, 64, 128, 256 or 512 times the value columns rounded up to 8, and the
    # kept inputs of the convolutions of its q, k and v channels
    assert ops.delta_state_floats(1, 5, 3, 3) == 32 * 8 + 13 * 2
    assert ops.delta_state_floats(2, 48, 40, 4) == 2 * (64 * 40 + 136 * 3)
    assert ops.delta_state_floats(3, 136, 41, 1) == 3 * 256 * 48
    assert ops.delta_state_floats(1, 300, 8, 2) == 512 * 8 + 608
    from rllm_b200.csrc import build
    try:
        lib = build.load("delta")
    except Exception:
        pytest.skip("the delta rule's library cannot be built here")
    lib.rllm_delta_state_floats.restype = __import__("ctypes").c_longlong
    for args in ((1, 5, 3, 3), (2, 48, 40, 4), (4, 128, 64, 1), (3, 136, 41, 6), (1, 300, 8, 2)):
        assert lib.rllm_delta_state_floats(*args) == ops.delta_state_floats(*args)


@pytest.mark.parametrize("manager", [CacheManager, NativeCacheManager])
def test_both_cache_managers_take_the_model(manager):
    needs, owners = _model("stack").cache_needs()
    cm = manager(needs, owners, 8, 256, 3)
    assert [g.need.window for g in cm.paged] == [13, 30, 6, 0] and len(cm.stateful) == 4
    slots = cm.append("a", 50)
    assert len(slots) == 4 and all(len(s) == 50 for s in slots)
    cm.append("a", 150)
    cm.release_passed("a")                                          # three windows have passed most of the 200 tokens
    assert [cm.n_free_pages(g) > 32 - 25 for g in range(4)] == [True, True, True, False]
    cm.append("b", 9)
    assert cm.state_slot("a") != cm.state_slot("b")
    cm.free("a")
    cm.free("b")
    cm.check_invariants()


def test_parts_keep_one_stacked_product_and_their_run_of_the_table():
    cfg = CASES["odd_sizes"]
    model = _model("odd_sizes")
    w = rc.make_weights(cfg, 3)
    model.load_tensors(dict(w))
    mx = model.blocks[1].mixer
    assert mx.w_both.shape[0] % 8 == 0 and mx.split % 8 == 0
    assert mx.left.w_qkv.data_ptr() == mx.w_both.data_ptr()                              # views, not copies
    assert mx.right.w_in.data_ptr() == mx.w_both.data_ptr() + mx.split * cfg["width"] * 4
    qk = 33
    assert torch.equal(mx.w_both[:9], w["l1.mix.left.q"]) and torch.equal(mx.w_both[9:18], w["l1.mix.left.k"])
    assert torch.equal(mx.right.w_in[qk:2 * qk], w["l1.mix.right.k"])
    b, a = mx.right.offs[4], mx.right.offs[5]
    assert torch.equal(mx.right.w_in[b:b + 5], w["l1.mix.right.b"]) and torch.equal(mx.right.w_in[a:a + 5], w["l1.mix.right.a"])
    assert not mx.right.w_in[a + 5:].any()
    side = model.blocks[1].side
    assert torch.equal(side.table, w["side.embed"][:, 5:10]) and side.padded == 8
    assert torch.equal(side.w_gate[:5], w["l1.side.gate"]) and not side.w_gate[5:].any() and not side.w_proj[:, 5:].any()
    assert model.final_norm.alpha == float(w["final.norm.alpha"])


# ---------------------------------------------------------------- the plain implementation's own pieces

def test_plain_attention_counts_the_token_itself_and_mixes_unnormed_keys():
    mx = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.0, "mask": {"size": 3}}
    w = {"a.q": torch.eye(2, dtype=F64), "a.k": torch.eye(2, dtype=F64), "a.o": torch.eye(2, dtype=F64),
         "a.q.norm": torch.ones(2, dtype=F64), "a.k.norm": 9 * torch.ones(2, dtype=F64)}
    h = torch.stack([torch.arange(6, dtype=F64), torch.ones(6, dtype=F64)], 1)
    out = pr.attention(h, w, "a.", mx, 1e-6)                        # scale 0: the mean of the visible values
    assert torch.allclose(out[:, 0], torch.tensor([0.0, 0.5, 1.0, 2.0, 3.0, 4.0], dtype=F64))
    mx = dict(mx, mask={"size": 1})
    assert torch.allclose(pr.attention(h, w, "a.", mx, 1e-6), h)


def test_plain_convolution_weighs_the_current_token_with_its_last_tap():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    out = pr.causal_conv_silu(x, torch.tensor([[2.0, 3.0]], dtype=F64))
    want = torch.tensor([[3.0], [32.0], [320.0]], dtype=F64)
    assert torch.allclose(out, want / (1 + torch.exp(-want)))


def test_plain_delta_rule_reads_its_own_write_and_corrects_towards_the_value():
    g = torch.Generator().manual_seed(1)
    k = pr.unit(torch.randn(5, 1, 4, generator=g, dtype=F64))
    v = torch.randn(5, 1, 3, generator=g, dtype=F64)
    one = torch.ones(5, 1, dtype=F64)
    # full strength, no decay: what is read along the key just written is its value, whatever was there before
    assert torch.allclose(pr.delta_rule(k, k, v, one, one), v, atol=1e-5)
    # no write: nothing; half strength, first token: half the value
    assert not pr.delta_rule(k, k, v, 0 * one, one).any()
    half = pr.delta_rule(k, k, v, 0.5 * one, one)
    assert torch.allclose(half[0], 0.5 * v[0], atol=1e-5)
    # the decay comes before the correction: token 1 sees g S_0
    q = torch.randn(2, 1, 4, generator=g, dtype=F64)
    o = pr.delta_rule(q, k[:2], v[:2], one[:2] * 0.7, torch.tensor([[0.9], [0.4]], dtype=F64))
    S = torch.outer(k[0, 0], 0.7 * v[0, 0]) * 0.4
    S = S + torch.outer(k[1, 0], 0.7 * (v[1, 0] - S.T @ k[1, 0]))
    assert torch.allclose(o[1, 0], S.T @ q[1, 0])


def test_plain_chunk_form_is_the_recurrence():
    """What a chunk of tokens does to the memory, written with the chunk's products, against the literal recurrence."""
    g = torch.Generator().manual_seed(2)
    T, dk, dv = 8, 5, 3
    q, k = torch.randn(T, 1, dk, generator=g, dtype=F64), pr.unit(torch.randn(T, 1, dk, generator=g, dtype=F64))
    v, S0 = torch.randn(T, 1, dv, generator=g, dtype=F64), torch.randn(dk, dv, generator=g, dtype=F64)
    beta, dec = torch.rand(T, 1, generator=g, dtype=F64), torch.rand(T, 1, generator=g, dtype=F64)
    S = S0.clone()
    want = []
    for t in range(T):
        S = dec[t] * S
        S = S + torch.outer(k[t, 0], beta[t] * (v[t, 0] - S.T @ k[t, 0]))
        want.append(S.T @ q[t, 0])
    c = torch.cumprod(dec[:, 0], 0)
    d = torch.tensor([[float(torch.prod(dec[j + 1:i + 1])) if j <= i else 0.0 for j in range(T)] for i in range(T)], dtype=F64)
    u = []
    for i in range(T):
        r = beta[i] * (v[i, 0] - c[i] * (S0.T @ k[i, 0]))
        for j in range(i):
            r = r - beta[i] * d[i, j] * (k[i, 0] @ k[j, 0]) * u[j]
        u.append(r)
    for i in range(T):
        o = c[i] * (S0.T @ q[i, 0]) + sum(d[i, j] * (q[i, 0] @ k[j, 0]) * u[j] for j in range(i + 1))
        assert torch.allclose(o, want[i])
    end = c[-1] * S0 + sum(d[-1, j] * torch.outer(k[j, 0], u[j]) for j in range(T))
    assert torch.allclose(end, S)


def test_plain_router_keeps_the_groups_with_the_largest_single_score():
    s = torch.tensor([0.30, 0.01, 0.20, 0.19, 0.02, 0.28], dtype=F64)
    idx, margin = pr.choose(s, 2, 3, 2)                             # groups {0,1}, {2,3}, {4,5}: best 0.30, 0.20, 0.28
    assert idx == [0, 5] and math.isclose(margin, 0.08)             # the second group's 0.19 and 0.20 do not count together
    assert pr.choose(s, 2, 1, 1)[0] == [0, 5] and pr.choose(s, 3, 1, 1)[0] == [0, 5, 2]
    assert pr.choose(s, 2, 3, 1)[0] == [0, 1]


def test_plain_unit_clamps_the_gate_above_only():
    w = {"u.gate": torch.tensor([[1.0]], dtype=F64), "u.up": torch.tensor([[1.0]], dtype=F64), "u.down": torch.tensor([[1.0]], dtype=F64)}
    h = torch.tensor([[-5.0], [0.5], [5.0]], dtype=F64)
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    want = torch.tensor([[f(-5.0, -2.0)], [f(0.5, 0.5)], [f(2.0, 2.0)]], dtype=F64)
    assert torch.allclose(pr.clamped_unit(h, w, "u.", 2.0), want)
