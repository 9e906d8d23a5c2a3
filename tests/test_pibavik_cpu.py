"""Pibavik without a GPU: the configuration and its errors, the model as data, tensor names and shapes, what the layers ask of
the cache (Python and C++ managers, keys that another layer reads through a longer window), state sizes, how parts keep
their tensors, and the plain implementation's own pieces."""
import copy
import math

import pytest
import torch

import pibavik_cases as pc
import plain_pibavik as pp
from pibavik_cases import CASES
from rllm_b200.cache import CacheManager
from rllm_b200.cache.native import NativeCacheManager
from rllm_b200.config import ConfigError, PibavikConfig, config_from_dict
from rllm_b200.csrc import ops
from rllm_b200.models.model import DecoderModel, expected_tensors
from rllm_b200.parts import PagedKVNeed, Runtime, StateNeed

F64 = torch.float64


@pytest.mark.parametrize("name", list(CASES))
def test_configuration_round_trip_and_tensor_list(name):
    cfg = CASES[name]
    c = config_from_dict(cfg)
    assert isinstance(c, PibavikConfig)
    assert c.to_dict() == cfg and config_from_dict(c.to_dict()) == c
    exp = expected_tensors(c.model_spec())
    want = pc.tensor_shapes(cfg)
    assert set(exp) == set(want)
    for n, (shape, _) in want.items():
        assert tuple(exp[n][0]) == tuple(shape), n


def test_the_model_as_data():
    spec = config_from_dict(CASES["stack"]).model_spec()
    assert all(ls.block == "pre_norm" for ls in spec.layers)
    assert [ls.mixer.kind for ls in spec.layers] == ["attention", "parallel", "latent_attention", "attention", "parallel"]
    assert [ls.ffn is None for ls in spec.layers] == [False, False, False, True, False]
    assert [e.cache_of for e in spec.run_order] == [None, None, None, 0, None]
    a, b = spec.layers[0].mixer.params, spec.layers[3].mixer.params
    assert a["slopes"] == (0.25, 0.0625, 0.015625, 0.00390625) and (a["window"], b["window"]) == (13, 45)
    assert a["own_kv"] and not b["own_kv"] and a["cache_window"] == b["cache_window"] == 45
    p = spec.layers[1].mixer.params
    left, right = p["left"].params, p["right"].params
    assert (p["left_scale"], p["right_scale"]) == (0.7, 0.8) and left["qk_norm"] == "head" and left["gate_per_head"]
    assert spec.layers[1].position.params["dims"] == 12 and spec.layers[1].position.params["base"] == 2000.0
    assert spec.layers[0].position is None and spec.layers[2].position is None
    assert (right["num_heads"], right["v_head_dim"], right["state"], right["groups"], right["conv"], right["norm_groups"]) == (4, 32, 48, 2, 4, 2)
    f = spec.layers[0].ffn.params
    assert (f["activation"], f["weigh_input"], f["normalize"], f["score"], f["shared_size"]) == ("relu2", True, False, "sigmoid", 40)
    assert spec.layers[1].ffn.params["shared_size"] == 0
    assert spec.embedding.params["scale"] == 3.0 and not spec.lm_head.params.get("tied_to") and spec.max_position == 0
    bare = config_from_dict(CASES["pair_unrotated"]).model_spec()
    assert bare.layers[0].position is None and bare.layers[0].ffn is None


def _broken(name, edit):
    cfg = copy.deepcopy(CASES[name])
    edit(cfg)
    return cfg


_mx = lambda c, i=0: c["layers"][i]["mixer"]
_mlp = lambda c: c["layers"][0]["mlp"]


@pytest.mark.parametrize("name,edit,word", [
    ("stack", lambda c: _mx(c).update(kv_heads=3), "kv_heads"),
    ("stack", lambda c: _mx(c).pop("scale"), "scale"),
    ("stack", lambda c: _mx(c)["mask"].update(size=0), "size"),
    ("stack", lambda c: _mx(c, 3).update(kv_from=3), "kv_from"),
    ("stack", lambda c: _mx(c, 3).update(kv_from=1), "kv_from"),
    ("stack", lambda c: _mx(c, 3).update(dim=30), "head sizes"),
    ("shared_keys", lambda c: _mx(c, 3).update(kv_from=1), "kv_from"),
    ("stack", lambda c: _mx(c, 2).pop("kv_rank"), "kv_rank"),
    ("stack", lambda c: _mx(c, 2).update(q_rank=0), "q_rank"),
    ("stack", lambda c: _mx(c, 1).pop("right"), "right"),
    ("stack", lambda c: _mx(c, 1).pop("left_scale"), "left_scale"),
    ("stack", lambda c: _mx(c, 1)["left"]["rot"].update(dims=34), "dims"),
    ("stack", lambda c: _mx(c, 1)["left"]["rot"].update(dims=3), "dims"),
    ("stack", lambda c: _mx(c, 1)["right"].update(groups=3), "groups"),
    ("stack", lambda c: _mx(c, 1)["right"].update(norm_groups=7), "norm_groups"),
    ("stack", lambda c: _mx(c, 1)["right"].update(conv=0), "conv"),
    ("stack", lambda c: c["layers"][0].update(type="mamba2"), "mamba2"),
    ("stack", lambda c: _mlp(c).update(kind="dense"), "dense"),
    ("stack", lambda c: _mlp(c)["expert"].pop("ff"), "ff"),
    ("stack", lambda c: _mlp(c)["shared"].update(ff=0), "ff"),
    ("stack", lambda c: _mlp(c)["router"].update(top=9), "top"),
    ("stack", lambda c: c["norm"].update(eps=0.0), "eps"),
    ("stack", lambda c: c.pop("vocab"), "vocab"),
    ("stack", lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(name, edit, word):
    with pytest.raises(ConfigError) as e:
        config_from_dict(_broken(name, edit))
    assert word in str(e.value)


def _model(name, dtype=torch.float32):
    return DecoderModel(config_from_dict(CASES[name]).model_spec(), Runtime(torch.device("cpu"), dtype))


def test_what_the_layers_ask_of_the_cache():
    needs, owners = _model("stack").cache_needs()
    assert owners == [None, None, None, 0, None]
    assert needs[0] == needs[3] == PagedKVNeed(2, 32, 45, 0, 0)           # the reader's window is the longer one
    assert needs[1] == (PagedKVNeed(2, 32, 30, 0, 16), StateNeed((ops.ssd_state_floats(4, 32, 48, 2, 4),), torch.float32))
    assert needs[2] == PagedKVNeed(1, 48, values_in_keys=48)
    needs, _ = _model("shared_keys_all").cache_needs()
    assert needs[0] == needs[1] == PagedKVNeed(1, 24, 0, 0, 0)            # a reader that sees everything
    needs, _ = _model("sloped_padded", torch.bfloat16).cache_needs()
    assert needs[0] == PagedKVNeed(1, 128, 21, 0, 0) and needs[1] == PagedKVNeed(3, 64, 9, 0, 0)
    needs, _ = _model("latent", torch.bfloat16).cache_needs()
    assert needs[0] == PagedKVNeed(1, 64, values_in_keys=64)


def test_state_sizes():
    # S of every head, then taps - 1 + 8 rows of the convolution's inputs; a multiple of 4
    assert ops.ssd_state_floats(2, 4, 8, 1, 4) == 2 * 4 * 8 + 11 * (8 + 16)
    assert ops.ssd_state_floats(1, 3, 5, 1, 1) == -(-(15 + 8 * 13) // 4) * 4


@pytest.mark.parametrize("manager", [CacheManager, NativeCacheManager])
def test_both_cache_managers_keep_keys_for_the_longest_reader(manager):
    needs, owners = _model("shared_keys").cache_needs()
    cm = manager(needs, owners, 8, 512, 3)
    assert [g.need.window for g in cm.paged] == [19]
    cm.append("a", 300)
    before = cm.n_free_pages(0)
    assert cm.release_passed("a") == 256 // 8 and cm.n_free_pages(0) == before + 32     # runs of 128 keys behind 300 + 1 - 19
    needs, owners = _model("stack").cache_needs()
    cm = manager(needs, owners, 8, 256, 3)
    assert [g.need.window for g in cm.paged] == [45, 30, 0, 9] and len(cm.stateful) == 2
    cm.append("a", 50)
    cm.append("a", 150)
    cm.release_passed("a")
    cm.append("b", 9)
    assert cm.state_slot("a") != cm.state_slot("b")
    cm.free("a")
    cm.free("b")
    cm.check_invariants()


def test_sides_keep_one_product_at_each_end():
    cfg = CASES["odd_sizes"]
    model = _model("odd_sizes")
    w = pc.make_weights(cfg, 3)
    model.load_tensors(dict(w))
    mx = model.blocks[1].mixer
    assert mx.w_both.shape[0] % 8 == 0 and mx.split % 8 == 0
    assert mx.left.w_qkv.data_ptr() == mx.w_both.data_ptr()                              # views, not copies
    assert mx.right.w_in.data_ptr() == mx.w_both.data_ptr() + mx.split * cfg["width"] * 4
    assert torch.equal(mx.w_both[:27], w["l1.mix.left.q"]) and torch.equal(mx.w_both[47:50], w["l1.mix.left.g"])
    n = w["l1.mix.right.in"].shape[0]
    assert torch.equal(mx.right.w_in[:n], w["l1.mix.right.in"]) and not mx.right.w_in[n:].any()
    assert torch.equal(mx.w_ends, torch.cat([w["l1.mix.left.o"], w["l1.mix.right.o"]], 1))
    assert mx.left.w_o is None and mx.right.w_o is None
    assert torch.equal(mx.right.conv_w, w["l1.mix.right.conv"].t()) and torch.allclose(mx.right.A, torch.exp(w["l1.mix.right.A_log"]))


def test_padded_heads_and_latents_hold_zeros():
    cfg = CASES["sloped_padded"]
    model = _model("sloped_padded", torch.bfloat16)
    w = pc.make_weights(cfg, 4, torch.bfloat16)
    model.load_tensors(dict(w))
    att = model.blocks[1].mixer                                             # heads of 16 and 56, stored as 64
    q = att.w_qkv[:3 * 64].view(3, 64, -1)
    assert torch.equal(q[:, :16].reshape(48, -1), w["l1.mix.q"]) and not q[:, 16:].any()
    v = att.w_qkv[6 * 64:].view(3, 64, -1)
    assert torch.equal(v[:, :56].reshape(168, -1), w["l1.mix.v"]) and not v[:, 56:].any()
    o = att.w_o.view(-1, 3, 64)
    assert torch.equal(o[:, :, :56].reshape(-1, 168), w["l1.mix.o"]) and not o[:, :, 56:].any()
    cfg = CASES["latent"]
    model = _model("latent", torch.bfloat16)
    w = pc.make_weights(cfg, 5, torch.bfloat16)
    model.load_tensors(dict(w))
    lat = model.blocks[0].mixer
    assert lat.w_qc.shape == (3, 64, 16) and not lat.w_qc[:, 36:].any() and lat.w_uv.shape == (3, 24, 64) and not lat.w_uv[:, :, 36:].any()
    assert torch.equal(lat.w_qc[1, :36].t(), w["l0.mix.uk"][16:32])


# ---------------------------------------------------------------- the plain implementation's own pieces

def test_plain_attention_counts_the_token_itself_and_takes_the_slope_off():
    q, k = torch.zeros(5, 2, 1, dtype=F64), torch.zeros(5, 1, 1, dtype=F64)
    v = torch.arange(5, dtype=F64).view(5, 1, 1)
    out = pp.attend(q, k, v, 1.0, window=2)                                  # equal scores: the mean of the visible values
    assert torch.allclose(out[:, 0, 0], torch.tensor([0.0, 0.5, 1.5, 2.5, 3.5], dtype=F64))
    assert torch.equal(pp.attend(q, k, v, 1.0, window=1)[:, 1, 0], v[:, 0, 0])
    out = pp.attend(q, k, v, 1.0, slope=torch.tensor([math.log(2.0), 0.0], dtype=F64))      # every step back halves the weight
    assert torch.allclose(out[2, :, 0], torch.tensor([(2 + 0.5 + 0) / 1.75, 1.0], dtype=F64))
    assert pp.slopes(8)[0] == 0.5 and pp.slopes(8)[7] == 2.0 ** -8 and pp.slopes(1)[0] == 2.0 ** -8


def test_plain_rotation_pairs_halves_and_depends_on_the_distance_only():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 1, 6, generator=g, dtype=F64), torch.randn(1, 1, 6, generator=g, dtype=F64)
    rq, rk = pp.rotate(q.repeat(9, 1, 1), 4, 100.0), pp.rotate(k.repeat(9, 1, 1), 4, 100.0)
    assert torch.allclose(rq[3, 0] @ rk[1, 0], rq[8, 0] @ rk[6, 0]) and torch.equal(rq[:, :, 4:], q.repeat(9, 1, 1)[:, :, 4:])
    e = pp.rotate(torch.tensor([[[1.0, 0, 0, 0]]], dtype=F64).repeat(2, 1, 1), 4, 100.0)[1, 0]
    assert torch.allclose(e, torch.tensor([math.cos(1), 0, math.sin(1), 0], dtype=F64))


def test_plain_recurrence_decays_before_it_writes():
    x, B, C = torch.tensor([[[2.0]], [[5.0]]], dtype=F64), torch.ones(2, 1, 1, dtype=F64), torch.ones(2, 1, 1, dtype=F64)
    y = pp.state_space(x, B, C, torch.tensor([[3.0], [0.5]], dtype=F64), torch.tensor([2.0], dtype=F64), torch.tensor([10.0], dtype=F64))
    assert torch.allclose(y[:, 0, 0], torch.tensor([6.0 + 20, 6 * math.exp(-1.0) + 2.5 + 50], dtype=F64))


def test_plain_chunk_form_is_the_recurrence():
    """A chunk written with the decays' running sums and the chunk's products, against the literal recurrence."""
    g = torch.Generator().manual_seed(2)
    T, N, P = 9, 4, 3
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    x, B, C, dt = rnd(T, 1, P), rnd(T, 1, N), rnd(T, 1, N), torch.rand(T, 1, generator=g, dtype=F64)
    A, D = torch.tensor([1.7], dtype=F64), torch.zeros(1, dtype=F64)
    want = pp.state_space(x, B, C, dt, A, D)[:, 0]
    cut = 4                                              # the state before the chunk
    S = torch.zeros((N, P), dtype=F64)
    for t in range(cut):
        S = torch.exp(-A * dt[t]) * S + dt[t] * torch.outer(B[t, 0], x[t, 0])
    L = torch.cumsum(-A * dt[cut:, 0], 0)
    for i in range(T - cut):
        y = torch.exp(L[i]) * (S.T @ C[cut + i, 0])
        for j in range(i + 1):
            y = y + (C[cut + i, 0] @ B[cut + j, 0]) * torch.exp(L[i] - L[j]) * dt[cut + j, 0] * x[cut + j, 0]
        assert torch.allclose(y, want[cut + i])


def test_plain_convolution_weighs_the_current_token_with_its_last_tap():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    out = pp.causal_conv_silu(x, torch.tensor([[2.0, 3.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    want = torch.tensor([[3.5], [32.5], [320.5]], dtype=F64)
    assert torch.allclose(out, want / (1 + torch.exp(-want)))


def test_plain_experts_weigh_their_input():
    w = {"m.router": torch.tensor([[0.0], [-1.0]], dtype=F64), "m.e0.up": torch.tensor([[2.0], [-1.0]], dtype=F64),
         "m.e0.down": torch.tensor([[1.0, 1.0]], dtype=F64), "m.e1.up": torch.zeros(2, 1, dtype=F64), "m.e1.down": torch.zeros(1, 2, dtype=F64)}
    out = pp.experts(torch.tensor([[3.0]], dtype=F64), w, "m.", {"router": {"top": 1}})
    assert torch.allclose(out, torch.tensor([[(0.5 * 6.0) ** 2]], dtype=F64))                # sigmoid(0) = 1/2 inside the square
    assert pp.choose(torch.tensor([0.3, 0.9, 0.5], dtype=F64), 2)[0] == [1, 2]
