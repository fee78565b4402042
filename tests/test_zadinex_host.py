"""Host-side tests of the Zadinex entry of the model registry (no GPU): config parsing and refusals through the C ABI, and sanity of the plain
float64 restatement the GPU tests compare against: it is causal, and its mechanisms do by hand what they say."""
import ctypes as C
import json
import math

import pytest
import torch

import koifish_b200 as kf
from koifish_b200 import _lib as L
import zadinex_ref as ref
from zadinex_models import attn, config, dense, layer, moe, tokens, weights, wkv

D = torch.float64


def dims(cfg):
    lib = kf.load()
    info, err = L.ModelInfo(), C.c_void_p()
    st = lib.kf_config_dims(json.dumps(cfg).encode(), C.byref(info), C.byref(err))
    msg = C.cast(err, C.c_char_p).value.decode() if err.value else ""
    if err.value:
        lib.kf_string_free(err)
    return st, info, msg


def small():
    return config([layer(wkv(), moe()), layer(attn(heads=3, kv_heads=1, vdim=20), None), layer(attn(), dense())], width=24, vocab=50)


def test_config_is_parsed_by_its_registry_entry():
    st, info, msg = dims({"hf_config": small(), "gpt": {"max_seq_len": 96, "max_batch": 3, "compute_dtype": "float32"}})
    assert st == kf.KF_OK, msg
    assert (info.n_layers, info.n_embd, info.vocab, info.max_seq_len, info.max_batch) == (3, 24, 50, 96, 3)
    st, info, msg = dims(small())  # the bare config.json
    assert st == kf.KF_OK and info.n_layers == 3, msg


def test_optional_keys_may_be_null_or_absent():
    cfg = small()
    a = cfg["layers"][1]["mixer"]
    a["rot"] = None
    a.pop("kv_heads"), a.pop("scale"), a.pop("vdim"), a.pop("v_mix")
    cfg["layers"][2]["mixer"]["rot"].pop("dims")
    cfg["layers"][0]["mixer"].pop("w_rank")
    cfg["layers"][0]["mlp"]["router"].pop("groups")
    cfg["layers"][0]["mlp"]["router"]["identity"] = None
    cfg["layers"][0]["mlp"]["expert"]["limit"] = None
    cfg["layers"][1].pop("mlp")
    st, _, msg = dims({"hf_config": cfg})
    assert st == kf.KF_OK, msg


@pytest.mark.parametrize("edit, words", [
    (lambda c: c["layers"][0].update(type="mingru"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(dim=600), "<= 512"),
    (lambda c: c["layers"][0]["mixer"].update(w_rank=0), "w_rank"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "kv_heads must divide heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=600), "<= 512"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=21), "kv_heads x vdim"),      # the two blending layers then differ
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "at most dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].pop("base"), "rot.base is missing"),
    (lambda c: c["layers"][0]["mlp"].update(kind="table"), "is not built"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top <= keep"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=2), "must divide"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "keep <= count"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff is missing"),
    (lambda c: c["layers"][2]["mlp"].pop("ff"), "ff is missing"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_refusals(edit, words):
    cfg = small()
    edit(cfg)
    st, _, msg = dims({"hf_config": cfg})
    assert st != kf.KF_OK and words in msg, msg


def test_no_device_no_model():
    if torch.cuda.is_available():
        pytest.skip("a GPU is present")
    with pytest.raises(kf.KoifishError):
        kf.Context(0)


# ------------------------------------------------------------------------------------------------------------ the oracle itself
def test_oracle_is_causal():
    cfg = small()
    W = weights(cfg, seed=1)
    a = tokens(40, cfg["vocab"], 2)
    b = list(a)
    b[25] = (a[25] + 1) % cfg["vocab"]
    la, lb = ref.forward(cfg, W, a), ref.forward(cfg, W, b)
    assert torch.allclose(la[:25], lb[:25], atol=1e-12) and not torch.allclose(la[25:], lb[25:])
    assert torch.allclose(ref.forward(cfg, W, a[:11]), la[:11], atol=1e-12)


def test_scan_by_hand():
    """one head, one key channel, one value: the first read-out sees the bonus alone, the second the undecayed first product"""
    r, k, v, d = (torch.tensor(x, dtype=D).view(3, 1, 1) for x in ([1.0, 2.0, 3.0], [5.0, 7.0, 11.0], [0.5, -1.0, 2.0], [0.9, 0.5, 0.25]))
    o = ref.wkv_scan(r, k, v, d, torch.tensor([[0.1]]))[:, 0, 0].tolist()
    s1 = 5 * 0.5
    s2 = 0.5 * s1 + 7 * -1.0
    u = float(torch.tensor(0.1))
    assert o == pytest.approx([u * 5 * 0.5, 2 * (s1 + u * 7 * -1.0), 3 * (s2 + u * 11 * 2.0)])


def test_scan_in_two_parts_equals_one():
    g = torch.Generator().manual_seed(1)
    r, k, v, d = (torch.rand(9, 2, 4, dtype=D, generator=g) for _ in range(4))
    u = torch.rand(2, 4, generator=g)
    S = torch.zeros(2, 4, 4, dtype=D)
    parts = [ref.wkv_scan(r[a:b], k[a:b], v[a:b], d[a:b], u, S) for a, b in ((0, 4), (4, 9))]
    assert torch.allclose(torch.cat(parts), ref.wkv_scan(r, k, v, d, u), atol=1e-12)


def test_norm_and_mix_by_hand():
    x = torch.tensor([[1.0, -2.0], [0.5, 3.0]], dtype=D)
    y = ref.dyt(x, torch.tensor(2.0), torch.tensor([3.0, 1.0]), torch.tensor([0.25, -1.0]))
    assert y[0].tolist() == pytest.approx([3 * math.tanh(2.0) + 0.25, math.tanh(-4.0) - 1.0])
    z = ref.token_mix(x, torch.tensor([0.25, 1.0]))
    assert torch.allclose(z, torch.tensor([[0.75, 0.0], [0.625, -2.0]], dtype=D))


def test_rotation_pairs_and_angles():
    x = torch.zeros(3, 1, 6, dtype=D)
    x[:, 0, 1], x[:, 0, 5] = 1.0, 7.0
    y = ref.rotate(x, 4, 100.0)  # pairs (0, 2), (1, 3); entries 4 and 5 pass
    for t in range(3):
        a = t * 100.0 ** -0.5
        assert y[t, 0].tolist() == pytest.approx([0, math.cos(a), 0, math.sin(a), 0, 7.0])


def test_sink_takes_its_share():
    """zero queries: every key weighs the same, and a sink of ln(c) weighs as c keys without a value"""
    m = dict(heads=1, kv_heads=1, dim=4, vdim=4, scale=1.0)
    g = torch.Generator().manual_seed(3)
    W = {"q": torch.zeros(4, 4), "k": torch.randn(4, 4, generator=g), "v": torch.eye(4), "sink": torch.tensor([math.log(3.0)]), "o": torch.eye(4)}
    h = torch.randn(6, 4, dtype=D, generator=g)
    out = ref.attention(h, m, W, "", 1e-5, {})
    for i in range(6):
        assert torch.allclose(out[i], h[:i + 1].sum(0) / (i + 1 + 3.0), atol=1e-6)


def test_values_are_blended_with_the_first_blending_layer():
    m = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=1.0, v_mix=True)
    W = {"q": torch.zeros(2, 2), "k": torch.eye(2), "v": torch.eye(2), "sink": torch.tensor([-1e4]), "o": torch.eye(2), "vmix": torch.tensor(0.25)}
    h = torch.tensor([[1.0, 2.0]], dtype=D)
    carried = {}
    assert torch.allclose(ref.attention(h, m, W, "", 1e-5, carried), h)                                    # its own number is not used
    assert torch.allclose(ref.attention(3 * h, m, W, "", 1e-5, carried), 0.75 * 3 * h + 0.25 * h)          # blends
    assert torch.allclose(ref.attention(5 * h, m, W, "", 1e-5, carried), 0.75 * 5 * h + 0.25 * h)          # with the FIRST layer, not the last
    assert torch.allclose(ref.attention(5 * h, dict(m, v_mix=False), W, "", 1e-5, carried), 5 * h)


def test_routing_by_hand():
    z = torch.log(torch.tensor([0.05, 0.3, 0.1, 0.15, 0.2, 0.2], dtype=D))
    zero = torch.zeros(6)
    assert ref.route(z, zero, 2, 1, 1)[0][0] == 1
    got, w = ref.route(z, zero, 2, 3, 1)                     # groups (0, 1), (2, 3), (4, 5): the largest entry decides, not the sum
    assert got == [1, 0] and w.tolist() == pytest.approx([0.3 / 0.35, 0.05 / 0.35])
    corr = torch.tensor([-1.0, -1.0, -0.9, -0.8, -0.9, -0.95])  # all choice values negative: a closed group must not win with a zero
    got, w = ref.route(z, corr, 3, 3, 2)                     # choice: -.95 -.7 | -.8 -.65 | -.7 -.75
    assert got[0] == 3 and set(got) <= {0, 1, 2, 3, 4, 5} and w.sum().item() == pytest.approx(1.0)
    got, w = ref.route(z, torch.tensor([5.0, 0, 0, 0, 0, 0]), 1, 1, 1)
    assert got == [0] and w.tolist() == pytest.approx([1.0])  # the correction chooses, the weight ignores it


def test_experts_pass_through_outputs_return_their_input():
    cfg = config([layer(wkv(), moe(experts=2, identity=2, top=1, groups=None))], width=8)
    W = weights(cfg, seed=6)
    W["l0.mlp.correction"] = torch.tensor([0.0, 0.0, 0.0, 9.0])
    h = torch.randn(3, 8, dtype=D, generator=torch.Generator().manual_seed(1))
    assert torch.allclose(ref.experts_ff(h, cfg["layers"][0]["mlp"], W, "l0.mlp."), h)


def test_expert_clamps():
    W = {"gate": torch.eye(2), "up": torch.eye(2), "down": torch.eye(2)}
    out = ref.expert(torch.tensor([[5.0, -5.0]], dtype=D), W, "", 1.5)[0].tolist()
    s = lambda z: 1 / (1 + math.exp(-z))
    assert out == pytest.approx([1.5 * s(1.702 * 1.5) * 2.5, -5 * s(-1.702 * 5) * (-0.5)])  # the gate is not clamped from below
