"""Host-side tests of the Gadilix entry of the model registry (no GPU): config parsing and refusals through the C ABI, and sanity of the
plain float64 restatement the GPU tests compare against: it is causal, its window, blocks, shift and expert table do what they say, and the
shaped weights of the GPU tests do what they are meant to."""
import ctypes as C
import json

import pytest
import torch

import koifish_b200 as kf
from koifish_b200 import _lib as L
import gadilix_ref as ref
from gadilix_models import attn, config, layer, moe, tokens, weights


def dims(cfg):
    lib = kf.load()
    info, err = L.ModelInfo(), C.c_void_p()
    st = lib.kf_config_dims(json.dumps(cfg).encode(), C.byref(info), C.byref(err))
    msg = C.cast(err, C.c_char_p).value.decode() if err.value else ""
    if err.value:
        lib.kf_string_free(err)
    return st, info, msg


def small():
    return config([layer(attn(), moe()), layer(attn(heads=3, kv_heads=1), None), layer(attn(), moe(), weights_of=0)], width=24, vocab=50)


def test_config_is_parsed_by_its_registry_entry():
    st, info, msg = dims({"hf_config": small(), "gpt": {"max_seq_len": 96, "max_batch": 3, "compute_dtype": "float32"}})
    assert st == kf.KF_OK, msg
    assert (info.n_layers, info.n_embd, info.vocab, info.max_seq_len, info.max_batch) == (3, 24, 50, 96, 3)
    st, info, msg = dims(small())  # the bare config.json
    assert st == kf.KF_OK and info.n_layers == 3, msg


def test_optional_keys_may_be_null_or_absent():
    cfg = small()
    a = cfg["layers"][1]["mixer"]
    a["mask"] = None
    a.pop("kv_heads"), a.pop("scale"), a.pop("vdim")
    cfg["layers"][0]["mixer"]["mask"]["pool"] = None
    cfg["layers"][0]["mlp"]["shared"] = None
    cfg["layers"][2]["mlp"].pop("shared")
    cfg["layers"][1].pop("mlp")
    cfg["layers"][1]["weights_of"] = None
    cfg.pop("residual_mult")
    st, _, msg = dims({"hf_config": cfg})
    assert st == kf.KF_OK, msg


@pytest.mark.parametrize("edit, words", [
    (lambda c: c["layers"][0].update(type="mingru"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads must divide heads"),
    (lambda c: c["layers"][0]["mixer"].update(dim=600), "<= 512"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "mask.size is missing"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size must be positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(pool=-1), "pool not negative"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "is not built"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top <= experts"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff is missing"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff is missing"),
    (lambda c: c["layers"][2].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][2].update(weights_of=2), "weights_of"),
    (lambda c: c["layers"][2].update(weights_of=-2), "weights_of"),
    (lambda c: c["layers"][0].update(weights_of=2), "weights_of"),  # a circle
    (lambda c: c["layers"][2].update(weights_of=1), "other sizes"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=11), "other sizes"),
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


def test_window_and_blocks_by_hand():
    assert ref.visible(4, 5, 3) == ([], [0, 1, 2, 3, 4])
    assert ref.visible(6, 5, 3) == ([], [2, 3, 4, 5, 6])         # positions 0 and 1 have left, their block has not: nobody sees them
    assert ref.visible(7, 5, 3) == ([0], [3, 4, 5, 6, 7])        # block 0 = positions 0 .. 2, 2 <= 7 - 5
    assert ref.visible(9, 5, 3) == ([0], [5, 6, 7, 8, 9])
    assert ref.visible(10, 5, 3) == ([0, 1], [6, 7, 8, 9, 10])
    assert ref.visible(3, 1, 1) == ([0, 1, 2], [3])              # window 1, blocks of one position: everything, as plain attention
    assert ref.visible(5, 2, 4) == ([0], [4, 5]) and ref.visible(4, 2, 4) == ([], [3, 4])   # blocks longer than the window
    assert ref.visible(3, 0, 0) == ([], [0, 1, 2, 3]) and ref.visible(9, 3, 0) == ([], [7, 8, 9])


def test_blocks_of_one_equal_plain_attention():
    m = attn(heads=2, kv_heads=1, dim=4, vdim=3, window=1, pool=1)
    W = weights(config([layer(m)], width=6), seed=4)
    h = torch.randn(9, 6, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    plain = {k: v for k, v in m.items() if k != "mask"}
    assert torch.allclose(ref.attention(h, m, W, "l0.mix.", 1e-5), ref.attention(h, plain, W, "l0.mix.", 1e-5), atol=1e-12)


def test_equal_scores_average_what_is_visible():
    """zero queries: every visible token and block weighs the same; the gate's logit is zero: one half of that"""
    m = attn(heads=1, kv_heads=1, dim=4, vdim=4, window=3, pool=2)
    E, T = 4, 11
    g = torch.Generator().manual_seed(3)
    W = {"q": torch.zeros(4, E), "k": torch.randn(4, E, generator=g), "v": torch.eye(4), "q.norm": torch.ones(4), "k.norm": torch.ones(4), "g": torch.zeros(1, E), "o": torch.eye(4)}
    h = torch.randn(T, E, dtype=torch.float64, generator=g)
    out = ref.attention(h, m, W, "", 1e-5)
    for i in range(T):
        blocks, toks = ref.visible(i, 3, 2)
        parts = [h[2 * b:2 * b + 2].mean(0) for b in blocks] + [h[j] for j in toks]
        assert torch.allclose(out[i], 0.5 * torch.stack(parts).mean(0), atol=1e-12)


def test_shift_by_hand():
    h = torch.tensor([[1.0, 2.0], [3.0, -1.0], [0.0, 4.0]], dtype=torch.float64)
    z = ref.token_shift(h, torch.tensor([0.25, 1.0]))
    assert torch.allclose(z, torch.tensor([[0.75, 0.0], [2.5, 2.0], [0.75, -1.0]], dtype=torch.float64))


def test_experts_follow_the_table():
    cfg = config([layer(attn(), moe(experts=4, top=3, ff=5, shared=0))], width=8, vocab=12)
    W = weights(cfg, seed=6)
    x = torch.randn(1, 8, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    out = ref.experts(x, [7], cfg["layers"][0]["mlp"], W, "l0.mlp.")
    want = sum(ref.gated(W, "l0.mlp.e%d." % e, x) for e in W["l0.mlp.table"][7].tolist()) / 3
    assert torch.allclose(out, want, atol=1e-12) and len(set(W["l0.mlp.table"][7].tolist())) == 3


def test_shared_layers_use_their_owner():
    cfg = config([layer(), layer(attn(window=5), None, weights_of=0), layer(attn(), None, weights_of=1)], width=12)
    assert [ref.owner(cfg, i) for i in range(3)] == [0, 0, 0]
    assert set(k.split(".")[0] for k in weights(cfg)) == {"embed", "head", "final", "l0"}
