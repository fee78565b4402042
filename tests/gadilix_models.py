"""Small random Gadilix models for the tests: layer entries, a config.json, weights drawn on the bf16 grid (optionally shaped so that a fault
shows), bf16 bit patterns, random token lists."""
import numpy as np
import torch


def attn(heads=4, kv_heads=2, dim=12, vdim=10, window=9, pool=4, scale=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5)
    if window:
        m["mask"] = {"size": window}
        if pool:
            m["mask"]["pool"] = pool
    return m


def moe(experts=6, top=2, ff=12, shared=20):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def layer(mixer=None, mlp=None, weights_of=None):
    ly = {"type": "attention", "mixer": mixer or attn(), "mlp": mlp}
    if weights_of is not None:
        ly["weights_of"] = weights_of
    return ly


def config(layers, width=48, vocab=96, eps=1e-5, mult=0.6):
    return {"architecture": "Gadilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": list(layers)}


def bf16_grid(t):
    return t.to(torch.bfloat16).to(torch.float32)


def weights(cfg, seed=0, q_gain=1.0, g_bias=0.0):
    """q_gain scales the norm weights of the queries (a peaked softmax); g_bias is added to one column of the gate's weight"""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, r, c, s=None):
        W[name] = bf16_grid(torch.randn(r, c, generator=g) * (s if s is not None else c ** -0.5))

    def vec(name, n, mean=0.0, s=0.3):
        W[name] = bf16_grid(mean + s * torch.randn(n, generator=g))

    def one(name, mean=1.0, s=0.3):  # a single number, shape []
        W[name] = bf16_grid(mean + s * torch.randn(1, generator=g))[0]

    mat("embed", V, E, 1.0)
    one("embed.norm")
    mat("head", V, E)
    one("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        if ly.get("weights_of") is not None:
            continue
        p, m, q = "l%d." % i, ly["mixer"], "l%d.mix." % i
        H, G, dk = m["heads"], m.get("kv_heads") or m["heads"], m["dim"]
        dv = m.get("vdim") or dk
        one(p + "norm1")
        vec(p + "shift", E, 0.4, 0.4)
        mat(q + "q", H * dk, E), mat(q + "k", G * dk, E), mat(q + "v", G * dv, E)
        vec(q + "q.norm", dk, q_gain, 0.3 * q_gain), vec(q + "k.norm", dk, 1.0, 0.3)
        mat(q + "g", H, E, 2.0 * E ** -0.5)
        if g_bias:
            W[q + "g"][:, 0] = bf16_grid(W[q + "g"][:, 0] + g_bias)
        mat(q + "o", E, H * dv)
        f = ly.get("mlp")
        if not f:
            continue
        one(p + "norm2")
        X, F, top = f["router"]["experts"], f["expert"]["ff"], f["router"]["top"]
        W[p + "mlp.table"] = torch.stack([torch.randperm(X, generator=g)[:top] for _ in range(V)]).to(torch.int32)
        for e in ["e%d" % k for k in range(X)] + (["shared"] if f.get("shared") else []):
            n = f["shared"]["ff"] if e == "shared" else F
            mat("%smlp.%s.gate" % (p, e), n, E), mat("%smlp.%s.up" % (p, e), n, E), mat("%smlp.%s.down" % (p, e), E, n)
    return W


def bits(t):
    return (t.contiguous().view(torch.int32).numpy().astype(np.uint32) >> 16).astype(np.uint16)


def st_entries(W):
    """(name, dtype, array) of every tensor as a checkpoint stores it"""
    return [(k, "I32", v.numpy()) if v.dtype == torch.int32 else (k, "BF16", bits(v).reshape(tuple(v.shape))) for k, v in W.items()]


def set_all(model, W):
    for k, v in W.items():
        if v.dtype == torch.int32:
            model.set_tensor(k, v.numpy())
        else:
            model.set_tensor(k, bits(v).reshape(-1, v.shape[-1]) if v.dim() > 1 else bits(v).reshape(-1))


def tokens(n, vocab, seed):
    return np.random.RandomState(seed).randint(0, vocab, n).tolist()
