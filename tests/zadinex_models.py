"""Small random Zadinex models for the tests: layer entries, a config.json, weights drawn on the bf16 grid (optionally shaped so that a fault
shows), bf16 bit patterns, random token lists."""
import numpy as np
import torch


def wkv(heads=3, dim=10, rank=6):
    return "wkv", {"heads": heads, "dim": dim, "w_rank": rank}


def attn(heads=4, kv_heads=2, dim=12, vdim=10, rot_dims=8, base=10000.0, scale=None, v_mix=True):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, v_mix=v_mix)
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return "attention", m


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, identity=3, top=3, ff=12, groups=(3, 2), limit=0.8):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    x = {"ff": ff}
    if limit:
        x["limit"] = limit
    return {"kind": "moe", "expert": x, "router": r}


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(layers, width=48, vocab=96, eps=1e-5):
    return {"architecture": "Zadinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}


def bf16_grid(t):
    return t.to(torch.bfloat16).to(torch.float32)


def weights(cfg, seed=0, decay=-1.0, bonus=0.5, sink=1.0, lam=0.5, correction=0.1):
    """decay: mean of w0, the logarithm of the decay's rate (-6: the first tokens still matter hundreds of steps later; 2: almost nothing is
    kept); bonus, sink: means of u and of the sinks; lam: mean share of the first layer's values; correction: spread of the choice's shift"""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, r, c, s=None):
        W[name] = bf16_grid(torch.randn(r, c, generator=g) * (s if s is not None else c ** -0.5))

    def vec(name, n, mean=0.0, s=0.3):
        W[name] = bf16_grid(mean + s * torch.randn(n, generator=g))

    def one(name, mean, s):  # a single number, shape []
        W[name] = bf16_grid(mean + s * torch.randn(1, generator=g))[0]

    def norm(name):
        vec(name, E, 1.0, 0.3), vec(name + ".b", E, 0.0, 0.2), one(name + ".alpha", 0.7, 0.1)

    mat("embed", V, E, 1.0)
    mat("head", V, E)
    norm("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        p, m, q = "l%d." % i, ly["mixer"], "l%d.mix." % i
        norm(p + "norm1")
        vec(p + "ls1", E, 0.8, 0.3)
        if ly["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                vec(q + "mu." + s, E, 0.5, 0.4)
                mat(q + s, n, E) if s != "w" else mat(q + "w1", m["w_rank"], E)
            mat(q + "w2", n, m["w_rank"]), vec(q + "w0", n, decay, 0.5)
            W[q + "u"] = bf16_grid(bonus + 0.5 * torch.randn(m["heads"], m["dim"], generator=g))
            vec(q + "norm", n, 1.0, 0.3), mat(q + "o", E, n)
        else:
            H, G, dk = m["heads"], m.get("kv_heads") or m["heads"], m["dim"]
            dv = m.get("vdim") or dk
            mat(q + "q", H * dk, E), mat(q + "k", G * dk, E), mat(q + "v", G * dv, E)
            if m.get("v_mix"):
                one(q + "vmix", lam, 0.2)
            vec(q + "sink", H, sink, 0.5), mat(q + "o", E, H * dv)
        f = ly.get("mlp")
        if not f:
            continue
        norm(p + "norm2")
        vec(p + "ls2", E, 0.8, 0.3)
        if f["kind"] == "dense":
            mat(p + "mlp.gate", f["ff"], E, 2.0 * E ** -0.5), mat(p + "mlp.up", f["ff"], E), mat(p + "mlp.down", E, f["ff"])
            continue
        X, F = f["router"]["experts"], f["expert"]["ff"]
        outs = X + f["router"].get("identity", 0)
        mat(p + "mlp.router", outs, E, 2.0 * E ** -0.5), vec(p + "mlp.correction", outs, 0.0, correction)
        for e in range(X):
            mat("%smlp.e%d.gate" % (p, e), F, E, 2.0 * E ** -0.5), mat("%smlp.e%d.up" % (p, e), F, E, 2.0 * E ** -0.5), mat("%smlp.e%d.down" % (p, e), E, F)
    return W


def bits(t):
    return (t.contiguous().view(torch.int32).numpy().astype(np.uint32) >> 16).astype(np.uint16)


def st_entries(W):
    """(name, dtype, array) of every tensor as a checkpoint stores it"""
    return [(k, "BF16", bits(v).reshape(tuple(v.shape))) for k, v in W.items()]


def set_all(model, W):
    for k, v in W.items():
        model.set_tensor(k, bits(v).reshape(-1, v.shape[-1]) if v.dim() > 1 else bits(v).reshape(-1))


def tokens(n, vocab, seed):
    return np.random.RandomState(seed).randint(0, vocab, n).tolist()
