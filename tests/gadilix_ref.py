"""Plain float64 restatement of the Gadilix stack, one function per mechanism, token-by-token loops where a mechanism has a mask or looks
back.  It shares no code with the library: it is what the GPU tests compare the framework against.

    x_0 = norm(embed[token]; g_embed);   norm(y; g) = y / sqrt(mean(y^2) + eps) * g  with ONE number g for the whole row
    layer:  h = x,  z_t = h_t + s * (h_{t-1} - h_t)  element by element (h_{-1} = 0);
            x <- x + m * norm(attention(z); g_1);   x <- x + m * norm(ff(x); g_2)      (the feed-forward reads x, not shifted)
    attention:  q, k, v = W_q z, W_k z, W_v z; q and k of every head RMS-normed over the head (weights shared by the heads);
                position i sees the tokens j with 0 <= i - j < S, and for every block b of P positions with bP + P - 1 <= i - S one
                key and one value: the means of the block's keys and values; one softmax over all of them with scores scale * q.k;
                head h's result times sigmoid((W_g z)_h); W_o on the heads side by side
    ff:         the experts of a token stand in a table row of the token's id, each with weight 1 / top; expert and shared expert are
                W_d (silu(W_g x) * (W_u x)); the shared one runs for every token and is added
    logits = W_head norm(x; g_final)
A layer that names another one in `weights_of` runs on that layer's tensors.
"""
import torch

D = torch.float64


def rmsnorm(y, g, eps):
    """g: one number, or a weight per entry"""
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * g.to(D)


def silu(z):
    return z * torch.sigmoid(z)


def lin(W, name, h):
    return h @ W[name].to(D).T


def owner(cfg, i):
    """the layer whose tensors layer i runs on"""
    seen = set()
    while cfg["layers"][i].get("weights_of") is not None:
        assert i not in seen
        seen.add(i)
        i = cfg["layers"][i]["weights_of"]
    return i


def token_shift(h, s):
    """h [T, E]: each token moves by the share s (per entry) towards the token before it; the first one towards zero"""
    out = torch.empty_like(h)
    for t in range(h.shape[0]):
        prev = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out[t] = h[t] + (prev - h[t]) * s.to(D)
    return out


def visible(i, size, pool):
    """(blocks, tokens) that position i sees; size 0: every earlier token; pool 0: no blocks"""
    if not size:
        return [], list(range(i + 1))
    toks = [j for j in range(i + 1) if i - j < size]
    blocks = [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size] if pool else []
    return blocks, toks


def attention(z, m, W, p, eps):
    """z [T, E] (shifted input) -> [T, E]"""
    T = z.shape[0]
    H, G = m["heads"], m.get("kv_heads") or m["heads"]
    dk, dv = m["dim"], m.get("vdim") or m["dim"]
    mask = m.get("mask") or {}
    S, P = mask.get("size", 0), mask.get("pool", 0)
    scale = m["scale"] if m.get("scale") is not None else dk ** -0.5
    q = rmsnorm(lin(W, p + "q", z).view(T, H, dk), W[p + "q.norm"], eps)
    k = rmsnorm(lin(W, p + "k", z).view(T, G, dk), W[p + "k.norm"], eps)
    v = lin(W, p + "v", z).view(T, G, dv)
    gate = torch.sigmoid(lin(W, p + "g", z))  # [T, H]
    kv_of = [h // (H // G) for h in range(H)]  # the kv head of every query head
    means = [(k[b * P:(b + 1) * P].mean(0), v[b * P:(b + 1) * P].mean(0)) for b in range(T // P)] if P else []
    out = torch.zeros(T, H, dv, dtype=D)
    for i in range(T):
        blocks, toks = visible(i, S, P)
        keys = torch.stack([means[b][0] for b in blocks] + [k[j] for j in toks])[:, kv_of]  # [n, H, dk]
        vals = torch.stack([means[b][1] for b in blocks] + [v[j] for j in toks])[:, kv_of]
        w = torch.softmax((keys * q[i]).sum(-1) * scale, 0)  # [n, H]
        out[i] = gate[i][:, None] * (w[:, :, None] * vals).sum(0)
    return lin(W, p + "o", out.reshape(T, H * dv))


def gated(W, p, x):
    return lin(W, p + "down", silu(lin(W, p + "gate", x)) * lin(W, p + "up", x))


def experts(x, toks, f, W, p):
    """x [T, E], toks the token ids"""
    top = f["router"]["top"]
    out = torch.zeros_like(x)
    for t, tok in enumerate(toks):
        for e in W[p + "table"][tok].tolist():
            out[t] += gated(W, "%se%d." % (p, e), x[t:t + 1])[0] / top
    if f.get("shared"):
        out = out + gated(W, p + "shared.", x)
    return out


def forward(cfg, W, toks, layers=None):
    """logits [T, vocab]; `layers` (a list) receives the stream after every layer"""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = rmsnorm(W["embed"].to(D)[toks], W["embed.norm"], eps)
    for i, ly in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        x = x + m * rmsnorm(attention(token_shift(x, W[p + "shift"]), ly["mixer"], W, p + "mix.", eps), W[p + "norm1"], eps)
        if ly.get("mlp"):
            x = x + m * rmsnorm(experts(x, toks, ly["mlp"], W, p + "mlp."), W[p + "norm2"], eps)
        if layers is not None:
            layers.append(x)
    return lin(W, "head", rmsnorm(x, W["final.norm"], eps))
