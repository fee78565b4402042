"""Plain float64 restatement of the Zadinex stack, one function per mechanism, a loop over tokens where a mechanism looks back.  It shares no
code with the library: it is what the GPU tests compare the framework against.

    x_0 = embed[token]
    layer:  x <- x + ls1 * mixer(dyt_1(x));   x <- x + ls2 * ff(dyt_2(x)),     dyt(x) = tanh(alpha x) * w + b  entry by entry
    wkv:        m_s = h_t + mu_s * (h_{t-1} - h_t)  for s in r, k, v, g, w  (h_{-1} = 0);  r, k, v = W_s m_s per head;
                decay d = exp(-exp(W_2 tanh(W_1 m_w) + w0)) per key channel;
                o_t = S^T r + (r . (u * k)) v  with the state BEFORE the token;  S <- diag(d) S + k v^T;
                o of a head over its rms, times the norm weight, times silu(W_g m_g);  W_o on the heads side by side
    attention:  q, k rotated by halves, then each head over its own rms (no weight); v blended with the first blending layer's v of the
                same token; softmax over all j <= i with e^{sink_h} added to the denominator; W_o on the heads side by side
    ff dense:   W_d (gelu(W_g h) * (W_u h))
    ff experts: s = softmax(W_r h) over experts and pass-through outputs; choice by s + correction inside the best groups (a group ranks by
                its largest choice value); weights s over the sum of the chosen s; an expert is W_d (g sigmoid(1.702 g) (u + 1)) with
                g = min(W_g h, L), u = clamp(W_u h, -L, L); the last outputs of the router pass h through
    logits = W_head dyt_f(x)
"""
import math

import torch

D = torch.float64


def dyt(x, alpha, w, b):
    return torch.tanh(alpha.to(D) * x) * w.to(D) + b.to(D)


def norm(W, name, x):
    return dyt(x, W[name + ".alpha"], W[name], W[name + ".b"])


def over_rms(y, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def lin(W, name, h):
    return h @ W[name].to(D).T


def token_mix(h, mu):
    """h [T, E]: each token moves by the share mu (per entry) towards the token before it; the first one towards zero"""
    out = torch.empty_like(h)
    for t in range(h.shape[0]):
        prev = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out[t] = h[t] + (prev - h[t]) * mu.to(D)
    return out


def wkv_scan(r, k, v, d, u, state=None):
    """r, k, d [T, H, N], v [T, H, P], u [H, N] -> o [T, H, P]; `state` [H, N, P] is updated in place when given"""
    T, H, N = k.shape
    S = torch.zeros(H, N, v.shape[2], dtype=D) if state is None else state
    o = torch.zeros(T, H, v.shape[2], dtype=D)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h].to(D)[:, None] * kv).T @ r[t, h]
            S[h] = d[t, h][:, None] * S[h] + kv
    return o


def wkv(h, m, W, p, eps):
    T, H, N = h.shape[0], m["heads"], m["dim"]
    mix = {s: token_mix(h, W[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = (lin(W, p + s, mix[s]).view(T, H, N) for s in "rkv")
    z = torch.tanh(mix["w"] @ W[p + "w1"].to(D).T) @ W[p + "w2"].to(D).T + W[p + "w0"].to(D)
    o = over_rms(wkv_scan(r, k, v, torch.exp(-torch.exp(z)).view(T, H, N), W[p + "u"]), eps).reshape(T, H * N)
    return lin(W, p + "o", o * W[p + "norm"].to(D) * silu(lin(W, p + "g", mix["g"])))


def rotate(x, dims, base):
    """x [T, heads, d]: pairs (i, i + dims / 2) turned by t * base^(-2i / dims), t = 0 .. T - 1"""
    y, half = x.clone(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = t * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            y[t, :, i] = x[t, :, i] * c - x[t, :, i + half] * s
            y[t, :, i + half] = x[t, :, i + half] * c + x[t, :, i] * s
    return y


def attention(h, m, W, p, eps, carried):
    """carried: {} at the first layer; the first layer that blends values leaves its own there"""
    T, H = h.shape[0], m["heads"]
    G, dk = m.get("kv_heads") or H, m["dim"]
    dv = m.get("vdim") or dk
    q, k = lin(W, p + "q", h).view(T, H, dk), lin(W, p + "k", h).view(T, G, dk)
    v = lin(W, p + "v", h).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        dims = rot.get("dims") or dk
        q, k = rotate(q, dims, rot["base"]), rotate(k, dims, rot["base"])
    q, k = over_rms(q, eps), over_rms(k, eps)
    if m.get("v_mix"):
        if "v" in carried:
            lam = W[p + "vmix"].to(D)
            v = (1.0 - lam) * v + lam * carried["v"].view(T, G, dv)
        else:
            carried["v"] = v.reshape(T, G * dv)
    scale = m["scale"] if m.get("scale") is not None else dk ** -0.5
    out = torch.zeros(T, H, dv, dtype=D)
    for i in range(T):
        for hd in range(H):
            g = hd // (H // G)
            s = (k[:i + 1, g] @ q[i, hd]) * scale
            sink = W[p + "sink"][hd].to(D)
            top = torch.maximum(s.max(), sink)
            w = torch.exp(s - top)
            out[i, hd] = (w / (w.sum() + torch.exp(sink - top))) @ v[:i + 1, g]
    return lin(W, p + "o", out.reshape(T, H * dv))


def dense_ff(h, W, p):
    return lin(W, p + "down", gelu(lin(W, p + "gate", h)) * lin(W, p + "up", h))


def expert(h, W, p, limit):
    g, u = lin(W, p + "gate", h), lin(W, p + "up", h)
    if limit:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return lin(W, p + "down", g * torch.sigmoid(1.702 * g) * (u + 1.0))


def route(z, correction, top, groups, keep):
    """one token's router logits -> (chosen outputs, their weights)"""
    s = torch.softmax(z, -1)
    choice = (s + correction.to(D)).tolist()
    n, per = len(choice), len(choice) // groups
    ranked = sorted(range(groups), key=lambda g: -max(choice[g * per:(g + 1) * per]))
    open_ = [e for e in range(n) if e // per in ranked[:keep]]
    chosen = sorted(open_, key=lambda e: -choice[e])[:top]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20)


def experts_ff(h, f, W, p):
    r = f["router"]
    E, g = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    z = lin(W, p + "router", h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(*route(z[t], W[p + "correction"], r["top"], g["count"], g["keep"])):
            out[t] += w * (h[t] if e >= E else expert(h[t:t + 1], W, "%se%d." % (p, e), f["expert"].get("limit"))[0])
    return out


def forward(cfg, W, toks, layers=None):
    """logits [T, vocab]; `layers` (a list) receives the stream after every layer"""
    eps = cfg["norm"]["eps"]
    x = W["embed"].to(D)[toks]
    carried = {}
    for i, ly in enumerate(cfg["layers"]):
        p, m = "l%d." % i, ly["mixer"]
        h = norm(W, p + "norm1", x)
        y = wkv(h, m, W, p + "mix.", eps) if ly["type"] == "wkv" else attention(h, m, W, p + "mix.", eps, carried)
        x = x + W[p + "ls1"].to(D) * y
        f = ly.get("mlp")
        if f:
            h = norm(W, p + "norm2", x)
            x = x + W[p + "ls2"].to(D) * (dense_ff(h, W, p + "mlp.") if f["kind"] == "dense" else experts_ff(h, f, W, p + "mlp."))
        if layers is not None:
            layers.append(x)
    return lin(W, "head", norm(W, "final.norm", x))
