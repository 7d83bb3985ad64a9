"""Plain, slow implementation of the Netezen design in double precision, one function per mechanism. Shares no code with
the package: the tests compare the framework with it. Also makes small configurations and random weights for it."""
import json
import math
import os

import torch


def unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


# ---- rotation ---------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(frequency of every pair, factor on cosine and sine)."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return f, 1.0

    def place(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(place(s["fast"])), 0)
    hi = min(math.ceil(place(s["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot):
    """x [T, heads, D]: dimensions 2i and 2i + 1 of the first ``dims`` turn together, by position times frequency i."""
    f, amp = frequencies(rot)
    out = x.clone()
    for p in range(x.shape[0]):
        for i, fi in enumerate(f):
            c, s = math.cos(p * fi) * amp, math.sin(p * fi) * amp
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            out[p, :, 2 * i] = u * c - v * s
            out[p, :, 2 * i + 1] = v * c + u * s
    return out


# ---- attention --------------------------------------------------------------------------------------------------------
def sees(i, j, window, keep_first=0):
    return j <= i and (i - j < window or j < keep_first)


def masked_softmax(q, k, v, scale, window, keep_first=0, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H * V]. ``sink`` [H]: its exponential joins the denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, window, keep_first)]
        for h in range(H):
            g = h // (H // G)
            s = k[js, g] @ q[i, h] * scale
            top = max(float(s.max()), float(sink[h]) if sink is not None else -math.inf)
            e = torch.exp(s - top)
            out[i, h] = e @ v[js, g] / (e.sum() + (math.exp(float(sink[h]) - top) if sink is not None else 0.0))
    return out.reshape(T, -1)


def grouped_attention(h, w, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = rotate((h @ w["q"].T).view(T, H, D), m["rot"]), rotate((h @ w["k"].T).view(T, G, D), m["rot"])
    v = (h @ w["v"].T).view(T, G, V)
    return masked_softmax(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"]) @ w["o"].T


def latent_attention(h, w, m, eps):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = ((unit(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).view(T, H, D + R)
    ckr = h @ w["dkv"].T
    c = unit(ckr[:, :C], eps) * w["dkv.norm"]
    k_rot = rotate(ckr[:, None, C:], m["rot"]).expand(T, H, R)
    q = torch.cat([q[..., :D], rotate(q[..., D:], m["rot"])], -1)
    k = torch.cat([(c @ w["uk"].T).view(T, H, D), k_rot], -1)
    v = (c @ w["uv"].T).view(T, H, V)
    return masked_softmax(q, k, v, m["scale"], m["mask"]["size"], sink=w["sink"]) @ w["o"].T


MIXERS = {"attention": grouped_attention, "latent_attention": latent_attention}


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def squared_relu_ff(h, w):
    z = h @ w["up"].T
    return (torch.where(z > 0, z, torch.zeros_like(z)) ** 2) @ w["down"].T


def clamped_ff(h, w, limit):
    g = torch.minimum(h @ w["gate"].T, torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def route(h, w, top):
    """[(expert, weight), ...] of one token."""
    z = w["router"] @ h
    e = torch.exp(z - z.max())
    s = e / e.sum()
    choice = (s + w["correction"]).tolist()
    chosen = sorted(range(len(choice)), key=lambda i: -choice[i])[:top]
    total = sum(float(s[i]) for i in chosen) + 1e-20
    return [(i, float(s[i]) / total) for i in chosen]


def under(w, name):
    return {k[len(name) + 1:]: v for k, v in w.items() if k.startswith(name + ".")}


def mixture_ff(h, w, mlp):
    out = []
    for t in range(h.shape[0]):
        x = h[t]
        y = sum(p * clamped_ff(x, under(w, f"e{i}"), mlp["expert"]["limit"])
                for i, p in route(x, w, mlp["router"]["top"]))
        if mlp.get("shared"):
            s = under(w, "shared")
            y = y + sigmoid(s["sg"] @ x) * clamped_ff(x, s, mlp["shared"]["limit"])
        out.append(y)
    return torch.stack(out)


def feed_forward(h, w, mlp):
    return squared_relu_ff(h, w) if mlp["kind"] == "dense" else mixture_ff(h, w, mlp)


# ---- model ------------------------------------------------------------------------------------------------------------
def connect(x, hc, sublayer, mult):
    """x [streams, T, W] -> the streams behind a sublayer."""
    S = x.shape[0]
    y = sublayer(sum(hc["in"][s] * x[s] for s in range(S)))
    return torch.stack([sum(hc["mix"][s, t] * x[s] for s in range(S)) + mult * hc["out"][t] * y for t in range(S)])


def logits(cfg, weights, tokens, stream=None):
    """Logits of every position [T, vocab]; ``stream`` (a list) collects the sum of the streams after every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = torch.stack([W["embed"][torch.as_tensor(list(tokens))]] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        w = under(W, f"l{i}")
        x = connect(x, under(w, "hc1"), lambda u: MIXERS[layer["type"]](
            unit(u, eps) * (1 + w["norm1"]), under(w, "mix"), layer["mixer"], eps), mult)
        if layer["mlp"] is not None:
            x = connect(x, under(w, "hc2"), lambda u: feed_forward(
                unit(u, eps) * (1 + w["norm2"]), under(w, "mlp"), layer["mlp"]), mult)
        if stream is not None:
            stream.append(x.sum(0))
    return (unit(x.sum(0), eps) * (1 + W["final.norm"])) @ W["embed"].T


def greedy(cfg, weights, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(logits(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]
