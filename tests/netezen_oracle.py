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


def rotate(x, rot, positions=None):
    """x [T, heads, D]: dimensions 2i and 2i + 1 of the first ``dims`` turn together, by position times frequency i."""
    f, amp = frequencies(rot)
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=x.dtype) if positions is None else torch.as_tensor(positions, dtype=x.dtype)
    for i, fi in enumerate(f):
        c, s = (torch.cos(p * fi) * amp)[:, None], (torch.sin(p * fi) * amp)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
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
    experts, shared = [under(w, f"e{i}") for i in range(mlp["router"]["experts"])], under(w, "shared")
    out = []
    for x in h:
        y = sum(p * clamped_ff(x, experts[i], mlp["expert"]["limit"]) for i, p in route(x, w, mlp["router"]["top"]))
        if shared:
            y = y + sigmoid(shared["sg"] @ x) * clamped_ff(x, shared, mlp["shared"]["limit"])
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


# ---- small models -----------------------------------------------------------------------------------------------------
def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, limit=1.3, shared=None):
    """shared: (ff, limit)"""
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit),
                shared=dict(zip(("ff", "limit"), shared)) if shared else None)


def attn_layer(heads, kv_heads, dim, vdim, dims, window, keep, mlp, base=500.0, scaling=None, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window, keep_first=keep),
                          scale=scale if scale is not None else dim ** -0.5,
                          rot=dict(base=base, dims=dims, **({"scaling": scaling} if scaling else {})))}


def latent_layer(heads, dim, rot, vdim, kv_rank, q_rank, window, mlp, base=300.0, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                          mask=dict(size=window), scale=scale if scale is not None else (dim + rot) ** -0.5,
                          rot=dict(base=base, dims=rot))}


def model(layers, vocab=97, width=40, eps=1e-5, streams=2, mult=0.6):
    return {"architecture": "Netezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "streams": streams, "residual_mult": mult}


CONFIGS = {
    # sizes on 16-byte boundaries, every mechanism
    "aligned": model([attn_layer(4, 2, 24, 40, 16, 37, 5, moe(8, 2, 24, shared=(40, 0.7)),
                                 scaling=dict(factor=4.0, original=64, fast=8.0, slow=0.5)),
                      latent_layer(3, 24, 16, 16, 40, 32, 50, dense(72)),
                      attn_layer(6, 3, 40, 24, 40, 150, 3, None)], width=48, vocab=120, streams=4),
    # nothing is a multiple of eight, layers differ in every size, experts without a shared one
    "odd": model([latent_layer(5, 11, 6, 9, 13, 7, 9, moe(5, 3, 11, shared=(7, 2.5))),
                  attn_layer(3, 1, 10, 13, 6, 20, 1, dense(37), scale=0.4),
                  latent_layer(2, 21, 10, 6, 30, 27, 33, None),
                  attn_layer(6, 2, 7, 5, 4, 3, 70, moe(3, 3, 9, limit=0.4), base=30.0,
                             scaling=dict(factor=3.0, original=500, fast=32.0, slow=1.0))],
                 width=45, vocab=101, eps=1e-3, streams=3, mult=1.0),
    # one kind of layer only; many query heads per key head, windows at and beyond the tiles' size, one stream
    "attention": model([attn_layer(20, 1, 64, 128, 32, 129, 130, dense(40)),
                        attn_layer(4, 4, 128, 64, 128, 128, 0, moe(35, 7, 16))], width=64, streams=1, mult=0.8),
    "latent": model([latent_layer(20, 64, 64, 128, 136, 48, 128, dense(64)),
                     latent_layer(3, 128, 32, 64, 64, 40, 200, moe(16, 1, 32, shared=(16, 1.0))),
                     latent_layer(2, 16, 8, 8, 24, 16, 1, None)], width=56, streams=5, mult=0.45),
    # heads and latents beyond what the tensor-core kernels take
    "wide": model([attn_layer(2, 1, 136, 200, 50, 70, 6, dense(24)),
                   latent_layer(2, 24, 16, 136, 632, 24, 90, moe(9, 4, 8, shared=(12, 0.9)))], width=32, streams=2),
}


def tensor_shapes(cfg):
    W, S, out = cfg["width"], cfg["streams"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            mix = {"q": (H * D, W), "k": (m["kv_heads"] * D, W), "v": (m["kv_heads"] * V, W), "o": (W, H * V)}
        else:
            R, C, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            mix = {"dq": (Q, W), "dq.norm": (Q,), "uq": (H * (D + R), Q), "dkv": (C + R, W), "dkv.norm": (C,),
                   "uk": (H * D, C), "uv": (H * V, C), "sink": (H,), "o": (W, H * V)}
        out.update({f"l{i}.mix.{k}": v for k, v in mix.items()})
        gated = lambda pre, ff: {pre + "gate": (ff, W), pre + "up": (ff, W), pre + "down": (W, ff)}
        ff = {}
        if mlp is not None and mlp["kind"] == "dense":
            ff = {"up": (mlp["ff"], W), "down": (W, mlp["ff"])}
        elif mlp is not None:
            E = mlp["router"]["experts"]
            ff = {"router": (E, W), "correction": (E,)}
            for e in range(E):
                ff.update(gated(f"e{e}.", mlp["expert"]["ff"]))
            if mlp["shared"]:
                ff.update({**gated("shared.", mlp["shared"]["ff"]), "shared.sg": (1, W)})
        out.update({f"l{i}.mlp.{k}": v for k, v in ff.items()})
        for q in (1, 2)[:1 if mlp is None else 2]:
            out.update({f"l{i}.norm{q}": (W,), f"l{i}.hc{q}.in": (S,), f"l{i}.hc{q}.out": (S,), f"l{i}.hc{q}.mix": (S, S)})
    out["final.norm"] = (W,)
    return out


def random_weights(cfg, seed=0, decided=False):
    """bf16 weights under which faults show: queries large enough that single keys dominate a softmax (a key lost or let in
    changes the output), sinks of the scores' size, a correction that changes the choice of experts, mixing matrices that
    are neither symmetric nor near one, no unit or zero constant. ``decided``: corrections so far apart that hardly a choice
    hangs on the rounding of the router's input (which may be bf16)."""
    g = torch.Generator().manual_seed(seed)
    S, out = cfg["streams"], {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g)
        if name.endswith((".norm1", ".norm2", "final.norm")):
            t = 0.3 * r
        elif name.endswith("norm"):
            t = 1 + 0.3 * r
        elif name.endswith(".sink"):
            t = 1 + r
        elif name.endswith(".correction"):
            t = 0.4 * torch.rand(*shape, generator=g)
            if decided:
                t = torch.argsort(t) * (1.0 / shape[0])
        elif name.endswith(".mix") and ".hc" in name:
            t = 0.7 * torch.eye(S) + 0.3 * r
        elif ".hc" in name:
            t = 0.6 + 0.4 * r
        elif name == "embed":
            t = r
        else:
            t = r * shape[-1] ** -0.5
            if name.endswith((".mix.q", ".mix.uq")):
                t = 2.5 * t
            elif name.endswith(".router") and decided:
                t = 0.25 * t
        out[name] = t.to(torch.bfloat16)
    return out


def save(cfg, weights, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)
