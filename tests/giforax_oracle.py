"""Plain, slow implementation of the Giforax design in double precision, one function per mechanism. Shares no code with
the package: the tests compare the framework with it. Also makes small configurations and random weights for it."""
import json
import math
import os

import torch


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def under(w, name):
    return {k[len(name) + 1:]: v for k, v in w.items() if k.startswith(name + ".")}


# ---- attention --------------------------------------------------------------------------------------------------------
def rotate(x, rot, positions=None):
    """x [T, heads, D]: of the first ``dims`` dimensions, i and i + dims / 2 turn together."""
    dims, out = rot["dims"], x.clone()
    p = torch.arange(x.shape[0], dtype=x.dtype) if positions is None else torch.as_tensor(positions, dtype=x.dtype)
    for i in range(dims // 2):
        a = p * rot["base"] ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i], out[..., i + dims // 2] = u * c - v * s, v * c + u * s
    return out


def visible(i, j, chunk):
    return j <= i and i // chunk == j // chunk


def sigmoid_attention(q, k, v, scale, key_bias, chunk):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: every visible key counts with the sigmoid of its score."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    mask = torch.tensor([[visible(i, j, chunk) for j in range(T)] for i in range(T)], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = (sigmoid(q[:, h] @ k[:, g].T * scale + key_bias[h]) * mask) @ v[:, g]
    return out


def keys_and_values(h, w, m, eps):
    T, G = h.shape[0], m["kv_heads"]
    return unit(rotate((h @ w["k"].T).view(T, G, -1), m["rot"]), eps), (h @ w["v"].T).view(T, G, -1)


def attention(h, w, m, eps, kv):
    q = unit(rotate((h @ w["q"].T).view(h.shape[0], m["heads"], -1), m["rot"]), eps)
    a = sigmoid_attention(q, *kv, m["scale"], w["pb"], m["mask"]["size"])
    a = a * sigmoid(h @ w["g"].T)[:, :, None]
    return a.flatten(1) @ w["o"].T


# ---- recurrence -------------------------------------------------------------------------------------------------------
def min_gru(h, w, state=None):
    """(outputs [T, W], the state behind the last token)"""
    z, u = sigmoid(h @ w["z"].T + w["z.b"]), h @ w["x"].T + w["x.b"]
    s = torch.zeros_like(u[0]) if state is None else state
    candidate = torch.where(u >= 0, u + 0.5, sigmoid(u))
    gate = h @ w["g"].T
    rows = []
    for t in range(h.shape[0]):
        s = (1 - z[t]) * s + z[t] * candidate[t]
        rows.append(s * gate[t] * sigmoid(gate[t]))
    return torch.stack(rows) @ w["o"].T, s


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def expert(h, w, limit):
    g = torch.minimum(h @ w["gate"].T, torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def route(h, w_router, top):
    """[(expert, weight), ...] of one token."""
    s = sigmoid(w_router @ h).tolist()
    return [(e, s[e]) for e in sorted(range(len(s)), key=lambda e: -s[e])[:top]]


def mixture(h, w, mlp):
    experts = [under(w, f"e{i}") for i in range(mlp["router"]["experts"])]
    out = torch.stack([sum(expert(p * x, experts[e], mlp["expert"]["limit"])
                           for e, p in route(x, w["router"], mlp["router"]["top"])) for x in h])
    if mlp.get("shared"):
        out = out + expert(h, under(w, "shared"), mlp["shared"]["limit"])
    return out


# ---- model ------------------------------------------------------------------------------------------------------------
def depth_average(weights, rows):
    return sum(weights[j] * rows[j] for j in range(len(rows)))


def logits(cfg, weights, tokens, stream=None):
    """Logits of every position [T, vocab]; ``stream`` (a list) collects the residual stream behind every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda x, w, name: layer_norm(x, w[name], w[name + ".b"], eps)
    x = W["embed"][torch.as_tensor(list(tokens))] * cfg["embedding"]["scale"]
    kept, results = {}, [x]
    for i, layer in enumerate(cfg["layers"]):
        w, m = under(W, f"l{i}"), layer["mixer"]
        mix, h = under(w, "mix"), norm(x, w, "norm1")
        if layer["type"] == "mingru":
            y, _ = min_gru(h, mix)
        else:
            kept[i] = kept[m["kv_from"]] if "kv_from" in m else keys_and_values(h, mix, m, eps)
            y = attention(h, mix, m, eps, kept[i])
        x = x + norm(y, w, "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(mixture(norm(x, w, "norm2"), under(w, "mlp"), layer["mlp"]), w, "norm2b")
        results.append(x)
        x = depth_average(w["dwa"], results)
        if stream is not None:
            stream.append(x)
    return norm(x, W, "final.norm") @ W["head"].T


def greedy(cfg, weights, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(logits(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ---- small models -----------------------------------------------------------------------------------------------------
def moe(experts, top, ff, limit=1.1, shared=None):
    """shared: (ff, limit)"""
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit),
                shared=dict(zip(("ff", "limit"), shared)) if shared else None)


def attn_layer(heads, kv_heads, dim, vdim, dims, chunk, mlp, base=400.0, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=chunk), rot=dict(base=base, dims=dims),
             scale=scale if scale is not None else 2.0 * dim ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gru_layer(width, mlp):
    return {"type": "mingru", "mixer": dict(width=width), "mlp": mlp}


def model(layers, vocab=97, width=40, eps=1e-5, scale=0.7):
    return {"architecture": "Giforax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


CONFIGS = {
    # sizes on 16-byte boundaries, every mechanism; two layers read the keys of a layer before them, under other chunks
    "aligned": model([gru_layer(64, moe(6, 2, 24, shared=(40, 0.8))),
                      attn_layer(4, 2, 24, 40, 16, 37, moe(8, 3, 24, shared=(32, 1.5))),
                      attn_layer(4, 2, 24, 40, 16, 150, None, kv_from=1, scale=0.6),
                      gru_layer(48, None),
                      attn_layer(4, 2, 24, 40, 16, 16, moe(5, 1, 16), kv_from=1)], width=48, vocab=120),
    # nothing is a multiple of eight, layers differ in every size, experts without a shared one
    "odd": model([attn_layer(3, 1, 11, 13, 6, 20, moe(5, 2, 11, limit=0.7), scale=0.4),
                  gru_layer(29, moe(3, 3, 13, limit=0.4, shared=(7, 2.5))),
                  attn_layer(6, 2, 7, 5, 4, 3, None, base=30.0),
                  attn_layer(6, 2, 7, 5, 4, 90, moe(7, 1, 9, shared=(21, 0.3)), base=30.0, kv_from=2),
                  gru_layer(51, moe(4, 2, 10))], width=45, vocab=101, eps=1e-3, scale=1.0),
    # attention only; many query heads per key head, chunks at and beyond the tiles' size
    "attention": model([attn_layer(20, 1, 64, 128, 32, 128, moe(9, 2, 16)),
                        attn_layer(4, 4, 128, 64, 128, 129, moe(35, 7, 16)),
                        attn_layer(20, 1, 64, 128, 32, 400, None, kv_from=0)], width=64, scale=1.7),
    # recurrences only
    "recurrent": model([gru_layer(136, moe(16, 4, 32, shared=(16, 1.0))), gru_layer(40, None), gru_layer(7, moe(2, 1, 24))],
                       width=56, scale=0.3),
    # heads beyond what the tensor-core kernels take
    "wide": model([attn_layer(2, 1, 136, 200, 50, 70, moe(4, 2, 24)),
                   attn_layer(2, 1, 136, 200, 50, 33, moe(9, 4, 8, shared=(12, 0.9)), kv_from=0)], width=32),
}


def tensor_shapes(cfg):
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"])}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        if layer["type"] == "mingru":
            I = m["width"]
            mix = {"z": (I, W), "z.b": (I,), "x": (I, W), "x.b": (I,), "g": (I, W), "o": (W, I)}
        else:
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mix = {"q": (H * D, W), "pb": (H,), "g": (H, W), "o": (W, H * V)}
            if "kv_from" not in m:
                mix.update(k=(G * D, W), v=(G * V, W))
        out.update({f"l{i}.mix.{k}": v for k, v in mix.items()})
        gated = lambda pre, ff: {pre + "gate": (ff, W), pre + "up": (ff, W), pre + "down": (W, ff)}
        if mlp is not None:
            ff = {"router": (mlp["router"]["experts"], W)}
            for e in range(mlp["router"]["experts"]):
                ff.update(gated(f"e{e}.", mlp["expert"]["ff"]))
            if mlp.get("shared"):
                ff.update(gated("shared.", mlp["shared"]["ff"]))
            out.update({f"l{i}.mlp.{k}": v for k, v in ff.items()})
        for norm in ("norm1", "norm1b") + (() if mlp is None else ("norm2", "norm2b")):
            out.update({f"l{i}.{norm}": (W,), f"l{i}.{norm}.b": (W,)})
        out[f"l{i}.dwa"] = (i + 2,)
    out.update({"final.norm": (W,), "final.norm.b": (W,)})
    return out


def random_weights(cfg, seed=0, decided=False):
    """bf16 weights under which faults show: a key bias that makes most weights small, so that single keys stand out, update
    gates between short and long memories, depth averages in which every layer's result counts, no unit or zero constant.
    ``decided``: the constant part of a router's input ranks the experts, what depends on the token changes the weights and
    hardly the ranks: no choice hangs on the rounding of that input (which may be bf16)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g)
        leaf = name.split(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            t = 1 + 0.3 * r
        elif leaf in ("norm1.b", "norm2.b", "norm1b.b", "norm2b.b") or name == "final.norm.b":
            t = 0.3 * r
        elif leaf == "dwa":
            t = 0.3 * r + torch.tensor([0.2] * (shape[0] - 1) + [0.8])
        elif leaf == "mix.pb":
            t = -2.0 + 0.7 * r
        elif leaf == "mix.z.b":
            t = -2.0 + 1.5 * r
        elif leaf == "mix.x.b":
            t = 0.5 * r
        elif name == "embed":
            t = r
        else:
            t = r * shape[-1] ** -0.5
            if leaf == "mlp.router":
                t = 2 * t
            elif leaf in ("mix.z", "mix.x"):
                t = 1.5 * t
        out[name] = t.to(torch.bfloat16)
    for i, layer in enumerate(cfg["layers"] if decided else ()):
        if layer["mlp"] is not None:
            out[f"l{i}.norm2.b"] *= 5
            r, b = (out[f"l{i}.{k}"].float() for k in ("mlp.router", "norm2.b"))
            rank, along = torch.randperm(r.shape[0], generator=g).float(), b / (b @ b)
            r = 0.02 * (r - torch.outer(r @ b, along)) + torch.outer(0.8 - 0.6 * rank, along)
            out[f"l{i}.mlp.router"] = r.to(torch.bfloat16)
    return out


def save(cfg, weights, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)
