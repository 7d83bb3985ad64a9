"""Plain, slow implementation of the Kebopel design in double precision, one function per mechanism. Shares no code with
the package: the tests compare the framework with it. Also makes small configurations and random weights for it."""
import json
import math
import os

import torch


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- embedding ------------------------------------------------------------------------------------------------------
def bigram_row(previous, token, spec):
    """Row of the pair table; ``previous`` None stands for "no token before"."""
    if previous is None:
        return spec["buckets"]
    return (previous * spec["mul_prev"] + token * spec["mul_cur"]) % spec["buckets"]


def embedding(tokens, table, pairs, spec):
    rows = [bigram_row(tokens[t - 1] if t else None, tokens[t], spec) for t in range(len(tokens))]
    return table[torch.as_tensor(tokens)] + pairs[torch.as_tensor(rows)]


# ---- parts of the mixers ----------------------------------------------------------------------------------------------
def short_conv(u, weight):
    """Per channel over time, zeros before the start, last tap = current token, no bias and no activation."""
    taps = weight.shape[1]
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += weight[:, j] * u[t - taps + 1 + j]
    return out


def query_temperature(position, spec):
    return 1 + spec["coef"] * math.log((position + 1) // spec["every"] + 1)


def distance_slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def causal_softmax(q, k, v, scale, bias=False, sink=False):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H * V], query by query and head by head. ``bias``: slope times
    distance is taken off the scores; ``sink``: one more key with score 0 and value 0."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        for i in range(T):
            row = s[i, :i + 1]
            if bias:
                row = row - distance_slope(h, H) * torch.arange(i, -1, -1, dtype=q.dtype)
            top = max(float(row.max()), 0.0)
            e = torch.exp(row - top)
            out[i, h] = e @ v[:i + 1, g] / (e.sum() + (math.exp(-top) if sink else 0.0))
    return out.reshape(T, -1)


def lightning(q, k, v, decay):
    """q, k [T, H, N], v [T, H, V]: S <- decay S + k v^T, o = S^T q, one token after the other."""
    T, H, N = q.shape
    S = torch.zeros(H, N, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out).reshape(T, -1)


# ---- mixers -----------------------------------------------------------------------------------------------------------
def convolved_attention(h, w, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"]) for n in "qkv")
    q = rms_norm(q.view(T, H, D), w["q.norm"], eps)
    k = rms_norm(k.view(T, G, D), w["k.norm"], eps)
    temp = torch.tensor([query_temperature(p, m["q_temp"]) for p in range(T)], dtype=h.dtype)
    return causal_softmax(q * temp[:, None, None], k, v.view(T, G, V), m["scale"]) @ w["o"].T


def biased_attention(h, w, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).view(T, H, D)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).view(T, G, D)
    v = (h @ w["v"].T).view(T, G, V)
    return causal_softmax(q, k, v, m["scale"], bias=True, sink=True) @ w["o"].T


def lightning_attention(h, w, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[n].T).view(T, H, -1) for n in "qkv")
    o = lightning(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms_norm(o, w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


def side_by_side(h, w, m, eps):
    side = lambda s: {k[len(s) + 1:]: v for k, v in w.items() if k.startswith(s + ".")}
    return (m["left_scale"] * biased_attention(h, side("left"), m["left"], eps)
            + m["right_scale"] * lightning_attention(h, side("right"), m["right"], eps))


def feed_forward(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"attention": convolved_attention, "parallel": side_by_side}


# ---- model ------------------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """[(layer, a pass begins here that is not the loop's first)] in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for p in range(loop["times"]):
        out += [(i, p > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def logits(cfg, weights, tokens, stream=None):
    """Logits of every position [T, vocab]; ``stream`` (a list) collects the residual stream after every layer run."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    first = x = embedding(list(tokens), W["embed"], W["bigram"], cfg["embedding"]["bigram"])
    for i, again in layer_runs(cfg):
        part = lambda kind: {k[len(f"l{i}.{kind}."):]: v for k, v in W.items() if k.startswith(f"l{i}.{kind}.")}
        layer = cfg["layers"][i]
        if again:
            x = x + first
        h = rms_norm(x, W[f"l{i}.norm1"], eps)
        y = MIXERS[layer["type"]](h, part("mix"), layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, part("mlp"))
        x = x + y
        if stream is not None:
            stream.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(cfg, weights, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(logits(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ---- small models -----------------------------------------------------------------------------------------------------
def attn_layer(heads, kv_heads, dim, vdim, ff, conv=3, coef=0.4, every=16, scale=None):
    return {"type": "attention",
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv,
                          scale=scale if scale is not None else dim ** -0.5, q_temp=dict(coef=coef, every=every)),
            "mlp": None if ff is None else dict(kind="dense", ff=ff)}


def parallel_layer(left, right, decay, ff, scales=(0.7, 0.55), scale=None):
    """left: (heads, kv_heads, dim, vdim), right: (heads, dim, vdim)"""
    return {"type": "parallel",
            "mixer": dict(left=dict(zip(("heads", "kv_heads", "dim", "vdim"), left),
                                    scale=scale if scale is not None else left[2] ** -0.5),
                          right=dict(zip(("heads", "dim", "vdim"), right), decay=list(decay)),
                          left_scale=scales[0], right_scale=scales[1]),
            "mlp": None if ff is None else dict(kind="dense", ff=ff)}


def model(layers, vocab=97, width=40, eps=1e-5, loop=None, bigram=(61, 13, 5)):
    return {"architecture": "Kebopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "loop": loop,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}}


CONFIGS = {
    # sizes on 16-byte boundaries; the loop ends before the last layer
    "aligned": model([parallel_layer((4, 2, 24, 40), (3, 16, 24), (0.5, 0.97, 0.999), 72), attn_layer(6, 2, 40, 24, 88),
                      parallel_layer((6, 1, 72, 96), (2, 40, 72), (0.9, 0.995), 64, (0.4, 1.3))],
                     width=48, vocab=120, loop=dict(start=0, stop=2, times=3)),
    # nothing is a multiple of eight, layers differ in every size, two have no feed-forward, one query head per key head
    "odd": model([attn_layer(3, 3, 10, 13, 37, conv=2, every=7), parallel_layer((5, 1, 11, 9), (3, 7, 5), (0.3, 0.9, 0.99), None,
                                                                         (1.5, -0.6)),
                  attn_layer(2, 1, 21, 6, None, conv=5, coef=-0.2, every=50, scale=0.3),
                  parallel_layer((4, 2, 6, 12), (4, 13, 10), (0.8, 1.0, 0.95, 0.998), 29, (0.9, 0.8), scale=0.5)],
                 width=45, vocab=101, eps=1e-3, loop=dict(start=1, stop=4, times=2), bigram=(50, 1000003, 777)),
    # one kind of layer only; many query heads per key head; no convolution state; no loop
    "attention": model([attn_layer(20, 1, 64, 128, 40, conv=1), attn_layer(4, 4, 128, 64, 64, conv=4)], width=64),
    "parallel": model([parallel_layer((16, 2, 128, 128), (2, 136, 72), (0.99, 0.8), 40),
                       parallel_layer((3, 3, 16, 16), (5, 16, 130), (0.1, 0.9, 0.7, 0.999, 0.97), None)],
                      width=56, loop=dict(start=1, stop=2, times=2)),
}


def tensor_shapes(cfg):
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, W)
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "attention":
            Q, K, V = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            mix = {"q": (Q, W), "k": (K, W), "v": (V, W), "q.b": (Q,), "k.b": (K,), "v.b": (V,), "q.conv": (Q, m["conv"]),
                   "k.conv": (K, m["conv"]), "v.conv": (V, m["conv"]), "q.norm": (m["dim"],), "k.norm": (m["dim"],),
                   "o": (W, m["heads"] * m["vdim"])}
        else:
            l, r = m["left"], m["right"]
            Q, K, V = l["heads"] * l["dim"], l["kv_heads"] * l["dim"], l["kv_heads"] * l["vdim"]
            N, P = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            mix = {"left.q": (Q, W), "left.k": (K, W), "left.v": (V, W), "left.q.norm": (Q,), "left.k.norm": (K,),
                   "left.o": (W, l["heads"] * l["vdim"]), "right.q": (N, W), "right.k": (N, W), "right.v": (P, W),
                   "right.g": (P, W), "right.o": (W, P), "right.norm": (P,)}
        out.update({f"l{i}.mix.{k}": v for k, v in mix.items()})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.mlp.gate": (ff, W), f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff)})
    out.update({"final.norm": (W,), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0):
    """bf16 weights under which faults show: query norms large enough that single keys dominate a softmax (a key lost or
    let in changes the output), no unit or zero constant, biases and taps of the size of what they are added to."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g)
        if name.endswith("q.norm"):
            t = 2.0 + 0.5 * r
        elif name.endswith(("norm", "norm1")):
            t = 1 + 0.3 * r
        elif name.endswith(".b"):
            t = 0.5 * r
        elif name in ("embed", "bigram"):
            t = r
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def save(cfg, weights, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)
