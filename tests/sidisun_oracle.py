"""Plain, slow implementation of the Sidisun design in double precision, one function per mechanism. Shares no code with
the package: the tests compare the framework with it. Also makes small configurations and random weights for it."""
import json
import math
import os

import torch


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def rotary_frequencies(rot):
    """(frequency per pair, factor on cos and sin); with 'scaling' the YaRN blend of kept and interpolated ones."""
    n, base = rot["dims"], float(rot["base"])
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(freq, dtype=torch.float64), 1.0

    def turns_to_dim(t):
        return n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(turns_to_dim(s["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1


def rotate(x, position, rot):
    """One vector (or a stack of them) at one position; half-split pairs, the rest passes."""
    freq, mag = rotary_frequencies(rot)
    half = rot["dims"] // 2
    c, s = torch.cos(position * freq) * mag, torch.sin(position * freq) * mag
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def latent_attention(h, w, m, eps):
    """h [T, width] -> [T, width], query by query."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_unit(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T
    q = q.view(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms_unit(down[:, :K], eps) * w["dkv.norm"]
    kr = torch.stack([rotate(down[t, K:], t, m["rot"]) for t in range(T)])
    k = (c @ w["uk"].T).view(T, H, D)
    v = (c @ w["uv"].T).view(T, H, V)
    rows = []
    for t in range(T):
        qr = rotate(q[t, :, D:], t, m["rot"])
        s = (torch.einsum("hd,jhd->hj", q[t, :, :D], k[:t + 1]) + qr @ kr[:t + 1].T) * m["scale"]
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        p = p / p.sum(-1, keepdim=True)
        rows.append(torch.einsum("hj,jhv->hv", p, v[:t + 1]).reshape(-1))
    gate = 1 / (1 + torch.exp(-(h @ w["g"].T)))
    return (torch.stack(rows) * gate) @ w["o"].T


def short_conv(x, weight, bias):
    """Per channel over time, zeros before the start, last tap = current token; then silu."""
    T, taps = x.shape[0], weight.shape[1]
    out = []
    for t in range(T):
        y = bias.clone()
        for k in range(taps):
            j = t - (taps - 1 - k)
            if j >= 0:
                y = y + weight[:, k] * x[j]
        out.append(silu(y))
    return torch.stack(out)


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, P], B and C [T, H, N], dt [T, H] (after softplus): the recurrence, one token after the other."""
    T, H, P = x.shape
    S = torch.zeros(H, B.shape[-1], P, dtype=x.dtype)
    out = []
    for t in range(T):
        for h in range(H):
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, h], x[t, h])
        out.append(torch.stack([S[h].T @ C[t, h] + D[h] * x[t, h] for h in range(H)]))
    return torch.stack(out)


def grouped_norm(x, groups, weight, eps):
    n = x.shape[-1] // groups
    return torch.cat([rms_unit(x[..., g * n:(g + 1) * n], eps) for g in range(groups)], -1) * weight


def mamba2(h, w, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ w["in"].T
    z, rest, dt = proj[:, :inner], proj[:, inner:inner + inner + 2 * G * N], proj[:, -H:]
    act = short_conv(rest, w["conv"], w["conv.b"])
    x = act[:, :inner].view(T, H, P)
    B, C = (act[:, inner + i * G * N: inner + (i + 1) * G * N].view(T, G, N) for i in (0, 1))
    of = [h_ // (H // G) for h_ in range(H)]
    y = state_space(x, B[:, of], C[:, of], softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    y = y.reshape(T, inner) * silu(z)
    return grouped_norm(y, m["norm_groups"], w["norm"], eps) @ w["o"].T


def feed_forward(h, w, eps):
    a, b, c, e = w["act"]
    z = h @ w["up"].T
    return (a * rms_unit(z, eps) + b * rms_unit(z * z, eps) + c * rms_unit(z * z * z, eps) + e) @ w["down"].T


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


def logits(cfg, weights, tokens, stream=None):
    """Logits of every position [T, vocab]; ``stream`` (a list) collects the residual stream after every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        part = lambda kind: {k[len(f"l{i}.{kind}."):]: v for k, v in W.items() if k.startswith(f"l{i}.{kind}.")}
        x = x + rms_unit(MIXERS[layer["type"]](x, part("mix"), layer["mixer"], eps), eps) * W[f"l{i}.norm1"]
        if layer["mlp"] is not None:
            x = x + rms_unit(feed_forward(x, part("mlp"), eps), eps) * W[f"l{i}.norm2"]
        if stream is not None:
            stream.append(x)
    return (rms_unit(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(logits(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ---- small models -------------------------------------------------------------------------------------------------
def attn_layer(heads, dim, rot, vdim, kv_rank, q_rank, ff, scale=None, base=10000.0, scaling=None):
    return {"type": "latent_attention",
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                          scale=scale if scale is not None else (dim + rot) ** -0.5,
                          rot=dict(base=base, dims=rot, scaling=scaling)),
            "mlp": None if ff is None else dict(kind="dense", ff=ff)}


def mamba_layer(heads, vdim, state, groups, ff, conv=4, norm_groups=1):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv,
                                            norm_groups=norm_groups),
            "mlp": None if ff is None else dict(kind="dense", ff=ff)}


def model(layers, vocab=97, width=40, eps=1e-5, logit_scale=0.5):
    return {"architecture": "Sidisun", "vocab": vocab, "width": width, "logit_scale": logit_scale, "norm": {"eps": eps},
            "layers": layers}


YARN = dict(factor=4.0, original=64, fast=16.0, slow=1.0)
CONFIGS = {
    # sizes on 16-byte boundaries: every tensor-core form applies
    "aligned": model([mamba_layer(4, 24, 32, 2, 72, norm_groups=2), attn_layer(5, 24, 16, 40, 48, 32, 88, scaling=YARN),
                      mamba_layer(4, 24, 32, 1, None, conv=3)], width=48, vocab=120),
    # nothing is a multiple of eight, layers differ in every size, one has no feed-forward, no rotary scaling
    "odd": model([attn_layer(3, 10, 6, 14, 21, 19, 37), mamba_layer(6, 7, 11, 3, 29, conv=2, norm_groups=3),
                  attn_layer(2, 13, 4, 9, 30, 17, None, base=500.0, scaling=dict(YARN, factor=1.0)),
                  mamba_layer(2, 12, 20, 2, 33, conv=5)], width=45, vocab=101, eps=1e-3, logit_scale=1.75),
    # one kind of layer only
    "attention": model([attn_layer(4, 16, 8, 16, 24, 24, 40), attn_layer(20, 64, 64, 72, 136, 40, 64, scaling=YARN)]),
    "recurrent": model([mamba_layer(3, 16, 16, 1, 40), mamba_layer(2, 64, 136, 1, 40, conv=1)]),
}


def tensor_shapes(cfg):
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "latent_attention":
            H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
            mix = {"dq": (m["q_rank"], W), "dq.norm": (m["q_rank"],), "uq": (H * (D + R), m["q_rank"]),
                   "dkv": (m["kv_rank"] + R, W), "dkv.norm": (m["kv_rank"],), "uk": (H * D, m["kv_rank"]),
                   "uv": (H * V, m["kv_rank"]), "g": (H * V, W), "o": (W, H * V)}
        else:
            I, GN = m["heads"] * m["vdim"], m["groups"] * m["state"]
            mix = {"in": (2 * I + 2 * GN + m["heads"], W), "conv": (I + 2 * GN, m["conv"]), "conv.b": (I + 2 * GN,),
                   "dt_bias": (m["heads"],), "A_log": (m["heads"],), "D": (m["heads"],), "norm": (I,), "o": (W, I)}
        out.update({f"l{i}.mix.{k}": v for k, v in mix.items()})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff), f"l{i}.mlp.act": (4,)})
    out.update({"final.norm": (W,), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0):
    """bf16 weights under which faults show: queries large enough that single keys dominate a softmax (a key lost or let
    in changes the output), decays slow enough that a state remembers hundreds of tokens, no unit or zero constant."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g)
        leaf = name.split(".", 2)[-1] if ".mix." in name else name
        if name.endswith(("norm", "norm1", "norm2")):
            t = 1 + 0.3 * r
        elif leaf == "uq":
            t = 2.5 * r * shape[1] ** -0.5
        elif leaf == "A_log":
            t = -1.0 + 0.7 * r
        elif leaf == "dt_bias":
            t = -3.0 + 0.7 * r
        elif leaf == "D":
            t = 0.5 + 0.5 * r
        elif leaf == "conv.b" or name.endswith("mlp.act"):
            t = 0.4 * r
        else:
            t = r * (shape[-1] ** -0.5 if name != "embed" else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def save(cfg, weights, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)
