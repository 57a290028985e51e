"""Plain, slow float64 implementation of the Sumolorn decoder, one function per mechanism, written from the equations and
sharing no code with the package: the yardstick for the kernels, the ragged step function and the engine.

Notation: h is a sublayer's normalised input [L, width]; all products are W h with W stored [out, in]; positions count
from 0.  A layer is x <- x + mixer(n1(x)), then (where it has a feed-forward) x <- x + ff(n2(x)), with
n(x) = rms(x) (1 + w).  A span of layers may run several times in a row.  Every recurrence walks the tokens one by one.
"""
import json
import math
import os

import torch

F64 = torch.float64
ALPHA = 1.702


# ----------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def frequencies(rot):
    """One angle per turn of position for every pair; with `scaling`, pairs of a long wave are slowed down by `factor`,
    those of a short wave stay, the ones between are mixed linearly in (original / wavelength)."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, pos, rot, interleaved):
    """x [L, H, d]: the first `dims` channels of every head turn by position x frequency; pair i is (i, i + dims / 2), or
    (2i, 2i + 1) when interleaved."""
    out = x.clone()
    n = rot["dims"] // 2
    p = torch.as_tensor(pos, dtype=F64)
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n)
        c, s = torch.cos(p * f)[:, None], torch.sin(p * f)[:, None]
        u, v = x[:, :, a], x[:, :, b]
        out[:, :, a] = u * c - v * s
        out[:, :, b] = v * c + u * s
    return out


def causal_conv(x, w):
    """x [L, C], w [C, taps] with the last column on the current token; zeros before the first token."""
    L = x.shape[0]
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(L):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * x[t - taps + 1 + j]
    return out


def weigh(scores, pos, size, sink):
    """scores [L, L] of one head -> softmax weights over the visible keys; a sink score joins the denominator only."""
    p = torch.as_tensor(pos)
    dist = p[:, None] - p[None, :]
    seen = (dist >= 0) & (dist < size) if size else dist >= 0
    s = scores.masked_fill(~seen, -math.inf)
    m = s.max(1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink)
    e = torch.exp(s - m)
    return e / (e.sum(1, keepdim=True) + (0.0 if sink is None else torch.exp(sink - m)))


# ----------------------------------------------------------------------------------------------- mixers
def attention(h, W, p, mx, pos):
    """Grouped key / value heads, rotate-half positions on a part of the head, soft-capped scores, a sliding window, a sink
    per head, one sigmoid gate per head."""
    L = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rotate((h @ W[p + "q"].T).view(L, H, d), pos, mx["rot"], False)
    k = rotate((h @ W[p + "k"].T).view(L, G, d), pos, mx["rot"], False)
    v = (h @ W[p + "v"].T).view(L, G, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    heads = []
    for n in range(H):
        g = n // (H // G)
        s = softcap(q[:, n] @ k[:, g].T * mx["scale"], mx["softcap"])
        heads.append(weigh(s, pos, mx["mask"]["size"], W[p + "sink"][n]) @ v[:, g] * gate[:, n:n + 1])
    return torch.cat(heads, 1) @ W[p + "o"].T


def latent_attention(h, W, p, mx, eps, pos):
    """Queries through a normalised latent; keys and values rebuilt from a normalised latent of the key side plus one rotated
    part that the heads share; interleaved pairs, no window, a sink per head, one sigmoid gate per head."""
    L = h.shape[0]
    H, d, r, dv, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    cq = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(L, H, d + r)
    low = h @ W[p + "dkv"].T
    c = rms(low[:, :R], eps) * W[p + "dkv.norm"]
    kr = rotate(low[:, None, R:], pos, mx["rot"], True)[:, 0]
    qr = rotate(q[:, :, d:], pos, mx["rot"], True)
    k = (c @ W[p + "uk"].T).view(L, H, d)
    v = (c @ W[p + "uv"].T).view(L, H, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    heads = []
    for n in range(H):
        s = (q[:, n, :d] @ k[:, n].T + qr[:, n] @ kr.T) * mx["scale"]
        heads.append(weigh(s, pos, 0, W[p + "sink"][n]) @ v[:, n] * gate[:, n:n + 1])
    return torch.cat(heads, 1) @ W[p + "o"].T


def convolved_attention(h, W, p, mx, eps, pos):
    """q, k, v each pass a short causal convolution; then positions (rotate-half), then q and k heads of unit RMS; a sliding
    window, ordinary softmax."""
    L = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = causal_conv(h @ W[p + "q"].T, W[p + "q.conv"]).view(L, H, d)
    k = causal_conv(h @ W[p + "k"].T, W[p + "k.conv"]).view(L, G, d)
    v = causal_conv(h @ W[p + "v"].T, W[p + "v.conv"]).view(L, G, dv)
    q, k = rms(rotate(q, pos, mx["rot"], False), eps), rms(rotate(k, pos, mx["rot"], False), eps)
    heads = []
    for n in range(H):
        g = n // (H // G)
        heads.append(weigh(q[:, n] @ k[:, g].T * mx["scale"], pos, mx["mask"]["size"], None) @ v[:, g])
    return torch.cat(heads, 1) @ W[p + "o"].T


def gated_linear_attention(h, W, p, mx, eps):
    """Per head a matrix S [d, dv], zero at the start; every token multiplies row i by sigmoid(z_i)^(1 / tau), adds
    outer(k, v) and reads S^T q (q scaled by d^-1/2); the read-out has unit RMS per head, a weight over dv that the heads
    share and a silu gate."""
    L = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T).view(L, H, d) * d ** -0.5
    k = (h @ W[p + "k"].T).view(L, H, d)
    v = (h @ W[p + "v"].T).view(L, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = (sigmoid(z) ** (1.0 / mx["tau"])).view(L, H, d)
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    o = torch.zeros(L, H, dv, dtype=h.dtype)
    for t in range(L):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    g = h @ W[p + "g"].T
    o = (rms(o, eps) * W[p + "norm"]).reshape(L, H * dv) * (g * sigmoid(g))
    return o @ W[p + "o"].T


def pair(h, W, p, mx, eps, pos):
    a = convolved_attention(h, W, p + "left.", mx["left"], eps, pos)
    b = gated_linear_attention(h, W, p + "right.", mx["right"], eps)
    return 0.5 * (rms(a, eps) * W[p + "left.out"] + rms(b, eps) * W[p + "right.out"])


def clamped_ff(h, W, p, limit):
    g = (h @ W[p + "gate"].T).clamp(max=limit)
    u = (h @ W[p + "up"].T).clamp(min=-limit, max=limit)
    return (g * sigmoid(ALPHA * g) * (u + 1.0)) @ W[p + "down"].T


# ----------------------------------------------------------------------------------------------- the model
def runs(cfg):
    """The layers in the order they run."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def mixer(h, W, p, ly, eps, pos):
    if ly["type"] == "attention":
        return attention(h, W, p, ly["mixer"], pos)
    if ly["type"] == "latent_attention":
        return latent_attention(h, W, p, ly["mixer"], eps, pos)
    return pair(h, W, p, ly["mixer"], eps, pos)


def forward(cfg, W, tokens, layers_out=None):
    """Logits [L, vocab] of one sequence; `layers_out` (a list) receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    pos = list(range(len(tokens)))
    x = W["embed"][torch.tensor(tokens)]
    for i in runs(cfg):
        ly, p = cfg["layers"][i], f"l{i}."
        x = x + mixer(rms(x, eps) * (1.0 + W[p + "norm1"]), W, p + "mix.", ly, eps, pos)
        if ly["mlp"] is not None:
            x = x + clamped_ff(rms(x, eps) * (1.0 + W[p + "norm2"]), W, p + "mlp.", ly["mlp"]["limit"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * (1.0 + W["final.norm"])) @ W["head"].T * cfg["logit_scale"]


# ----------------------------------------------------------------------------------------------- test models
def dense(ff=56, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _rot(dims, base, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, cap=8.0, window=12, rot_dims=8, base=1000.0,
                    scaling=(4.0, 1.0, 4.0, 64), mlp="dense"):
    return {"type": "attention", "mlp": dense() if mlp == "dense" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                      "mask": {"size": window}, "rot": _rot(rot_dims, base, scaling)}}


def latent_layer(heads=3, dim=16, rot_dim=8, vdim=8, kv_rank=24, q_rank=32, scale=0.25, base=500.0, mlp="dense"):
    return {"type": "latent_attention", "mlp": dense() if mlp == "dense" else mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale, "rot": _rot(rot_dim, base)}}


def parallel_layer(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, window=9, rot_dims=8, base=300.0, conv=3, g_heads=2, g_dim=8,
                   g_vdim=16, tau=8.0, rank=8, mlp="dense"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv,
            "mask": {"size": window}, "rot": _rot(rot_dims, base)}
    return {"type": "parallel", "mlp": dense() if mlp == "dense" else mlp, "_rank": rank,
            "mixer": {"left": left, "right": {"heads": g_heads, "dim": g_dim, "vdim": g_vdim, "tau": tau}}}


def make_config(layers, width=48, vocab=96, eps=1e-5, logit_scale=0.5, loop=None):
    cfg = {"architecture": "Sumolorn", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab,
           "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_weights(cfg, seed=0):
    """name -> bf16-representable fp32 tensors in the checkpoint's naming."""
    gen = torch.Generator().manual_seed(seed)
    W, Wd = {}, cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=gen) * (s / math.sqrt(i))

    def vec(n, mean=0.0, std=0.2):
        return mean + torch.randn(n, generator=gen) * std

    W["embed"] = torch.randn(cfg["vocab"], Wd, generator=gen)
    W["head"] = lin(cfg["vocab"], Wd)
    W["final.norm"] = vec(Wd)
    for i, ly in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", ly["mixer"], ly["mlp"]
        W[p + "norm1"] = vec(Wd)
        if mlp is not None:
            W[p + "norm2"] = vec(Wd)
            W[p + "mlp.gate"], W[p + "mlp.up"] = lin(mlp["ff"], Wd, 1.5), lin(mlp["ff"], Wd, 1.5)
            W[p + "mlp.down"] = lin(Wd, mlp["ff"])
        p += "mix."
        if ly["type"] == "attention":
            H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
            W[p + "q"], W[p + "k"], W[p + "v"] = lin(H * d, Wd, 2.0), lin(G * d, Wd, 2.0), lin(G * dv, Wd)
            W[p + "sink"], W[p + "g"], W[p + "o"] = vec(H, 0.0, 1.5), lin(H, Wd, 2.0), lin(Wd, H * dv)
        elif ly["type"] == "latent_attention":
            H, d, r, dv, R, Q = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"], mx["q_rank"]
            W[p + "dq"], W[p + "dq.norm"], W[p + "uq"] = lin(Q, Wd), vec(Q, 1.0), lin(H * (d + r), Q, 2.0)
            W[p + "dkv"], W[p + "dkv.norm"] = lin(R + r, Wd, 1.5), vec(R, 1.0)
            W[p + "uk"], W[p + "uv"] = lin(H * d, R, 2.0), lin(H * dv, R)
            W[p + "sink"], W[p + "g"], W[p + "o"] = vec(H, 0.0, 1.5), lin(H, Wd, 2.0), lin(Wd, H * dv)
        else:
            lm, rm = mx["left"], mx["right"]
            H, G, d, dv = lm["heads"], lm["kv_heads"], lm["dim"], lm["vdim"]
            q = p + "left."
            for n, rows, s in (("q", H * d, 2.0), ("k", G * d, 2.0), ("v", G * dv, 1.0)):
                W[q + n] = lin(rows, Wd, s)
                W[q + n + ".conv"] = torch.randn(rows, lm["conv"], generator=gen) * 0.6
            W[q + "o"], W[q + "out"] = lin(Wd, H * dv), vec(Wd, 1.0)
            r, H, d, dv = p + "right.", rm["heads"], rm["dim"], rm["vdim"]
            W[r + "q"], W[r + "k"], W[r + "v"] = lin(H * d, Wd, 1.5), lin(H * d, Wd, 1.5), lin(H * dv, Wd)
            W[r + "g"], W[r + "o"] = lin(H * dv, Wd, 1.5), lin(Wd, H * dv)
            W[r + "norm"], W[r + "out"] = vec(dv, 1.0), vec(Wd, 1.0)
            W[r + "a1"] = lin(ly.get("_rank", 8), Wd, 1.5)
            W[r + "a2"], W[r + "a2.b"] = lin(H * d, ly.get("_rank", 8), 1.5), vec(H * d, 0.5, 1.5)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def write_checkpoint(folder, cfg, W):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    plain = dict(cfg, layers=[{k: v for k, v in ly.items() if k != "_rank"} for ly in cfg["layers"]])   # the rank: tensors tell
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(plain, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in W.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def to64(W):
    return {k: v.to(F64) for k, v in W.items()}
