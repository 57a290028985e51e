"""Plain, slow float64 implementation of the Sodurax decoder, one function per mechanism, written from the equations and
sharing no code with the package: the yardstick for the kernels, the ragged step function and the engine.

Notation: h is a sublayer's input [L, width]; all products are W h with W stored [out, in]; positions count from 0.  A
layer is x <- x + n_o(mixer(n_i(x))), then (where it has a feed-forward) x <- x + n_o'(ff(n_i'(x))), every n an
elementwise squashing norm with parameters of its own.  A layer may run on another layer's tensors.
"""
import json
import math
import os

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------------------------- small pieces
def squash(x, W, name):
    """Elementwise norm: tanh(a x) w + b with a scalar a and vectors w, b."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def rotate_half(x, pos, rot):
    """x [L, H, d]: channel i < dims/2 of every head is paired with channel i + dims/2 and turned by the angle
    pos * base^(-2i/dims) / factor; the channels from `dims` on pass."""
    dims, base = rot["dims"], float(rot["base"])
    factor = float((rot.get("scaling") or {"factor": 1.0})["factor"])
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = float(pos[t]) * base ** (-2.0 * i / dims) / factor
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def visible(i, j, mask):
    """Does position i see position j?  Sliding window of `size` positions plus the first `keep_first` of the sequence."""
    if j > i:
        return False
    return mask is None or i - j < mask["size"] or j < mask.get("keep_first", 0)


# ----------------------------------------------------------------------------------------------- mixer
def attention(h, W, p, mx, pos):
    """Grouped-query softmax attention: biases on q, k, v; rotary positions on a part of the head; window + kept first
    keys; every output channel times sigmoid(W_g h)."""
    L = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rotate_half((h @ W[p + "q"].T + W[p + "q.b"]).view(L, H, d), pos, mx["rot"])
    k = rotate_half((h @ W[p + "k"].T + W[p + "k.b"]).view(L, G, d), pos, mx["rot"])
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(L, G, dv)
    ok = torch.tensor([[visible(int(i), int(j), mx.get("mask")) for j in pos] for i in pos])
    out = torch.zeros(L, H, dv, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        s = ((q[:, n] @ k[:, g].T) * mx["scale"]).masked_fill(~ok, float("-inf"))
        out[:, n] = torch.softmax(s, -1) @ v[:, g]
    gate = torch.sigmoid(h @ W[p + "g"].T)
    return (out.reshape(L, H * dv) * gate) @ W[p + "o"].T


# ----------------------------------------------------------------------------------------------- feed-forward
def choose(z, corr, router):
    """z [E] router logits, corr [E] -> (chosen experts, their weights).  s = sigmoid(z); choice scores s + corr; a group's
    score is the sum of its two largest choice scores; experts outside the best `keep` groups cannot be chosen; the weights
    are s itself."""
    s = torch.sigmoid(z)
    c = (s + corr).tolist()
    E = len(c)
    gr = router.get("groups") or {"count": 1, "keep": 1}
    n = E // gr["count"]
    score = [sum(sorted(c[g * n:(g + 1) * n], reverse=True)[:2]) for g in range(gr["count"])]
    best = sorted(range(gr["count"]), key=lambda g: -score[g])[:gr["keep"]]
    open_ = [e for e in range(E) if e // n in best]
    chosen = sorted(open_, key=lambda e: -c[e])[:router["top"]]
    return chosen, s[chosen]


def routed_ff(h, W, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, w = choose(W[p + "router"] @ h[t], W[p + "correction"], mlp["router"])
        for e, we in zip(chosen, w):
            z = torch.clamp(W[f"{p}e{e}.up"] @ h[t], min=0.0)
            out[t] += we * (W[f"{p}e{e}.down"] @ (z * z))
    return out


# ----------------------------------------------------------------------------------------------- the model
def forward(cfg, W, tokens, trace=None):
    """Token ids -> logits [L, vocab] (W: tensor name -> float64).  `trace` collects the stream after every layer."""
    x = W["embed"][torch.tensor(tokens)]
    pos = torch.arange(len(tokens))
    for i, ly in enumerate(cfg["layers"]):
        j = i
        while "weights_of" in cfg["layers"][j]:
            j = cfg["layers"][j]["weights_of"]
        p = f"l{j}."
        x = x + squash(attention(squash(x, W, p + "norm1"), W, p + "mix.", ly["mixer"], pos), W, p + "norm1b")
        if ly.get("mlp") is not None:
            x = x + squash(routed_ff(squash(x, W, p + "norm2"), W, p + "mlp.", ly["mlp"]), W, p + "norm2b")
        if trace is not None:
            trace.append(x.clone())
    return squash(x, W, "final.norm") @ W["embed"].T


# ----------------------------------------------------------------------------------------------- test models
def layer(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=8, base=1000.0, factor=4.0, scale=0.3, window=11, keep=3,
          mlp=True):
    rot = {"dims": rot_dims, "base": base}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if window:
        mixer["mask"] = {"size": window, "keep_first": keep}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def again(j):
    """A layer that runs on layer j's tensors."""
    return {"weights_of": j}


def make_config(layers, width=48, vocab=61, eps=1e-5, experts=8, top=2, ff=24, groups=2, keep_groups=1):
    router = {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep_groups}}
    out = []
    for ly in layers:
        if "weights_of" in ly:
            out.append(dict(out[ly["weights_of"]], weights_of=ly["weights_of"]))
        else:
            out.append(dict(ly, mlp={"kind": "moe", "expert": {"ff": ff}, "router": router} if ly["mlp"] else None))
    return {"architecture": "Sodurax", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_weights(cfg, seed=0):
    """Random tensors of every name and shape the file format has, rounded to bfloat16 as a checkpoint holds them."""
    g = torch.Generator().manual_seed(seed)
    Wd = cfg["width"]

    def mat(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s * i ** -0.5)

    def vec(n, mean, s):
        return torch.randn(n, generator=g) * s + mean

    def norm(name, out_scale):
        W[name], W[name + ".b"] = vec(Wd, out_scale, 0.3), vec(Wd, 0.0, 0.2)
        W[name + ".alpha"] = torch.tensor(0.5 + torch.rand((), generator=g).item())

    W = {"embed": torch.randn(cfg["vocab"], Wd, generator=g)}
    norm("final.norm", 1.0)
    for i, ly in enumerate(cfg["layers"]):
        if "weights_of" in ly:
            continue
        mx, p = ly["mixer"], f"l{i}.mix."
        H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        for n in ("norm1", "norm1b"):
            norm(f"l{i}.{n}", 1.0)
        W[p + "q"], W[p + "k"], W[p + "v"] = mat(H * d, Wd), mat(G * d, Wd), mat(G * dv, Wd)
        W[p + "q.b"], W[p + "k.b"], W[p + "v.b"] = vec(H * d, 0, 0.5), vec(G * d, 0, 0.5), vec(G * dv, 0, 0.5)
        W[p + "g"], W[p + "o"] = mat(H * dv, Wd, 2.0), mat(Wd, H * dv, 2.0)
        mlp = ly.get("mlp")
        if mlp is None:
            continue
        for n in ("norm2", "norm2b"):
            norm(f"l{i}.{n}", 1.0)
        q, E, f = f"l{i}.mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
        for e in range(E):
            W[f"{q}e{e}.up"], W[f"{q}e{e}.down"] = mat(f, Wd, 1.5), mat(Wd, f)
        W[q + "router"], W[q + "correction"] = mat(E, Wd, 2.0), vec(E, -0.3, 0.4)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def to64(W):
    return {k: v.to(F64) for k, v in W.items()}


def write_checkpoint(folder, cfg, W):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in W.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)
