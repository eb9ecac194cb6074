"""The Milozen decoder, written plainly: one function per mechanism, float64 torch on the CPU, whole sequences at once,
no cache.  It shares no code with the package; the tests compare the package against it.

A model is ``(config, tensors)``: the dictionary of config.json and the tensors by name.

Notation: ``X [s, n, width]`` the parallel residual streams of one sequence, position ``i`` of a query, ``j`` of a key,
``H`` heads, ``d`` / ``r`` the unrotated / rotated size of a query or key, ``v`` a value's size, ``kr`` a latent's.
"""
import json
import math
import os
import struct

import torch

F = torch.float64


def t64(t):
    return t.to(F)


# ----------------------------------------------------------------------------- norms

def layer_norm(x, w, eps):
    mean = x.mean(-1, keepdim=True)
    dev = x - mean
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ----------------------------------------------------------------------------- parallel streams

def streams_read(X, a):
    """``u = sum_s a[s] X_s`` (``a [s]``): what a sublayer's norm gets."""
    return torch.einsum("s,snh->nh", a, X)


def streams_write(X, M, b, y):
    """``X'_t = sum_s M[s, t] X_s + b[t] y``: the new streams, all from the old ones."""
    return torch.einsum("st,snh->tnh", M, X) + b[:, None, None] * y[None]


# ----------------------------------------------------------------------------- latent attention

def rotate_neighbours(x, pos, dims, base):
    """x [n, ..., D]; numbers 2i and 2i + 1 of the last axis form a pair that turns by ``p * base^(-2i / dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        ang = pos.to(F) * base ** (-2.0 * i / dims)
        while ang.dim() < x.dim() - 1:
            ang = ang.unsqueeze(1)
        c, s = torch.cos(ang), torch.sin(ang)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_visible(n, size=None):
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    ok = j <= i
    return ok if size is None else ok & (i - j < size)


def latent_rows(h, w, m, pos, eps):
    """What a layer with a latent of its own caches: the normed latent ``c [n, kr]`` and the rotated key part ``[n, r]``."""
    kr = m["kv_rank"]
    row = h @ w["dkv"].T
    return rms_norm(row[:, :kr], w["dkv.norm"], eps), rotate_neighbours(row[:, kr:], pos, m["rot"]["dims"], m["rot"]["base"])


def latent_queries(h, w, m, pos, eps):
    H, d, r = m["heads"], m["dim"], m["rot_dim"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(h.shape[0], H, d + r)
    return q[..., :d], rotate_neighbours(q[..., d:], pos, m["rot"]["dims"], m["rot"]["base"])


def attend(qu, qr, ku, kr, v, ok, scale):
    """qu [n, H, d], qr [n, H, r], ku [L, H, d], kr [L, r] (one for all heads), v [L, H, v] -> [n, H, v]."""
    s = (torch.einsum("nhd,lhd->hnl", qu, ku) + torch.einsum("nhr,lr->hnl", qr, kr)) * scale
    return torch.einsum("hnl,lhv->nhv", torch.softmax(s.masked_fill(~ok[None], -math.inf), dim=-1), v)


def latent_attention(h, w, m, pos, eps, rows):
    """``rows``: what ``latent_rows`` gives, of this layer or of the layer whose cache it reads."""
    n = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    c, k_rot = rows
    qu, qr = latent_queries(h, w, m, pos, eps)
    ku = (c @ w["uk"].T).reshape(n, H, d)
    v = (c @ w["uv"].T).reshape(n, H, vd)
    o = attend(qu, qr, ku, k_rot, v, window_visible(n, (m.get("mask") or {}).get("size")), m["scale"])
    return (o.reshape(n, H * vd) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------------------- feed-forwards

def dense_ff(h, w):
    g = h @ w["gate"].T
    return (g * torch.sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def expert(x, w, e, limit):
    g = torch.clamp(x @ w[f"e{e}.gate"].T, max=limit)
    u = torch.clamp(x @ w[f"e{e}.up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[f"e{e}.down"].T


def route(h, w_router, top, forced=None):
    """Chosen experts ``[n, top]`` (largest score first) and their scores, which are not divided by their sum."""
    s = torch.sigmoid(h @ w_router.T)
    ids = forced if forced is not None else torch.topk(s, top, dim=-1).indices
    return ids, torch.gather(s, 1, ids)


def moe_ff(h, w, mlp, forced=None):
    """The score multiplies the expert's INPUT; outputs are summed as they are."""
    ids, scores = route(h, w["router"], mlp["router"]["top"], forced)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(ids[t].tolist(), scores[t]):
            out[t] += expert((s * h[t])[None], w, e, mlp["expert"]["limit"])[0]
    return out


# ----------------------------------------------------------------------------- the whole model

def local(tensors, prefix):
    return {k[len(prefix):]: t64(v) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, ids, layers_out=None, forced=None):
    """Logits [n, vocab] (float64) of one sequence.  ``layers_out``: a list that receives the sum of the streams after
    every layer.  ``forced``: for every mixture-of-experts layer in order, the experts ``[n, top]`` to use instead of the
    router's choice."""
    forced = list(forced) if forced is not None else None
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(ids))
    x0 = t64(tensors["embed"])[torch.tensor(list(ids), dtype=torch.long)] * cfg["embedding"]["scale"]
    X = torch.stack([x0] * cfg["streams"])
    kept = {}                                                   # latents of the layers that have their own
    for li, l in enumerate(cfg["layers"]):
        p = f"l{li}."
        w, m = local(tensors, p + "mix."), l["mixer"]
        hc = local(tensors, p + "hc1.")
        h = layer_norm(streams_read(X, hc["in"]), t64(tensors[p + "norm1"]), eps)
        if m.get("kv_from") is None:
            kept[li] = latent_rows(h, w, m, pos, eps)
        y = latent_attention(h, w, m, pos, eps, kept[li if m.get("kv_from") is None else m["kv_from"]])
        X = streams_write(X, hc["mix"], hc["out"], y)
        mlp = l.get("mlp")
        if mlp is not None:
            hc, wf = local(tensors, p + "hc2."), local(tensors, p + "mlp.")
            h = layer_norm(streams_read(X, hc["in"]), t64(tensors[p + "norm2"]), eps)
            y = dense_ff(h, wf) if mlp["kind"] == "dense" else moe_ff(h, wf, mlp, forced.pop(0) if forced else None)
            X = streams_write(X, hc["mix"], hc["out"], y)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return layer_norm(X.sum(0), t64(tensors["final.norm"]), eps) @ t64(tensors["embed"]).T


# ----------------------------------------------------------------------------- reading a folder

_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16, "F64": torch.float64}


def read_folder(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    tensors = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        tensors[name] = torch.frombuffer(bytearray(data[a:b]), dtype=_DT[info["dtype"]]).reshape(info["shape"]).clone()
    return cfg, tensors


def greedy(config, tensors, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(config, tensors, ids)[-1])))
    return ids[len(prompt):]
