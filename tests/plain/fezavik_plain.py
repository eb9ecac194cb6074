"""The Fezavik decoder, written plainly: one function per mechanism, float64 torch on the CPU, whole sequences at once,
no cache.  It shares no code with the package; the tests compare the package against it.

A model is ``(config, tensors)``: the dictionary of config.json and the tensors by name.

Notation: ``x [n, width]`` the residual stream of one sequence, ``h`` a sublayer's input, position ``i`` of a query, ``j``
of a key, ``H`` / ``G`` query and key/value heads, ``E`` experts with tensors, ``I`` identity experts.
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

def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sandwich(x, f, w_in, w_out, eps):
    """``x + norm_out(f(norm_in(x)))``: a sublayer between two norms."""
    return x + rms_norm(f(rms_norm(x, w_in, eps)), w_out, eps)


# ----------------------------------------------------------------------------- positions

def frequencies(dims, base, scaling=None):
    """One per pair.  ``scaling`` (factor, low, high, original): by the wavelength, kept, divided, or in between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            turns = scaling["original"] / wave              # full turns within the original context
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = f * (s + (1.0 - s) / scaling["factor"])
        out.append(f)
    return out


def rotate(x, pos, freqs, neighbours):
    """x [n, ..., D]: pair ``i`` is numbers ``(2i, 2i + 1)`` (``neighbours``) or ``(i, i + m)``, ``m`` pairs in all, and turns
    by ``pos * freqs[i]``; numbers behind the pairs stay."""
    out = x.clone()
    m = len(freqs)
    for i, f in enumerate(freqs):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + m)
        ang = (pos.to(F) * f).reshape([-1] + [1] * (x.dim() - 2))
        u, v = x[..., a], x[..., b]
        out[..., a] = u * torch.cos(ang) - v * torch.sin(ang)
        out[..., b] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


# ----------------------------------------------------------------------------- attention

def window_visible(n, size=None):
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    ok = j <= i
    return ok if size is None else ok & (i - j < size)


def sink_softmax(s, ok, sink):
    """s [H, n, L]: weights ``exp(s_j) / (exp(sink_h) + sum exp(s))`` over the visible keys; they add up to less than one."""
    full = torch.cat([s.masked_fill(~ok[None], -math.inf), sink[:, None, None].expand(-1, s.shape[1], 1)], dim=-1)
    return torch.softmax(full, dim=-1)[..., :-1]


def window_of(m):
    return (m.get("mask") or {}).get("size")


def attention(h, w, m, pos, eps):
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot")
    freqs = frequencies(rot["dims"], rot["base"], rot.get("scaling")) if rot else []
    q = rotate(rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(n, H, d), pos, freqs, True)
    k = rotate(rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(n, G, d), pos, freqs, True)
    v = (h @ w["v"].T).reshape(n, G, vd)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    p = sink_softmax(torch.einsum("nhd,lhd->hnl", q, k) * m["scale"], window_visible(n, window_of(m)), w["sink"])
    return torch.einsum("hnl,lhv->nhv", p, v).reshape(n, H * vd) @ w["o"].T


def latent_attention(h, w, m, pos, eps):
    n, H, d, r, vd, kr = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freqs = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(n, H, d + r)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :kr], w["dkv.norm"], eps)
    k_rot = rotate(down[:, kr:], pos, freqs, False)
    q_rot = rotate(q[..., d:], pos, freqs, False)
    ku, v = (c @ w["uk"].T).reshape(n, H, d), (c @ w["uv"].T).reshape(n, H, vd)
    s = (torch.einsum("nhd,lhd->hnl", q[..., :d], ku) + torch.einsum("nhr,lr->hnl", q_rot, k_rot)) * m["scale"]
    o = torch.einsum("hnl,lhv->nhv", sink_softmax(s, window_visible(n, window_of(m)), w["sink"]), v)
    o = o * torch.sigmoid(h @ w["g"].T)[..., None]              # one gate per head
    return o.reshape(n, H * vd) @ w["o"].T


# ----------------------------------------------------------------------------- recurrence

def forget_gate(h, w):
    """``[n, heads * dim]``, between the channel's lower bound and 1."""
    low = w["lower"]
    return low + (1.0 - low) * torch.sigmoid(h @ w["f"].T + w["f.b"])


def hgrn2_states(q, f, v, S=None):
    """q, f [n, H, d], v [n, H, vd] -> o [n, H, vd], token by token; what the gate lets go is what is written."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F) if S is None else S
    out = []
    for t in range(q.shape[0]):
        S = f[t][..., None] * S + (1.0 - f[t])[..., None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def hgrn2(h, w, m, eps):
    n, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    z = h @ w["q"].T
    q = (z * torch.sigmoid(z)).reshape(n, H, d)
    o, _ = hgrn2_states(q, forget_gate(h, w).reshape(n, H, d), (h @ w["v"].T).reshape(n, H, vd))
    return rms_norm(o, w["norm"], eps).reshape(n, H * vd) @ w["o"].T


# ----------------------------------------------------------------------------- experts

def expert(x, w, e):
    g = x @ w[f"e{e}.gate"].T
    return (g * torch.sigmoid(g) * (x @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T


def route(h, w, top, forced=None):
    """Chosen experts ``[n, top]`` (largest choice score first) and their weights: the softmax over ALL experts, not divided
    by what was chosen; the correction takes part in the choice alone."""
    s = torch.softmax(h @ w["router"].T, dim=-1)
    ids = forced if forced is not None else torch.topk(s + w["correction"], top, dim=-1).indices
    return ids, torch.gather(s, 1, ids)


def moe_ff(h, w, mlp, forced=None):
    ids, weights = route(h, w, mlp["router"]["top"], forced)
    out = torch.zeros_like(h)
    for e in torch.unique(ids).tolist():
        t, j = (ids == e).nonzero(as_tuple=True)                # the tokens that use it, and as which of their choices
        out[t] += weights[t, j, None] * (expert(h[t], w, e) if e < mlp["router"]["experts"] else h[t])
    return out


# ----------------------------------------------------------------------------- the whole model

def local(tensors, prefix):
    return {k[len(prefix):]: t64(v) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, ids, layers_out=None, forced=None):
    """Logits [n, vocab] (float64) of one sequence.  ``layers_out``: a list that receives the stream after every layer.
    ``forced``: for every mixture-of-experts layer in order, the experts ``[n, top]`` to use instead of the router's choice."""
    forced = list(forced) if forced is not None else None
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(ids))
    x = t64(tensors["embed"])[torch.tensor(list(ids), dtype=torch.long)]
    for li, l in enumerate(cfg["layers"]):
        p = f"l{li}."
        w, m = local(tensors, p + "mix."), l["mixer"]
        mix = {"attention": lambda h: attention(h, w, m, pos, eps), "latent_attention": lambda h: latent_attention(h, w, m, pos, eps),
               "hgrn2": lambda h: hgrn2(h, w, m, eps)}[l["type"]]
        x = sandwich(x, mix, t64(tensors[p + "norm1"]), t64(tensors[p + "norm1b"]), eps)
        if l.get("mlp") is not None:
            wf, choice = local(tensors, p + "mlp."), forced.pop(0) if forced else None
            x = sandwich(x, lambda h: moe_ff(h, wf, l["mlp"], choice), t64(tensors[p + "norm2"]), t64(tensors[p + "norm2b"]), eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, t64(tensors["final.norm"]), eps) @ t64(tensors["head"]).T


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
        tensors[name] = t64(torch.frombuffer(bytearray(data[a:b]), dtype=_DT[info["dtype"]]).reshape(info["shape"]))
    return cfg, tensors


def greedy(config, tensors, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(config, tensors, ids)[-1])))
    return ids[len(prompt):]
