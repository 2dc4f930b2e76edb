"""Plain, slow reference of the Vogerax design: one function per mechanism, no batching, no cache, no kernels.

``forward`` runs one whole sequence and returns its logits; ``layers_out`` collects the residual after every layer.  Weights are a
dict of float tensors under the checkpoint's tensor names.  The arithmetic type is that of the weights (float64 in the tests), and
nothing is imported from the package.
"""
import math

import torch


def rms(x, eps):
    """Rows divided by the square root of (mean square + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def group_norm(x, w, eps, groups):
    """Every one of ``groups`` equal parts of a row by its own root mean square."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * w


def silu(x):
    return x * torch.sigmoid(x)


def relu2(x):
    return torch.clamp(x, min=0) ** 2


# ------------------------------------------------------------------ rotations
def frequencies(dims, base):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)


def linear_frequencies(dims, base, factor):
    return frequencies(dims, base) / factor


def yarn_frequencies(dims, base, factor, original, fast, slow):
    """Slow turns are divided by ``factor``, fast ones kept, a ramp in between; and the factor of cosines and sines."""
    def dim_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim_of(fast)), 0), min(math.ceil(dim_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(frequencies(dims, base).tolist()):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1


def rotation(rot):
    """(angles per position, factor of cosines and sines) of a config's "rot"."""
    s = rot.get("scaling")
    if not s:
        return frequencies(rot["dims"], rot["base"]), 1.0
    if "original" in s:
        return yarn_frequencies(rot["dims"], rot["base"], s["factor"], s["original"], s["fast"], s["slow"])
    return linear_frequencies(rot["dims"], rot["base"], s["factor"]), 1.0


def rotate(x, pos, freq, amp=1.0):
    """The first 2 len(freq) dimensions of ``x`` [T, heads, d]: dimension i with i + len(freq)."""
    n = len(freq)
    a = pos.to(torch.float64)[:, None] * freq[None, :]
    c, s = ((f(a) * amp).to(x)[:, None, :] for f in (torch.cos, torch.sin))
    u, v = x[..., :n], x[..., n: 2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


# ------------------------------------------------------------------ attention
def softmax_over(scores, seen, sink=None):
    """Softmax of ``scores`` [H, q, k] over the keys that are ``seen`` [q, k]; ``sink`` [H]: one more term below the line."""
    s = scores.masked_fill(~seen[None], float("-inf"))
    if sink is None:
        return torch.softmax(s, dim=-1)
    s = torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1).to(s)], dim=-1)
    return torch.softmax(s, dim=-1)[..., :-1]


def attend(q, k, v, seen, scale, sink=None):
    """``q`` [Tq, H, a], ``k`` [Tk, G, a], ``v`` [Tk, G, b] -> [Tq, H, b]."""
    share = q.shape[1] // k.shape[1]
    k, v = (x.repeat_interleave(share, dim=1) for x in (k, v))
    return torch.einsum("hqk,khb->qhb", softmax_over(torch.einsum("qha,kha->hqk", q, k) * scale, seen, sink), v)


def causal(qpos, n):
    return torch.arange(n)[None, :] <= qpos[:, None]


def pooled(x, pool):
    """Means of the whole blocks of ``pool`` rows."""
    n = len(x) // pool
    return x[: n * pool].reshape(n, pool, *x.shape[1:]).mean(dim=1)


def window_and_blocks(qpos, n, size, pool):
    """What rows at ``qpos`` see of ``n`` tokens, and of their whole blocks."""
    d = qpos[:, None] - torch.arange(n)[None, :]
    last = torch.arange(n // pool) * pool + pool - 1
    return (d >= 0) & (d < size), last[None, :] <= qpos[:, None] - size


def pooled_window_attend(q, k, v, qpos, size, pool, scale):
    near, far = window_and_blocks(qpos, len(k), size, pool)
    return attend(q, torch.cat([k, pooled(k, pool)]), torch.cat([v, pooled(v, pool)]), torch.cat([near, far], dim=1), scale)


def attention(w, p, m, eps, h):
    t, pos = len(h), torch.arange(len(h))
    q, k = ((h @ w[p + n].T).reshape(t, c, -1) for n, c in (("q", m["heads"]), ("k", m["kv_heads"])))
    freq, amp = rotation(m["rot"])
    mask, qr, kr = m.get("mask"), rotate(q, pos, freq, amp), rotate(k, pos, freq, amp)
    if mask and mask.get("pool"):
        o = pooled_window_attend(qr, kr, k, pos, mask["size"], mask["pool"], m["scale"])
    else:
        o = attend(qr, kr, k, window_and_blocks(pos, t, mask["size"], t)[0] if mask else causal(pos, t), m["scale"])
    return o.reshape(t, -1) @ w[p + "o"].T


def left(w, p, m, eps, h):
    t, pos = len(h), torch.arange(len(h))
    q, k, v = ((h @ w[p + n].T).reshape(t, c, -1) for n, c in (("q", m["heads"]), ("k", m["kv_heads"]), ("v", m["kv_heads"])))
    q, k = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"]
    freq, amp = rotation(m["rot"])
    turn = frequencies(m["vdim"], m["rot"]["base"])
    o = attend(rotate(q, pos, freq, amp), rotate(k, pos, freq, amp), rotate(v, pos, turn), causal(pos, t), m["scale"], w[p + "sink"])
    o = rotate(o, -pos, turn)
    return (o.reshape(t, -1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ retention
def retention_scan(q, k, v, decay, state=None):
    """``q``, ``k`` [T, H, a], ``v`` [T, H, b], ``decay`` [H] -> ([T, H, b], state [H, a, b])."""
    s = torch.zeros(*k.shape[1:], v.shape[-1]).to(k) if state is None else state
    out = []
    for j in range(len(q)):
        s = decay[:, None, None] * s + k[j][:, :, None] * v[j][:, None, :]
        out.append(torch.einsum("hab,ha->hb", s, q[j]))
    return torch.stack(out), s


def right(w, p, m, eps, h):
    t, pos = len(h), torch.arange(len(h))
    q, k, v = ((h @ w[p + n].T).reshape(t, m["heads"], -1) for n in "qkv")
    freq, amp = rotation(m["rot"])
    q, k = rotate(q, pos, freq, amp), rotate(k, pos, freq, amp) * m["dim"] ** -0.5
    o, _ = retention_scan(q, k, v, torch.tensor(m["decay"], dtype=torch.float64).to(q))
    return (rms(o, eps).reshape(t, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(w, p, m, eps, h):
    a, b = left(w, p + "left.", m["left"], eps, h), right(w, p + "right.", m["right"], eps, h)
    return (rms(a, eps) * w[p + "left.out"] + rms(b, eps) * w[p + "right.out"]) / 2


# ------------------------------------------------------------------ feed-forwards
def feed(w, p, h):
    return relu2(h @ w[p + "up"].T) @ w[p + "down"].T


def routed(w, p, m, h):
    scores = torch.softmax(h @ w[p + "router"].T, dim=-1)
    out = torch.zeros_like(h)
    for i in range(len(h)):
        for e in torch.sort(scores[i], descending=True, stable=True).indices[: m["router"]["top"]].tolist():
            out[i] += scores[i, e] * feed(w, f"{p}e{e}.", h[i])
    return out + feed(w, p + "shared.", h) if m.get("shared") else out


def feed_forward(w, p, m, h):
    return routed(w, p, m, h) if m["kind"] == "moe" else feed(w, p, h)


# ------------------------------------------------------------------ the whole
def owner(cfg, i):
    """The layer whose tensors layer ``i`` uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(w, cfg, tokens, layers_out=None):
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    norm = lambda x, name: group_norm(x, w[name], eps, groups)                       # noqa: E731
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        mixer = {"attention": attention, "parallel": parallel}[layer["type"]]
        x = x + norm(mixer(w, p + "mix.", layer["mixer"], eps, norm(x, p + "norm1")), p + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(w, p + "mlp.", layer["mlp"], norm(x, p + "norm2")), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ w["head"].T
