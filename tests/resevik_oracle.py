"""Plain, slow statement of the Resevik decoder on whole sequences (PyTorch, CPU, fp32 or fp64), one function per
mechanism. It shares no code with the package: the tests compare the product path with it. ``p`` maps checkpoint names to
tensors, ``cfg`` is the parsed configuration; sequences are [T, width] with positions 0 .. T - 1.

``low`` marks every value that a bf16 model may hold in bf16 (projection inputs and outputs, activations of the recurrence's
inputs, cached keys and values, attention outputs). It is the identity; inside ``rounding()`` it rounds to bf16, which shows
how much of a difference such rounding alone explains."""
import contextlib
import math

import torch

_ROUND = [False]


def low(x):
    return x.to(torch.bfloat16).to(x.dtype) if _ROUND[0] else x


@contextlib.contextmanager
def rounding():
    _ROUND[0] = True
    try:
        yield
    finally:
        _ROUND[0] = False


def linear(x, w):
    return low(low(x) @ w.t())


def silu(z):
    return z * torch.sigmoid(z)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate(x, base, dims, layout):
    """x [T, heads, d], row t at position t; the first ``dims`` channels turn, pairs (i, i + dims / 2) for layout "half" and
    (2 i, 2 i + 1) for "pairs"."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = t * float(base) ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            iu, iv = (i, i + dims // 2) if layout == "half" else (2 * i, 2 * i + 1)
            u, v = x[t, :, iu], x[t, :, iv]
            out[t, :, iu] = u * c - v * s
            out[t, :, iv] = v * c + u * s
    return out


def decayed_recurrence(q, k, v, decay, S=None):
    """q / k [T, H, N], v [T, H, P], decay [H] -> o [T, H, P] and the final state [H, N, P]."""
    T, H, N = q.shape
    P = v.shape[-1]
    S = torch.zeros(H, N, P, dtype=q.dtype) if S is None else S.clone()
    o = torch.zeros(T, H, P, dtype=q.dtype)
    g = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def lightning(h, p, pre, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = low(silu(linear(h, p[pre + "q"]))).reshape(T, H, N)
    k = low(silu(linear(h, p[pre + "k"]))).reshape(T, H, N)
    v = low(silu(linear(h, p[pre + "v"]))).reshape(T, H, P)
    o, _ = decayed_recurrence(q, k, v, m["decay"])
    o = unit_rms(low(o.reshape(T, H * P)), eps) * p[pre + "norm"]
    return linear(o * torch.sigmoid(linear(h, p[pre + "g"])), p[pre + "o"])


def retention(h, p, pre, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = rotate(linear(h, p[pre + "q"]).reshape(T, H, N), rot["base"], rot["dims"], "half")
    k = rotate(linear(h, p[pre + "k"]).reshape(T, H, N), rot["base"], rot["dims"], "half") * N ** -0.5
    v = linear(h, p[pre + "v"]).reshape(T, H, P)
    o, _ = decayed_recurrence(q, k, v, m["decay"])
    o = unit_rms(low(o), eps).reshape(T, H * P)
    return linear(o * silu(linear(h, p[pre + "g"])), p[pre + "o"])


def window_attention(h, p, pre, m, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    rot, win = m["rot"], m["mask"]["size"]
    raw = linear(h, p[pre + "k"]).reshape(T, G, D)
    q = low(unit_rms(rotate(linear(h, p[pre + "q"]).reshape(T, H, D), rot["base"], rot["dims"], "pairs"), eps))
    k = low(unit_rms(rotate(raw, rot["base"], rot["dims"], "pairs"), eps))
    out = torch.zeros(T, H, D, dtype=h.dtype)
    for i in range(T):
        lo = max(0, i - win + 1)
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * m["scale"]
            out[i, hd] = torch.softmax(s, 0) @ raw[lo:i + 1, g]
    return linear(out.reshape(T, H * D), p[pre + "o"])


MIXERS = {"lightning": lightning, "retention": retention, "attention": window_attention}


def route(h, w, top):
    """Chosen experts [T, top] and their weights."""
    s = torch.sigmoid(low(h) @ w.t())
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return order, s.gather(-1, order)


def expert(h, p, pre):
    return linear(low(silu(linear(h, p[pre + "gate"])) * linear(h, p[pre + "up"])), p[pre + "down"])


def mixture(h, p, pre, m):
    ids, weights = route(h, p[pre + "router"], m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        for slot in range(ids.shape[1]):
            rows = (ids[:, slot] == e).nonzero()[:, 0]
            if rows.numel():
                out[rows] = out[rows] + expert(weights[rows, slot, None] * h[rows], p, f"{pre}e{e}.")
    return out


def runs(cfg):
    """(layer, whether a pass other than the first starts here) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for t in range(times):
        order += [(i, t > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def forward(tokens, p, cfg):
    """Logits [T, vocab] and the stream after every layer run [runs, T, width]."""
    eps = cfg["norm"]["eps"]
    x0 = p["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x, stream = x0, []
    for i, again in runs(cfg):
        if again:
            x = x + x0
        spec = cfg["layers"][i]
        h = unit_rms(x, eps) * p[f"l{i}.norm1"]
        y = MIXERS[spec["type"]](h, p, f"l{i}.mix.", spec["mixer"], eps)
        if spec.get("mlp") is not None:
            y = y + mixture(h, p, f"l{i}.mlp.", spec["mlp"])
        x = x + y
        stream.append(x)
    return low(unit_rms(x, eps) * p["final.norm"]) @ p["head"].t(), torch.stack(stream)
