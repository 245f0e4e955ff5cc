"""Plain, slow statement of the Vosezen decoder on whole sequences (PyTorch, CPU, fp32 or fp64), one function per
mechanism. It shares no code with the package: the tests compare the product path with it. ``p`` maps checkpoint names to
tensors, ``cfg`` is the parsed configuration; sequences are [T, width] with positions 0 .. T - 1.

``low`` marks every value that a bf16 model may hold in bf16 (projection inputs and outputs, normed queries and keys, cached
rows, attention and expert outputs). It is the identity; inside ``rounding()`` it rounds to bf16, which shows how much of a
difference such rounding alone explains."""
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


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1 + w)


def rotate_pairs(x, base):
    """x [T, heads, d], row t at position t; channels (2 i, 2 i + 1) turn by t * base^(-2 i / d)."""
    T, _, d = x.shape
    out = x.clone()
    for i in range(d // 2):
        a = torch.arange(T, dtype=torch.float64) * float(base) ** (-2.0 * i / d)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def temperature(T, m):
    """Factor of the queries at positions 0 .. T - 1."""
    t = m.get("q_temp")
    if t is None:
        return torch.ones(T, dtype=torch.float64)
    return torch.tensor([1 + t["coef"] * math.log((p + 1) // t["every"] + 1) for p in range(T)], dtype=torch.float64)


def attend(q, k, v, scale, softcap=None, sink=None):
    """Causal attention of one head, q / k [T, d], v [T, dv]. ``sink``: a further score without a value."""
    T = q.shape[0]
    s = (q @ k.t()) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.expand(T, 1).to(s.dtype)], 1)
    w = torch.softmax(s, -1)
    return w[:, :T] @ v


def keys_values(h, p, pre, m, eps, maps):
    """(normed keys [T, G, maps, dim], values [T, G, vdim]) as the cache holds them."""
    T, G = h.shape[0], m["kv_heads"]
    k = unit_rms(linear(h, p[pre + "k"]).reshape(T, G, maps, m["dim"]), eps) * p[pre + "k.norm"]
    return low(k), linear(h, p[pre + "v"]).reshape(T, G, m["vdim"])


def queries(h, p, pre, m, eps, maps):
    T = h.shape[0]
    q = unit_rms(linear(h, p[pre + "q"]).reshape(T, m["heads"], maps, m["dim"]), eps) * p[pre + "q.norm"]
    return low(q * temperature(T, m).to(q.dtype)[:, None, None, None])


def gated_output(o, h, p, pre):
    """One gate per head, then the output projection; o [T, H, vdim]."""
    g = torch.sigmoid(linear(h, p[pre + "g"]))
    return linear(low(o * g[:, :, None]).reshape(o.shape[0], -1), p[pre + "o"])


def difference_factor(p, pre, m):
    """lambda: how much of the second map is taken off the first."""
    return torch.exp((p[pre + "lq1"] * p[pre + "lk1"]).sum()) - torch.exp((p[pre + "lq2"] * p[pre + "lk2"]).sum()) + m["diff"]


def difference_attention(h, p, pre, m, eps, kv):
    q, (k, v) = queries(h, p, pre, m, eps, 2), kv
    lam, rep = difference_factor(p, pre, m), m["heads"] // m["kv_heads"]
    out = []
    for hd in range(m["heads"]):
        a = [low(attend(q[:, hd, i], k[:, hd // rep, i], v[:, hd // rep], m["scale"], m.get("softcap"))) for i in (0, 1)]
        out.append(low(unit_rms(a[0] - lam * a[1], eps) * (1 - m["diff"])))
    return gated_output(torch.stack(out, 1), h, p, pre)


def sink_attention(h, p, pre, m, eps, kv):
    q, (k, v) = queries(h, p, pre, m, eps, 1), kv
    rep = m["heads"] // m["kv_heads"]
    out = [attend(q[:, hd, 0], k[:, hd // rep, 0], v[:, hd // rep], m["scale"], m.get("softcap"), p[pre + "sink"][hd])
           for hd in range(m["heads"])]
    return gated_output(low(torch.stack(out, 1)), h, p, pre)


def latent_attention(h, p, pre, m, eps):
    T, H, dn, dr, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    cq = low(unit_rms(linear(h, p[pre + "dq"]), eps) * p[pre + "dq.norm"])
    q = linear(cq, p[pre + "uq"]).reshape(T, H, dn + dr)
    d = linear(h, p[pre + "dkv"])
    c = low(unit_rms(d[:, :r], eps) * p[pre + "dkv.norm"])
    kr = low(rotate_pairs(d[:, None, r:], m["rot"]["base"]))[:, 0]
    qr = low(rotate_pairs(q[:, :, dn:], m["rot"]["base"]))
    kn, v = linear(c, p[pre + "uk"]).reshape(T, H, dn), linear(c, p[pre + "uv"]).reshape(T, H, m["vdim"])
    out = [attend(torch.cat([q[:, hd, :dn], qr[:, hd]], 1), torch.cat([kn[:, hd], kr], 1), v[:, hd], m["scale"]) for hd in range(H)]
    return linear(low(torch.stack(out, 1)).reshape(T, -1), p[pre + "o"])


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def route(h, w, correction, router):
    """Chosen outputs [T, top] and their weights. Outputs behind the experts are identities."""
    s = torch.softmax(low(h) @ w.t(), -1)
    choice = s + correction
    n, count = choice.shape[1], router["groups"]["count"]
    best = choice.reshape(-1, count, n // count).amax(-1)
    kept = torch.argsort(best, dim=-1, descending=True, stable=True)[:, :router["groups"]["keep"]]
    allowed = torch.zeros_like(best, dtype=torch.bool).scatter(1, kept, True).repeat_interleave(n // count, 1)
    ids = torch.argsort(choice.masked_fill(~allowed, float("-inf")), dim=-1, descending=True, stable=True)[:, :router["top"]]
    return ids, s.gather(1, ids) * router["scale"]


def plain_mlp(h, p, pre):
    return linear(low(gelu(linear(h, p[pre + "up"]))), p[pre + "down"])


def mixture(h, p, pre, m):
    r = m["router"]
    ids, weights = route(h, p[pre + "router"], p[pre + "correction"], r)
    out = plain_mlp(h, p, pre + "shared.") if m.get("shared") else torch.zeros_like(h)
    for e in range(r["experts"] + r["identity"]):
        for slot in range(r["top"]):
            rows = (ids[:, slot] == e).nonzero()[:, 0]
            if rows.numel():
                y = plain_mlp(h[rows], p, f"{pre}e{e}.") if e < r["experts"] else low(h[rows])
                out[rows] = out[rows] + weights[rows, slot, None] * y
    return out


def mixer(kind, i, h, p, m, eps, kept):
    """Layer i's mixer; ``kept`` holds the keys and values of the layers run so far."""
    pre = f"l{i}.mix."
    if kind == "latent_attention":
        return latent_attention(h, p, pre, m, eps)
    kept[i] = kept[m["kv_from"]] if m.get("kv_from") is not None else keys_values(h, p, pre, m, eps, 2 if kind == "attention" else 1)
    return (difference_attention if kind == "attention" else sink_attention)(h, p, pre, m, eps, kept[i])


def forward(tokens, p, cfg):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    x, stream, kept = p["embed"][torch.as_tensor(tokens)], [], {}
    for i, spec in enumerate(cfg["layers"]):
        x = x + centred_norm(mixer(spec["type"], i, x, p, spec["mixer"], eps, kept), p[f"l{i}.norm1"], eps)
        if spec.get("mlp") is not None:
            x = x + centred_norm(mixture(x, p, f"l{i}.mlp.", spec["mlp"]), p[f"l{i}.norm2"], eps)
        stream.append(x)
    return low(centred_norm(x, p["final.norm"], eps)) @ p["embed"].t(), torch.stack(stream)
