"""Plain, slow statement of the Duvivik decoder on whole sequences (PyTorch, CPU, fp32 or fp64), one function per
mechanism. It shares no code with the package: the tests compare the product path with it. ``p`` maps checkpoint names to
tensors, ``cfg`` is the parsed configuration; sequences are [T, width] with positions 0 .. T - 1.

``low`` marks every value that a bf16 model may hold in bf16 (projection inputs and outputs, convolution outputs, cached
latents, attention outputs). It is the identity; inside ``rounding()`` it rounds to bf16, which shows how much of a
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


def layer_norm(x, w, b, eps):
    m = x.mean(-1, keepdim=True)
    var = ((x - m) ** 2).mean(-1, keepdim=True)
    return (x - m) / torch.sqrt(var + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_pairs(x, base, pos=None):
    """Interleaved rotation of the whole last dimension; x [T, ..., dims], row t at position t (or pos[t])."""
    T, dims = x.shape[0], x.shape[-1]
    out = x.clone()
    for t in range(T):
        at = t if pos is None else int(pos[t])
        for i in range(dims // 2):
            a = at * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, ..., 2 * i].clone(), x[t, ..., 2 * i + 1].clone()
            out[t, ..., 2 * i] = u * c - v * s
            out[t, ..., 2 * i + 1] = v * c + u * s
    return out


def causal_conv(x, w, b):
    """Depthwise: out[t, c] = b[c] + sum_j w[c, j] x[t - (taps - 1) + j, c], zeros before the start; then silu."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = b.clone()
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                acc = acc + w[:, j] * x[src]
        out[t] = acc
    return low(out * torch.sigmoid(out))


def ssd_recurrence(x, B, C, dt, A_log, D, S=None):
    """x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P] and the final state [H, N, P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if S is None else S.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].t() @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    v = y * (z * torch.sigmoid(z))
    parts = [rms(c, eps) for c in v.chunk(groups, -1)]
    return torch.cat(parts, -1) * w


def mamba2(h, p, pre, m, eps):
    inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
    u = linear(h, p[pre + "in"])
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * gn], u[:, 2 * inner + 2 * gn:]
    assert dt.shape[1] == m["heads"]
    xbc = causal_conv(xbc, p[pre + "conv"], p[pre + "conv.b"])
    T = h.shape[0]
    x = xbc[:, :inner].reshape(T, m["heads"], m["vdim"])
    B = xbc[:, inner:inner + gn].reshape(T, m["groups"], m["state"])
    C = xbc[:, inner + gn:].reshape(T, m["groups"], m["state"])
    v = dt + p[pre + "dt_bias"]
    dt = torch.logaddexp(v, torch.zeros_like(v))
    y, _ = ssd_recurrence(x, B, C, dt, p[pre + "A_log"], p[pre + "D"])
    y = gated_group_norm(low(y.reshape(T, inner)), z, p[pre + "norm"], m["norm_groups"], eps)
    return linear(y, p[pre + "o"])


def latent_kv(h, p, pre, m, eps):
    """What a layer with its own down-projection leaves for itself and for the layers that read it."""
    u = linear(h, p[pre + "dkv"])
    r = m["kv_rank"]
    c = rms(u[:, :r], eps) * p[pre + "dkv.norm"]
    return low(c), low(rotate_pairs(u[:, r:], m["rot"]["base"]))


def latent_attention(h, p, pre, m, c, kr):
    T, H, dn, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = linear(h, p[pre + "q"]).reshape(T, H, dn + dr)
    qr = low(rotate_pairs(q[..., dn:], m["rot"]["base"]))
    k = linear(c, p[pre + "uk"]).reshape(T, H, dn)
    v = linear(c, p[pre + "uv"]).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        for hd in range(H):
            s = (k[:i + 1, hd] @ q[i, hd, :dn] + kr[:i + 1] @ qr[i, hd]) * m["scale"]
            out[i, hd] = torch.softmax(s, 0) @ v[:i + 1, hd]
    return linear(out.reshape(T, H * dv), p[pre + "o"])


def clamped_glu(h, p, pre, limit):
    g = torch.minimum(linear(h, p[pre + "gate"]) + p[pre + "gate.b"], torch.tensor(limit, dtype=h.dtype))
    u = (linear(h, p[pre + "up"]) + p[pre + "up.b"]).clamp(-limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), p[pre + "down"]) + p[pre + "down.b"]


def forward(tokens, p, cfg):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = p["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    cached, stream = {}, []
    for i, spec in enumerate(cfg["layers"]):
        pre, m = f"l{i}.mix.", spec["mixer"]
        if spec["type"] == "mamba2":
            y = mamba2(x, p, pre, m, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                cached[i] = latent_kv(x, p, pre, m, eps)
            y = latent_attention(x, p, pre, m, *cached[i if src is None else src])
        x = layer_norm(alpha * x + y, p[f"l{i}.norm1"], p[f"l{i}.norm1.b"], eps)
        if spec["mlp"] is not None:
            y = clamped_glu(x, p, f"l{i}.mlp.", spec["mlp"]["limit"])
            x = layer_norm(alpha * x + y, p[f"l{i}.norm2"], p[f"l{i}.norm2.b"], eps)
        stream.append(x)
    x = layer_norm(x, p["final.norm"], p["final.norm.b"], eps)
    return low(x) @ p["head"].t(), torch.stack(stream)
