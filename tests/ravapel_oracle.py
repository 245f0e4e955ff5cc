"""Plain, slow statement of the Ravapel decoder on whole sequences (PyTorch, CPU, fp32 or fp64), one function per mechanism. It
shares no code with the package: the tests compare the product path with it. ``p`` maps checkpoint names to tensors, ``cfg`` is
the parsed configuration; sequences are [T, width] with positions 0 .. T - 1.

``low`` marks every value that a bf16 model may hold in bf16 (projection inputs and outputs, what the input convolution leaves
behind, normed queries and keys, cached rows, attention weights as factors of the values, the heads' results, the gated units). It
is the identity; inside ``rounding()`` it rounds to bf16, and inside ``rounding(seed)`` it moves every value by as much at random,
which shows how much of a difference such rounding alone explains."""
import contextlib

import torch

_ROUND = [None]


def low(x):
    how = _ROUND[0]
    if how is None:
        return x
    if how is True:
        return x.to(torch.bfloat16).to(x.dtype)
    return x * (1 + (2 * torch.rand(x.shape, generator=how, dtype=x.dtype) - 1) * 2.0 ** -9)


@contextlib.contextmanager
def rounding(seed=None):
    _ROUND[0] = True if seed is None else torch.Generator().manual_seed(seed)
    try:
        yield
    finally:
        _ROUND[0] = None


def linear(x, w, b=None):
    y = low(x) @ w.t()
    return low(y if b is None else y + b)


def silu(z):
    return z / (1 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1 + w)


def embedding(tokens, p, cfg):
    """Token vector + vector of the pair (previous token, token) + vector of the position."""
    e = cfg["embedding"]["bigram"]
    rows = []
    for t, tok in enumerate(tokens):
        pair = e["buckets"] if t == 0 else (tokens[t - 1] * e["mul_prev"] + tok * e["mul_cur"]) % e["buckets"]
        rows.append(p["embed"][tok] + p["bigram"][pair] + p["pos"][t])
    return torch.stack(rows)


def input_convolution(h, w):
    """h_t + sum over the taps of w[:, j] h_{t - taps + 1 + j}; w [width, taps]."""
    T, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] = out[t] + w[:, j] * h[s]
    return out


def forget(z, lower):
    """Forget gates between the bound and one."""
    return lower + (1 - lower) / (1 + torch.exp(-z))


def gated_state(q, f, v):
    """One head: S <- diag(f) S + (1 - f) v^T, o = S^T q; q, f [T, N], v [T, P]."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + (1 - f[t])[:, None] * v[t][None, :]
        out.append(q[t] @ S)
    return torch.stack(out)


def hgrn2(h, p, pre, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = low(silu(linear(h, p[pre + "q"]))).reshape(T, H, N)
    f = forget(low(h) @ p[pre + "f"].t() + p[pre + "f.b"], p[pre + "lower"]).reshape(T, H, N)
    v = linear(h, p[pre + "v"]).reshape(T, H, P)
    o = torch.stack([low(gated_state(q[:, i], f[:, i], v[:, i])) for i in range(H)], 1)
    return linear((unit_rms(o, eps) * p[pre + "norm"]).reshape(T, H * P), p[pre + "o"])


def rotate_halves(x, base, dims):
    """x [T, heads, d], row t at position t; channels (i, i + dims / 2) turn by t * base^(-2 i / dims)."""
    T, half = x.shape[0], dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(T, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, w = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - w * s
        out[:, :, i + half] = w * c + u * s
    return out


def visible(T, chunk):
    """[T, T]: row i sees column j."""
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // chunk == i[:, None] // chunk)


def sigmoid_attend(q, k, v, scale, bias, seen):
    """One head: every visible key counts with the sigmoid of its score; nothing is divided by the sum of the weights."""
    w = 1 / (1 + torch.exp(-((q @ k.t()) * scale + bias)))
    return low(torch.where(seen, w, torch.zeros_like(w))) @ v


def sigmoid_attention(h, p, pre, m, eps):
    T, H, G, D, DV = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(linear(h, p[pre + "q"]).reshape(T, H, D), eps) * p[pre + "q.norm"]
    k = unit_rms(linear(h, p[pre + "k"]).reshape(T, G, D), eps) * p[pre + "k.norm"]
    q, k = (low(rotate_halves(t, m["rot"]["base"], m["rot"]["dims"])) for t in (q, k))
    v = linear(h, p[pre + "v"]).reshape(T, G, DV)
    seen = visible(T, m["mask"]["size"])
    o = [sigmoid_attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], p[pre + "pb"][i], seen) for i in range(H)]
    return linear(torch.stack(o, 1).reshape(T, H * DV), p[pre + "o"])


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, i, f):
    """One head: q, k [T, N], v [T, P], logarithms of the input and forget gates i, f [T]."""
    N, P = q.shape[1], v.shape[1]
    S, n, m, out = torch.zeros(N, P, dtype=q.dtype), torch.zeros(N, dtype=q.dtype), torch.zeros((), dtype=q.dtype), []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + put * k[t][:, None] * v[t][None, :]
        n = keep * n + put * k[t]
        m = new
        out.append((q[t] @ S) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def memory_gates(h, p, pre, cap):
    """Logarithms of the input and forget gates, [T, heads] each."""
    i = soft_cap(low(h) @ p[pre + "i"].t() + p[pre + "i.b"], cap)
    z = soft_cap(low(h) @ p[pre + "f"].t() + p[pre + "f.b"], cap)
    return i, -torch.log(1 + torch.exp(-z))


def mlstm(h, p, pre, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, p[pre + "q"]).reshape(T, H, N) * N ** -0.5
    k, v = linear(h, p[pre + "k"]).reshape(T, H, N), linear(h, p[pre + "v"]).reshape(T, H, P)
    i, f = memory_gates(h, p, pre, float(m["gate_cap"]))
    o = torch.stack([low(matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])) for a in range(H)], 1)
    o = unit_rms(o, eps).reshape(T, H * P) * p[pre + "norm"]
    return linear(o / (1 + torch.exp(-linear(h, p[pre + "g"]))), p[pre + "o"])


def parallel(h, p, pre, m, eps):
    left, right = sigmoid_attention(h, p, pre + "left.", m["left"], eps), mlstm(h, p, pre + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def gated_mlp(h, p, pre):
    a = silu(linear(h, p[pre + "gate"], p[pre + "gate.b"])) * linear(h, p[pre + "up"], p[pre + "up.b"])
    return linear(low(a), p[pre + "down"], p[pre + "down.b"])


def layer(x, i, spec, p, eps):
    pre = f"l{i}."
    h = low(input_convolution(low(centred_norm(x, p[pre + "norm1"], eps)), p[pre + "canon1"]))
    y = (hgrn2 if spec["type"] == "hgrn2" else parallel)(h, p, pre + "mix.", spec["mixer"], eps)
    x = x + centred_norm(y, p[pre + "norm1b"], eps)
    if spec.get("mlp") is not None:
        y = gated_mlp(centred_norm(x, p[pre + "norm2"], eps), p, pre + "mlp.")
        x = x + centred_norm(y, p[pre + "norm2b"], eps)
    return x


def enter_pass(x, x0, w):
    """Stream at the start of a pass of the loop."""
    return low(torch.cat([x, x0], 1)) @ w.t()


def forward(tokens, p, cfg):
    """Logits [T, vocab] and the stream after every layer run [runs, T, width]."""
    tokens, eps, n = [int(t) for t in tokens], cfg["norm"]["eps"], len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    x0 = embedding(tokens, p, cfg)
    x, stream = x0, []

    def run(i):
        nonlocal x
        x = layer(x, i, cfg["layers"][i], p, eps)
        stream.append(x)
    for i in range(loop["start"]):
        run(i)
    for _ in range(loop["times"]):
        x = enter_pass(x, x0, p["loop.in"])
        for i in range(loop["start"], loop["stop"]):
            run(i)
    for i in range(loop["stop"], n):
        run(i)
    return low(centred_norm(x, p["final.norm"], eps)) @ p["head"].t(), torch.stack(stream)
