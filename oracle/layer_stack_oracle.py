"""Plain NumPy restatement of the layer-stack models (Keselix): one function per mechanism, token by token where
the mechanism is a recurrence, no caches except the ones a recurrence defines.  float64 by default, so that it
stands for the exact result.  It shares no code with the CUDA path and is slow on purpose.

A model is a configuration dict and a flat dict {tensor name: array}; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

F = np.float64


# ------------------------------------------------------------------ pieces ----
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rotate_interleaved(x, positions, base):
    """Rotates all of the last axis (even size n): dims (2i, 2i + 1) at position p by the angle p * base^(-2i/n)."""
    n = x.shape[-1]
    freq = base ** (-np.arange(0, n, 2, dtype=F) / n)
    ang = np.asarray(positions, F)[:, None] * freq[None, :]
    while ang.ndim < x.ndim:
        ang = ang[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * np.cos(ang) - v * np.sin(ang)
    out[..., 1::2] = v * np.cos(ang) + u * np.sin(ang)
    return out


def window_attention(q, k, v, scale, window):
    """q [T, H, n], k [T, H, n], v [T, H, m]: softmax over the keys j with 0 <= i - j < window."""
    T = q.shape[0]
    out = np.zeros((T, q.shape[1], v.shape[2]), F)
    for i in range(T):
        lo = max(0, i - window + 1)
        s = np.einsum("hn,jhn->hj", q[i], k[lo:i + 1]) * scale
        w = np.exp(s - s.max(-1, keepdims=True))
        w /= w.sum(-1, keepdims=True)
        out[i] = np.einsum("hj,jhm->hm", w, v[lo:i + 1])
    return out


def latent_attention(h, w, m, eps):
    """Attention whose keys and values are linear maps of a normalised latent shared by all heads, plus one
    rotated key part shared by all heads.  w: tensors of the mixer by their last name."""
    T = h.shape[0]
    H, n, r, nv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (h @ w["q"].T).reshape(T, H, n + r)
    q = np.concatenate([q[..., :n], rotate_interleaved(q[..., n:], pos, m["rot"]["base"])], -1)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    kr = rotate_interleaved(down[:, rank:], pos, m["rot"]["base"])
    k = np.concatenate([(c @ w["uk"].T).reshape(T, H, n), np.repeat(kr[:, None, :], H, axis=1)], -1)
    v = (c @ w["uv"].T).reshape(T, H, nv)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * nv) @ w["o"].T


def causal_conv(x, taps, bias):
    """Per-channel convolution over time: x [T, C], taps [C, K], the last column weighs the current row."""
    T, C = x.shape
    K = taps.shape[1]
    xp = np.concatenate([np.zeros((K - 1, C), x.dtype), x])
    return sum(xp[j:j + T] * taps[:, j] for j in range(K)) + bias


def selective_scan(u, dt, A, B, C, D):
    """S <- exp(dt A) S + dt u B; y = sum_n S C + D u.  u, dt [T, inner]; A [inner, state]; B, C [T, state]."""
    S = np.zeros(A.shape, F)
    y = np.empty(u.shape, F)
    for t in range(u.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * u[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * u[t]
    return y


def mamba1(h, w, m):
    inner, state, rank = m["inner"], m["state"], m["dt_rank"]
    xz = h @ w["in"].T
    u = silu(causal_conv(xz[:, :inner], w["conv"], w["conv.b"]))
    p = u @ w["x"].T
    dt = softplus(p[:, :rank] @ w["dt"].T + w["dt.b"])
    y = selective_scan(u, dt, -np.exp(w["A_log"]), p[:, rank:rank + state], p[:, rank + state:], w["D"])
    return (y * silu(xz[:, inner:])) @ w["o"].T


def dense_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# ------------------------------------------------------------------- model ----
def layer_schedule(config):
    """[(layer index, first layer of a pass)] in the order the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] +
            [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] +
            [(i, False) for i in range(b, n)])


def forward(config, weights, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer run)."""
    W = {k: np.asarray(v, F) for k, v in weights.items()}
    eps, mult = config["norm"]["eps"], config["residual_mult"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}

    x = W["embed"][np.asarray(tokens)]
    x0 = x
    trail = []
    for i, first in layer_schedule(config):
        if first:
            x = np.concatenate([x, x0], -1) @ W["loop.in"].T
        layer, p = config["layers"][i], f"l{i}."
        h = rms_norm(x, W[p + "norm1"], eps)
        w = sub(p + "mix.")
        y = latent_attention(h, w, layer["mixer"], eps) if layer["type"] == "latent_attention" else \
            mamba1(h, w, layer["mixer"])
        x = x + mult * rms_norm(y, W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            y = dense_mlp(rms_norm(x, W[p + "norm2"], eps), sub(p + "mlp."))
            x = x + mult * rms_norm(y, W[p + "norm2b"], eps)
        trail.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, np.stack(trail)) if return_layers else logits


def generate_greedy(config, weights, prompt, steps):
    """Greedy continuation by recomputing the whole sequence every step; ties go to the highest index, as in the
    framework's sampler."""
    toks, out = list(prompt), []
    for _ in range(steps):
        last = forward(config, weights, toks)[-1]
        t = int(len(last) - 1 - np.argmax(last[::-1]))
        out.append(t)
        toks.append(t)
    return out


# ---------------------------------------------------- small random models ----
def tensor_shapes(config):
    """{name: shape} of every tensor of a configuration."""
    d, V = config["width"], config["vocab"]
    s = {"embed": (V, d)}
    if config.get("loop"):
        s["loop.in"] = (d, 2 * d)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        s[p + "norm1"] = s[p + "norm1b"] = (d,)
        if layer["type"] == "mamba1":
            n = m["inner"]
            s[p + "mix.in"], s[p + "mix.conv"], s[p + "mix.conv.b"] = (2 * n, d), (n, m["conv"]), (n,)
            s[p + "mix.x"], s[p + "mix.dt"] = (m["dt_rank"] + 2 * m["state"], n), (n, m["dt_rank"])
            s[p + "mix.dt.b"], s[p + "mix.A_log"], s[p + "mix.D"] = (n,), (n, m["state"]), (n,)
            s[p + "mix.o"] = (d, n)
        else:
            H = m["heads"]
            s[p + "mix.q"] = (H * (m["dim"] + m["rot_dim"]), d)
            s[p + "mix.dkv"], s[p + "mix.dkv.norm"] = (m["kv_rank"] + m["rot_dim"], d), (m["kv_rank"],)
            s[p + "mix.uk"], s[p + "mix.uv"] = (H * m["dim"], m["kv_rank"]), (H * m["vdim"], m["kv_rank"])
            s[p + "mix.o"] = (d, H * m["vdim"])
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            s[p + "norm2"] = s[p + "norm2b"] = (d,)
            s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (f, d), (f, d), (d, f)
    s["final.norm"], s["head"] = (d,), (V, d)
    return s


def to_bf16_grid(a):
    """float32 values rounded to the nearest bfloat16 (ties to even)."""
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    b = (b + 0x7FFF + ((b >> 16) & 1)) & np.uint32(0xFFFF0000)
    return b.view(np.float32)


def random_weights(config, seed, gain=1.0):
    """bf16-exact random weights under which every mechanism contributes: norms around one, decays from slow to
    fast, scores spread enough that single keys matter."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if "norm" in leaf:
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf == "mix.A_log":
            a = np.log(rng.uniform(0.02, 4.0, shape))
        elif leaf == "mix.dt.b":
            a = rng.uniform(-4.0, 0.5, shape)
        elif leaf == "mix.D":
            a = rng.standard_normal(shape)
        elif leaf in ("mix.conv", "mix.conv.b"):
            a = 0.5 * rng.standard_normal(shape)
        elif leaf == "embed":
            a = rng.standard_normal(shape)
        elif leaf in ("mix.q", "mix.dkv"):
            a = 2.0 * gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        else:
            a = gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = to_bf16_grid(a)
    return out
