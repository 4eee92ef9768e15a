"""Plain NumPy restatement of Bavutar models: layers of grouped softmax attention without rotation, gated delta-rule
mixers with a decay per key channel, and Mamba-2 mixers, each followed by a squared-relu feed-forward, with a layer norm
behind every residual sum.  One function per mechanism, recurrences token by token, float64.  It shares no code with the
CUDA path and is slow on purpose.

A model is a configuration dict and a flat dict {tensor name: array}; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np

from oracle.layer_stack_oracle import F, causal_conv, rms_norm, sigmoid, silu, softplus, to_bf16_grid


# ------------------------------------------------------------------ pieces ----
def layer_norm(x, weight, bias, eps):
    mu = x.mean(-1, keepdims=True)
    var = ((x - mu) ** 2).mean(-1, keepdims=True)
    return (x - mu) / np.sqrt(var + eps) * weight + bias


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def unit(x):
    """Unit vectors along the last axis, the fixed 1e-6 under the root."""
    return x / np.sqrt(np.sum(x * x, -1, keepdims=True) + 1e-6)


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, F) + 1.0) / every) + 1.0)


def causal_attention(q, k, v, scale):
    """q [T, H, n], k [T, G, n], v [T, G, m]: query head h reads key head h // (H / G); softmax over all j <= i."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.empty((T, H, v.shape[2]), F)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s[np.triu_indices(T, 1)] = -np.inf
        w = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (w / w.sum(-1, keepdims=True)) @ v[:, g]
    return out


def attention(h, w, m, eps, kv=None):
    """Returns (output, (keys, values)); ``kv`` are another layer's keys and values to be used instead of own ones."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, m["dim"])
    if m.get("q_temp"):
        q = q * query_temperature(np.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    if kv is None:
        kv = (rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, G, m["dim"]), (h @ w["v"].T).reshape(T, G, m["vdim"]))
    o = causal_attention(q, *kv, m["scale"])
    return o.reshape(T, -1) @ w["o"].T, kv


def delta_rule(q, k, v, g, beta):
    """Per head, token by token: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.
    q, k, g [T, H, n]; v [T, H, m]; beta [T, H]."""
    T, H, n = k.shape
    S = np.zeros((H, n, v.shape[2]), F)
    o = np.empty(v.shape, F)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hnm,hn->hm", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    return o


def channel_delta(h, w, m, eps):
    T, H, G, n, nv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda name: silu(causal_conv(h @ w[name].T, w[name + ".conv"], 0.0))
    spread = lambda x: np.repeat(x.reshape(T, G, n), H // G, axis=1)
    q = unit(spread(conv("q"))) * n ** -0.5
    k = unit(spread(conv("k")))
    v = conv("v").reshape(T, H, nv)
    beta = sigmoid(h @ w["b"].T)
    raw = ((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(T, H, n)
    g = np.exp(-np.exp(w["A_log"])[None, :, None] * softplus(raw))
    o = rms_norm(delta_rule(q, k, v, g, beta), w["norm"], eps)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, nv)
    return (o * gate).reshape(T, H * nv) @ w["o"].T


def state_space_dual(x, B, C, dt, A_log, D):
    """Per head, token by token: S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x.
    x [T, H, m]; B, C [T, G, n]; dt [T, H]."""
    T, H = dt.shape
    rep = H // B.shape[1]
    S = np.zeros((H, B.shape[2], x.shape[2]), F)
    y = np.empty(x.shape, F)
    for t in range(T):
        b, c = np.repeat(B[t], rep, 0), np.repeat(C[t], rep, 0)
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + (dt[t][:, None] * b)[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnm,hn->hm", S, c) + D[:, None] * x[t]
    return y


def mamba2(h, w, m, eps):
    T, H, nv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * nv
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    y = state_space_dual(x.reshape(T, H, nv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    y = (y.reshape(T, inner) * silu(z)).reshape(T, m["norm_groups"], -1)
    return (rms_norm(y, 1.0, eps).reshape(T, inner) * w["norm"]) @ w["o"].T


def dense_mlp(h, w):
    return squared_relu(h @ w["up"].T) @ w["down"].T


# ------------------------------------------------------------------- model ----
def forward(config, weights, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    W = {k: np.asarray(v, F) for k, v in weights.items()}
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}

    def norm(x, name):
        return layer_norm(x, W[name], W[name + ".b"], eps)

    x = W["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    trail, kept = [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        w = sub(p + "mix.")
        if layer["type"] == "attention":
            y, kept[i] = attention(x, w, m, eps, kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = {"channel_delta": channel_delta, "mamba2": mamba2}[layer["type"]](x, w, m, eps)
        x = norm(alpha * x + y, p + "norm1")
        if layer["mlp"] is not None:
            x = norm(alpha * x + dense_mlp(x, sub(p + "mlp.")), p + "norm2")
        trail.append(x)
    logits = softcap(norm(x, "final.norm") @ W["head"].T, config.get("logit_softcap"))
    return (logits, np.stack(trail)) if return_layers else logits


# ---------------------------------------------------- small random models ----
def tensor_shapes(config, ranks=(7, 5)):
    """{name: shape} of every tensor; ``ranks``: inner widths of the delta mixers' decay and gate projections."""
    d, V = config["width"], config["vocab"]
    s = {"embed": (V, d), "final.norm": (d,), "final.norm.b": (d,), "head": (V, d)}
    for i, layer in enumerate(config["layers"]):
        p, m, t = f"l{i}.", layer["mixer"], {}
        norms = ["norm1"] + (["norm2"] if layer["mlp"] is not None else [])
        for n in norms:
            t[n] = t[n + ".b"] = (d,)
        if layer["type"] == "attention":
            t["mix.q"] = (m["heads"] * m["dim"], d)
            t["mix.q.norm"] = (m["heads"] * m["dim"],)
            if m.get("kv_from") is None:
                t["mix.k"], t["mix.v"] = (m["kv_heads"] * m["dim"], d), (m["kv_heads"] * m["vdim"], d)
                t["mix.k.norm"] = (m["kv_heads"] * m["dim"],)
            t["mix.o"] = (d, m["heads"] * m["vdim"])
        elif layer["type"] == "channel_delta":
            H, n, nv = m["heads"], m["dim"], m["vdim"]
            for name, rows in (("q", m["kv_heads"] * n), ("k", m["kv_heads"] * n), ("v", H * nv)):
                t["mix." + name], t[f"mix.{name}.conv"] = (rows, d), (rows, m["conv"])
            t["mix.b"], t["mix.A_log"], t["mix.norm"], t["mix.dt_bias"] = (H, d), (H,), (nv,), (H * n,)
            t["mix.a1"], t["mix.a2"] = (ranks[0], d), (H * n, ranks[0])
            t["mix.g1"], t["mix.g2"] = (ranks[1], d), (H * nv, ranks[1])
            t["mix.o"] = (d, H * nv)
        else:
            H, inner = m["heads"], m["heads"] * m["vdim"]
            ch = inner + 2 * m["groups"] * m["state"]
            t["mix.in"], t["mix.conv"], t["mix.conv.b"] = (inner + ch + H, d), (ch, m["conv"]), (ch,)
            t["mix.dt_bias"] = t["mix.A_log"] = t["mix.D"] = (H,)
            t["mix.norm"], t["mix.o"] = (inner,), (d, inner)
        if layer["mlp"] is not None:
            t["mlp.up"], t["mlp.down"] = (layer["mlp"]["ff"], d), (d, layer["mlp"]["ff"])
        s.update({p + k: v for k, v in t.items()})
    return s


def random_weights(config, seed, gain=1.0, ranks=(7, 5)):
    """bf16-exact random weights under which every mechanism contributes: norms around one, decays from slow to fast,
    scores spread enough that single keys matter."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, ranks).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if leaf.endswith("norm.b") or leaf in ("norm1.b", "norm2.b"):
            a = 0.3 * rng.standard_normal(shape)
        elif leaf in ("mix.q.norm", "mix.k.norm"):
            a = 1.5 + 0.4 * rng.standard_normal(shape)
        elif "norm" in leaf:
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf == "mix.A_log":
            a = np.log(rng.uniform(0.05, 2.0, shape))
        elif leaf == "mix.dt_bias":
            a = rng.uniform(-4.0, 0.5, shape)
        elif leaf == "mix.D":
            a = rng.standard_normal(shape)
        elif leaf.endswith("conv") or leaf == "mix.conv.b":
            a = 0.6 * rng.standard_normal(shape)
        elif leaf == "embed":
            a = rng.standard_normal(shape)
        else:
            a = gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = to_bf16_grid(a)
    return out
